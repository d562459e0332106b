"""The state-space / chunk-attention / gated-linear decoder as a whole on the GPU against the plain restatement:
prompts, decoding, unequal batches, memory used again, far keys and chunk edges, first tokens, generation through
the framework's own entry points, the trace runner, the engine."""
import json
import os
import subprocess
import sys

import pytest
import torch

import moponex_plain as P
import tulezen_plain as T

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}

# odd sizes; groups of heads, norm parts that straddle heads, other taps; one and as many key heads as query heads; with
# and without rotation, slow-down, chunks, groups of experts, identity experts, shared expert, feed-forward
ODD = P.make_config([P.parallel_layer((6, 2, 12, 0.4, 9, (8, 100.0, 3.0)), (3, 20, 28, 4.0, 5), P.dense_mlp(44)),
                     P.ssm_layer(6, 10, 12, groups=3, conv=3, norm_groups=4, mlp=P.moe_mlp(7, 3, 20, identity=2, groups=(3, 2), shared=12)),
                     P.parallel_layer((2, 2, 9, 0.5, 0, None), (1, 8, 12, 1.0, 16), P.moe_mlp(5, 2, 12)),
                     P.ssm_layer(4, 16, 24, groups=4, conv=2, norm_groups=1),
                     P.parallel_layer((4, 1, 16, 0.3, 33, (16, 5000.0, None)), (2, 12, 8, 20.0, 8), P.moe_mlp(8, 4, 8, identity=4, groups=(4, 3)))],
                    width=52, vocab=83)
# sizes that fill or exceed the tensor-core tiles; two heads per tile and one
WIDE = P.make_config([P.ssm_layer(4, 64, 128, groups=2, mlp=P.moe_mlp(12, 3, 40, identity=4, groups=(4, 2), shared=72)),
                      P.parallel_layer((20, 1, 64, 0.12, 130, (48, 20000.0, 2.0)), (2, 128, 136, 12.0, 16), P.dense_mlp(136)),
                      P.ssm_layer(3, 136, 70, groups=1, norm_groups=3), P.parallel_layer((4, 2, 100, 0.1, 64, (100, 300.0, None)), (3, 50, 64, 2.0, 24)),
                      P.ssm_layer(5, 40, 20, groups=5, norm_groups=5, mlp=P.dense_mlp(64))], width=192, vocab=334, eps=1e-6, mult=1.0, logit_scale=1.0)
# head sizes the tensor-core kernels do not have; heads, ranks, groups and taps of one; no bigram rows
HUGE = P.make_config([P.parallel_layer((2, 1, 140, 0.08, 20, (40, 1000.0, 8.0)), (1, 136, 24, 6.0, 1), P.moe_mlp(3, 1, 16)),
                      P.ssm_layer(1, 8, 136, conv=5), P.parallel_layer((1, 1, 2, 1.0, 1, (2, 10.0, None)), (1, 1, 1, 9.0, 3), P.dense_mlp(24)),
                      P.ssm_layer(2, 1, 1, conv=1, norm_groups=2)], width=40, vocab=64, bigram=None)
CONFIGS = {"odd": ODD, "wide": WIDE, "huge": HUGE}


def make(cfg, dtype, seed=1, change=None):
    from energonai_b200.registry import build_model
    from energonai_b200.utils import processing_Moponex
    tensors = P.make_tensors(cfg, seed)
    if change:
        change(tensors)
    model = build_model("Moponex", config_dict=P.with_ranks(cfg), dtype=DTYPES[dtype])
    model.load_state_dict(processing_Moponex(tensors, model))
    return model.cuda().eval(), tensors


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def check(got, want, dtype):
    """Row by row, the mean over the vocabulary taken off.  A row in ten, or one, may be further off: a close call of a
    router falls the other way now and then in 16 bits, and the first tokens of a recurrence are badly
    conditioned (a memory of one key gives (q.k) v, and q.k may be near zero)."""
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all()
    d = got - want
    err = ((d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std(-1).mean()).sort().values
    most, worst, typical = (3e-5, 2e-4, 1e-5) if dtype == "float32" else (0.12, 0.8, 0.03)
    n = err.numel()
    assert float(err[-1]) < worst and float(err[n // 2]) < (typical if n > 2 else worst), err
    assert float(err[n - 1 - max(1, n // 10)] if n > 2 else err[0]) < most, err


def prompt_logits(model, toks):
    return model.logits(model.prompt(torch.tensor([toks], device="cuda"), reserve=4))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,n", [("odd", 1), ("odd", 2), ("odd", 129), ("odd", 300), ("wide", 127), ("wide", 400), ("huge", 70)])
def test_prompt(name, n, dtype):
    cfg = CONFIGS[name]
    model, t = make(cfg, dtype)
    toks, seen = tokens(cfg, n), []
    x = model.prompt(torch.tensor([toks], device="cuda"), on_layer=lambda i, s: seen.append(s.clone()))
    want, streams = P.forward(cfg, t, toks)
    check(model.logits(x), want, dtype)
    assert len(seen) == len(streams)
    for a, b in zip(seen, streams):
        check(a[:, :cfg["width"]], b, dtype)
        assert a.dtype == torch.float32 and float(a[:, cfg["width"]:].abs().sum()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,start,n", [("odd", 1, 200), ("odd", 127, 140), ("odd", 128, 140), ("wide", 2, 20), ("wide", 250, 280), ("huge", 38, 60)])
def test_decoding_token_by_token(name, start, n, dtype):
    """A prompt and the steps behind it against the whole, and against one prompt."""
    cfg = CONFIGS[name]
    model, t = make(cfg, dtype)
    toks = tokens(cfg, n)
    want, _ = P.forward(cfg, t, toks)
    got = [prompt_logits(model, toks[:start])]
    for k in range(start, n):
        got.append(model.step(torch.tensor([toks[k]], device="cuda")))
    got = torch.cat(got)
    check(got, want, dtype)
    check(prompt_logits(model, toks), got, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,lens", [("odd", (1, 37, 12, 190)), ("wide", (3, 260)), ("odd", (70, 71, 69)), ("wide", (1, 1, 2))])
def test_unequal_batch_against_each_alone(name, lens, dtype):
    cfg = CONFIGS[name]
    model, t = make(cfg, dtype)
    more, S = 20, max(lens)
    toks = [tokens(cfg, n + more, seed=n + r) for r, n in enumerate(lens)]
    ids = torch.zeros(len(lens), S, dtype=torch.long)
    mask = torch.zeros_like(ids)
    for r, n in enumerate(lens):
        ids[r, S - n:], mask[r, S - n:] = torch.tensor(toks[r][:n]), 1
    x = model.prompt(ids.cuda(), mask, reserve=2).view(len(lens), S, -1)
    assert torch.isfinite(x).all()
    got = [[model.logits(x[r, S - n:].contiguous())] for r, n in enumerate(lens)]
    live = list(range(len(lens)))
    for k in range(more):
        if k == 8:                                       # one request ends, its state goes
            drop = live[1]
            model.state.keep([i for i, r in enumerate(live) if r != drop])
            live.remove(drop)
        lg = model.step(torch.tensor([toks[r][lens[r] + k] for r in live], device="cuda"))
        for i, r in enumerate(live):
            got[r].append(lg[i:i + 1])
    for r, n in enumerate(lens):
        out = torch.cat(got[r])
        check(out, P.forward(cfg, t, toks[r])[0][:out.shape[0]], dtype)
        model.state = model.new_state()
        alone = [prompt_logits(model, toks[r][:n])]
        for k in range(out.shape[0] - n):
            alone.append(model.step(torch.tensor([toks[r][n + k]], device="cuda")))
        check(out, torch.cat(alone), dtype)


def test_float16():
    """The third number format: tensor-core products and attention, recurrences on the CUDA cores."""
    from energonai_b200.registry import build_model
    from energonai_b200.utils import processing_Moponex
    t = P.make_tensors(ODD, 1)
    model = build_model("Moponex", config_dict=P.with_ranks(ODD), dtype=torch.float16)
    model.load_state_dict(processing_Moponex(t, model))
    model, toks = model.cuda().eval(), tokens(ODD, 60)
    got = [prompt_logits(model, toks[:40])] + [model.step(torch.tensor([x], device="cuda")) for x in toks[40:]]
    check(torch.cat(got), P.forward(ODD, t, toks)[0], "float16")


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_sequences_at_once(dtype):
    """More rows than one pass of the weight-streaming products takes, and than they serve."""
    model, t = make(ODD, dtype)
    for B in (40, 150):
        toks = [tokens(ODD, 14, seed=r) for r in range(B)]
        model.prompt(torch.tensor([x[:9] for x in toks], device="cuda"), reserve=8)
        got = torch.stack([model.step(torch.tensor([x[k] for x in toks], device="cuda")) for k in range(9, 14)], 1)
        some = sorted({0, 1, 7, 8, 15, 16, 31, 32, 33, B - 1, *range(2, B, 5)})
        check(got[some].flatten(0, 1), torch.cat([P.forward(ODD, t, toks[r])[0][9:] for r in some]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_and_caches_are_used_again(dtype):
    """Later batches in the memory of earlier ones, of other content and length."""
    model, t = make(ODD, dtype)
    a, b = tokens(ODD, 150, seed=1), tokens(ODD, 50, seed=2)
    for toks in (a, b, a[:7], b):
        want, _ = P.forward(ODD, t, toks)
        got = [prompt_logits(model, toks[:5])] + [model.step(torch.tensor([x], device="cuda")) for x in toks[5:]]
        check(torch.cat(got), want, dtype)


def loud(t):
    """Token 7 gets keys that stand out, token 8 queries that ask for them; sinks leave them room, and the recurrences
    hold on to what they have."""
    W = t["embed"].shape[1]
    g = torch.Generator().manual_seed(99)
    key, ask = torch.randn(W, generator=g) * 1.5, torch.randn(W, generator=g) * 1.5
    t["embed"][7], t["embed"][8] = key.bfloat16(), ask.bfloat16()
    key, ask = key / key.norm(), ask / ask.norm()
    for name in [k for k in t if k.endswith("left.k") or k.endswith("right.k")]:
        q, k = t[name[:-1] + "q"].float(), t[name].float()
        k += torch.outer(torch.randn(k.shape[0], generator=g), key)
        rows = min(q.shape[0], k.shape[0])
        q[:rows] += 2.0 * torch.outer(k[:rows] @ key, ask)
        t[name[:-1] + "q"], t[name] = q.bfloat16(), k.bfloat16()
    for name in [k for k in t if k.endswith("a2.b")]:
        t[name] += 4.0
    for name in [k for k in t if k.endswith("A_log")]:
        t[name] -= 1.5
    for name in [k for k in t if k.endswith("left.sink")]:
        t[name] -= 1.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,at,ask", [("wide", 0, 600), ("wide", 1, 128), ("wide", 127, 600), ("wide", 128, 600), ("wide", 255, 256), ("wide", 511, 600),
                                         ("wide", 130, 259), ("wide", 129, 130), ("wide", 64, 127), ("wide", 63, 64), ("odd", 9, 17), ("odd", 8, 9), ("odd", 0, 33),
                                         ("odd", 33, 65), ("odd", 32, 33)])
def test_a_key_far_back_and_at_the_edges_of_chunks(name, at, ask, dtype):
    """In prompts and in decoding: far keys, the first of a chunk from its last position, the last of the chunk before
    from its first."""
    cfg = CONFIGS[name]
    model, t = make(cfg, dtype, change=loud)
    n = ask + 1
    toks = [x if x not in (7, 8) else 9 for x in tokens(cfg, n, seed=3)]
    toks[at], toks[ask] = 7, 8
    want, _ = P.forward(cfg, t, toks)
    without = list(toks)
    without[at] = 9
    moved = float((P.forward(cfg, t, without)[0][-1] - want[-1]).std() / want[-1].std())
    assert moved > (1e-3 if dtype == "float32" else 0.0), moved                     # the far token does show
    check(prompt_logits(model, toks), want, dtype)
    few = min(3, n - 1)
    got = prompt_logits(model, toks[:-few])
    for x in toks[-few:]:
        got = model.step(torch.tensor([x], device="cuda"))
    check(got, want[-1:], dtype)


def test_chunks_are_counted_from_the_first_token_of_each_sequence():
    """Left padding moves no chunk: sequences of every offset in one batch, decoded over a chunk's end."""
    model, t = make(ODD, "float32", change=loud)
    lens, more = list(range(4, 22)), 16
    S = max(lens)
    toks = [tokens(ODD, n + more, seed=n) for n in lens]
    ids, mask = torch.zeros(len(lens), S, dtype=torch.long), torch.zeros(len(lens), S, dtype=torch.long)
    for r, n in enumerate(lens):
        ids[r, S - n:], mask[r, S - n:] = torch.tensor(toks[r][:n]), 1
    x = model.prompt(ids.cuda(), mask, reserve=more).view(len(lens), S, -1)
    got = [[model.logits(x[r, S - n:].contiguous())] for r, n in enumerate(lens)]
    for k in range(more):
        lg = model.step(torch.tensor([s[n + k] for s, n in zip(toks, lens)], device="cuda"))
        for r in range(len(lens)):
            got[r].append(lg[r:r + 1])
    for r in range(len(lens)):
        check(torch.cat(got[r]), P.forward(ODD, t, toks[r])[0], "float32")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("cfg", [ODD, HUGE])
def test_greedy_generation_eager_and_replayed(cfg, dtype):
    model, t = make(cfg, dtype, seed=4)
    prompts = [tokens(cfg, n, seed=n) for n in (4, 21, 13)]
    new, S = 60, 21
    ids = torch.zeros(3, S, dtype=torch.long)
    mask = torch.zeros_like(ids)
    for r, p in enumerate(prompts):
        ids[r, S - len(p):], mask[r, S - len(p):] = torch.tensor(p), 1
    call = lambda: model(input_ids=ids.cuda(), attention_mask=mask.cuda(), max_tokens=S + new, top_k=1)
    first = call()
    assert model._decode_state["graph"] is not None and first.shape == (3, S + new)
    again = call()                                       # the captured step and the state serve a second call
    model.use_cuda_graph = False
    eager = call()
    assert torch.equal(first, again) and torch.equal(first, eager)
    if dtype == "float32":
        for r, p in enumerate(prompts):
            want, gap = P.greedy(cfg, t, p, new)
            assert gap > 1e-5 and first[r, S - len(p):].tolist() == want
    assert model.state.length == S + new - 1
    short = model(input_ids=ids.cuda(), attention_mask=mask.cuda(), top_k=1)
    assert torch.equal(short, first[:, S])               # without max_tokens: the next token


def test_a_sequence_goes_on_behind_a_generation():
    """The state a replayed generation leaves, the previous token among it, is that of its tokens."""
    model, t = make(ODD, "float32", seed=4)
    toks = tokens(ODD, 10)
    out = model(input_ids=torch.tensor([toks], device="cuda"), max_tokens=30, top_k=1)[0].tolist()
    got = model.step(torch.tensor([out[-1]], device="cuda"))
    check(got, P.forward(ODD, t, out)[0][-1:], "float32")


def test_sampling_stays_within_top_k():
    model, t = make(ODD, "float32")
    toks = tokens(ODD, 10)
    torch.manual_seed(0)
    out = model(input_ids=torch.tensor([toks] * 4, device="cuda"), max_tokens=22, top_k=3, temperature=0.8)
    assert out.shape == (4, 22)
    for row in out.tolist():
        lg, _ = P.forward(ODD, t, row)
        for k in range(10, 22):
            assert row[k] in lg[k - 1].topk(3).indices.tolist()


def test_padding_shifts_no_position():
    """A left-padded prompt and the same without padding: chunks, rotations, bigram rows and states count from the
    first token."""
    model, _ = make(ODD, "float32")
    ids = torch.tensor([tokens(ODD, 12)], device="cuda")
    mask = torch.ones_like(ids)
    mask[0, :4] = 0
    padded = model(input_ids=ids, attention_mask=mask, max_tokens=30, top_k=1)
    plain = model(input_ids=ids[:, 4:], max_tokens=26, top_k=1)
    assert torch.equal(padded[:, 4:], plain)


def save(folder, cfg, seed):
    t = P.make_tensors(cfg, seed)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(P.file_config(cfg), f)
    T.save_safetensors(os.path.join(folder, "model.safetensors"), t)
    return t


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner(tmp_path, dtype):
    t = save(str(tmp_path / "m"), ODD, 6)
    a, b, c = tokens(ODD, 140, seed=1), tokens(ODD, 18, seed=2), tokens(ODD, 6, seed=3)
    steps = [dict(entries=[dict(id="p", tokens=a[:135], want=[0, 134]), dict(id="q", tokens=b[:9], want=[8])], end=[])]
    want = [[(a, 0), (a, 134), (b, 8)]]
    for k in range(5):
        steps.append(dict(entries=[dict(id="q", tokens=[b[9 + k]], want=[0]), dict(id="p", tokens=[a[135 + k]], want=[0] if k != 2 else [])],
                          end=["p"] if k == 4 else []))
        want.append([(b, 9 + k)] + ([(a, 135 + k)] if k != 2 else []))
    steps.append(dict(entries=[dict(id="q", tokens=[b[14]], want=[])], end=["q"]))
    want.append([])
    steps.append(dict(entries=[dict(id="p", tokens=c, want=[5])], end=["p"]))
    want.append([(c, 5)])
    out = tmp_path / "out"
    out.mkdir()
    text = "".join(json.dumps(dict(s, step=i)) + "\n" for i, s in enumerate(steps))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "200"], input=text, capture_output=True, text=True, timeout=200)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [ln for ln in r.stdout.splitlines() if ln.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    logits = {id(x): P.forward(ODD, t, x)[0] for x in (a, b, c)}
    got, ref = [], []
    for i, w in enumerate(want):
        path = out / f"{i}.f32"
        assert path.exists() == bool(w)
        if w:
            got.append(torch.frombuffer(bytearray(path.read_bytes()), dtype=torch.float32).view(len(w), ODD["vocab"]))
            ref += [logits[id(x)][k] for x, k in w]
    check(torch.cat(got), torch.stack(ref), dtype)


def test_part_of_a_batch_goes_on_by_itself():
    """Trace sessions split a batch; both halves keep their own state, the previous token among it."""
    from energonai_b200.trace import TraceSession
    model, t = make(ODD, "float32")
    a, b = tokens(ODD, 40, seed=1), tokens(ODD, 30, seed=2)
    s = TraceSession(model, torch.device("cuda"))
    run = lambda entries: s.run([dict(id=i, tokens=x, want=[len(x) - 1]) for i, x in entries])
    la, lb = P.forward(ODD, t, a)[0], P.forward(ODD, t, b)[0]
    check(run([("a", a[:20]), ("b", b[:10])]), torch.stack([la[19], lb[9]]), "float32")
    for k in range(3):
        check(run([("a", [a[20 + k]])]), la[20 + k:21 + k], "float32")
    for k in range(5):
        check(run([("b", [b[10 + k]])]), lb[10 + k:11 + k], "float32")
    check(run([("b", [b[15]]), ("a", [a[23]])]), torch.stack([lb[15], la[23]]), "float32")


def test_engine_serves_the_design(tmp_path):
    """launch_engine + BatchManagerForGeneration: requests of several lengths, batched by the scheduler."""
    save(str(tmp_path), ODD, 4)
    env = dict(os.environ, PYTHONPATH=ROOT + os.pathsep + os.path.join(ROOT, "tests"), MASTER_ADDR="127.0.0.1")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "tests", "engine_check_moponex_gpu.py"), str(tmp_path)], cwd=ROOT, env=env,
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and "engine moponex ok" in r.stdout, r.stdout[-2000:] + r.stderr[-4000:]


def test_no_wait_ran_out():
    from energonai_b200.gemm import device_status
    assert device_status()[0] == 0
