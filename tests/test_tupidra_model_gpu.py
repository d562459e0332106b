"""The latent-attention / selective-scan / capped-attention decoder as a whole on the GPU against the plain restatement:
prompts, decoding, unequal batches, memory used again, far keys and the edges of windows, first tokens, generation
through the framework's own entry points, the trace runner, the engine."""
import json
import os
import subprocess
import sys

import pytest
import torch

import tulezen_plain as T
import tupidra_plain as P

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}

# odd sizes; groups of heads and one key head per query head; with and without window, kept positions, cap, slowed
# rotation and feed-forward; value heads larger and smaller than key heads; latents of another layer; taps of one
ODD = P.make_config([P.scan_layer(44, 6, 5, 3, P.dense_mlp(44)), P.attention_layer(6, 2, 12, 20, 0.3, 4.0, (9, 3), P.dense_mlp(36)),
                     P.latent_layer(3, 12, 6, 10, 20, 18, 0.25, 100.0, (4.0, 30, 4.0, 0.5)), P.attention_layer(2, 2, 9, 9, 0.3),
                     P.latent_layer(5, 20, 6, 24, 12, 18, 0.2, 100.0, (4.0, 30, 4.0, 0.5), kv_from=2, mlp=P.dense_mlp(20)), P.scan_layer(24, 20, 9, 1)],
                    width=52, vocab=83, taps=3)
# sizes that fill or exceed the tensor-core tiles; more than 16 heads on one latent or key head; more kept positions than the window has
WIDE = P.make_config([P.attention_layer(20, 1, 64, 64, 0.12, 30.0, (130, 5), P.dense_mlp(136)),
                      P.latent_layer(18, 100, 28, 128, 200, 228, 0.09, 20000.0, (8.0, 64, 16.0, 1.0), mlp=P.dense_mlp(64)), P.scan_layer(200, 16, 24, 4, P.dense_mlp(72)),
                      P.latent_layer(4, 40, 28, 60, 64, 228, 0.12, 20000.0, (8.0, 64, 16.0, 1.0), kv_from=1), P.attention_layer(4, 2, 100, 80, 0.1, 50.0, (64, 70)),
                      P.scan_layer(136, 40, 16, 2)], width=192, vocab=334, eps=1e-6)
# sizes the tensor-core kernels do not have, and the smallest ones
HUGE = P.make_config([P.latent_layer(2, 120, 20, 140, 9, 500, 0.1, 1000.0), P.attention_layer(2, 1, 140, 20, 0.08, 2.0, (20, 1), P.dense_mlp(24)), P.scan_layer(8, 130, 1, 5),
                      P.attention_layer(1, 1, 2, 3, 1.0, 1.0, (1, 0)), P.scan_layer(3, 1, 2, 2, P.dense_mlp(8)), P.latent_layer(1, 1, 2, 4, 2, 3, 1.0, 10.0)],
                     width=40, vocab=64, taps=1)
# large heads and latents on the tensor cores; those kernels for the prompt or for the steps only; latents from far below
MIXED = P.make_config([P.latent_layer(3, 130, 62, 100, 24, 512, 0.09, 500.0, mlp=P.dense_mlp(40)), P.latent_layer(2, 40, 8, 32, 16, 580, 0.14, 900.0, (2.0, 50, 8.0, 1.0)),
                       P.attention_layer(3, 3, 30, 70, 0.2, 9.0, (50, 0)), P.latent_layer(20, 24, 62, 40, 20, 512, 0.16, 500.0, kv_from=0, mlp=P.dense_mlp(24)),
                       P.latent_layer(1, 200, 8, 32, 16, 580, 0.1, 900.0, (2.0, 50, 8.0, 1.0), kv_from=1), P.latent_layer(2, 150, 6, 50, 8, 40, 0.1, 80.0)],
                      width=80, vocab=101, taps=2)
CONFIGS = {"odd": ODD, "wide": WIDE, "huge": HUGE, "mixed": MIXED}


def make(cfg, dtype, seed=1, change=None):
    from energonai_b200.registry import build_model
    from energonai_b200.utils import processing_Tupidra
    tensors = P.make_tensors(cfg, seed)
    if change:
        change(tensors)
    model = build_model("Tupidra", config_dict=cfg, dtype=DTYPES.get(dtype, torch.float16))
    model.load_state_dict(processing_Tupidra(tensors, model))
    return model.cuda().eval(), tensors


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def check(got, want, dtype):
    """Row by row, the mean over the vocabulary taken off; a row in ten, or one, may be further off (a norm of few numbers
    that are near zero is badly conditioned)."""
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all()
    d = got - want
    err = ((d - d.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt() / want.std(-1).mean()).sort().values
    most, worst, typical = (3e-5, 2e-4, 1e-5) if dtype == "float32" else (0.08, 0.3, 0.03)
    n = err.numel()
    assert float(err[-1]) < worst and float(err[n // 2]) < (typical if n > 2 else worst), err
    assert float(err[n - 1 - max(1, n // 10)] if n > 2 else err[0]) < most, err


def prompt_logits(model, toks):
    return model.logits(model.prompt(torch.tensor([toks], device="cuda"), reserve=4))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,n", [("odd", 1), ("odd", 2), ("odd", 129), ("odd", 300), ("wide", 127), ("wide", 400), ("huge", 70), ("mixed", 300)])
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
@pytest.mark.parametrize("name,start,n", [("odd", 1, 200), ("odd", 127, 140), ("odd", 128, 140), ("wide", 2, 20), ("wide", 125, 150), ("wide", 250, 280), ("huge", 38, 60), ("mixed", 140, 170)])
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


def left_padded(toks):
    S = max(map(len, toks))
    ids, mask = torch.zeros(len(toks), S, dtype=torch.long), torch.zeros(len(toks), S, dtype=torch.long)
    for r, x in enumerate(toks):
        ids[r, S - len(x):], mask[r, S - len(x):] = torch.tensor(x), 1
    return ids, mask


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,lens", [("odd", (1, 37, 12, 190)), ("wide", (3, 260)), ("odd", (70, 71, 69)), ("wide", (1, 1, 2)), ("huge", (2, 30, 1))])
def test_unequal_batch_against_each_alone(name, lens, dtype):
    cfg = CONFIGS[name]
    model, t = make(cfg, dtype)
    more, S = 20, max(lens)
    toks = [tokens(cfg, n + more, seed=n + r) for r, n in enumerate(lens)]
    ids, mask = left_padded([x[:n] for x, n in zip(toks, lens)])
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
    model, t = make(ODD, "float16")
    toks = tokens(ODD, 60)
    got = [prompt_logits(model, toks[:40])] + [model.step(torch.tensor([x], device="cuda")) for x in toks[40:]]
    check(torch.cat(got), P.forward(ODD, t, toks)[0], "float16")


@pytest.mark.parametrize("dtype", DTYPES)
def test_many_sequences_at_once(dtype):
    """More rows than the weight-streaming products serve, several sequences per CTA of the scan's step."""
    model, t = make(ODD, dtype)
    for B in (40, 150):
        toks = [tokens(ODD, 14, seed=r) for r in range(B)]
        model.prompt(torch.tensor([x[:9] for x in toks], device="cuda"), reserve=8)
        got = torch.stack([model.step(torch.tensor([x[k] for x in toks], device="cuda")) for k in range(9, 14)], 1)
        some = sorted({0, 1, 7, 8, 15, 16, 31, 32, 33, B - 1, *range(2, B, 9)})
        check(got[some].flatten(0, 1), torch.cat([P.forward(ODD, t, toks[r])[0][9:] for r in some]), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_state_and_caches_are_used_again(dtype):
    """Later batches in the memory of earlier ones, of other content and length."""
    model, t = make(ODD, dtype)
    a, b = tokens(ODD, 100, seed=1), tokens(ODD, 40, seed=2)
    for toks in (a, b, a[:7], b):
        want, _ = P.forward(ODD, t, toks)
        got = [prompt_logits(model, toks[:5])] + [model.step(torch.tensor([x], device="cuda")) for x in toks[5:]]
        check(torch.cat(got), want, dtype)


def loud(t):
    """Token 7 gets keys that stand out, token 8 queries that ask for them; the recurrences hold on to what they have."""
    W = t["embed"].shape[1]
    g = torch.Generator().manual_seed(99)
    key, ask = torch.randn(W, generator=g) * 1.5, torch.randn(W, generator=g) * 1.5
    t["embed"][7], t["embed"][8] = key.bfloat16(), ask.bfloat16()
    key, ask = key / key.norm(), ask / ask.norm()
    for name in [k for k in t if k.endswith("mix.k")]:
        q, k = t[name[:-1] + "q"].float(), t[name].float()
        k += torch.outer(torch.randn(k.shape[0], generator=g), key)
        share = k.repeat(q.shape[0] // k.shape[0] + 1, 1)[:q.shape[0]]
        q += torch.outer(share @ key, ask)
        t[name[:-1] + "q"], t[name] = q.bfloat16(), k.bfloat16()
    source = None
    for name in [k for k in t if k.endswith("mix.uk")]:
        p = name[:-2]
        if p + "dkv" in t:
            source = torch.zeros(t[p + "dkv"].shape[0])
            source[:t[name].shape[1]] = torch.randn(t[name].shape[1], generator=g)
            t[p + "dkv"] = (t[p + "dkv"].float() + torch.outer(source, key)).bfloat16()
        asks = torch.randn(t[p + "dq"].shape[0], generator=g)
        t[p + "dq"] = (t[p + "dq"].float() + torch.outer(asks, ask)).bfloat16()
        H = t[p + "sink"].shape[0]
        uq, uk = t[p + "uq"].float().view(H, -1, t[p + "uq"].shape[1]), t[name].float().view(H, -1, t[name].shape[1])
        toward = uk @ source[:uk.shape[2]]
        uq[:, :uk.shape[1]] += toward[:, :, None] * (asks / asks.norm() ** 2)[None, None]
        t[p + "uq"] = uq.view(-1, uq.shape[2]).bfloat16()
    for name in [k for k in t if k.endswith("A_log")]:
        t[name] -= 1.0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,at,ask", [("wide", 0, 500), ("wide", 4, 300), ("wide", 5, 300), ("wide", 127, 256), ("wide", 128, 257), ("wide", 255, 256), ("wide", 130, 259),
                                         ("wide", 129, 259), ("odd", 0, 33), ("odd", 2, 40), ("odd", 3, 40), ("odd", 20, 28), ("odd", 20, 29), ("odd", 32, 33)])
def test_a_key_far_back_and_at_the_edges(name, at, ask, dtype):
    """In prompts and in decoding: far keys, kept positions and the first one that is not, just inside and outside windows."""
    cfg = CONFIGS[name]
    model, t = make(cfg, dtype, change=loud)
    n = ask + 1
    toks = [x if x not in (7, 8) else 9 for x in tokens(cfg, n, seed=3)]
    toks[at], toks[ask] = 7, 8
    want, _ = P.forward(cfg, t, toks)
    without = list(toks)
    without[at] = 9
    moved = float((P.forward(cfg, t, without)[0][-1] - want[-1]).std() / want[-1].std())
    assert moved > 1e-2, moved                           # the far token does show
    check(prompt_logits(model, toks), want, dtype)
    few = min(3, n - 1)
    got = prompt_logits(model, toks[:-few])
    for x in toks[-few:]:
        got = model.step(torch.tensor([x], device="cuda"))
    check(got, want[-1:], dtype)


EDGE_CASES = [(40, 3), (130, 1), (128, 140), (64, 0)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("size,keep", EDGE_CASES)
def test_every_edge_of_a_window_alone(size, keep, dtype):
    """One attention layer and nothing else that looks back further than two tokens: a token moves the last logits exactly when
    the window or the kept positions have it, and the values are those of the restatement."""
    cfg = P.make_config([P.attention_layer(3, 1, 24, 16, 0.5, 6.0, (size, keep))], width=48, vocab=50, taps=2)
    model, t = make(cfg, dtype, change=loud)
    for n in (size + 2, size + keep + 5, 2 * size + keep + 70):
        last = n - 1
        ats = {last - size + 2, last - size + 1, last - size, last - size - 1, 0, keep - 1, keep, keep + 1}
        for at in sorted(a for a in ats if 0 <= a < last - 4):
            toks = [9 if x in (7, 8) else x for x in tokens(cfg, n, seed=n)]
            toks[last] = 8
            base = P.forward(cfg, t, toks)[0][-1]
            toks[at] = 7
            want = P.forward(cfg, t, toks)[0]
            reach = [last - j < size or j < keep for j in (at, at + 1)]             # (the convolution carries it one token on)
            moved = float((want[-1] - base).std() / base.std())
            assert (moved > 0) == any(reach) and (moved > 1e-5 or not reach[0]), (n, at, moved)
            check(prompt_logits(model, toks)[-1:], want[-1:], dtype)
            prompt_logits(model, toks[:-2])
            for x in toks[-2:]:
                got = model.step(torch.tensor([x], device="cuda"))
            check(got, want[-1:], dtype)


def test_positions_count_from_the_first_token_of_each_sequence():
    """Left padding moves no window, kept position, angle or state: sequences of every offset in one batch, decoded over
    a window's end."""
    model, t = make(ODD, "float32", change=loud)
    lens, more = list(range(1, 18)), 16
    S = max(lens)
    toks = [tokens(ODD, n + more, seed=n) for n in lens]
    ids, mask = left_padded([x[:n] for x, n in zip(toks, lens)])
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
    new, S = 40, 21
    ids, mask = left_padded(prompts)
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
    """The state a replayed generation leaves is that of its tokens."""
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


def save(folder, cfg, seed):
    t = P.make_tensors(cfg, seed)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
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
    """Trace sessions split a batch; both halves keep their own state."""
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
    r = subprocess.run([sys.executable, os.path.join(ROOT, "tests", "engine_check_tupidra_gpu.py"), str(tmp_path)], cwd=ROOT, env=env,
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and "engine tupidra ok" in r.stdout, r.stdout[-2000:] + r.stderr[-4000:]


def test_no_wait_ran_out():
    from energonai_b200.gemm import device_status
    assert device_status()[0] == 0
