"""The latent-attention decoder as a whole on the GPU against the plain restatement: prompts, decoding
through the ring caches, batches, memory that is used again, generation through the framework's own
entry points, the trace runner."""
import json
import os
import subprocess
import sys

import pytest
import torch

import tulezen_plain as P

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
DTYPES = {"float32": torch.float32, "bfloat16": torch.bfloat16}

# odd sizes, unequal windows and head sizes, a layer without feed-forward, latents shared with a wider
# window than their own layer's, a single expert that is always chosen
ODD = P.make_config([dict(heads=3, dim=20, vdim=28, rank=40, window=9, scale=0.3, moe=(5, 2, 12, 0.7)),
                     dict(heads=2, dim=8, vdim=8, rank=24, window=33, scale=0.5, moe=None),
                     dict(heads=5, dim=12, vdim=4, rank=40, window=70, scale=0.2, kv_from=0, moe=(1, 1, 20, 1.5)),
                     dict(heads=1, dim=64, vdim=40, rank=24, window=1, scale=0.2, kv_from=1, moe=(9, 9, 8, 0.4))], width=76, vocab=101)
# tensor-core sizes, a long window
WIDE = P.make_config([dict(heads=18, dim=128, vdim=96, rank=200, window=150, scale=0.09, moe=(16, 4, 64, 1.0)),
                      dict(heads=4, dim=100, vdim=128, rank=200, window=64, scale=0.1, kv_from=0, moe=(3, 1, 136, 2.0))], width=192, vocab=333)
# sizes the tensor-core kernels do not have
HUGE = P.make_config([dict(heads=2, dim=136, vdim=16, rank=520, window=40, scale=0.08, moe=(4, 2, 16, 1.0))], width=64, vocab=64)
CONFIGS = {"odd": ODD, "wide": WIDE, "huge": HUGE}


def make(cfg, dtype, seed=1):
    from energonai_b200.registry import build_model
    from energonai_b200.utils import processing_Tulezen
    tensors = P.make_tensors(cfg, seed)
    model = build_model("Tulezen", config_dict=cfg, dtype=DTYPES[dtype])
    model.load_state_dict(processing_Tulezen(tensors, model))
    return model.cuda().eval(), tensors


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def check(got, want, dtype):
    """Row by row.  In 32-bit every row has to fit; in bfloat16 a row in which two experts' scores are
    closer than the rounding may choose another expert than the exact arithmetic does."""
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all()
    err = (got - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
    if dtype == "float32":
        assert float(err.max()) < 2e-5, err
    else:
        assert float(err.median()) < 0.03 and float(err.quantile(0.85)) < 0.1, err.sort().values


def prompt_logits(model, toks):
    x = model.prompt(torch.tensor([toks], device="cuda"), reserve=4)
    return model.logits(x)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,n", [("odd", 1), ("odd", 2), ("odd", 40), ("odd", 150), ("wide", 100), ("wide", 300), ("huge", 70)])
def test_prompt(name, n, dtype):
    cfg = CONFIGS[name]
    model, t = make(cfg, dtype)
    toks = tokens(cfg, n)
    seen = []
    x = model.prompt(torch.tensor([toks], device="cuda"), on_layer=lambda i, s: seen.append(s.clone()))
    want, streams = P.forward(cfg, t, toks)
    check(model.logits(x), want, dtype)
    assert len(seen) == len(streams)
    for a, b in zip(seen, streams):
        check(a[:, :cfg["width"]], b, dtype)
        assert a.dtype == torch.float32 and float(a[:, cfg["width"]:].abs().sum()) == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,start,n", [("odd", 1, 170), ("odd", 8, 40), ("odd", 33, 60), ("wide", 2, 20), ("wide", 149, 170), ("huge", 38, 60)])
def test_decoding_token_by_token(name, start, n, dtype):
    """From prompts shorter and longer than the windows, through several turns of the rings."""
    cfg = CONFIGS[name]
    model, t = make(cfg, dtype)
    toks = tokens(cfg, n)
    want, _ = P.forward(cfg, t, toks)
    got = [prompt_logits(model, toks[:start])]
    for k in range(start, n):
        got.append(model.step(torch.tensor([toks[k]], device="cuda")))
    check(torch.cat(got), want, dtype)
    check(prompt_logits(model, toks), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name,lens", [("odd", (1, 37, 12, 90)), ("wide", (3, 160)), ("odd", (70, 71, 69))])
def test_unequal_batch_against_each_alone(name, lens, dtype):
    cfg = CONFIGS[name]
    model, t = make(cfg, dtype)
    more, S = 20, max(lens)
    toks = [tokens(cfg, n + more, seed=n) for n in lens]
    ids = torch.zeros(len(lens), S, dtype=torch.long)
    mask = torch.zeros_like(ids)
    for r, n in enumerate(lens):
        ids[r, S - n:], mask[r, S - n:] = torch.tensor(toks[r][:n]), 1
    x = model.prompt(ids.cuda(), mask, reserve=2).view(len(lens), S, -1)
    got = [[model.logits(x[r, S - n:].contiguous())] for r, n in enumerate(lens)]
    live = list(range(len(lens)))
    for k in range(more):
        if k == 8:                                       # one request ends, its memory goes
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


def test_caches_are_used_again():
    """A second batch in the same memory, after the rings have turned, shorter and of another content."""
    model, t = make(ODD, "float32")
    a, b = tokens(ODD, 120, seed=1), tokens(ODD, 50, seed=2)
    for toks in (a, b, a[:7], b):
        want, _ = P.forward(ODD, t, toks)
        got = [prompt_logits(model, toks[:5])] + [model.step(torch.tensor([x], device="cuda")) for x in toks[5:]]
        check(torch.cat(got), want, "float32")


@pytest.mark.parametrize("dtype", DTYPES)
def test_greedy_generation_eager_and_replayed(dtype):
    cfg = CONFIGS["odd"]
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
    again = call()                                       # the captured step and the caches serve a second call
    model.use_cuda_graph = False
    eager = call()
    assert torch.equal(first, again) and torch.equal(first, eager)
    if dtype == "float32":
        for r, p in enumerate(prompts):
            want, gap = P.greedy(cfg, t, p, new)
            assert gap > 1e-4 and first[r, S - len(p):].tolist() == want
    assert model.state.length == S + new - 1
    short = model(input_ids=ids.cuda(), attention_mask=mask.cuda(), top_k=1)
    assert torch.equal(short, first[:, S])               # without max_tokens: the next token


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


def test_model_without_padding_after_one_with_padding():
    model, _ = make(ODD, "float32")
    ids = torch.tensor([tokens(ODD, 12)], device="cuda")
    mask = torch.ones_like(ids)
    mask[0, :4] = 0
    padded = model(input_ids=ids, attention_mask=mask, max_tokens=30, top_k=1)
    plain = model(input_ids=ids[:, 4:], max_tokens=26, top_k=1)
    assert torch.equal(padded[:, 4:], plain)
    full = model(input_ids=ids, max_tokens=30, top_k=1)
    model.use_cuda_graph = False
    assert torch.equal(full, model(input_ids=ids, max_tokens=30, top_k=1))


def save(folder, cfg, seed):
    t = P.make_tensors(cfg, seed)
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    P.save_safetensors(os.path.join(folder, "model.safetensors"), t)
    return t


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_runner(tmp_path, dtype):
    t = save(str(tmp_path / "m"), ODD, 6)
    a, b, c = tokens(ODD, 30, seed=1), tokens(ODD, 18, seed=2), tokens(ODD, 6, seed=3)
    steps = [dict(entries=[dict(id="p", tokens=a[:25], want=[0, 24]), dict(id="q", tokens=b[:9], want=[8])], end=[])]
    want = [[(a, 0), (a, 24), (b, 8)]]
    for k in range(5):
        steps.append(dict(entries=[dict(id="q", tokens=[b[9 + k]], want=[0]), dict(id="p", tokens=[a[25 + k]], want=[0] if k != 2 else [])],
                          end=["p"] if k == 4 else []))
        want.append([(b, 9 + k)] + ([(a, 25 + k)] if k != 2 else []))
    steps.append(dict(entries=[dict(id="q", tokens=[b[14]], want=[])], end=["q"]))
    want.append([])
    steps.append(dict(entries=[dict(id="p", tokens=c, want=[5])], end=["p"]))
    want.append([(c, 5)])
    out = tmp_path / "out"
    out.mkdir()
    text = "".join(json.dumps(dict(s, step=i)) + "\n" for i, s in enumerate(steps))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out),
                        "--max-tokens", "64"], input=text, capture_output=True, text=True, timeout=200)
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


def test_engine_serves_the_design(tmp_path):
    """launch_engine + BatchManagerForGeneration: requests of several lengths, batched by the scheduler."""
    save(str(tmp_path), ODD, 4)
    env = dict(os.environ, PYTHONPATH=ROOT + os.pathsep + os.path.join(ROOT, "tests"), MASTER_ADDR="127.0.0.1")
    r = subprocess.run([sys.executable, os.path.join(ROOT, "tests", "engine_check_tulezen_gpu.py"), str(tmp_path)], cwd=ROOT, env=env,
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0 and "engine tulezen ok" in r.stdout, r.stdout[-2000:] + r.stderr[-4000:]


def test_no_wait_ran_out():
    from energonai_b200.gemm import device_status
    assert device_status()[0] == 0
