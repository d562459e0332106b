"""Throughput of the layer-listed decoders (latent attention / mixture of experts, matrix memory / grouped
attention, state space / chunk attention beside gated linear attention, selective state space / capped attention /
rotary latent attention beside dense feed-forwards) at sizes that resemble a real model's
layers (random weights), beside an OPT-shaped PipelineModel of equal width, heads, depth and weights per
token, and the time of every kernel next to its roofline and to the like kernel of another model.
`bench.py --design tulezen | mutolix | moponex | tupidra` prints the result as one JSON line."""
import json
import os
import statistics
import time

import torch

SIZES = {
    # window, kv_rank, experts ... of a layer; every second layer takes its latents from the one before
    "2048": dict(width=2048, heads=16, dim=128, kv_rank=512, window=1024, experts=64, top=6, ff=1408, layers=8, vocab=32768),
    "4096": dict(width=4096, heads=32, dim=128, kv_rank=512, window=4096, experts=32, top=4, ff=2048, layers=6, vocab=32768),
}
RUNS = [  # (size, batch, prompt, new tokens)
    ("2048", 8, 1024, 64), ("2048", 64, 1024, 64), ("4096", 16, 512, 64), ("4096", 2, 4096, 64),
]
FLUSH_BYTES = 400 << 20      # a timed kernel cycles through operand copies of at least this size


def peaks():
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    d = json.load(open(path)) if os.path.exists(path) else {}
    # sfu: special-function results per second, 16 per clock on each of 148 SMs at 1.965 GHz (nominal)
    return {"hbm": d.get("hbm_gbs", 6650.0) * 1e9, "tensor": d.get("bf16_tflops", 1590.0) * 1e12, "sfu": 16 * 148 * 1.965e9,
            "kind": "measured" if d else "fallback"}


def make_tulezen(z):
    from ..registry import build_model
    layer = {"type": "latent_attention",
             "mixer": {"heads": z["heads"], "dim": z["dim"], "vdim": z["dim"], "kv_rank": z["kv_rank"], "mask": {"size": z["window"]},
                       "scale": z["dim"] ** -0.5},
             "mlp": {"kind": "moe", "router": {"experts": z["experts"], "top": z["top"]}, "expert": {"ff": z["ff"], "limit": 7.0}}}
    layers = [dict(layer, mixer=dict(layer["mixer"], **({"kv_from": i - 1} if i % 2 else {}))) for i in range(z["layers"])]
    torch.manual_seed(1)
    return build_model("Tulezen", config_dict={"vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-5}, "layers": layers},
                       dtype=torch.bfloat16, device="cuda")


def make_opt(z, max_len):
    from ..model import create_pipeline_model
    torch.manual_seed(1)
    ffn = (z["top"] * z["ff"] * 3 // 2 + 7) // 8 * 8            # as many feed-forward weights per token
    with torch.device("cuda"):
        m = create_pipeline_model(depth=z["layers"], vocab_size=z["vocab"], hidden_size=z["width"], max_seq_len=max_len,
                                  num_heads=z["heads"], mlp_ratio=ffn / z["width"], activation=torch.nn.functional.relu,
                                  is_decoder=True, fused_qkv=True, dtype=torch.bfloat16)
    m.eos_token_id = -1
    return m.eval()


MUTOLIX_SIZES = {
    # alternating matrix-memory layers (no feed-forward) and attention layers (with one); m*: the memory's heads
    "2048": dict(width=2048, heads=16, kv_heads=4, dim=128, mheads=8, mdim=128, mvdim=256, ff=8192, layers=8, vocab=32768),
    "4096": dict(width=4096, heads=32, kv_heads=8, dim=128, mheads=16, mdim=128, mvdim=256, ff=16384, layers=6, vocab=32768),
}


def make_mutolix(z):
    from ..registry import build_model
    memory = {"type": "mlstm", "mixer": {"heads": z["mheads"], "dim": z["mdim"], "vdim": z["mvdim"], "gate_cap": 15.0}, "mlp": None}
    attention = {"type": "attention", "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"],
                                                "scale": z["dim"] ** -0.5, "q_temp": {"coef": 0.1, "every": 512}, "v_mix": True},
                 "mlp": {"kind": "dense", "ff": z["ff"]}}
    torch.manual_seed(1)
    return build_model("Mutolix", config_dict={"vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
                                               "layers": [memory, attention] * (z["layers"] // 2)}, dtype=torch.bfloat16, device="cuda")


def mutolix_as_opt(z):
    """The feed-forward size with which an OPT layer has as many weights as a layer here has on average."""
    w, h = z["width"], z["heads"] * z["dim"]
    memory = w * (2 * z["mheads"] * z["mdim"] + 3 * z["mheads"] * z["mvdim"] + w)
    attention = w * (2 * h + 2 * z["kv_heads"] * z["dim"] + 2 * w + 2 * z["ff"])
    ffn = ((memory + attention) / 2 / w - 4 * w) / 2
    return dict(z, top=1, ff=int(ffn / 1.5))


def timed_generation(model, vocab, B, S, new, reps=3):
    ids = torch.randint(0, vocab, (B, S), device="cuda")
    mask = torch.ones_like(ids)
    out = []
    for i in range(reps + 2):
        rec = {"allow_graph": True}
        model(input_ids=ids, attention_mask=mask, max_tokens=S + new, top_k=1, record=rec)
        torch.cuda.synchronize()
        if i >= 2:
            ev = rec["step_events"]
            steps = [a.elapsed_time(b) for a, b in zip(ev[3:-1], ev[4:])]
            out.append((ev[0].elapsed_time(ev[1]), statistics.median(steps)))
    pre, step = statistics.median(o[0] for o in out), statistics.median(o[1] for o in out)
    return {"prefill_ms": pre, "prefill_tokens_per_s": B * S / pre * 1e3, "step_ms": step, "decode_tokens_per_s": B / step * 1e3}


def time_calls(calls, reps=10):
    """Median time of one call, from replays of a graph that runs all of `calls` (operand copies that
    together exceed L2) back to back, at least eight of them."""
    calls = list(calls) * -(-8 // len(calls))
    for c in calls[:2]:
        c()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for c in calls:
            c()
    time.sleep(0.3)              # a kernel timed right behind a run of large products would find the clock lowered by the power cap
    ts = []
    for i in range(reps + 3):
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        g.replay()
        b.record()
        torch.cuda.synchronize()
        if i >= 3:
            ts.append(a.elapsed_time(b) * 1e3 / len(calls))
    return statistics.median(ts)


def copies(nbytes, most=64):
    return max(2, min(most, -(-FLUSH_BYTES // max(1, int(nbytes)))))


def kernel_table(z, B, S, T):
    """[(phase, kernel, like kernel or None, us, bytes, flops)] for batch B at S cached positions
    (generation step) and T prompt tokens in sequences of min(S, T)."""
    from ..attention import (attention_decode, attention_prefill, attention_prefill_window, latent_decode)
    from ..gemm import gemm
    from ..kernel.cuda_native.layer_norm import layer_norm_forward
    from ..moe import SortedRows, grouped_gemm, new_counts, per_head, route, skinny_experts
    from ..norm import rms_norm, rms_residual
    bf, dev = torch.bfloat16, "cuda"
    W, H, d, R, E, K, ff = z["width"], z["heads"], z["dim"], z["kv_rank"], z["experts"], z["top"], z["ff"]
    win = z["window"]
    keys = min(S, win)
    rnd = lambda *s, dtype=bf: (torch.randn(*s, device=dev, dtype=torch.float32) * 0.05).to(dtype)
    rows = []

    def add(phase, name, like, us, nbytes, flops=0.0):
        rows.append((phase, name, like, us, float(nbytes), float(flops)))

    def product(phase, name, M, N, Kd, like=None, out32=False):
        nb = 2 * (N * Kd + M * Kd) + (4 if out32 else 2) * M * N
        ws = [rnd(N, Kd) for _ in range(copies(2 * N * Kd, 32))]
        xs = [rnd(M, Kd) for _ in range(4)]
        us = time_calls([lambda w=w, x=xs[i % 4]: gemm(x, w, out_dtype=torch.float32 if out32 else None, static_weight=True)
                         for i, w in enumerate(ws)])
        add(phase, name, like, us, nb, 2.0 * M * N * Kd)

    # ---- generation step ----
    product("step", "gemm in_proj", B, H * d + R, W)
    product("step", "gemm out_proj", B, W, H * d)
    pos = torch.tensor([S - 1], dtype=torch.int32, device=dev)
    ring = [rnd(B, keys, R) for _ in range(copies(B * keys * R * 2))]
    q = rnd(B, H * R)
    add("step", "latent_decode", "attention_decode (OPT)", time_calls([lambda c=c: latent_decode(q, c, R, H, win, pos, 0.05) for c in ring]),
        2 * B * keys * R + 4 * B * H * R, 4.0 * B * H * keys * R)
    kv = [rnd(B, keys, 3 * H * d) for _ in range(copies(B * keys * 2 * H * d * 2))]
    add("step", "attention_decode (OPT)", None, time_calls([lambda c=c: attention_decode(
        c[:, :, 2 * H * d:], c[:, :, :H * d], c[:, :, H * d:2 * H * d], d, keys, q_in_cache=True) for c in kv]), 4 * B * keys * H * d)
    del kv
    w = rnd(R)
    x = rnd(B, R)
    add("step", "rms_norm to ring", "layer_norm (OPT)", time_calls([lambda c=c: rms_norm(x, w, 1e-5, write_out=False, ring=c, pos_device=pos)
                                                                    for c in ring]), 4 * B * R)
    del ring
    ups = [rnd(H, R, d) for _ in range(copies(H * R * d * 2, 48))]
    qh, o = rnd(B, H * d), rnd(B, H * R)
    add("step", "per_head key absorb", "gemm out_proj", time_calls([lambda w=w: per_head(qh, w) for w in ups]), 2 * (H * R * d + B * H * (R + d)))
    add("step", "per_head value up", "gemm out_proj", time_calls([lambda w=w: per_head(o, w.view(H, d, R)) for w in ups]),
        2 * (H * R * d + B * H * (R + d)))
    del ups
    xs, xt, y, nw = torch.randn(B, W, device=dev), rnd(B, W), rnd(B, W), rnd(W)
    routers = [rnd(E, W) for _ in range(16)]
    add("step", "rms_residual + router", "layer_norm (OPT)", time_calls([lambda r=r: rms_residual(y, nw, 1e-5, xs, xt=xt, offset=1.0, router=(r, E, K))
                                                                         for r in routers]), 12 * B * W + 2 * E * W)
    lw, lb = rnd(W), rnd(W)
    add("step", "layer_norm (OPT)", None, time_calls([lambda: layer_norm_forward(xt, lw, lb, 1e-5)] * 16), 4 * B * W)
    g = torch.Generator(device=dev).manual_seed(3)
    n_w = max(2, min(8, -(-FLUSH_BYTES // (6 * E * ff * W))))
    gu = [rnd(E, 2 * ff, W) for _ in range(n_w)]
    dn = [rnd(E, W, ff) for _ in range(n_w)]
    idx = torch.rand(B, E, device=dev, generator=g).topk(K, -1).indices.to(torch.int32)
    wts = torch.rand(B, K, device=dev)
    act_e = int(idx.unique().numel())
    a = rnd(B * K, ff)
    add("step", "experts gate_up", "gemm out_proj", time_calls([lambda w=w: skinny_experts(xt, w, idx, K, gate=(7.0, 1.702)) for w in gu]),
        2 * (act_e * 2 * ff * W + B * W + B * K * ff), 4.0 * B * K * ff * W)
    add("step", "experts down", "gemm out_proj", time_calls([lambda w=w: skinny_experts(a, w, idx, 1) for w in dn]),
        2 * (act_e * ff * W + B * K * (W + ff)), 2.0 * B * K * ff * W)
    ym = rnd(B * K, W)
    add("step", "rms_residual combine", "layer_norm (OPT)", time_calls([lambda: rms_residual(ym, nw, 1e-5, xs, xt=xt, offset=1.0, mix=(idx, None, wts))] * 16),
        10 * B * W + 2 * B * K * W)

    # ---- prompt ----
    seq = min(S, T)
    nB = T // seq
    product("prompt", "gemm in_proj", T, H * d + R, W)
    product("prompt", "gemm kv_up", T, 2 * H * d, R)
    product("prompt", "gemm out_proj", T, W, H * d)
    product("prompt", "gemm router", T, E, W, out32=True)
    q3, kv3 = rnd(nB, seq, H * d), rnd(nB, seq, 2 * H * d)
    n_c = 4
    pairs = sum(min(i + 1, win) for i in range(seq))
    add("prompt", "attention window", "attention causal (OPT)", time_calls([lambda: attention_prefill_window(q3, kv3[:, :, :H * d], kv3[:, :, H * d:], d, win)] * n_c),
        2 * T * 4 * H * d, 4.0 * nB * H * d * pairs)
    add("prompt", "attention causal (OPT)", None, time_calls([lambda: attention_prefill(q3, kv3[:, :, :H * d], kv3[:, :, H * d:], d)] * n_c),
        2 * T * 4 * H * d, 4.0 * nB * H * d * seq * (seq + 1) / 2)
    c = [rnd(T, R) for _ in range(copies(4 * T * R))]
    add("prompt", "rms_norm latent", "layer_norm (OPT)", time_calls([lambda t=t: rms_norm(t, w, 1e-5) for t in c]), 4 * T * R)
    del c
    xs = [torch.randn(T, W, device=dev) for _ in range(copies(12 * T * W, 8))]
    xts, ys = [rnd(T, W) for _ in xs], [rnd(T, W) for _ in xs]
    add("prompt", "rms_residual", "layer_norm (OPT)", time_calls([lambda x=x, t=t, y=y: rms_residual(y, nw, 1e-5, x, xt=t, offset=1.0)
                                                                  for x, t, y in zip(xs, xts, ys)]), 12 * T * W)
    add("prompt", "layer_norm (OPT)", None, time_calls([lambda t=t: layer_norm_forward(t, lw, lb, 1e-5) for t in xts + ys]), 4 * T * W)
    logits = torch.randn(T, E, device=dev)
    counts, n0, n1 = [new_counts(E, dev) for _ in range(3)]
    add("prompt", "moe route", None, time_calls([lambda: route(logits, E, K, counts=n0)] * 4), 4 * T * E + 12 * T * K)
    idx, wts, ranks = route(logits, E, K, counts=counts)
    keep = counts.clone()

    def sort_rows():
        n1.copy_(keep)
        return SortedRows(xts[0], idx, ranks, n1)
    plan = sort_rows()
    add("prompt", "moe plan + permute", "layer_norm (OPT)", time_calls([sort_rows] * 4), 2 * T * W * (1 + K))
    live = int(plan.live_tiles.item()) * 128
    add("prompt", "grouped gate_up", "gemm out_proj", time_calls([lambda w=w: grouped_gemm(plan.x, w, plan, gate=(7.0, 1.702)) for w in gu]),
        2 * (E * 2 * ff * W + T * K * (W + ff)), 4.0 * T * K * ff * W)
    act = grouped_gemm(plan.x, gu[0], plan, gate=(7.0, 1.702))
    add("prompt", "grouped down", "gemm out_proj", time_calls([lambda w=w: grouped_gemm(act, w, plan) for w in dn]),
        2 * (E * ff * W + T * K * (W + ff)), 2.0 * T * K * ff * W)
    ym = grouped_gemm(act, dn[0], plan)
    add("prompt", "rms_residual combine", "layer_norm (OPT)", time_calls([lambda x=x, t=t: rms_residual(ym, nw, 1e-5, x, xt=t, offset=1.0, mix=(idx, plan.rows, wts))
                                                                          for x, t in zip(xs, xts)]), 10 * T * W + 2 * T * K * W)
    return rows, {"active_experts": act_e, "sorted_rows": live, "routed_rows": T * K}


def mutolix_kernel_table(z, B, S, T):
    """As kernel_table, for the matrix-memory / grouped-attention decoder."""
    from ..attention import (attention_decode, attention_group_decode, attention_inputs, attention_prefill, attention_prefill_biased, distance_bias)
    from ..gemm import gemm, project_parts
    from ..kernel.cuda_native.layer_norm import layer_norm_forward
    from ..memory import head_norm_gate, memory_prompt, memory_step
    from ..norm import stream_update
    bf, dev = torch.bfloat16, "cuda"
    W, H, G, d, ff = z["width"], z["heads"], z["kv_heads"], z["dim"], z["ff"]
    MH, md, mv = z["mheads"], z["mdim"], z["mvdim"]
    rnd = lambda *s, dtype=bf: (torch.randn(*s, device=dev, dtype=torch.float32) * 0.05).to(dtype)
    rows = []

    def add(phase, name, like, us, nbytes, flops=0.0):
        rows.append((phase, name, like, us, float(nbytes), float(flops)))

    def product(phase, name, M, N, Kd, like=None, act=None, xielu=0, tail=0):
        N += tail
        nb = 2 * (N * Kd + M * Kd) + 2 * M * (N + tail)
        ws = [rnd(N, Kd) for _ in range(copies(2 * N * Kd, 32))]
        xs = [rnd(M, Kd) for _ in range(4)]
        bias, par = rnd(N), torch.tensor([0.7, 0.9], device=dev)
        if xielu or tail:
            call = lambda w, x: project_parts(x, w, bias=bias, xielu=(par, xielu) if xielu else None, tail_col=N - tail if tail else None)
        else:
            call = lambda w, x: gemm(x, w, bias=bias if act else None, act=act, static_weight=True)
        us = time_calls([lambda w=w, x=xs[i % 4]: call(w, x) for i, w in enumerate(ws)])
        add(phase, name, like, us, nb, 2.0 * M * N * Kd)

    qk, vg = MH * md, MH * mv
    n_mem, n_att = 2 * qk + 2 * vg + W, (H + 2 * G) * d + W
    nw, w32, lw, lb = rnd(W), torch.ones(W, device=dev), rnd(W), rnd(W)
    bias_h = tuple(torch.rand(H, device=dev) for _ in range(2))
    mbias = tuple(torch.zeros(MH, device=dev) + x for x in (0.0, 4.0))

    # ---- generation step ----
    product("step", "gemm in_proj (memory)", B, n_mem, W, tail=-(-2 * MH // 8) * 8)
    product("step", "gemm in_proj (attention)", B, n_att, W)
    product("step", "gemm out_proj", B, W, H * d)
    product("step", "gemm up + xielu", B, ff + W, W, like="gemm fc1 relu (OPT)", xielu=ff)
    product("step", "gemm fc1 relu (OPT)", B, ff + W, W, act="relu")
    product("step", "gemm down", B, W, ff)
    nb = 8 * B * MH * (md * mv + md)
    states = [[rnd(B, MH, md, mv, dtype=torch.float32), rnd(B, MH, md, dtype=torch.float32), torch.zeros(B, MH, device=dev)] for _ in range(copies(nb / 2))]
    row = rnd(B, 2 * qk + 2 * vg)
    gates, mnorm = rnd(B, 2 * MH, dtype=torch.float32), rnd(vg)
    q, k, v, g = row.split([qk, qk, vg, vg], 1)
    add("step", "memory_step", "attention_decode (OPT)", time_calls([lambda s=s: memory_step(q, k, v, g, gates, mbias, 15.0, md ** -0.5, mnorm, mv, 1e-6, s, MH)
                                                                     for s in states]), nb + 2 * B * (2 * qk + 3 * vg))
    del states
    pos = torch.tensor([S - 1], dtype=torch.int32, device=dev)
    kv = [rnd(B, S, 2 * G * d) for _ in range(copies(B * S * 2 * G * d * 2))]
    qr = rnd(B, H * d)
    add("step", "attention_group_decode", "attention_decode (OPT)", time_calls([lambda c=c: attention_group_decode(
        qr, c[:, :, :G * d], c[:, :, G * d:], d, pos, 0.09, bias=bias_h) for c in kv]), 4 * B * S * G * d + 4 * B * H * d)
    pr, qn, kn, lam = rnd(B, n_att), rnd(H * d), rnd(G * d), torch.full((1,), 0.5, device=dev)
    add("step", "attention_inputs", "layer_norm (OPT)", time_calls([lambda c=c: attention_inputs(
        pr, H, G, d, d, qn, H * d, kn, G * d, 1e-6, c[:, :, :G * d], c[:, :, G * d:], 1, temp=(0.1, 512), vmix=lam, v_first=kv[0][:, :, G * d:],
        pos_device=pos) for c in kv[1:]]), 4 * B * (H + 2 * G) * d + 2 * B * G * d)
    del kv
    kv = [rnd(B, S, 3 * H * d) for _ in range(copies(B * S * 2 * H * d * 2))]
    add("step", "attention_decode (OPT)", None, time_calls([lambda c=c: attention_decode(
        c[:, :, 2 * H * d:], c[:, :, :H * d], c[:, :, H * d:2 * H * d], d, S, q_in_cache=True) for c in kv]), 4 * B * S * H * d)
    del kv
    x, y, gr = torch.randn(B, W, device=dev), rnd(B, W), rnd(B, n_mem)[:, :W]
    add("step", "stream_update", "layer_norm (OPT)", time_calls([lambda: stream_update(x, 1e-6, y=y, gate=gr, w_out=w32, w_next=nw)] * 16), 14 * B * W)
    xt = rnd(B, W)
    add("step", "layer_norm (OPT)", None, time_calls([lambda: layer_norm_forward(xt, lw, lb, 1e-5)] * 16), 4 * B * W)

    # ---- prompt ----
    seq = min(S, T)
    nB = T // seq
    product("prompt", "gemm in_proj (memory)", T, n_mem, W, tail=-(-2 * MH // 8) * 8)
    product("prompt", "gemm in_proj (attention)", T, n_att, W)
    product("prompt", "gemm out_proj", T, W, H * d)
    product("prompt", "gemm up + xielu", T, ff + W, W, like="gemm fc1 relu (OPT)", xielu=ff)
    product("prompt", "gemm fc1 relu (OPT)", T, ff + W, W, act="relu")
    product("prompt", "gemm down", T, W, ff)
    projs = [rnd(T, n_mem) for _ in range(3)]
    gates = rnd(T, 2 * MH, dtype=torch.float32)
    state = [torch.empty(nB, MH, md, mv, device=dev), torch.empty(nB, MH, md, device=dev), torch.empty(nB, MH, device=dev)]
    add("prompt", "memory_chunks", "attention causal (OPT)", time_calls([lambda r=r: memory_prompt(
        *r[:, :2 * qk + vg].split([qk, qk, vg], 1), gates, mbias, 15.0, md ** -0.5, state, MH, chunked=True) for r in projs]),
        4 * T * (qk + vg) + 8 * T * MH + 4 * nB * MH * md * mv, 4.0 * T * MH * md * mv)
    os_ = [rnd(T, vg) for _ in range(4)]
    add("prompt", "head_norm_gate", "layer_norm (OPT)", time_calls([lambda o=o: head_norm_gate(o, projs[0][:, 2 * qk + vg:2 * qk + 2 * vg], mnorm, MH, mv, 1e-6)
                                                                    for o in os_]), 6 * T * vg)
    del projs, os_
    projs = [rnd(T, n_att) for _ in range(3)]
    caches = [rnd(nB, seq, 2 * G * d) for _ in range(2)]
    kc, vc = caches[0][:, :, :G * d], caches[0][:, :, G * d:]
    add("prompt", "attention_inputs", "layer_norm (OPT)", time_calls([lambda r=r: attention_inputs(
        r, H, G, d, d, qn, H * d, kn, G * d, 1e-6, kc, vc, seq, temp=(0.1, 512), vmix=lam, v_first=caches[1][:, :, G * d:]) for r in projs]),
        4 * T * (H + 2 * G) * d + 2 * T * G * d)
    del projs
    q3, kv3 = rnd(nB, seq, H * d), rnd(nB, seq, 2 * H * d)
    flops = 4.0 * nB * H * d * seq * (seq + 1) / 2
    add("prompt", "attention biased", "attention causal (OPT)", time_calls([lambda: attention_prefill_biased(q3, kc, vc, d, table)] * 4)
        if (table := distance_bias(*bias_h, seq)) is not None else 0.0, 2 * T * (2 * H + 2 * G) * d, flops)
    add("prompt", "distance_bias", None, time_calls([lambda: distance_bias(*bias_h, seq)] * 8), 4 * H * (seq + 256))
    add("prompt", "attention causal (OPT)", None, time_calls([lambda: attention_prefill(q3, kv3[:, :, :H * d], kv3[:, :, H * d:], d)] * 4),
        2 * T * 4 * H * d, flops)
    del q3, kv3, caches
    xs = [torch.randn(T, W, device=dev) for _ in range(copies(14 * T * W, 8))]
    ys = [rnd(T, W) for _ in xs]
    gs = [rnd(T, n_att)[:, -W:] for _ in range(2)]
    add("prompt", "stream_update", "layer_norm (OPT)", time_calls([lambda x=x, y=y, g=gs[i % 2]: stream_update(x, 1e-6, y=y, gate=g, w_out=w32, w_next=nw)
                                                                   for i, (x, y) in enumerate(zip(xs, ys))]), 14 * T * W)
    lns = [rnd(T, W) for _ in range(copies(4 * T * W, 8))]
    add("prompt", "layer_norm (OPT)", None, time_calls([lambda t=t: layer_norm_forward(t, lw, lb, 1e-5) for t in lns]), 4 * T * W)
    return rows, {}


MOPONEX_SIZES = {
    # alternating parallel layers (chunk attention | gated linear attention, dense feed-forward) and state-space layers
    # (routed experts); g*: the gated linear heads, s*: the state space's
    "2048": dict(width=2048, heads=16, kv_heads=4, dim=128, chunk=1024, gheads=8, gdim=128, gvdim=256, rank=16, ff=5632, sheads=64, svdim=64, state=128,
                 sgroups=1, norm_groups=1, experts=62, identity=2, groups=8, keep=4, top=6, eff=1024, shared=2048, layers=8, vocab=32768),
    "4096": dict(width=4096, heads=32, kv_heads=8, dim=128, chunk=2048, gheads=16, gdim=128, gvdim=256, rank=16, ff=11264, sheads=128, svdim=64, state=128,
                 sgroups=8, norm_groups=8, experts=30, identity=2, groups=4, keep=2, top=4, eff=2048, shared=4096, layers=6, vocab=32768),
}


def make_moponex(z):
    from ..registry import build_model
    par = {"type": "parallel", "mlp": {"kind": "dense", "ff": z["ff"]},
           "mixer": {"left": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5,
                              "mask": {"size": z["chunk"]}, "rot": {"dims": z["dim"] // 2, "base": 5e5, "scaling": {"factor": 4.0}}},
                     "right": {"heads": z["gheads"], "dim": z["gdim"], "vdim": z["gvdim"], "tau": 12.0, "rank": z["rank"]}}}
    ssm = {"type": "mamba2", "mixer": {"heads": z["sheads"], "vdim": z["svdim"], "state": z["state"], "groups": z["sgroups"], "conv": 4,
                                       "norm_groups": z["norm_groups"]},
           "mlp": {"kind": "moe", "expert": {"ff": z["eff"]}, "shared": {"ff": z["shared"]},
                   "router": {"experts": z["experts"], "top": z["top"], "identity": z["identity"], "groups": {"count": z["groups"], "keep": z["keep"]}}}}
    torch.manual_seed(1)
    return build_model("Moponex", dtype=torch.bfloat16, device="cuda", config_dict={
        "vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "residual_mult": 0.8, "logit_scale": 0.25, "layers": [par, ssm] * (z["layers"] // 2),
        "embedding": {"bigram": {"buckets": z["vocab"] - 1, "mul_prev": 1021, "mul_cur": 13}}})


def moponex_as_opt(z):
    """The feed-forward size with which an OPT layer has as many weights per token as a layer here has on average."""
    w = z["width"]
    par = w * (2 * z["heads"] * z["dim"] + z["kv_heads"] * z["dim"] + 2 * z["gheads"] * z["gdim"] + 3 * z["gheads"] * z["gvdim"] + 3 * z["ff"])
    ssm = w * (3 * z["sheads"] * z["svdim"] + 2 * z["sgroups"] * z["state"] + 2 * z["shared"] + 2 * z["top"] * z["eff"])
    ffn = ((par + ssm) / 2 / w - 4 * w) / 2
    return dict(z, top=1, ff=int(ffn / 1.5))


def moponex_kernel_table(z, B, S, T):
    """As kernel_table, for the state-space / chunk-attention / gated-linear decoder."""
    from ..attention import (attention_decode, attention_group_decode_chunk, attention_inputs, attention_prefill, attention_prefill_chunk, attention_rotary)
    from ..decay import gate_group_norm, gla_prompt, gla_step, short_conv, ssm_prompt, ssm_step
    from ..gemm import gemm, project_parts, project_unit
    from ..kernel.cuda_native.layer_norm import layer_norm_forward
    from ..memory import head_norm_gate, memory_prompt, memory_step
    from ..moe import RouterRule, SortedRows, grouped_gemm, new_counts, route, route_rule, skinny_experts
    from ..norm import rms_residual, stream_add, stream_update
    bf, f32, dev = torch.bfloat16, torch.float32, "cuda"
    W, H, G, d, ff = z["width"], z["heads"], z["kv_heads"], z["dim"], z["ff"]
    GH, gd, gv, rank = z["gheads"], z["gdim"], z["gvdim"], z["rank"]
    SH, sv, N, SG = z["sheads"], z["svdim"], z["state"], z["sgroups"]
    E, K, eff, n = z["experts"], z["top"], z["eff"], z["experts"] + z["identity"]
    rnd = lambda *s, dtype=bf: (torch.randn(*s, device=dev, dtype=torch.float32) * 0.05).to(dtype)
    rows = []

    def add(phase, name, like, us, nbytes, flops=0.0):
        rows.append((phase, name, like, us, float(nbytes), float(flops)))

    def product(phase, name, M, Nn, Kd, like=None, unit=None, act=None, tail=0, out32=False):
        Nn += tail
        cols = Nn // 2 if unit == "geglu" else Nn
        nb = 2 * (Nn * Kd + M * Kd) + (4 if out32 else 2) * M * (cols + tail)
        ws = [rnd(Nn, Kd) for _ in range(copies(2 * Nn * Kd, 32))]
        xs = [rnd(M, Kd) for _ in range(4)]
        bias = rnd(Nn)
        if unit:
            call = lambda w, x: project_unit(x, w, unit)
        elif tail:
            call = lambda w, x: project_parts(x, w, tail_col=Nn - tail)
        else:
            call = lambda w, x: gemm(x, w, bias=bias if act else None, act=act, out_dtype=f32 if out32 else None, static_weight=True)
        add(phase, name, like, time_calls([lambda w=w, x=xs[i % 4]: call(w, x) for i, w in enumerate(ws)]), nb, 2.0 * M * Nn * Kd)

    inner, chan = SH * sv, SH * sv + 2 * SG * N
    n_ssm, n_par = inner + chan, (H + G) * d + 2 * GH * (gd + gv) + rank
    qk, vg = GH * gd, GH * gv
    nw, w32, lw, lb = rnd(W), torch.ones(W, device=dev), rnd(W), rnd(W)
    per_head = [torch.full((SH,), v, device=dev) for v in (-2.0, -1.0, 1.0)]
    conv_w, conv_b, ssm_norm = rnd(4, chan), rnd(chan), rnd(inner)
    a2, a2b, gnorm = rnd(qk, rank), rnd(qk), rnd(vg)
    qn, kn, freq, sinks = rnd(d), rnd(d), torch.rand(d // 4, device=dev), torch.zeros(H, device=dev)
    corr = torch.rand(n, device=dev) * 0.01 - 1.0
    rule = RouterRule(n, E, corr, z["groups"], z["keep"])
    R = min(z["chunk"], S)
    mbias = tuple(torch.zeros(GH, device=dev) + x for x in (0.0, 4.0))

    def gemms(phase, M):
        product(phase, "gemm in_proj (state space)", M, n_ssm, W, tail=SH)
        product(phase, "gemm in_proj (parallel)", M, n_par, W)
        product(phase, "gemm out_proj", M, W, H * d)
        product(phase, "gemm gate_up + geglu", M, 2 * ff, W, like="gemm fc1 relu (OPT)", unit="geglu")
        product(phase, "gemm fc1 relu (OPT)", M, 2 * ff, W, act="relu")
        product(phase, "gemm down", M, W, ff)
        product(phase, "gemm shared up + gelu", M, z["shared"], W, like="gemm out_proj", unit="gelu")

    # ---- generation step ----
    gemms("step", B)
    pos = torch.tensor([S - 1], dtype=torch.int32, device=dev)
    nb = 8 * B * SH * N * sv
    states = [rnd(B, SH, N, sv, dtype=f32) for _ in range(copies(nb / 2))]
    row, dt, ring = rnd(B, n_ssm), rnd(B, SH, dtype=f32), rnd(B, 4, chan)
    add("step", "ssm_step", "memory_step (Mutolix)", time_calls([lambda s=s: ssm_step(row[:, inner:], conv_w, conv_b, ring, pos, dt, *per_head, s, SH, SG, N, sv)
                                                                 for s in states]), nb + 2 * B * (6 * chan + inner))
    del states
    y = rnd(B, inner)
    add("step", "gate_group_norm", "layer_norm (OPT)", time_calls([lambda: gate_group_norm(y, row[:, :inner], ssm_norm, 1e-6, SH, sv, z["norm_groups"])] * 16), 6 * B * inner)
    nb = 8 * B * GH * gd * gv
    states = [rnd(B, GH, gd, gv, dtype=f32) for _ in range(copies(nb / 2))]
    row = rnd(B, n_par)
    q, k, v, g, low = row[:, (H + G) * d:].split([qk, qk, vg, vg, rank], 1)
    add("step", "gla_step", "memory_step (Mutolix)", time_calls([lambda s=s: gla_step(q, k, v, g, low, a2, a2b, 12.0, gd ** -0.5, gnorm, gv, 1e-6, s, GH) for s in states]),
        nb + 2 * B * (2 * qk + 3 * vg) + 2 * qk * rank)
    gates = rnd(B, 2 * GH, dtype=f32)
    extra = [[rnd(B, GH, gd, dtype=f32), torch.zeros(B, GH, device=dev)] for _ in states]
    add("step", "memory_step (Mutolix)", None, time_calls([lambda s=s, e=e: memory_step(q, k, v, g, gates, mbias, 15.0, gd ** -0.5, gnorm, gv, 1e-6, [s] + e, GH)
                                                           for s, e in zip(states, extra)]), nb + 2 * B * (2 * qk + 3 * vg))
    del states, extra
    kv = [rnd(B, R, 2 * G * d) for _ in range(copies(B * R * 2 * G * d * 2))]
    qr = rnd(B, H * d)
    add("step", "attention_group_decode chunk", "attention_decode (OPT)", time_calls([lambda c=c: attention_group_decode_chunk(
        qr, c[:, :, :G * d], c[:, :, G * d:], d, pos, 0.09, z["chunk"], sinks=sinks) for c in kv]), 4 * B * (((S - 1) % z["chunk"]) + 1) * G * d + 4 * B * H * d)
    add("step", "attention_rotary", "layer_norm (OPT)", time_calls([lambda c=c: attention_rotary(row, H, G, d, d, qn, kn, 1e-6, freq, c[:, :, :G * d], c[:, :, G * d:], 1,
                                                                                                 pos_device=pos) for c in kv]), 4 * B * H * d + 6 * B * G * d)
    del kv
    kv = [rnd(B, R, 3 * H * d) for _ in range(copies(B * R * 2 * H * d * 2))]
    add("step", "attention_decode (OPT)", None, time_calls([lambda c=c: attention_decode(
        c[:, :, 2 * H * d:], c[:, :, :H * d], c[:, :, H * d:2 * H * d], d, R, q_in_cache=True) for c in kv]), 4 * B * R * H * d)
    del kv
    x, y, y2 = torch.randn(B, W, device=dev), rnd(B, W), rnd(B, W)
    add("step", "stream_add", "layer_norm (OPT)", time_calls([lambda: stream_add(x, 1e-6, y=y, scale=0.8, w_next=nw)] * 16), 12 * B * W)
    add("step", "stream_add, two rows", "layer_norm (OPT)", time_calls([lambda: stream_add(x, 1e-6, y=y, w=w32, y2=y2, w2=w32, scale=0.8, w_next=nw)] * 16), 14 * B * W)
    routers = [rnd(n + 8, W) for _ in range(16)]
    add("step", "stream_add + router", "rms_residual + router (Tulezen)", time_calls([lambda r=r: stream_add(x, 1e-6, y=y, scale=0.8, w_next=nw, router=(r, rule, K, True))
                                                                                      for r in routers]), 12 * B * W + 2 * (n + 1) * W)
    xt = rnd(B, W)
    add("step", "rms_residual + router (Tulezen)", None, time_calls([lambda r=r: rms_residual(y, nw, 1e-5, x, xt=xt, router=(r, n, K)) for r in routers]), 12 * B * W + 2 * n * W)
    add("step", "layer_norm (OPT)", None, time_calls([lambda: layer_norm_forward(xt, lw, lb, 1e-5)] * 16), 4 * B * W)
    n_w = max(2, min(8, -(-FLUSH_BYTES // (4 * E * eff * W))))
    ups, downs = [rnd(E, eff, W) for _ in range(n_w)], [rnd(E, W, eff) for _ in range(n_w)]
    idx, w, _, gate = route_rule(torch.randn(B, n + 1, device=dev), rule, K, gated=True)
    live = idx[idx < E]
    act_e, pairs = int(live.unique().numel()), int(live.numel())
    a = rnd(B * K, eff)
    add("step", "experts up + gelu", "gemm out_proj", time_calls([lambda u=u: skinny_experts(xt, u, idx, K, unit="gelu") for u in ups]),
        2 * (act_e * eff * W + B * W + pairs * eff), 2.0 * pairs * eff * W)
    add("step", "experts down", "gemm out_proj", time_calls([lambda u=u: skinny_experts(a, u, idx, 1) for u in downs]), 2 * (act_e * eff * W + pairs * (W + eff)),
        2.0 * pairs * eff * W)
    ym, sh = rnd(B * K, W), rnd(B, W)
    add("step", "stream_add of a mixture", "layer_norm (OPT)", time_calls([lambda: stream_add(
        x, 1e-6, y=ym, mix=(idx, None, w), ident=xt, experts=E, shared=sh, gate=gate, scale=0.8, w_next=nw)] * 16), 12 * B * W + 2 * (pairs + B) * W)

    # ---- prompt ----
    seq = min(S, T)
    nB = T // seq
    gemms("prompt", T)
    product("prompt", "gemm decay logits", T, qk, rank, out32=True)
    projs = [rnd(T, n_ssm) for _ in range(3)]
    ring = rnd(nB, 4, chan)
    add("prompt", "short_conv", "layer_norm (OPT)", time_calls([lambda r=r: short_conv(r[:, inner:], conv_w, conv_b, ring, nB) for r in projs]), 4 * T * chan)
    xbc, dt = [short_conv(r[:, inner:], conv_w, conv_b, ring, nB) for r in projs], rnd(T, SH, dtype=f32)
    state = torch.empty(nB, SH, N, sv, device=dev)
    add("prompt", "ssm_chunks", "memory_chunks (Mutolix)", time_calls([lambda r=r: ssm_prompt(r, dt, *per_head, state, SH, SG, N, sv, chunked=True) for r in xbc]),
        2 * T * (chan + inner) + 4 * T * SH + 4 * nB * SH * N * sv, 4.0 * T * SH * N * sv)
    ys = [rnd(T, inner) for _ in range(3)]
    add("prompt", "gate_group_norm", "layer_norm (OPT)", time_calls([lambda y=y, r=r: gate_group_norm(y, r[:, :inner], ssm_norm, 1e-6, SH, sv, z["norm_groups"])
                                                                     for y, r in zip(ys, projs)]), 6 * T * inner)
    del projs, xbc, ys, state
    projs = [rnd(T, n_par) for _ in range(3)]
    zl = rnd(T, qk, dtype=f32) + 2.0
    state = torch.empty(nB, GH, gd, gv, device=dev)
    part = lambda r: r[:, (H + G) * d:(H + G) * d + 2 * qk + vg].split([qk, qk, vg], 1)
    add("prompt", "gla_chunks", "memory_chunks (Mutolix)", time_calls([lambda r=r: gla_prompt(*part(r), zl, 12.0, gd ** -0.5, state, GH, chunked=True) for r in projs]),
        4 * T * (qk + vg) + 4 * T * qk + 4 * nB * GH * gd * gv, 4.0 * T * GH * gd * gv)
    gates, ms = rnd(T, 2 * GH, dtype=f32), [state, torch.empty(nB, GH, gd, device=dev), torch.empty(nB, GH, device=dev)]
    add("prompt", "memory_chunks (Mutolix)", None, time_calls([lambda r=r: memory_prompt(*part(r), gates, mbias, 15.0, gd ** -0.5, ms, GH, chunked=True) for r in projs]),
        4 * T * (qk + vg) + 8 * T * GH + 4 * nB * GH * gd * gv, 4.0 * T * GH * gd * gv)
    os_ = [rnd(T, vg) for _ in range(4)]
    add("prompt", "head_norm_gate", "layer_norm (OPT)", time_calls([lambda o=o: head_norm_gate(o, projs[0][:, -vg - rank:-rank], gnorm, GH, gv, 1e-6, silu=True) for o in os_]),
        6 * T * vg)
    rb = rnd(nB, min(z["chunk"], seq), 2 * G * d)
    add("prompt", "attention_rotary", "layer_norm (OPT)", time_calls([lambda r=r: attention_rotary(
        r, H, G, d, d, qn, kn, 1e-6, freq, rb[:, :, :G * d], rb[:, :, G * d:], seq, keys=True) for r in projs]), 4 * T * (H + G) * d + 4 * nB * rb.shape[1] * G * d)
    del projs, os_, state, ms
    q3, k3, v3, kv3 = rnd(nB, seq, H * d), rnd(nB, seq, G * d), rnd(nB, seq, G * d), rnd(nB, seq, 2 * H * d)
    c = z["chunk"]
    seen = sum(i % c + 1 for i in range(seq))
    add("prompt", "attention chunk", "attention causal (OPT)", time_calls([lambda: attention_prefill_chunk(q3, k3, v3, d, c, sinks=sinks)] * 4), 2 * T * (2 * H + 2 * G) * d,
        4.0 * nB * H * d * seen)
    add("prompt", "attention causal (OPT)", None, time_calls([lambda: attention_prefill(q3, kv3[:, :, :H * d], kv3[:, :, H * d:], d)] * 4), 2 * T * 4 * H * d,
        4.0 * nB * H * d * seq * (seq + 1) / 2)
    del q3, k3, v3, kv3
    xs = [torch.randn(T, W, device=dev) for _ in range(copies(12 * T * W, 8))]
    ys = [rnd(T, W) for _ in xs]
    add("prompt", "stream_add", "layer_norm (OPT)", time_calls([lambda x=x, y=y: stream_add(x, 1e-6, y=y, scale=0.8, w_next=nw) for x, y in zip(xs, ys)]), 12 * T * W)
    add("prompt", "stream_add, two rows", "layer_norm (OPT)", time_calls([lambda x=x, y=y: stream_add(x, 1e-6, y=y, w=w32, y2=ys[0], w2=w32, scale=0.8, w_next=nw)
                                                                          for x, y in zip(xs[1:], ys[1:])]), 14 * T * W)
    add("prompt", "layer_norm (OPT)", None, time_calls([lambda t=t: layer_norm_forward(t, lw, lb, 1e-5) for t in ys]), 4 * T * W)
    logits = torch.randn(T, n + 8, device=dev)
    counts, n0, n1 = [new_counts(E, dev) for _ in range(3)]
    add("prompt", "moe route by rule", "moe route (Tulezen)", time_calls([lambda: route_rule(logits, rule, K, counts=n0, gated=True)] * 4), 4 * T * n + 12 * T * K)
    n2 = new_counts(n, dev)
    add("prompt", "moe route (Tulezen)", None, time_calls([lambda: route(logits, n, K, counts=n2)] * 4), 4 * T * n + 12 * T * K)
    idx, w, ranks, gate = route_rule(logits, rule, K, counts=counts, gated=True)
    keep = counts.clone()

    def sort_rows():
        n1.copy_(keep)
        return SortedRows(ys[0], idx, ranks, n1)
    plan = sort_rows()
    pairs = int((idx < E).sum())
    add("prompt", "moe plan + permute", "layer_norm (OPT)", time_calls([sort_rows] * 4), 2 * T * W + 2 * pairs * W)
    add("prompt", "grouped up + gelu", "gemm out_proj", time_calls([lambda u=u: grouped_gemm(plan.x, u, plan, unit="gelu") for u in ups]),
        2 * (E * eff * W + pairs * (W + eff)), 2.0 * pairs * eff * W)
    act = grouped_gemm(plan.x, ups[0], plan, unit="gelu")
    add("prompt", "grouped down", "gemm out_proj", time_calls([lambda u=u: grouped_gemm(act, u, plan) for u in downs]),
        2 * (E * eff * W + pairs * (W + eff)), 2.0 * pairs * eff * W)
    ym = grouped_gemm(act, downs[0], plan)
    add("prompt", "stream_add of a mixture", "layer_norm (OPT)", time_calls([lambda x=x, y=y: stream_add(
        x, 1e-6, y=ym, mix=(idx, plan.rows, w), ident=y, experts=E, shared=ys[0], gate=gate, scale=0.8, w_next=nw) for x, y in zip(xs[1:], ys[1:])]),
        12 * T * W + 2 * (pairs + T) * W)
    return rows, {"active_experts": act_e, "sorted_rows": int(plan.live_tiles.item()) * 128, "routed_rows": pairs}


TUPIDRA_SIZES = {
    # a selective state space (inner, state, dt_rank), a capped attention (heads on kv_heads, window, keep) and two rotary latent
    # attentions (l*: heads of ldim + rot / lvdim, q_rank, kv_rank), the second on the latents of the first; every layer
    # with a dense feed-forward beside its mixer
    "2048": dict(width=2048, inner=4096, state=16, dt_rank=128, heads=16, kv_heads=4, dim=128, window=1024, keep=64, lheads=32, ldim=64, rot=32, lvdim=64,
                 q_rank=768, kv_rank=256, ff=5632, layers=8, vocab=32768),
    "4096": dict(width=4096, inner=8192, state=16, dt_rank=256, heads=32, kv_heads=8, dim=128, window=4096, keep=64, lheads=32, ldim=128, rot=64, lvdim=128,
                 q_rank=1536, kv_rank=512, ff=11264, layers=8, vocab=32768),
}


def make_tupidra(z):
    from ..registry import build_model
    ff = {"kind": "dense", "ff": z["ff"]}
    scan = {"type": "mamba1", "mlp": ff, "mixer": {"inner": z["inner"], "state": z["state"], "dt_rank": z["dt_rank"], "conv": 4}}
    att = {"type": "attention", "mlp": ff, "mixer": {"heads": z["heads"], "kv_heads": z["kv_heads"], "dim": z["dim"], "vdim": z["dim"], "scale": z["dim"] ** -0.5,
                                                     "softcap": 50.0, "mask": {"size": z["window"], "keep_first": z["keep"]}}}
    mix = {"heads": z["lheads"], "dim": z["ldim"], "rot_dim": z["rot"], "vdim": z["lvdim"], "q_rank": z["q_rank"], "kv_rank": z["kv_rank"],
           "scale": (z["ldim"] + z["rot"]) ** -0.5,
           "rot": {"dims": z["rot"], "base": 1e5, "scaling": {"factor": 16.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    layers = []
    for i in range(0, z["layers"], 4):
        layers += [scan, att, {"type": "latent_attention", "mlp": ff, "mixer": mix}, {"type": "latent_attention", "mlp": ff, "mixer": dict(mix, kv_from=i + 2)}]
    torch.manual_seed(1)
    return build_model("Tupidra", config_dict={"vocab": z["vocab"], "width": z["width"], "norm": {"eps": 1e-6}, "canon": {"taps": 4}, "layers": layers},
                       dtype=torch.bfloat16, device="cuda")


def tupidra_as_opt(z):
    """The feed-forward size with which an OPT layer has as many weights as a layer here has on average."""
    w, h = z["width"], z["heads"] * z["dim"]
    scan = z["inner"] * (3 * w + 2 * z["dt_rank"] + 2 * z["state"])
    att = w * (3 * h + 2 * z["kv_heads"] * z["dim"])
    lh, key = z["lheads"], z["ldim"] + z["rot"]
    latent = w * (z["q_rank"] + 2 * lh * z["lvdim"]) + lh * (key * z["q_rank"] + (z["ldim"] + z["lvdim"]) * z["kv_rank"])
    latents = w * (z["kv_rank"] + z["rot"])
    ffn = ((scan + att + 2 * latent + latents) / 4 / w + 3 * z["ff"] - 4 * w) / 2
    return dict(z, top=1, ff=int(ffn / 1.5))


def tupidra_kernel_table(z, B, S, T):
    """As kernel_table, for the selective-scan / capped-attention / rotary-latent decoder."""
    from ..attention import (LATENT_WIDTHS, PROMPT_HEADS, attention_decode, attention_group_decode, attention_group_decode_capped, attention_prefill, attention_prefill_biased,
                             attention_prefill_capped, attention_prefill_gated, attention_rotary, attention_values, distance_bias, distance_slopes, latent_decode,
                             latent_inputs, rotate_heads, sigmoid_gate)
    from ..decay import selective_scan, selective_step, short_conv, short_conv_step, ssm_prompt, ssm_step
    from ..gemm import gemm, project_parts, project_unit
    from ..kernel.cuda_native.layer_norm import layer_norm_forward
    from ..moe import per_head
    from ..norm import rms_norm, stream_add, stream_conv
    bf, f32, dev = torch.bfloat16, torch.float32, "cuda"
    W, H, G, d, ff, C, N, dr = (z[k] for k in ("width", "heads", "kv_heads", "dim", "ff", "inner", "state", "dt_rank"))
    LH, ld, rot, lv, qr, kr = (z[k] for k in ("lheads", "ldim", "rot", "lvdim", "q_rank", "kv_rank"))
    dk, R = min(h for h in PROMPT_HEADS if h[0] >= ld + rot and h[1] >= lv)[0], min(w for w in LATENT_WIDTHS if w >= kr + rot)
    win, keep = z["window"], z["keep"]
    rnd = lambda *s, dtype=bf: (torch.randn(*s, device=dev, dtype=torch.float32) * 0.05).to(dtype)
    rows = []

    def add(phase, name, like, us, nbytes, flops=0.0, sfu=0.0):
        rows.append((phase, name, like, us, float(nbytes), float(flops), float(sfu)))

    def product(phase, name, M, Nn, Kd, like=None, unit=None, act=None, tail=0, out32=False, bias=False):
        Nn += tail
        cols = Nn // 2 if unit == "geglu" else Nn
        nb = 2 * (Nn * Kd + M * Kd) + (4 if out32 else 2) * M * (cols + tail)
        ws = [rnd(Nn, Kd) for _ in range(copies(2 * Nn * Kd, 32))]
        xs = [rnd(M, Kd) for _ in range(4)]
        b = rnd(Nn)
        if unit:
            call = lambda w, x: project_unit(x, w, unit)
        elif tail:
            call = lambda w, x: project_parts(x, w, tail_col=Nn - tail)
        else:
            call = lambda w, x: gemm(x, w, bias=b if act or bias else None, act=act, out_dtype=f32 if out32 else None, static_weight=True)
        add(phase, name, like, time_calls([lambda w=w, x=xs[i % 4]: call(w, x) for i, w in enumerate(ws)]), nb, 2.0 * M * Nn * Kd)

    def gemms(phase, M):
        product(phase, "gemm in_proj (scan)", M, 2 * C, W)
        product(phase, "gemm x_proj", M, dr, C, tail=2 * N)
        product(phase, "gemm in_proj (attention)", M, (2 * H + 2 * G) * d, W, bias=True)
        product(phase, "gemm in_proj (latent)", M, qr + R + LH * lv, W)
        product(phase, "gemm query up", M, LH * dk, qr)
        product(phase, "gemm gate_up + geglu", M, 2 * ff, W, like="gemm fc1 relu (OPT)", unit="geglu")
        product(phase, "gemm fc1 relu (OPT)", M, 2 * ff, W, act="relu")
        product(phase, "gemm out (scan | mlp)", M, W, C + ff)
        product(phase, "gemm out (attention | mlp)", M, W, H * d + ff, bias=True)

    scan_p = [torch.full((C,), -3.0, device=dev), torch.rand(C, N, device=dev), torch.ones(C, device=dev)]
    conv_w, conv_b, dtw = rnd(4, C), rnd(C), rnd(C, dr)
    k1, k2, lw, lb, nw = torch.rand(4, W, device=dev), torch.rand(4, W, device=dev), rnd(W), rnd(W), rnd(W)
    slopes, rule = distance_slopes(H, dev), dict(window=win, keep=keep, cap=50.0)
    sinks, freq, qn, cn = torch.zeros(LH, device=dev), torch.rand(rot // 2, device=dev), rnd(qr), rnd(kr)
    pos = torch.tensor([S - 1], dtype=torch.int32, device=dev)
    held = min(win, S)
    seen = held + min(keep, max(0, S - held))

    # ---- generation step ----
    gemms("step", B)
    nb = 8 * B * C * N
    states = [rnd(B, C, N, dtype=f32) for _ in range(copies(nb / 2))]
    xz, low, bc, x1 = rnd(B, 2 * C), rnd(B, dr), rnd(B, 2 * N, dtype=f32), rnd(B, C)
    ring = rnd(B, 4, C)
    add("step", "short_conv_step", "layer_norm (OPT)", time_calls([lambda: short_conv_step(xz[:, :C], conv_w, conv_b, ring, pos)] * 16), 12 * B * C)
    add("step", "selective_step", "ssm_step (Moponex)", time_calls([lambda s=s: selective_step(x1, xz[:, C:], low, dtw, bc, *scan_p, s) for s in states]),
        nb + 6 * B * C + 2 * C * dr + 4 * C * N)
    SH, sn = C // 64, max(8, N)
    smalls = [s.view(B, SH, sn, -1) for s in states] if N * 64 % sn == 0 else None
    per = [torch.full((SH,), v, device=dev) for v in (-2.0, -1.0, 1.0)]
    sw, sb, srow, sring, sdt = rnd(4, C + 2 * sn), rnd(C + 2 * sn), rnd(B, C + 2 * sn), rnd(B, 4, C + 2 * sn), rnd(B, SH, dtype=f32)
    add("step", "ssm_step (Moponex)", None, time_calls([lambda s=s: ssm_step(srow, sw, sb, sring, pos, sdt, *per, s, SH, 1, sn, 64) for s in smalls]),
        nb + 2 * B * (6 * (C + 2 * sn) + C))
    del states, smalls
    kv = [rnd(B, keep + held, 2 * G * d) for _ in range(copies(B * held * 2 * G * d * 2))]
    pr = rnd(B, (2 * H + 2 * G) * d)
    q, k, v, g = pr.split([H * d, G * d, G * d, H * d], 1)
    add("step", "attention_group_decode capped", "attention_group_decode (Mutolix)", time_calls([lambda c=c: attention_group_decode_capped(
        q, c[:, :, :G * d], c[:, :, G * d:], d, pos, 0.09, slopes=slopes, gate=g, **rule) for c in kv]), 4 * B * seen * G * d + 6 * B * H * d)
    bias_h = tuple(torch.rand(H, device=dev) for _ in range(2))
    qc, last = q.contiguous(), torch.tensor([held - 1], dtype=torch.int32, device=dev)
    add("step", "attention_group_decode (Mutolix)", None, time_calls([lambda c=c: attention_group_decode(
        qc, c[:, :, :G * d], c[:, :, G * d:], d, last, 0.09, bias=bias_h) for c in kv]), 4 * B * held * G * d + 4 * B * H * d)
    add("step", "attention_values", "attention_rotary (Moponex)", time_calls([lambda c=c: attention_values(
        k, v, G, d, 1e-6, c[:, :, :G * d], c[:, :, G * d:], keep, 1, pos_device=pos) for c in kv]), 10 * B * G * d)
    hn, hf = rnd(d), torch.rand(d // 4, device=dev)
    add("step", "attention_rotary (Moponex)", None, time_calls([lambda c=c: attention_rotary(pr, H, G, d, d, hn, hn, 1e-6, hf, c[:, :, :G * d], c[:, :, G * d:], 1,
                                                                                             pos_device=pos) for c in kv]), 4 * B * H * d + 6 * B * G * d)
    del kv
    cache = [rnd(B, S, R) for _ in range(copies(B * S * R * 2))]
    qa = rnd(B, LH * R)
    lat = lambda sk: time_calls([lambda c=c: latent_decode(qa, c, R, LH, 0, pos, 0.05, sinks=sk) for c in cache])
    add("step", "latent_decode with sinks", "latent_decode (Tulezen)", lat(sinks), 2 * B * S * R + 4 * B * LH * R, 4.0 * B * LH * S * R)
    add("step", "latent_decode (Tulezen)", None, lat(None), 2 * B * S * R + 4 * B * LH * R, 4.0 * B * LH * S * R)
    pl = rnd(B, qr + R + LH * lv)
    row = lambda c, **kw: dict(cols=R, rot_col=kr, count=kr, norm=cn, freq=freq, factor=1.2, ring=c, **kw)
    add("step", "latent_inputs", "rms_norm to ring (Tulezen)", time_calls([lambda c=c: latent_inputs(pl, qr, qr, qn, 1e-6, row=row(c), pos_device=pos) for c in cache]),
        4 * B * (qr + R))
    rn = rnd(R)
    add("step", "rms_norm to ring (Tulezen)", None, time_calls([lambda c=c: rms_norm(pl[:, :R], rn, 1e-5, write_out=False, ring=c, pos_device=pos) for c in cache]), 4 * B * R)
    del cache
    qh, o, vo, gl = rnd(B, LH * dk), rnd(B, LH * R), rnd(B, LH * lv), pl[:, qr + R:]
    add("step", "rotate_heads", "attention_rotary (Moponex)", time_calls([lambda: rotate_heads(qh, LH, dk, ld, freq, 1.2, 1, pos_device=pos)] * 16), 4 * B * LH * rot)
    ups = [rnd(LH, R, dk) for _ in range(copies(LH * R * dk * 2, 48))]
    add("step", "per_head key absorb", "gemm query up", time_calls([lambda w=w: per_head(qh, w) for w in ups]), 2 * (LH * R * dk + B * LH * (R + dk)))
    add("step", "per_head value up", "gemm query up", time_calls([lambda w=w: per_head(o, w.view(-1)[:LH * lv * R].view(LH, lv, R)) for w in ups]),
        2 * (LH * R * lv + B * LH * (R + lv)))
    del ups
    add("step", "sigmoid_gate", "layer_norm (OPT)", time_calls([lambda: sigmoid_gate(vo, gl)] * 16), 6 * B * LH * lv)
    x, y, xt, rr = torch.randn(B, W, device=dev), rnd(B, W), rnd(B, W), rnd(B, 4, W)
    add("step", "stream_conv", "stream_add (Moponex)", time_calls([lambda: stream_conv(x, k1, rr, 1e-6, B, y=y, k2=k2, pos_device=pos)] * 16), 22 * B * W + 32 * W)
    add("step", "stream_add (Moponex)", None, time_calls([lambda: stream_add(x, 1e-6, y=y, w_next=nw)] * 16), 12 * B * W)
    add("step", "layer_norm (OPT)", None, time_calls([lambda: layer_norm_forward(xt, lw, lb, 1e-5)] * 16), 4 * B * W)

    # ---- prompt ----
    seq = min(S, T)
    nB = T // seq
    gemms("prompt", T)
    product("prompt", "gemm step logits", T, C, dr, out32=True)
    product("prompt", "gemm kv up", T, LH * (dk + lv), R)
    xzs, zs, bc = [rnd(T, 2 * C) for _ in range(3)], rnd(T, C, dtype=f32), rnd(T, 2 * N, dtype=f32)
    ring = rnd(nB, 4, C)
    add("prompt", "short_conv", "layer_norm (OPT)", time_calls([lambda r=r: short_conv(r[:, :C], conv_w, conv_b, ring, nB) for r in xzs]), 4 * T * C)
    state = torch.empty(nB, C, N, device=dev)
    add("prompt", "selective_scan", "ssm_chunks (Moponex)", time_calls([lambda r=r: selective_scan(r[:, :C], r[:, C:], zs, bc, *scan_p, state) for r in xzs]),
        10 * T * C + 8 * T * N + 4 * nB * C * N, 0.0, float(T) * C * N)
    del xzs, zs, state
    sx, sdt, sst = rnd(T, C + 256), rnd(T, SH, dtype=f32), torch.empty(nB, SH, 128, 64, device=dev)
    add("prompt", "ssm_chunks (Moponex)", None, time_calls([lambda: ssm_prompt(sx, sdt, *per, sst, SH, 1, 128, 64, chunked=True)] * 4),
        2 * T * (2 * C + 256) + 4 * T * SH + 4 * nB * C * 128, 4.0 * T * C * 128)
    del sx, sst
    q3, kv3, g3 = rnd(nB, seq, H * d), rnd(nB, seq, 2 * G * d), rnd(nB, seq, H * d)
    k3, v3 = kv3[:, :, :G * d], kv3[:, :, G * d:]
    pairs = sum(min(i + 1, win) + min(keep, max(0, i + 1 - win)) for i in range(seq))
    full = seq * (seq + 1) / 2
    add("prompt", "attention capped", "attention biased (Mutolix)", time_calls([lambda: attention_prefill_capped(q3, k3, v3, d, d, slopes=slopes, gate=g3, **rule)] * 4),
        2 * T * (3 * H + 2 * G) * d, 4.0 * nB * H * d * pairs)
    table = distance_bias(*bias_h, seq)
    add("prompt", "attention biased (Mutolix)", None, time_calls([lambda: attention_prefill_biased(q3, k3, v3, d, table)] * 4), 2 * T * (2 * H + 2 * G) * d, 4.0 * nB * H * d * full)
    cb = rnd(nB, keep + min(win, seq), 2 * G * d)
    kvs = [rnd(T, 2 * G * d) for _ in range(copies(T * G * d * 10, 16))]
    add("prompt", "attention_values", "attention_rotary (Moponex)", time_calls([lambda r=r: attention_values(
        r[:, :G * d], r[:, G * d:], G, d, 1e-6, cb[:, :, :G * d], cb[:, :, G * d:], keep, seq) for r in kvs]), 4 * T * G * d + 4 * nB * cb.shape[1] * G * d + 2 * nB * cb.shape[1] * G * d)
    projs = [rnd(T, (H + G) * d) for _ in range(3)]
    add("prompt", "attention_rotary (Moponex)", None, time_calls([lambda r=r: attention_rotary(
        r, H, G, d, d, hn, hn, 1e-6, hf, cb[:, :, :G * d], cb[:, :, G * d:], seq, keys=True) for r in projs]), 4 * T * (H + G) * d + 4 * nB * cb.shape[1] * G * d)
    del q3, kv3, g3, k3, v3, kvs, cb, projs
    q3, kv3, g3 = rnd(nB, seq, LH * dk), rnd(nB, seq, LH * (dk + lv)), rnd(nB, seq, LH * lv)
    k3, v3 = kv3[:, :, :LH * dk], kv3[:, :, LH * dk:]
    add("prompt", "attention latent", "attention causal (OPT)", time_calls([lambda: attention_prefill_gated(q3, k3, v3, dk, lv, sinks=sinks, gate=g3)] * 4),
        2 * T * (2 * dk + 3 * lv) * LH, 2.0 * nB * LH * (dk + lv) * full)
    del kv3, g3, k3, v3
    q4, kv4 = rnd(nB, seq, H * d), rnd(nB, seq, 2 * H * d)
    add("prompt", "attention causal (OPT)", None, time_calls([lambda: attention_prefill(q4, kv4[:, :, :H * d], kv4[:, :, H * d:], d)] * 4), 8 * T * H * d, 4.0 * nB * H * d * full)
    del q4, kv4
    pls, lc = [rnd(T, qr + R + LH * lv) for _ in range(3)], rnd(nB, seq, R)
    add("prompt", "latent_inputs", "rms_norm latent (Tulezen)", time_calls([lambda r=r: latent_inputs(r, qr, qr, qn, 1e-6, row=row(lc, keep_rows=True), rows_per_batch=seq) for r in pls]),
        T * (4 * qr + 6 * R))
    cs = [rnd(T, R) for _ in range(copies(4 * T * R))]
    add("prompt", "rms_norm latent (Tulezen)", None, time_calls([lambda t=t: rms_norm(t, rn, 1e-5, ring=lc, rows_per_batch=seq) for t in cs]), 6 * T * R)
    del pls, cs, lc
    qs = [q3.view(T, -1)] + [rnd(T, LH * dk) for _ in range(3)]
    add("prompt", "rotate_heads", "attention_rotary (Moponex)", time_calls([lambda r=r: rotate_heads(r, LH, dk, ld, freq, 1.2, seq) for r in qs]), 4 * T * LH * rot)
    del qs, q3
    xs = [torch.randn(T, W, device=dev) for _ in range(copies(14 * T * W, 8))]
    ys, rr = [rnd(T, W) for _ in xs], rnd(nB, 4, W)
    add("prompt", "stream_conv", "stream_add (Moponex)", time_calls([lambda x=x, y=y: stream_conv(x, k1, rr, 1e-6, nB, y=y, k2=k2) for x, y in zip(xs, ys)]), 14 * T * W)
    add("prompt", "stream_add (Moponex)", None, time_calls([lambda x=x, y=y: stream_add(x, 1e-6, y=y, w_next=nw) for x, y in zip(xs, ys)]), 12 * T * W)
    add("prompt", "layer_norm (OPT)", None, time_calls([lambda t=t: layer_norm_forward(t, lw, lb, 1e-5) for t in ys]), 4 * T * W)
    return rows, {}


DESIGNS = {
    "tupidra": dict(sizes=TUPIDRA_SIZES, runs=RUNS, make=make_tupidra, as_opt=tupidra_as_opt, table=tupidra_kernel_table),
    "moponex": dict(sizes=MOPONEX_SIZES, runs=RUNS, make=make_moponex, as_opt=moponex_as_opt, table=moponex_kernel_table),
    "tulezen": dict(sizes=SIZES, runs=RUNS, make=make_tulezen, as_opt=lambda z: z, table=kernel_table),
    "mutolix": dict(sizes=MUTOLIX_SIZES, runs=RUNS, make=make_mutolix, as_opt=mutolix_as_opt, table=mutolix_kernel_table),
}


def table_with_fractions(rows):
    pk = peaks()
    out = []
    for phase, name, like, us, *work in rows:
        times = {what: n / pk[what] * 1e6 for what, n in zip(("hbm", "tensor", "sfu"), work)}
        bound = max(times, key=times.get)
        out.append({"phase": phase, "kernel": name, "us": round(us, 2), "roofline_us": round(times[bound], 2), "frac": round(times[bound] / us, 3), "like": like,
                    "bound": bound})
    by = {(r["phase"], r["kernel"]): r["frac"] for r in out}
    for r in out:
        if r["like"]:
            r["like_frac"] = by[(r["phase"], r["like"])]
            r["ratio_to_like"] = round(r["frac"] / r["like_frac"], 2)
    return out


def run(design="tulezen", kernels=True, generation=True):
    from ..gemm import device_status
    D = DESIGNS[design]
    res = {"design": design, "dtype": "bf16", "data": "synthetic, random weights", "peaks": peaks(), "sizes": D["sizes"], "generation": [],
           "kernels": {}}
    if kernels:
        with torch.inference_mode():
            for (name, B, S, T) in (("2048", 64, 2048, 8192), ("4096", 16, 4096, 8192)):
                rows, info = D["table"](D["sizes"][name], B, S, T)
                res["kernels"][f"width {name}, batch {B}, {S} positions, {T} prompt tokens"] = dict(info, table=table_with_fractions(rows))
                torch.cuda.empty_cache()
    if generation:
        for name, B, S, new in D["runs"]:
            z = D["sizes"][name]
            line = {"size": name, "batch": B, "prompt": S, "new_tokens": new}
            for what, make in ((design, lambda: D["make"](z)), ("opt", lambda: make_opt(D["as_opt"](z), S + new))):
                model = make()
                line[what] = timed_generation(model, z["vocab"], B, S, new)
                model._decode_state = None
                del model
                torch.cuda.empty_cache()
            res["generation"].append(line)
    status = device_status()
    res["device_status"] = list(status)
    return res
