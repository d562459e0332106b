"""Kernels of the matrix-memory / grouped-attention decoder against the plain restatement."""
import pytest
import torch

import mutolix_plain as P

pytestmark = pytest.mark.gpu


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def rel(got, want):
    """Largest error of a row, over the root mean square of that row or of all rows (the larger one)."""
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all()
    size = want.pow(2).mean(-1).sqrt()
    return float(((got - want).pow(2).mean(-1).sqrt() / size.clamp(min=float(want.pow(2).mean().sqrt()))).max())


# ---- products with xIELU -------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, torch.float16])
@pytest.mark.parametrize("M,N,K,cols", [(1, 48, 40, 24), (17, 136, 264, 136), (32, 72, 64, 0), (64, 264, 96, 128), (300, 520, 200, 264)])
def test_product_with_bias_and_xielu_on_its_first_columns(dtype, M, N, K, cols):
    from energonai_b200.gemm import project_parts, xielu_params
    x, w, b = rnd(M, K, seed=1).to(dtype), rnd(N, K, seed=2, scale=K ** -0.5).to(dtype), rnd(N, seed=3).to(dtype)
    act = xielu_params(0.7, -1.1)
    z = x.double() @ w.double().T + b.double()
    want = z.clone()
    want[:, :cols] = P.xielu(z[:, :cols], torch.tensor(0.7, dtype=torch.float64), torch.tensor(-1.1, dtype=torch.float64))
    tol = {torch.float32: 1e-6, torch.bfloat16: 6e-3, torch.float16: 1e-3}[dtype]
    got = project_parts(x.cuda(), w.cuda(), bias=b.cuda(), xielu=(act.cuda(), cols))
    assert got.dtype == dtype and rel(got, want) < tol
    # the last columns in fp32, with and without activation
    got, tail = project_parts(x.cuda(), w.cuda(), bias=b.cuda(), xielu=(act.cuda(), cols), tail_col=N - 16)
    assert tail.dtype == torch.float32 and rel(got, want[:, :N - 16]) < tol and rel(tail, want[:, N - 16:]) < (1e-6 if dtype == torch.float32 else 2e-6 if cols <= N - 16 else 1e-4)
    got, tail = project_parts(x.cuda(), w.cuda(), tail_col=8)
    assert rel(got, z[:, :8] - b.double()[:8]) < tol and rel(tail, z[:, 8:] - b.double()[8:]) < 2e-6


# ---- norms around a sublayer ----------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rows,width,count", [(1, 40, 36), (5, 2056, 2056), (3, 4096, 4090), (2, 16384, 16384)])
def test_stream_update(dtype, rows, width, count):
    from energonai_b200.norm import stream_update
    pad = lambda t: torch.nn.functional.pad(t, (0, width - count))
    y, g, src, x0 = (pad(rnd(rows, count, seed=s)).to(dtype) for s in (1, 2, 3, 4))
    wo, wn = pad(1 + rnd(count, seed=5)), pad(1 + rnd(count, seed=6)).to(dtype)
    eps, tol = 1e-3, 3e-6 if dtype == torch.float32 else 6e-3
    d = lambda t: t[..., :count].double()
    dev = lambda t: t.cuda()
    # start of the stream
    x = torch.empty(rows, width, device="cuda")
    h = stream_update(x, eps, count, src=dev(src), src_scale=2.5, w_next=dev(wn))
    want = d(src) * 2.5
    assert rel(x[:, :count], want) < 1e-6 and float(x[:, count:].abs().sum()) == 0
    want_h = P.rms_norm(want, d(wn), eps)
    assert rel(h[:, :count], want_h) < tol
    # between two sublayers, with and without gate
    for gate in (g, None):
        x = x0.float().cuda()
        h = stream_update(x, eps, count, y=dev(y), gate=dev(gate) if gate is not None else None, w_out=dev(wo), w_next=dev(wn))
        s = d(y) * torch.sigmoid(d(gate)) if gate is not None else d(y)
        want = d(x0) + P.rms_norm(s, d(wo), eps)
        assert rel(x[:, :count], want) < 3e-6 and rel(h[:, :count], P.rms_norm(want, d(wn), eps)) < tol
    # the last one
    x = x0.float().cuda()
    assert stream_update(x, eps, count, y=dev(y), gate=dev(g), w_out=dev(wo)) is None
    assert rel(x[:, :count], d(x0) + P.rms_norm(d(y) * torch.sigmoid(d(g)), d(wo), eps)) < 3e-6


# ---- queries, keys, values ------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,d,dk", [(4, 2, 20, 24), (3, 3, 64, 64), (16, 1, 100, 128), (1, 1, 5, 8)])
def test_attention_inputs(dtype, H, G, d, dk):
    from energonai_b200.attention import attention_inputs
    B, S, cap, eps, tol = 2, 9, 12, 1e-3, 2e-6 if dtype == torch.float32 else 6e-3
    heads = lambda t, n: torch.nn.functional.pad(t.view(*t.shape[:-1], n, d), (0, dk - d)).reshape(*t.shape[:-1], n * dk)
    q, k, v, vf = (rnd(B * S, n * d, seed=s).to(dtype) for s, n in ((1, H), (2, G), (3, G), (4, G)))
    wq, wk = (1 + rnd(H * d, seed=5)).to(dtype), (1 + rnd(G * d, seed=6)).to(dtype)
    proj = torch.cat([heads(q, H), heads(k, G), heads(v, G), rnd(B * S, 16, seed=7).to(dtype)], 1).cuda()
    first = torch.tensor([0, 4], dtype=torch.int32, device="cuda")
    vmix = torch.tensor([0.3], device="cuda")
    for pos in (None, 3):
        cache = torch.zeros(B, cap, 2 * G * dk, dtype=dtype, device="cuda")
        other = torch.zeros_like(cache)
        p0 = pos or 0
        other[:, p0:p0 + S, G * dk:] = heads(vf, G).view(B, S, -1).cuda()
        kc, vc = cache[:, :, :G * dk], cache[:, :, G * dk:]
        got = attention_inputs(proj, H, G, dk, dk, heads(wq, H).cuda(), H * d, heads(wk, G).cuda(), G * d, eps, kc, vc, S, temp=(0.4, 3),
                               vmix=vmix, v_first=other[:, :, G * dk:], first=first,
                               pos_device=None if pos is None else torch.tensor([pos], dtype=torch.int32, device="cuda"))
        want_q = P.rms_norm(q.double(), wq.double(), eps).view(B, S, -1)
        want_k = P.rms_norm(k.double(), wk.double(), eps)
        want_v = (0.7 * v.double() + 0.3 * vf.double())
        t = P.query_temperature(p0 + S, 0.4, 3)
        got_q = got.view(B, S, H, dk)
        for b in range(B):
            for s in range(S):
                p = p0 + s - int(first[b])
                if p >= 0:
                    assert rel(got_q[b, s, :, :d].reshape(1, -1), want_q[b, s:s + 1] * t[p]) < tol
        assert float(got_q[..., d:].abs().sum()) == 0
        n = min(S, cap - p0)
        for c, w in ((kc, want_k), (vc, want_v)):
            c = c.reshape(B, cap, G, dk)
            assert rel(c[:, p0:p0 + n, :, :d].reshape(B * n, -1), w.view(B, S, -1)[:, :n].reshape(B * n, -1)) < tol
            assert float(c[:, :p0].abs().sum()) == 0 and float(c[:, p0 + n:].abs().sum()) == 0


# ---- attention -------------------------------------------------------------------------------------------
def attention_case(B, S, H, G, d, dv, r_sign=1.0, seed=0):
    """Random heads with one loud query and a loud key far away, so that a misplaced bias, sink or
    group shows."""
    q, k, v = rnd(B, S, H, d, seed=seed), rnd(B, S, G, d, seed=seed + 1), rnd(B, S, G, dv, seed=seed + 2)
    far = k[:, 1 if S > 1 else 0].clone()
    q[:, -1] = far.repeat_interleave(H // G, 1) * 3.0
    v[:, 1 if S > 1 else 0] *= 4.0
    r1 = torch.rand(H, generator=torch.Generator().manual_seed(seed + 3)) * 2 * r_sign
    r2 = torch.rand(H, generator=torch.Generator().manual_seed(seed + 4)) * 0.5
    return q, k, v, r1, r2


def attention_want(q, k, v, r1, r2, scale, first):
    out = []
    for b in range(q.shape[0]):
        f = first[b]
        n = q.shape[1] - f
        y = P.sink_attention(q[b, f:].double(), k[b, f:].double(), v[b, f:].double(), scale, P.distance_bias(n, r1.double(), r2.double()))
        out.append(y.reshape(n, -1))
    return out


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float16])
@pytest.mark.parametrize("B,S,H,G,D,sign", [(1, 1, 2, 1, 64, 1), (1, 130, 4, 2, 64, 1), (2, 257, 6, 2, 128, 1), (1, 700, 4, 4, 128, 1), (1, 300, 4, 1, 64, -1),
                                            (1, 1100, 2, 1, 128, 1)])
def test_prompt_attention_with_bias_and_sink(dtype, B, S, H, G, D, sign):
    from energonai_b200.attention import attention_plain, attention_prefill_biased, distance_bias
    q, k, v, r1, r2 = attention_case(B, S, H, G, D, D, sign)
    q, k, v = (t.to(dtype) for t in (q, k, v))
    first = [0] + [S // 3] * (B - 1)
    scale = D ** -0.5
    flat = lambda t: t.reshape(B, S, -1).cuda()
    mask = torch.zeros(B, S, dtype=dtype)
    for b, f in enumerate(first):
        mask[b, :f] = -10000.0
    table = distance_bias(r1.cuda(), r2.cuda(), S)
    want_bias = r1[:, None].double() * torch.log2(1 + r2[:, None].double() * torch.arange(S))
    assert float((table[:, :S].cpu() - want_bias).abs().max()) < 1e-4
    got = attention_prefill_biased(flat(q), flat(k), flat(v), D, table, mask=mask.cuda() if any(first) else None, scale=scale).cpu()
    plain = attention_plain(flat(q).float(), flat(k).float(), flat(v).float(), H, D, D, scale=scale, kv_heads=G, bias=(r1.cuda(), r2.cuda()), sink=True,
                            first=torch.tensor(first, dtype=torch.int32, device="cuda")).cpu()
    for b, w in enumerate(attention_want(q, k, v, r1, r2, scale, first)):
        assert rel(plain[b, first[b]:], w) < 1e-4
        assert rel(got[b, first[b]:], w) < (2e-2 if dtype == torch.bfloat16 else 3e-3)
        assert torch.isfinite(got).all()


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float16])
@pytest.mark.parametrize("B,S,H,G,D,nsplit", [(1, 1, 1, 1, 64, 1), (2, 63, 4, 2, 64, 1), (3, 64, 6, 2, 128, 2), (2, 65, 16, 1, 64, None), (1, 700, 40, 2, 128, 3),
                                              (2, 1000, 8, 8, 128, None), (2, 321, 12, 1, 64, 5)])
def test_step_attention_of_head_groups(dtype, B, S, H, G, D, nsplit):
    from energonai_b200.attention import attention_group_decode, attention_plain
    q, k, v, r1, r2 = attention_case(B, S, H, G, D, D, seed=7)
    q, k, v = (t.to(dtype) for t in (q, k, v))
    first = [0] + [S // 2] * (B - 1)
    cache = torch.full((B, S + 70, 2 * G * D), 3.0, dtype=dtype, device="cuda")
    cache[:, :S, :G * D], cache[:, :S, G * D:] = k.reshape(B, S, -1).cuda(), v.reshape(B, S, -1).cuda()
    pos, fd, bias = torch.tensor([S - 1], dtype=torch.int32, device="cuda"), torch.tensor(first, dtype=torch.int32, device="cuda"), (r1.cuda(), r2.cuda())
    kc, vc = cache[:, :, :G * D], cache[:, :, G * D:]
    ql = q[:, -1].reshape(B, -1).cuda()
    want = attention_want(q, k, v, r1, r2, 0.1, first)
    for _ in range(2):                                   # (the split counters are zero again)
        got = attention_group_decode(ql, kc, vc, D, pos, 0.1, first=fd, bias=bias, nsplit=nsplit)
        for b in range(B):
            assert rel(got[b:b + 1], want[b][-1:]) < (2e-2 if dtype == torch.bfloat16 else 3e-3)
    plain = attention_plain(ql.float().view(B, 1, -1), kc.float(), vc.float(), H, D, D, scale=0.1, first=fd, pos_device=pos, kv_heads=G, bias=bias, sink=True)
    for b in range(B):
        assert rel(plain[b], want[b][-1:]) < 1e-4
    bare = attention_group_decode(ql, kc, vc, D, pos, 0.1, first=fd, bias=None, sink=False, nsplit=nsplit)
    for b in range(B):
        s = torch.einsum("hd,jhd->hj", q[b, -1].double(), k[b, first[b]:].double().repeat_interleave(H // G, 1)) * 0.1
        w = torch.einsum("hj,jhd->hd", torch.softmax(s, -1), v[b, first[b]:].double().repeat_interleave(H // G, 1))
        assert rel(bare[b:b + 1], w.reshape(1, -1)) < (2e-2 if dtype == torch.bfloat16 else 3e-3)


def test_sink_takes_the_weight_when_every_score_is_low():
    from energonai_b200.attention import attention_group_decode, attention_prefill_biased, distance_bias
    S, D = 150, 64
    k = torch.ones(1, S, D, dtype=torch.bfloat16, device="cuda")
    v, z = torch.ones_like(k), torch.zeros(1, device="cuda")
    for level, want in ((-30.0, 0.0), (0.0, None), (30.0, 1.0)):
        q = torch.full((1, S, D), level / D, dtype=torch.bfloat16, device="cuda")
        got = attention_prefill_biased(q, k, v, D, distance_bias(z, z, S), scale=1.0)[0, :, 0].float().cpu()
        ref = torch.arange(1, S + 1) / torch.arange(2, S + 2) if want is None else torch.full((S,), want)
        assert float((got - ref).abs().max()) < 5e-3
        last = attention_group_decode(q[:, -1], k, v, D, torch.tensor([S - 1], dtype=torch.int32, device="cuda"), 1.0, bias=(z, z))
        assert abs(float(last[0, 0]) - float(ref[-1])) < 5e-3


# ---- matrix memory ----------------------------------------------------------------------------------------
def memory_case(B, S, H, d, dv, seed=0, forget=4.0):
    q, k, v, g = (rnd(B, S, H, n, seed=seed + i) for i, n in enumerate((d, d, dv, dv)))
    gates = torch.cat([rnd(B * S, H, seed=seed + 5, scale=2.0), rnd(B * S, H, seed=seed + 6, scale=2.0)], 1)
    if S > 4:                                            # a token that is remembered, asked for at the end
        k[:, 2] *= 3.0
        gates.view(B, S, -1)[:, 2, :H] += 6.0
        q[:, -1] = k[:, 2]
    bias = (torch.full((H,), -0.5) + 0.3 * torch.arange(H), torch.full((H,), forget) - 0.7 * torch.arange(H))
    return q, k, v, g, gates, bias


def memory_want(q, k, v, gates, bias, cap, scale, first):
    """Per sequence: outputs and final (S, n, m) of the recurrence."""
    out = []
    for b in range(q.shape[0]):
        f, H = first[b], q.shape[2]
        a = gates.view(*q.shape[:2], -1)[b, f:].double()
        eye = torch.eye(H, dtype=torch.float64)
        i, lf = P.memory_gates(a[:, :H], eye, bias[0].double(), eye, bias[1].double(), cap)[0], P.memory_gates(
            a[:, H:2 * H], eye, bias[0].double(), eye, bias[1].double(), cap)[1]
        kk, vv = k[b, f:].double(), v[b, f:].double()
        o = P.memory_scan(q[b, f:].double() * scale, kk, vv, i, lf)
        n, m = kk.shape[0], torch.zeros(H, dtype=torch.float64)
        S, z = torch.zeros(H, kk.shape[2], vv.shape[2], dtype=torch.float64), torch.zeros(H, kk.shape[2], dtype=torch.float64)
        for t in range(n):
            new = torch.maximum(lf[t] + m, i[t])
            S = torch.exp(lf[t] + m - new)[:, None, None] * S + torch.exp(i[t] - new)[:, None, None] * kk[t][:, :, None] * vv[t][:, None, :]
            z = torch.exp(lf[t] + m - new)[:, None] * z + torch.exp(i[t] - new)[:, None] * kk[t]
            m = new
        out.append((o, S, z, m))
    return out


def heads_close(got, want, tol):
    """Head by head: the error of a head's rows over their own size (the head norm makes it matter)."""
    got, want = got.double().cpu(), want.double()
    assert torch.isfinite(got).all()
    for h in range(want.shape[1]):
        assert float((got[:, h] - want[:, h]).pow(2).mean().sqrt() / want[:, h].pow(2).mean().sqrt()) < tol, h


@pytest.mark.parametrize("path,dtype", [("scan", torch.float32), ("scan", torch.bfloat16), ("chunks", torch.bfloat16)])
@pytest.mark.parametrize("B,S,H,d,dv", [(1, 1, 1, 64, 8), (2, 5, 2, 64, 40), (1, 127, 2, 128, 128), (2, 128, 1, 64, 136), (1, 129, 3, 128, 64), (2, 300, 2, 64, 256),
                                        (1, 700, 2, 128, 200)])
@pytest.mark.parametrize("forget", [4.0, -3.0])
def test_memory_of_a_prompt_and_steps_behind_it(path, dtype, B, S, H, d, dv, forget):
    from energonai_b200.memory import head_norm_gate, memory_prompt, memory_step
    more, cap, scale, eps = 6, 9.0, d ** -0.5, 1e-4
    q, k, v, g, gates, bias = memory_case(B, S + more, H, d, dv, forget=forget)
    q, k, v, g = (t.to(dtype) for t in (q, k, v, g))
    first = [0] + [min(S - 1, S // 2 + 1)] * (B - 1)
    want = memory_want(q, k, v, gates, bias, cap, scale, first)
    proj = torch.cat([t.reshape(B, S + more, -1) for t in (q, k, v, g)], 2).cuda()
    G = gates.view(B, S + more, -1).cuda()
    n_cols = [H * d, H * d, H * dv, H * dv]
    state = [torch.full((B, H, d, dv), 7.0, device="cuda"), torch.full((B, H, d), 7.0, device="cuda"), torch.full((B, H), 7.0, device="cuda")]
    db = tuple(x.cuda() for x in bias)
    fd = torch.tensor(first, dtype=torch.int32, device="cuda")
    pq, pk, pv, pg = proj[:, :S].reshape(B * S, -1).split(n_cols, 1)
    o = memory_prompt(pq, pk, pv, G[:, :S].reshape(B * S, -1).contiguous(), db, cap, scale, state, H, first=fd if any(first) else None, chunked=path == "chunks")
    tol = 2e-5 if dtype == torch.float32 else 1.5e-2
    o4 = o.view(B, S, H, dv)
    for b in range(B):
        heads_close(o4[b, first[b]:], want[b][0][:S - first[b]], tol)
        assert torch.isfinite(o4[b].float()).all()
    norm = (1 + rnd(H * dv, seed=20, scale=0.3)).to(dtype)
    y = head_norm_gate(o, pg, norm.cuda(), H, dv, eps)
    ref = P.unit_rms(o.double().cpu().view(B * S, H, dv), eps).reshape(B * S, -1) * norm.double() * torch.sigmoid(pg.double().cpu())
    assert rel(y, ref) < (2e-6 if dtype == torch.float32 else 6e-3)
    for t in range(S, S + more):
        sq, sk, sv, sg = proj[:, t].split(n_cols, 1)
        y = memory_step(sq, sk, sv, sg, G[:, t].contiguous(), db, cap, scale, norm.cuda(), dv, eps, state, H)
        for b in range(B):
            ow = want[b][0][t - first[b]]
            ref = P.unit_rms(ow, eps).reshape(1, -1) * norm.double() * torch.sigmoid(g[b, t].double().reshape(1, -1))
            heads_close(y[b].view(1, H, dv), ref.view(1, H, dv), 3e-5 if dtype == torch.float32 else 1.5e-2)
    # the state itself is 32-bit on every path (what enters it is not rounded to 16 bits)
    for b in range(B):
        for got, ref in zip(state, want[b][1:]):
            heads_close(got[b].reshape(1, H, -1), ref.reshape(1, H, -1), 3e-5)


def test_memory_step_in_clusters_and_uneven_columns():
    """Batches small and large enough for every split of a head's columns, head sizes that do not split
    evenly."""
    from energonai_b200.memory import memory_step
    for B, H, d, dv in ((1, 1, 64, 512), (2, 3, 40, 264), (40, 8, 64, 72), (1, 2, 200, 2048)):
        q, k, v, g, gates, bias = memory_case(B, 1, H, d, dv, seed=B)
        state = [rnd(B, H, d, dv, seed=30), rnd(B, H, d, seed=31), rnd(B, H, seed=32).abs()]
        dev = [t.clone().cuda() for t in state]
        norm = 1 + rnd(H * dv, seed=33, scale=0.2)
        row = torch.cat([t.reshape(B, -1) for t in (q, k, v, g)], 1).cuda()
        y = memory_step(*row.split([H * d, H * d, H * dv, H * dv], 1), gates.cuda(), tuple(x.cuda() for x in bias), 5.0, 0.2, norm.cuda(), dv, 1e-5, dev, H)
        S, n, m = (t.double() for t in state)
        a = gates.double()
        i = 5 * torch.tanh((a[:, :H] + bias[0].double()) / 5)
        f = torch.nn.functional.logsigmoid(5 * torch.tanh((a[:, H:] + bias[1].double()) / 5))
        new = torch.maximum(f + m, i)
        ea, eb = torch.exp(f + m - new), torch.exp(i - new)
        S = ea[..., None, None] * S + eb[..., None, None] * k[:, 0].double()[..., :, None] * v[:, 0].double()[..., None, :]
        n = ea[..., None] * n + eb[..., None] * k[:, 0].double()
        qd = q[:, 0].double() * 0.2
        o = torch.einsum("bhdv,bhd->bhv", S, qd) / (torch.maximum((n * qd).sum(-1).abs(), torch.exp(-new)) + 1e-6)[..., None]
        want = P.unit_rms(o, 1e-5).reshape(B, -1) * norm.double() * torch.sigmoid(g.reshape(B, -1).double())
        assert rel(y, want) < 2e-5
        for got, ref in zip(dev, (S, n, new)):
            assert rel(got.reshape(B, -1), ref.reshape(B, -1)) < 2e-6


def test_no_wait_ran_out():
    from energonai_b200.gemm import device_status
    assert device_status()[0] == 0
