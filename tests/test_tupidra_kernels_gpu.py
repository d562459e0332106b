"""Kernels of the latent-attention / selective-scan / capped-attention decoder against the plain restatement."""
import pytest
import torch

import tupidra_plain as P

pytestmark = pytest.mark.gpu
F32, BF16, F16 = torch.float32, torch.bfloat16, torch.float16


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def rel(got, want):
    """Largest error of a row, over the root mean square of that row or of all rows (the larger one)."""
    got, want = got.double().cpu(), want.double().cpu()
    assert got.shape == want.shape and torch.isfinite(got).all()
    size = want.pow(2).mean(-1).sqrt()
    return float(((got - want).pow(2).mean(-1).sqrt() / size.clamp(min=float(want.pow(2).mean().sqrt()))).max())


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def tol(dtype, exact=3e-6):
    return {F32: exact, BF16: 8e-3, F16: 1.5e-3}[dtype]


# ---- residual step, norms and convolutions ------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("B,S,width,count,taps,real,two", [(1, 1, 40, 36, 4, 4, True), (2, 70, 72, 72, 4, 4, True), (3, 9, 136, 130, 2, 1, False), (1, 300, 2056, 2056, 3, 3, True),
                                                           (2, 37, 4096, 4090, 4, 4, True), (1, 20, 8200, 8200, 4, 4, True), (2, 50, 64, 64, 8, 6, True), (1, 40, 48, 48, 16, 13, False),
                                                           (40, 130, 64, 64, 4, 4, True)])
def test_stream_conv(dtype, B, S, width, count, taps, real, two):
    """Prompt rows, and the steps behind them out of the ring."""
    from energonai_b200.norm import stream_conv
    eps, steps = 1e-3, 3
    pad = lambda t: torch.nn.functional.pad(t, (0, width - count))
    n = S + steps
    x, y = pad(rnd(B, n, count, seed=1)), pad(rnd(B, n, count, seed=2)).to(dtype)
    first = [min(S - 1, 2 * b) for b in range(B)]
    norms, convs = [1 + 0.3 * rnd(count, seed=3 + k) for k in (0, 1)], [rnd(count, real, seed=5 + k, scale=0.5) for k in (0, 1)]
    tables = []
    for w, c in zip(norms, convs):
        k = torch.zeros(taps, width)
        k[taps - real:, :count] = c.T.clone()
        k[-1, :count] += 1
        k[:, :count] *= w
        tables.append(k.cuda())
    ring = torch.full((B, taps, width), float("nan"), dtype=dtype, device="cuda")
    flat = lambda t: t[:, :S].reshape(B * S, width).cuda()
    kw = dict(k2=tables[1] if two else None, first=i32(first))
    got = [t if t is None else t.view(B, S, width) for t in stream_conv(flat(x), tables[0], ring, eps, B, count, y=flat(y), **kw)]
    src = x.to(dtype)
    ring2 = torch.zeros_like(ring)
    from_src = stream_conv(None, tables[0], ring2, eps, B, count, src=flat(src), **kw)
    assert torch.equal(from_src[0].cpu(), flat(src).float().cpu())
    outs = [[g] if g is not None else None for g in got]
    for s in range(steps):
        row = lambda t: t[:, S + s].contiguous().cuda()
        for k, t in enumerate(stream_conv(row(x), tables[0], ring, eps, B, count, y=row(y), pos_device=i32(S + s), **kw)):
            if t is not None:
                outs[k].append(t.view(B, 1, width))
    some = sorted({0, 1, B // 2, B - 1} & set(range(B)))
    for b in some:
        f = first[b]
        new = x[b, f:, :count].double() + y[b, f:, :count].double()
        assert rel(torch.cat([o[b] for o in outs[0]])[f:, :count], new) < 1e-6
        for k in range(2 if two else 1):
            want = P.mixed_input(P.rms_norm(new, norms[k].double(), eps), convs[k].double())
            full = torch.cat([o[b] for o in outs[1 + k]])
            assert rel(full[f:, :count], want) < tol(dtype) and float(full[:, count:].float().abs().sum()) == 0
    assert two or got[2] is None


# ---- selective scan -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("B,S,inner,states,rank", [(1, 1, 8, 4, 8), (2, 33, 40, 16, 16), (1, 100, 72, 24, 8), (3, 31, 264, 8, 24), (2, 65, 16, 32, 8), (1, 40, 24, 64, 16),
                                                   (1, 20, 16, 128, 8), (1, 18, 8, 256, 8), (2, 17, 136, 4, 40), (70, 5, 24, 12, 8), (16, 40, 520, 16, 8), (64, 9, 640, 16, 8)])
def test_selective_scan_and_step(dtype, B, S, inner, states, rank):
    from energonai_b200.decay import selective_scan, selective_step
    steps = 3
    n = S + steps
    x, g, low = rnd(B, n, inner, seed=1).to(dtype), rnd(B, n, inner, seed=2).to(dtype), rnd(B, n, rank, seed=3).to(dtype)
    bc, w = rnd(B, n, 2 * states, seed=4), rnd(inner, rank, seed=5, scale=rank ** -0.5).to(dtype)
    bias, a_log, skip = rnd(inner, seed=6) - 2.0, rnd(inner, states, seed=7) - 1.5, rnd(inner, seed=8)
    first = [0] + [S // 3] * (B - 1)
    z = low.double() @ w.double().T
    dev = [t.cuda() for t in (bias, a_log, skip)]
    S_ = torch.full((B, inner, states), 7.0, device="cuda")
    flat = lambda t: t[:, :S].reshape(B * S, -1).cuda()
    wide = torch.zeros(B * S, inner + 16, dtype=dtype, device="cuda")              # the result as columns of wider rows
    out = selective_scan(flat(x), flat(g), flat(z.float()), flat(bc), *dev, S_, first=i32(first), out=wide[:, 8:8 + inner]).reshape(B, S, inner)
    assert float(wide[:, :8].float().abs().sum()) == 0 and float(wide[:, 8 + inner:].float().abs().sum()) == 0
    outs = [out]
    states_prompt = S_.clone()
    for s in range(steps):
        row = lambda t: t[:, S + s].contiguous().cuda()
        outs.append(selective_step(row(x), row(g), row(low), w.cuda(), row(bc), *dev, S_).view(B, 1, inner))
    got = torch.cat(outs, 1)
    for b in sorted({0, 1, B // 2, B - 1} & set(range(B))):
        d = lambda t: t[b, first[b]:].double()
        dt = torch.nn.functional.softplus(d(z) + bias.double(), threshold=1e9)
        B_, C_ = d(bc).split(states, 1)
        y, last = P.selective_scan(d(x), dt, -torch.exp(a_log.double()), B_, C_, skip.double())
        _, at_prompt = P.selective_scan(d(x)[:S - first[b]], dt[:S - first[b]], -torch.exp(a_log.double()), B_[:S - first[b]], C_[:S - first[b]], skip.double())
        assert rel(got[b, first[b]:], y * P.silu(d(g))) < tol(dtype, 5e-6)
        assert rel(S_[b], last) < (5e-6 if dtype == F32 else 5e-3) and rel(states_prompt[b], at_prompt) < 5e-6


def test_selective_scan_over_a_long_sequence():
    """Slow decays: the state remembers thousands of tokens, and rounding does not add up."""
    from energonai_b200.decay import selective_scan
    n, inner, states = 3000, 16, 16
    x, g, z, bc = rnd(n, inner, seed=1), rnd(n, inner, seed=2), rnd(n, inner, seed=3) - 4.0, rnd(n, 2 * states, seed=4)
    bias, a_log, skip = torch.zeros(inner), rnd(inner, states, seed=5) - 2.5, torch.ones(inner)
    S = torch.empty(1, inner, states, device="cuda")
    got = selective_scan(*(t.cuda() for t in (x, g, z, bc, bias, a_log, skip)), S)
    dt = torch.nn.functional.softplus(z.double())
    y, last = P.selective_scan(x.double(), dt, -torch.exp(a_log.double()), *bc.double().split(states, 1), skip.double())
    assert rel(got, y * P.silu(g.double())) < 2e-5 and rel(S[0], last) < 2e-5


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("taps,S,C", [(1, 5, 8), (2, 1, 40), (4, 9, 264), (6, 3, 16)])
def test_short_conv_of_steps(dtype, taps, S, C):
    from energonai_b200.decay import short_conv, short_conv_step
    B, steps = 3, 7
    x, w, b = rnd(B, S + steps, C, seed=1).to(dtype), rnd(C, taps, seed=2).to(dtype), rnd(C, seed=3).to(dtype)
    first = [0, min(1, S - 1), S - 1]
    ring = torch.full((B, taps, C), float("nan"), dtype=dtype, device="cuda")
    wt = w.T.contiguous().cuda()
    got = [short_conv(x[:, :S].reshape(B * S, C).cuda(), wt, b.cuda(), ring, B, first=i32(first)).view(B, S, C)]
    for s in range(steps):
        got.append(short_conv_step(x[:, S + s].contiguous().cuda(), wt, b.cuda(), ring, i32(S + s), first=i32(first)).view(B, 1, C))
    got = torch.cat(got, 1)
    for r in range(B):
        want = P.silu(P.causal_conv(x[r, first[r]:].double(), w.double()) + b.double())
        assert rel(got[r, first[r]:], want) < tol(dtype)


# ---- capped attention -------------------------------------------------------------------------------------------
def capped_case(dtype, B, n, H, G, d, seed=0, loud=1.0):
    q, k, v = (rnd(B, n, h * d, seed=seed + i).to(dtype) for i, h in enumerate((H, G, G)))
    return q * loud, k, v, rnd(B, n, H * d, seed=seed + 3).to(dtype)


def plain_capped(q, k, v, gate, H, G, scale, cap, size, keep):
    n = q.shape[0]
    o = P.capped_attention(q.double().view(n, H, -1), k.double().view(n, G, -1), v.double().view(n, G, -1), scale, cap, P.window_mask(n, size or None, keep)).reshape(n, -1)
    return o * torch.sigmoid(gate.double()) if gate is not None else o


CAPPED = [  # n, heads, key heads, window, kept, cap, loudness of the queries
    (5, 2, 1, 0, 0, 5.0, 1.0), (130, 4, 2, 0, 0, 0.0, 1.0), (300, 2, 2, 40, 3, 5.0, 4.0), (700, 3, 1, 100, 140, 50.0, 1.0), (700, 2, 1, 128, 128, 20.0, 30.0),
    (600, 2, 1, 129, 1, 3.0, 1.0), (513, 2, 1, 1, 2, 8.0, 1.0), (400, 20, 1, 130, 257, 30.0, 3.0), (260, 1, 1, 300, 7, 10.0, 1.0)]


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("n,H,G,size,keep,cap,loud", CAPPED)
def test_capped_attention_of_prompts_and_steps(dtype, n, H, G, size, keep, cap, loud):
    """The tensor-core kernels and the plain one, left padding, the ring behind kept rows, splits; series and exponential
    form of the cap (loud queries)."""
    from energonai_b200.attention import attention_group_decode_capped, attention_plain_capped, attention_prefill_capped, attention_values, distance_slopes, sigmoid_gate
    d, B, eps = 64, 2, 1e-5
    scale, first = 0.125, [0, min(n - 1, 37)]
    q, k, v, gate = capped_case(dtype, B, n, H, G, d, seed=n, loud=loud)
    slopes = distance_slopes(H, "cuda")
    assert torch.allclose(slopes.cpu().double(), P.slopes(H))
    rows = min(size, n) if size else n
    buf = torch.full((B, keep + rows, 2 * G * d), 3.0, dtype=dtype, device="cuda")
    kc, vc = buf[:, :, :G * d], buf[:, :, G * d:]
    proj = torch.cat([k, v], 2).reshape(B * n, -1).cuda()
    attention_values(proj[:, :G * d], proj[:, G * d:], G, d, eps, kc, vc, keep, n, first=i32(first))
    unit = P.unit_rms(v.double().view(B, n, G, d), eps).reshape(B, n, G * d)
    assert rel(proj[:, G * d:], unit.reshape(B * n, -1)) < tol(dtype)
    vn = proj[:, G * d:].reshape(B, n, G * d)
    for b in range(B):                                   # what the cache holds
        for p in range(first[b], n):
            if p - first[b] < keep:
                assert torch.equal(kc[b, p - first[b]].cpu(), k[b, p]) and torch.equal(vc[b, p - first[b]], vn[b, p])
            if n - p <= rows:
                assert torch.equal(kc[b, keep + p % rows].cpu(), k[b, p])
    rule = dict(window=size, keep=keep, scale=scale, slopes=slopes, cap=cap, first=i32(first))
    kd, gd = k.cuda(), gate.cuda()
    plain = attention_plain_capped(q.cuda(), kd, vn, H, d, d, kv_heads=G, sink=True, **rule)
    plain = sigmoid_gate(plain.view(B * n, -1), gd.view(B * n, -1)).view(B, n, -1)
    step_args = (q[:, -1].contiguous().cuda(), kc, vc)
    pos, last = i32(n - 1), gd[:, -1].contiguous()
    one = attention_plain_capped(q[:, -1:].cuda(), kc, vc, H, d, d, kept_rows=keep, kv_heads=G, sink=True, pos_device=pos, **rule)
    outs, steps = [plain], [sigmoid_gate(one.view(B, -1), last)]
    if dtype != F32:
        wide = torch.zeros(B, n, H * d + 64, dtype=dtype, device="cuda")
        outs.append(attention_prefill_capped(q.cuda(), kd, vn, d, d, gate=gd, out=wide[:, :, 64:], **rule))
        steps += [attention_group_decode_capped(*step_args, d, pos, gate=last, nsplit=s, **rule) for s in (1, 3)]
    for b in range(B):
        f = first[b]
        want = plain_capped(q[b, f:], k[b, f:], vn[b, f:].cpu(), gate[b, f:], H, G, scale, cap, size, keep)
        for o in outs:
            assert rel(o[b, f:], want) < tol(dtype, 2e-5)
        for o in steps:
            assert rel(o[b:b + 1], want[-1:]) < tol(dtype, 2e-5)


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("d,dv,sink", [(128, 64, True), (128, 128, False), (64, 64, False)])
def test_capped_attention_other_heads_and_no_sink(dtype, d, dv, sink):
    from energonai_b200.attention import attention_prefill_capped, distance_slopes
    n, H, G = 330, 4, 2
    q, k, v = rnd(1, n, H * d, seed=1).to(dtype), rnd(1, n, G * d, seed=2).to(dtype), rnd(1, n, G * dv, seed=3).to(dtype)
    got = attention_prefill_capped(q.cuda(), k.cuda(), v.cuda(), d, dv, window=70, keep=4, slopes=distance_slopes(H, "cuda"), cap=6.0, sink=sink, scale=0.1)
    s = torch.einsum("ihd,jhd->hij", q[0].double().view(n, H, d), k[0].double().view(n, G, d)[:, [0, 0, 1, 1]]) * 0.1
    s = 6.0 * torch.tanh(s / 6.0) - P.slopes(H)[:, None, None] * (torch.arange(n)[:, None] - torch.arange(n)[None, :])
    p = P.softmax_with_sink(s, P.window_mask(n, 70, 4), torch.zeros(H, dtype=torch.float64) if sink else None)
    want = torch.einsum("hij,jhd->ihd", p, v[0].double().view(n, G, dv)[:, [0, 0, 1, 1]]).reshape(n, -1)
    assert rel(got[0], want) < tol(dtype)


# ---- rotary latent attention ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("dims,base,scaling", [(16, 1e4, None), (2, 10.0, None), (64, 1e5, (16.0, 4096, 32.0, 1.0)), (8, 100.0, (4.0, 30, 4.0, 0.5)), (32, 5e5, (2.0, 100, 1.0, 1.0)),
                                               (12, 50.0, (8.0, 10, 100.0, 50.0))])
def test_rotation_tables_and_rotated_heads(dims, base, scaling):
    from energonai_b200.attention import rotate_heads, yarn_rotation
    d = dict(zip(("factor", "original", "fast", "slow"), scaling)) if scaling else None
    freq, factor = yarn_rotation(dims, base, scaling)
    want, wf = P.yarn(dims, base, d)
    assert torch.allclose(freq.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-6) and abs(factor - wf) < 1e-12
    B, S, H, cols, at = 2, 40, 3, dims + 24, 8
    first, start = [0, 5], 1000
    for dtype in (F32, BF16):
        x = rnd(B * S, H * cols, seed=1).to(dtype)
        got = rotate_heads(x.cuda().clone(), H, cols, at, freq.cuda(), factor, S, pos_device=i32(start), first=i32(first)).cpu().view(B, S, H, cols)
        y = x.view(B, S, H, cols)
        assert torch.equal(got[..., :at], y[..., :at]) and torch.equal(got[..., at + dims:], y[..., at + dims:])
        for b in range(B):
            ref = P.rotate(y[b, :, :, at:at + dims].double(), [start + s - first[b] for s in range(S)], {"dims": dims, "base": base, "scaling": d})
            assert rel(got[b, :, :, at:at + dims].reshape(S, -1), ref.reshape(S, -1)) < (2e-4 if dtype == F32 else 8e-3)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("q_cols,q_count,rank,kv,rot", [(24, 20, 64, 18, 6), (8, 8, 16, 3, 2), (768, 768, 320, 256, 32), (200, 193, 136, 100, 28)])
def test_latent_inputs(dtype, q_cols, q_count, rank, kv, rot):
    from energonai_b200.attention import latent_inputs, yarn_rotation
    B, S, eps, scaling = 2, 7, 1e-4, (4.0, 30, 4.0, 0.5)
    at = -(-kv // 8) * 8
    pad = lambda t, n: torch.nn.functional.pad(t, (0, n - t.shape[-1]))
    dq, c, kr = rnd(B * S, q_count, seed=1), rnd(B * S, kv, seed=2), rnd(B * S, rot, seed=3)
    proj = torch.cat([pad(dq, q_cols), pad(torch.cat([pad(c, at), kr], 1), rank), rnd(B * S, 16, seed=4)], 1).to(dtype)
    qn, cn = pad(1 + 0.3 * rnd(q_count, seed=5), q_cols).to(dtype), pad(1 + 0.3 * rnd(kv, seed=6), at).to(dtype)
    freq, factor = yarn_rotation(rot, 100.0, scaling)
    first, start = [0, 3], 20
    ring = torch.zeros(B, 4, rank, dtype=dtype, device="cuda")
    row = dict(cols=rank, rot_col=at, count=kv, norm=cn.cuda(), freq=freq.cuda(), factor=factor, ring=ring, keep_rows=True)
    q, rows = latent_inputs(proj.cuda(), q_cols, q_count, qn.cuda(), eps, row=row, rows_per_batch=S, pos_device=i32(start), first=i32(first))
    d = lambda t: t.to(dtype).double()
    assert rel(q[:, :q_count], P.rms_norm(d(dq), qn[:q_count].double(), eps)) < tol(dtype) and float(q[:, q_count:].float().abs().sum()) == 0
    rows = rows.view(B, S, rank)
    for b in range(B):
        part = slice(b * S, b * S + S)
        assert rel(rows[b, :, :kv], P.rms_norm(d(c)[part], cn[:kv].double(), eps)) < tol(dtype)
        want = P.rotate(d(kr)[part][:, None], [start + s - first[b] for s in range(S)], {"dims": rot, "base": 100.0, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling))})
        assert rel(rows[b, :, at:at + rot], want[:, 0]) < tol(dtype, 2e-5)
        assert float(rows[b, :, kv:at].float().abs().sum()) == 0 and float(rows[b, :, at + rot:].float().abs().sum()) == 0
        for s in range(S - 4, S):
            assert torch.equal(ring[b, (start + s) % 4], rows[b, s])
    alone, none = latent_inputs(proj.cuda(), q_cols, q_count, qn.cuda(), eps)      # a layer without latents of its own
    assert torch.equal(alone, q) and none is None


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("n,H,dk,dv", [(3, 2, 64, 64), (200, 3, 128, 64), (300, 2, 128, 128), (520, 1, 128, 64), (1, 1, 192, 128), (390, 3, 192, 128), (257, 2, 192, 64)])
def test_gated_prompt_attention_with_sinks(dtype, n, H, dk, dv):
    from energonai_b200.attention import attention_prefill_gated
    B, first = 2, [0, min(n - 1, 140)]
    q, k, v, g = (rnd(B, n, H * w, seed=i).to(dtype) for i, w in ((1, dk), (2, dk), (3, dv), (4, dv)))
    sinks = rnd(H, seed=5) * 2
    got = attention_prefill_gated(q.cuda(), k.cuda(), v.cuda(), dk, dv, sinks=sinks.cuda(), first=i32(first), gate=g.cuda(), scale=0.11)
    for b in range(B):
        m = n - first[b]
        d = lambda t, w: t[b, first[b]:].double().view(m, H, w)
        s = torch.einsum("ihd,jhd->hij", d(q, dk), d(k, dk)) * 0.11
        o = torch.einsum("hij,jhd->ihd", P.softmax_with_sink(s, P.window_mask(m, None, 0), sinks.double()), d(v, dv)).reshape(m, -1)
        assert rel(got[b, first[b]:], o * torch.sigmoid(g[b, first[b]:].double())) < tol(dtype)


@pytest.mark.parametrize("R,H,n", [(64, 3, 20), (192, 16, 130), (192, 20, 600), (320, 5, 700), (320, 33, 64), (512, 17, 300), (576, 3, 700), (576, 18, 130)])
def test_latent_decode_with_sinks(R, H, n):
    """The sink joins once, whatever the splits."""
    from energonai_b200.attention import attention_plain, latent_decode
    B, first, scale = 2, [0, n // 3], R ** -0.5
    q, c, sinks = rnd(B, H * R, seed=1).to(BF16), rnd(B, n + 5, R, seed=2).to(BF16), rnd(H, seed=3) * 2 + 2
    for nsplit in (1, 2, 3, 4, 9):
        got = latent_decode(q.cuda(), c.cuda(), R, H, 0, i32(n - 1), scale, first=i32(first), sinks=sinks.cuda(), nsplit=nsplit)
        for b in range(B):
            cc = c[b, first[b]:n].double()
            s = (q[b].double().view(H, 1, R) * cc[None]).sum(-1)[:, None] * scale
            p = P.softmax_with_sink(s, torch.ones(1, cc.shape[0], dtype=torch.bool), sinks.double())
            assert rel(got[b].view(H, R), (p[:, 0] @ cc)) < 8e-3, nsplit
    plain = attention_plain(q.cuda().view(B, 1, -1), c.cuda(), c.cuda(), H, R, R, scale=scale, first=i32(first), pos_device=i32(n - 1), shared_kv=True, chunk=0, sinks=sinks.cuda())
    assert rel(plain.view(B, -1), got) < 8e-3


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
def test_sigmoid_gate_and_strided_units(dtype):
    from energonai_b200.attention import sigmoid_gate
    from energonai_b200.gemm import project_unit
    y, g = rnd(37, 72, seed=1).to(dtype), rnd(37, 72, seed=2, scale=3.0).to(dtype)
    wide = torch.zeros(37, 136, dtype=dtype, device="cuda")
    sigmoid_gate(y.cuda(), g.cuda(), out=wide[:, 64:])
    assert rel(wide[:, 64:], y.double() * torch.sigmoid(g.double())) < tol(dtype, 1e-6) and float(wide[:, :64].float().abs().sum()) == 0
    for M in (3, 37, 300):                               # a feed-forward's unit into columns of wider rows
        x, a, b = rnd(M, 64, seed=3).to(dtype), rnd(72, 64, seed=4, scale=0.2).to(dtype), rnd(72, 64, seed=5, scale=0.2).to(dtype)
        w = torch.cat([a.view(-1, 1, 8, 64), b.view(-1, 1, 8, 64)], 1).reshape(144, 64)
        wide = torch.zeros(M, 136, dtype=dtype, device="cuda")
        project_unit(x.cuda(), w.cuda(), "geglu", out=wide[:, 64:])
        want = P.gelu_tanh(x.double() @ a.double().T) * (x.double() @ b.double().T)
        assert rel(wide[:, 64:], want) < tol(dtype) and float(wide[:, :64].float().abs().sum()) == 0
