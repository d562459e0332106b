"""Kernels of the state-space / chunk-attention / gated-linear decoder against the plain restatement."""
import pytest
import torch

import moponex_plain as P

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


def heads_close(got, want, tol):
    """Head by head: the error of a head's rows over their own size."""
    got, want = got.double().cpu(), want.double()
    assert got.shape == want.shape and torch.isfinite(got).all()
    for h in range(want.shape[1]):
        assert float((got[:, h] - want[:, h]).pow(2).mean().sqrt() / want[:, h].pow(2).mean().sqrt()) < tol, h


def firsts(B, S):
    return [0] + [min(S - 1, S // 2 + 1)] * (B - 1)


def i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


# ---- products with a unit -----------------------------------------------------------------------------------
def interleave(gate, up):
    return torch.cat([gate.view(-1, 1, 8, gate.shape[1]), up.view(-1, 1, 8, up.shape[1])], 1).reshape(-1, gate.shape[1])


@pytest.mark.parametrize("dtype", [F32, BF16, F16])
@pytest.mark.parametrize("M,N,K", [(1, 8, 40), (16, 136, 264), (31, 72, 64), (33, 64, 96), (130, 264, 200), (300, 1024, 512)])
def test_units_in_the_epilogue_of_a_product(dtype, M, N, K):
    from energonai_b200.gemm import project_unit
    x, g, u = rnd(M, K, seed=1).to(dtype), rnd(N, K, seed=2, scale=2 * K ** -0.5).to(dtype), rnd(N, K, seed=3, scale=K ** -0.5).to(dtype)
    tol = {F32: 2e-6, BF16: 6e-3, F16: 1e-3}[dtype]
    zg, zu = x.double() @ g.double().T, x.double() @ u.double().T
    assert rel(project_unit(x.cuda(), interleave(g, u).cuda(), "geglu"), P.gelu_tanh(zg) * zu) < tol
    assert rel(project_unit(x.cuda(), g.cuda(), "gelu"), P.gelu_erf(zg)) < tol


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("unit", ["gelu", "geglu"])
def test_units_of_experts(dtype, unit):
    from energonai_b200.moe import SortedRows, grouped_gemm, new_counts, route_rule, RouterRule, skinny_experts
    T, E, K, ff, top = 40, 5, 72, 48, 2
    x, gate, up = rnd(T, K, seed=1).to(dtype), rnd(E, ff, K, seed=2, scale=K ** -0.5).to(dtype), rnd(E, ff, K, seed=3, scale=K ** -0.5).to(dtype)
    w = up if unit == "gelu" else torch.stack([interleave(a, b) for a, b in zip(gate, up)])
    counts = new_counts(E, "cuda")
    idx, _, ranks, _ = route_rule(rnd(T, E + 3, seed=4).cuda(), RouterRule(E + 1, E), top, counts=counts)
    want = torch.zeros(T, top, ff, dtype=torch.float64)
    live = (idx < E).cpu()
    for t in range(T):
        for k in range(top):
            e = int(idx[t, k])
            if e < E:
                z = up[e].double() @ x[t].double()
                want[t, k] = P.gelu_erf(z) if unit == "gelu" else P.gelu_tanh(gate[e].double() @ x[t].double()) * z
    assert 0 < int((~live).sum())                        # some choices are the input itself: no rows
    tol = 2e-6 if dtype == F32 else 6e-3
    plan = SortedRows(x.cuda(), idx, ranks, counts)
    y = grouped_gemm(plan.x, w.cuda(), plan, unit=unit)
    assert int(counts.abs().sum()) == 0 and bool((plan.rows.cpu()[~live] == -1).all())
    assert rel(y[plan.rows.cpu()[live].long().cuda()], want[live]) < tol
    if dtype == BF16:
        y = skinny_experts(x.cuda(), w.cuda(), idx, top, unit=unit).view(T, top, ff)
        assert rel(y.cpu()[live], want[live]) < tol


# ---- router ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("T,E,identity,top,groups,keep", [(33, 16, 0, 4, 1, 1), (40, 13, 2, 3, 3, 2), (7, 5, 1, 2, 2, 1), (20, 60, 4, 40, 4, 3), (11, 130, 6, 40, 34, 20), (9, 3, 0, 1, 3, 1),
                                                          (12, 250, 6, 8, 8, 4)])
def test_router_rule(T, E, identity, top, groups, keep):
    from energonai_b200.moe import RouterRule, new_counts, route_rule
    n = E + identity
    z, corr, gate = rnd(T, n, seed=T, scale=2.0), rnd(n, seed=5, scale=0.3) - 1.5, rnd(T, seed=6)
    logits = torch.cat([z, gate[:, None], rnd(T, 3, seed=7)], 1).cuda()
    want_idx, want_w = P.choose(z.double(), corr.double(), top, groups, keep)
    rule = RouterRule(n, E, corr.cuda(), groups, keep)
    counts = new_counts(E, "cuda")
    idx, w, ranks, g = route_rule(logits, rule, top, counts=counts, gated=True)
    for t in range(T):
        assert idx[t].tolist() == want_idx[t]
    assert torch.allclose(w.cpu().double(), torch.stack(want_w), rtol=2e-5, atol=1e-7)
    assert torch.allclose(g.cpu(), torch.sigmoid(gate), rtol=1e-5)
    per = counts.view(E, -1)[:, 0].cpu()
    for e in range(E):
        r = sorted(ranks.cpu()[idx.cpu() == e].tolist())
        assert r == list(range(int(per[e])))
    assert bool((ranks.cpu()[idx.cpu() >= E] == -1).all())
    # padding gets no expert
    idx, w, _, g = route_rule(logits[:T // 2 * 2], rule, top, first=i32([1, T // 2]), rows_per_batch=T // 2, gated=True)
    assert bool((idx[0] == -1).all()) and bool((idx[T // 2:] == -1).all()) and float(g[0]) == 0.0 and idx[1].tolist() == want_idx[1]


# ---- residual step ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,width,count", [(1, 40, 36), (5, 2056, 2056), (3, 4096, 4090), (2, 16384, 16384)])
def test_stream_add(dtype, rows, width, count):
    from energonai_b200.norm import stream_add
    pad = lambda t: torch.nn.functional.pad(t, (0, width - count))
    a, b, x0 = (pad(rnd(rows, count, seed=s)).to(dtype) for s in (1, 2, 3))
    wa, wb, wn = pad(1 + rnd(count, seed=4)), pad(1 + rnd(count, seed=5)), pad(1 + rnd(count, seed=6)).to(dtype)
    eps, m, s, tol = 1e-3, 0.3, 1.7, 3e-6 if dtype == F32 else 6e-3
    d = lambda t: t[..., :count].double()
    nxt = dict(w_next=wn.cuda(), next_scale=s)
    last = lambda x: P.rms_norm(x, d(wn), eps) * s
    # the start: one row, or two
    for second in (None, b):
        x = torch.empty(rows, width, device="cuda")
        h = stream_add(x, eps, count, src=a.cuda(), src2=None if second is None else second.cuda(), **nxt)
        want = d(a) + (0 if second is None else d(second))
        assert rel(x[:, :count], want) < 1e-6 and rel(h[:, :count], last(want)) < tol and float(x[:, count:].abs().sum()) == 0
    # a row; two rows normalised each by itself
    x = x0.float().cuda()
    h = stream_add(x, eps, count, y=a.cuda(), scale=m, **nxt)
    want = d(x0) + m * d(a)
    assert rel(x[:, :count], want) < 1e-6 and rel(h[:, :count], last(want)) < tol
    x = x0.float().cuda()
    h = stream_add(x, eps, count, y=a.cuda(), w=wa.cuda(), y2=b.cuda(), w2=wb.cuda(), scale=m, **nxt)
    want = d(x0) + m * (P.rms_norm(d(a), d(wa), eps) + P.rms_norm(d(b), d(wb), eps))
    assert rel(x[:, :count], want) < 3e-6 and rel(h[:, :count], last(want)) < tol
    # no norm behind it; a norm alone leaves x as it is
    x = x0.float().cuda()
    assert stream_add(x, eps, count, y=a.cuda(), scale=m) is None and rel(x[:, :count], d(x0) + m * d(a)) < 1e-6
    x = x0.float().cuda()
    assert rel(stream_add(x, eps, count, **nxt)[:, :count], last(d(x0))) < tol and torch.equal(x.cpu(), x0.float())


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("width,experts,identity,top,groups,keep,gated", [(64, 6, 2, 3, 2, 1, True), (2048, 30, 2, 6, 4, 3, True), (40, 4, 0, 1, 1, 1, False),
                                                                          (9000, 12, 4, 5, 4, 2, True)])
def test_stream_add_of_a_mixture_and_the_router_behind_it(dtype, width, experts, identity, top, groups, keep, gated):
    from energonai_b200.moe import RouterRule
    from energonai_b200.norm import stream_add
    T, n, eps, m = 6, experts + identity, 1e-4, 0.8
    g = torch.Generator().manual_seed(1)
    y, h0, sh, x0 = rnd(T * top, width, seed=1).to(dtype), rnd(T, width, seed=2).to(dtype), rnd(T, width, seed=3).to(dtype), rnd(T, width, seed=4)
    idx = torch.stack([torch.randperm(n, generator=g)[:top] for _ in range(T)]).to(torch.int32)
    idx[2, 0] = -1
    if identity:
        idx[3, 0] = n - 1
    w, gate = torch.rand(T, top, generator=g), torch.rand(T, generator=g)
    rows = torch.randperm(T * top, generator=g).view(T, top).to(torch.int32)
    wn, router, corr = (1 + rnd(width, seed=5)).to(dtype), rnd(n + 5, width, seed=6, scale=2 * width ** -0.5).to(dtype), rnd(n, seed=7) - 1.0
    for r in (None, rows):
        want = x0.double().clone()
        for t in range(T):
            for k in range(top):
                e = int(idx[t, k])
                if e >= 0:
                    want[t] += m * float(w[t, k]) * (h0[t] if e >= experts else y[int(r[t, k]) if r is not None else t * top + k]).double()
            if gated:
                want[t] += m * float(gate[t]) * sh[t].double()
        x = x0.cuda()
        h, (ri, rw, rg) = stream_add(x, eps, y=y.cuda(), mix=(idx.cuda(), None if r is None else r.cuda(), w.cuda()), ident=h0.cuda(), experts=experts,
                                     shared=sh.cuda() if gated else None, gate=gate.cuda() if gated else None, scale=m, w_next=wn.cuda(),
                                     router=(router.cuda(), RouterRule(n, experts, corr.cuda(), groups, keep), top, gated))
        assert rel(x, want) < 2e-6
        assert rel(h, P.rms_norm(want, wn.double(), eps)) < (3e-6 if dtype == F32 else 6e-3)
        z = h.double().cpu() @ router.double().T                         # (the router reads h as it is rounded)
        want_idx, want_w = P.choose(z[:, :n], corr.double(), top, groups, keep)
        assert [ri[t].tolist() for t in range(T)] == want_idx
        assert torch.allclose(rw.cpu().double(), torch.stack(want_w), rtol=1e-4, atol=1e-6)
        assert (rg is None) == (not gated) and (rg is None or torch.allclose(rg.cpu().double(), torch.sigmoid(z[:, n]), rtol=1e-4))


def test_stream_add_of_a_mixture_of_many_rows():
    from energonai_b200.norm import stream_add
    T, width, E, top = 700, 72, 5, 3
    g = torch.Generator().manual_seed(2)
    y, h0, sh, x0 = rnd(T * top, width, seed=1), rnd(T, width, seed=2), rnd(T, width, seed=3), rnd(T, width, seed=4)
    idx, w, gate = torch.randint(0, E + 2, (T, top), generator=g).to(torch.int32), torch.rand(T, top, generator=g), torch.rand(T, generator=g)
    rows = torch.where(idx[..., None] < E, y.view(T, top, width), h0[:, None])
    want = x0.double() + 0.5 * ((w[..., None].double() * rows.double()).sum(1) + gate[:, None].double() * sh.double())
    x = x0.cuda()
    stream_add(x, 1e-5, y=y.cuda(), mix=(idx.cuda(), None, w.cuda()), ident=h0.cuda(), experts=E, shared=sh.cuda(), gate=gate.cuda(), scale=0.5)
    assert rel(x, want) < 2e-6


# ---- bigram rows in the tail of a step ---------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
def test_greedy_step_with_bigram_rows(dtype):
    from energonai_b200.step import greedy_step
    B, V, h, buckets, mp, mc = 3, 50, 24, 37, 1000003, 77
    emb, table = rnd(V, h, seed=1).to(dtype).cuda(), rnd(buckets + 1, h, seed=2).to(dtype).cuda()
    out_ids = torch.randint(0, V, (B, 9), generator=torch.Generator().manual_seed(3)).cuda()
    before = out_ids.clone()
    kv, counter = i32([4, 5]), torch.zeros(1, dtype=torch.int32, device="cuda")
    hid, pair, tok = torch.empty(B, h, dtype=dtype, device="cuda"), torch.empty(B, h, dtype=dtype, device="cuda"), torch.empty(B, dtype=torch.int64, device="cuda")
    for col in (5, 6):
        logits = rnd(B, V, seed=col).cuda()
        new = logits.argmax(-1)
        greedy_step(logits, out_ids, tok, kv, counter, word_emb=emb, hidden_out=hid, add_pos=False, bigram=(table, mp, mc, buckets, pair))
        assert torch.equal(out_ids[:, col], new) and torch.equal(hid, emb[new])
        prev = (before[:, 4] if col == 5 else out_ids[:, 5]).tolist()
        rows = [P.bigram_rows([a, b], mp, mc, buckets)[1] for a, b in zip(prev, new.tolist())]
        assert torch.equal(pair, table[torch.tensor(rows, device="cuda")])
    assert kv.tolist() == [6, 7]


# ---- convolution ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("B,S,C,taps", [(1, 1, 8, 4), (2, 3, 40, 4), (2, 50, 1032, 4), (1, 17, 16, 2), (2, 33, 24, 3), (2, 20, 16, 1), (1, 40, 8, 7)])
def test_short_convolution(dtype, B, S, C, taps):
    from energonai_b200.decay import short_conv
    x, w, b = rnd(B, S, C + 16, seed=1).to(dtype), rnd(C, taps, seed=2).to(dtype), rnd(C, seed=3).to(dtype)
    first, R = firsts(B, S), min(taps, S)
    ring = torch.full((B, R, C), 9.0, dtype=dtype, device="cuda")
    out = short_conv(x.cuda().view(B * S, -1)[:, 8:8 + C], w.t().contiguous().cuda(), b.cuda(), ring, B, first=i32(first) if any(first) else None).view(B, S, C)
    for r in range(B):
        f = first[r]
        want = P.silu(P.short_conv(x[r, f:, 8:8 + C].double(), w.double(), b.double()))
        assert rel(out[r, f:], want) < (1e-6 if dtype == F32 else 6e-3)
        for p in range(max(f, S - R), S):
            assert torch.equal(ring[r, p % R].cpu(), x[r, p, 8:8 + C])
    assert torch.isfinite(out).all()


# ---- state space -----------------------------------------------------------------------------------------------------
def ssm_case(B, S, H, G, dk, dv, seed, speed):
    """Tokens of every kind of step size; one early token that stands out and is asked for by the last."""
    xbc = rnd(B, S, H * dv + 2 * G * dk, seed=seed)
    dt = rnd(B, S, H, seed=seed + 1, scale=1.5)
    if S > 4:
        at = H * dv
        xbc[:, 2, :at] *= 3.0
        xbc[:, -1, at + G * dk:] = 2.0 * xbc[:, 2, at:at + G * dk]
        dt[:, 2] += 3.0
    bias, a_log, skip = rnd(H, seed=seed + 2, scale=0.3) - 2.0, torch.linspace(speed - 2.0, speed, H), 0.5 + rnd(H, seed=seed + 3, scale=0.3)
    return xbc, dt, bias, a_log, skip


def ssm_want(xbc, dt, bias, a_log, skip, H, G, dk, dv, first):
    out = []
    for b in range(xbc.shape[0]):
        x, Bm, C = xbc[b, first[b]:].double().split([H * dv, G * dk, G * dk], 1)
        n = x.shape[0]
        step = torch.nn.functional.softplus(dt[b, first[b]:].double() + bias.double(), threshold=1e9)
        out.append(P.ssm_scan(x.view(n, H, dv), Bm.view(n, G, dk), C.view(n, G, dk), step, a_log.double(), skip.double()))
    return out


@pytest.mark.parametrize("path,dtype", [("scan", F32), ("scan", BF16), ("chunks", BF16)])
@pytest.mark.parametrize("B,S,H,G,dk,dv", [(1, 1, 2, 1, 64, 64), (2, 5, 4, 2, 64, 64), (2, 127, 3, 3, 128, 64), (1, 128, 2, 1, 64, 136), (2, 129, 4, 1, 128, 64),
                                           (2, 300, 6, 2, 64, 64), (1, 700, 2, 1, 128, 128), (1, 520, 2, 2, 128, 264)])
@pytest.mark.parametrize("speed", [-2.0, 3.0])
def test_state_space_prompt_and_steps_behind_it(path, dtype, B, S, H, G, dk, dv, speed):
    from energonai_b200.decay import ssm_prompt, ssm_step
    more, taps = 6, 1
    xbc, dt, bias, a_log, skip = ssm_case(B, S + more, H, G, dk, dv, seed=B + S, speed=speed)
    xbc = xbc.to(dtype)
    first = firsts(B, S)
    # (steps go through a convolution of one tap: silu(x))
    seen = xbc.clone()
    seen[:, S:] = P.silu(xbc[:, S:].double()).to(dtype)
    want = ssm_want(seen, dt, bias, a_log, skip, H, G, dk, dv, first)
    state = torch.full((B, H, dk, dv), 7.0, device="cuda")
    vecs, fd, D = [v.cuda() for v in (bias, a_log, skip)], i32(first), dt.cuda()
    y = ssm_prompt(xbc[:, :S].reshape(B * S, -1).cuda(), D[:, :S].reshape(B * S, H).contiguous(), *vecs, state, H, G, dk, dv, first=fd if any(first) else None,
                   chunked=path == "chunks").view(B, S, H, dv)
    tol = 2e-5 if dtype == F32 else 1.5e-2
    for b in range(B):
        heads_close(y[b, first[b]:], want[b][0][:S - first[b]], tol)
        assert torch.isfinite(y[b].float()).all()
    ring = torch.zeros(B, 1, xbc.shape[2], dtype=dtype, device="cuda")
    one, zero = torch.ones(1, xbc.shape[2], dtype=dtype, device="cuda"), torch.zeros(xbc.shape[2], dtype=dtype, device="cuda")
    for t in range(S, S + more):
        y = ssm_step(xbc[:, t].contiguous().cuda(), one, zero, ring, i32([t]), D[:, t].contiguous(), *vecs, state, H, G, dk, dv, first=fd)
        for b in range(B):
            heads_close(y[b].view(1, H, dv), want[b][0][t - first[b]].view(1, H, dv), 3e-5 if dtype == F32 else 1.5e-2)
    # what enters the state is not rounded to 16 bits
    for b in range(B):
        heads_close(state[b].reshape(1, H, -1), want[b][1].reshape(1, H, -1), 3e-5)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("taps,first,start", [(4, 0, 0), (4, 2, 2), (3, 1, 1), (2, 0, 0), (6, 3, 3)])
def test_state_space_step_carries_the_convolution(dtype, taps, first, start):
    """Token by token from the very first one; the ring wraps."""
    from energonai_b200.decay import ssm_step
    B, H, G, dk, dv, n = 2, 4, 2, 16, 24, 15
    C = H * dv + 2 * G * dk
    x, w, cb = rnd(B, n, C, seed=1).to(dtype), rnd(C, taps, seed=2).to(dtype), rnd(C, seed=3).to(dtype)
    _, dt, bias, a_log, skip = ssm_case(B, n, H, G, dk, dv, seed=4, speed=0.0)
    ring = torch.full((B, taps, C), 1e4, dtype=dtype, device="cuda")         # what a sequence of the past left there
    state = torch.zeros(B, H, dk, dv, device="cuda")
    got = []
    for t in range(n):
        got.append(ssm_step(x[:, t].cuda(), w.t().contiguous().cuda(), cb.cuda(), ring, i32([t + start]), dt[:, t].cuda().contiguous(), bias.cuda(), a_log.cuda(),
                            skip.cuda(), state, H, G, dk, dv, first=i32([first] * B)))
    got = torch.stack(got, 1)
    seen = torch.stack([P.silu(P.short_conv(x[b].double(), w.double(), cb.double())) for b in range(B)])
    want = ssm_want(seen, dt, bias, a_log, skip, H, G, dk, dv, [0] * B)
    for b in range(B):
        assert rel(got[b], want[b][0].reshape(n, -1)) < (2e-5 if dtype == F32 else 1.5e-2)


@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("rows,H,dv,pad,parts", [(3, 4, 24, 24, 1), (2, 3, 20, 64, 5), (5, 6, 8, 8, 2), (400, 8, 64, 64, 4), (2, 64, 64, 64, 1), (3, 8, 48, 64, 3)])
def test_gate_and_norm_in_equal_parts(dtype, rows, H, dv, pad, parts):
    """Parts that are heads, several heads, and that straddle heads."""
    from energonai_b200.decay import gate_group_norm
    heads = lambda t: torch.nn.functional.pad(t.view(-1, H, dv), (0, pad - dv)).reshape(-1, H * pad)
    y, z, w = rnd(rows, H * dv, seed=1).to(dtype), rnd(rows, H * dv, seed=2).to(dtype), (1 + rnd(H * dv, seed=3)).to(dtype)
    y[:, :7] *= 30.0
    got = gate_group_norm(heads(y).cuda(), heads(z).cuda(), heads(w[None])[0].cuda(), 1e-3, H, dv, parts).view(rows, H, pad)
    want = P.group_norm(y.double() * P.silu(z.double()), w.double(), parts, 1e-3)
    assert rel(got[..., :dv].reshape(rows, -1), want) < (3e-6 if dtype == F32 else 6e-3) and float(got[..., dv:].abs().sum()) == 0


# ---- gated linear attention --------------------------------------------------------------------------------------------
@pytest.mark.parametrize("path,dtype", [("scan", F32), ("scan", BF16), ("chunks", BF16)])
@pytest.mark.parametrize("B,S,H,dk,dv", [(1, 1, 1, 64, 8), (2, 5, 2, 64, 40), (1, 127, 2, 128, 128), (2, 128, 1, 64, 136), (1, 129, 3, 128, 64), (2, 300, 2, 64, 256),
                                         (1, 700, 2, 128, 200)])
@pytest.mark.parametrize("tau,shift", [(16.0, 2.0), (1.0, 0.0), (0.5, -6.0)])
def test_gated_linear_prompt_and_steps_behind_it(path, dtype, B, S, H, dk, dv, tau, shift):
    """Decays from slow to so fast that a block of 16 tokens spans more than the exponents' range."""
    from energonai_b200.decay import gla_prompt, gla_step
    from energonai_b200.memory import head_norm_gate
    more, eps, rank, scale = 5, 1e-4, 24, dk ** -0.5
    n = S + more
    q, k, v, g = (rnd(B, n, H * d, seed=S + i) for i, d in enumerate((dk, dk, dv, dv)))
    if S > 4:
        k[:, 2] *= 3.0
        q[:, -1], q[:, S - 1] = k[:, 2], k[:, 2]
    low, w2, b2 = rnd(B, n, rank, seed=S + 5), rnd(H * dk, rank, seed=6, scale=2 * rank ** -0.5), rnd(H * dk, seed=7) + shift
    q, k, v, g, low, w2, b2 = (t.to(dtype) for t in (q, k, v, g, low, w2, b2))
    z = low.double() @ w2.double().T + b2.double()
    log_a = (torch.nn.functional.logsigmoid(z) / tau).view(B, n, H, dk)
    first = firsts(B, S)
    want = [P.gla_scan(*(t[b, first[b]:].double().view(-1, H, d) * s for t, d, s in ((q, dk, scale), (k, dk, 1.0), (v, dv, 1.0))), log_a[b, first[b]:]) for b in range(B)]
    proj = torch.cat([q, k, v, g, low], 2).cuda()
    cols = [H * dk, H * dk, H * dv, H * dv, rank]
    state, fd = torch.full((B, H, dk, dv), 7.0, device="cuda"), i32(first)
    pq, pk, pv, pg, _ = proj[:, :S].reshape(B * S, -1).split(cols, 1)
    o = gla_prompt(pq, pk, pv, z[:, :S].reshape(B * S, -1).float().cuda(), tau, scale, state, H, first=fd if any(first) else None, chunked=path == "chunks")
    tol = 3e-5 if dtype == F32 else 1.5e-2
    for b in range(B):
        heads_close(o.view(B, S, H, dv)[b, first[b]:], want[b][0][:S - first[b]], tol)
        assert torch.isfinite(o.float()).all()
    norm = (1 + rnd(H * dv, seed=20, scale=0.3)).to(dtype)
    y = head_norm_gate(o, pg, norm.cuda(), H, dv, eps, silu=True)
    ref = P.unit_rms(o.double().cpu().view(B * S, H, dv), eps).reshape(B * S, -1) * norm.double() * P.silu(pg.double().cpu())
    assert rel(y, ref) < (3e-6 if dtype == F32 else 6e-3)
    for t in range(S, n):
        y = gla_step(*proj[:, t].split(cols, 1), w2.cuda(), b2.cuda(), tau, scale, norm.cuda(), dv, eps, state, H)
        for b in range(B):
            ref = P.unit_rms(want[b][0][t - first[b]], eps).reshape(1, -1) * norm.double() * P.silu(g[b, t].double().reshape(1, -1))
            heads_close(y[b].view(1, H, dv), ref.view(1, H, dv), 5e-5 if dtype == F32 else 1.5e-2)
    for b in range(B):
        heads_close(state[b].reshape(1, H, -1), want[b][1].reshape(1, H, -1), 3e-5)


def test_gated_linear_step_in_clusters_and_uneven_columns():
    from energonai_b200.decay import gla_step
    for B, H, dk, dv in ((1, 1, 64, 512), (2, 3, 40, 264), (40, 8, 64, 72), (1, 2, 200, 2048)):
        q, k, v, g, low = (rnd(B, n, seed=s) for s, n in enumerate((H * dk, H * dk, H * dv, H * dv, 8)))
        w2, b2, norm, S0 = rnd(H * dk, 8, seed=6), rnd(H * dk, seed=7), 1 + rnd(H * dv, seed=8, scale=0.2), rnd(B, H, dk, dv, seed=9)
        state = S0.clone().cuda()
        y = gla_step(*torch.cat([q, k, v, g, low], 1).cuda().split([H * dk, H * dk, H * dv, H * dv, 8], 1), w2.cuda(), b2.cuda(), 4.0, 0.2, norm.cuda(), dv, 1e-5, state, H)
        a = torch.sigmoid(low.double() @ w2.double().T + b2.double()).pow(0.25).view(B, H, dk)
        S = a[..., None] * S0.double() + k.double().view(B, H, dk, 1) * v.double().view(B, H, 1, dv)
        o = torch.einsum("bhdv,bhd->bhv", S, q.double().view(B, H, dk) * 0.2)
        assert rel(y, P.unit_rms(o, 1e-5).reshape(B, -1) * norm.double() * P.silu(g.double())) < 2e-5
        assert rel(state.reshape(B, -1), S.reshape(B, -1)) < 2e-6


# ---- attention over chunks -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [F32, BF16])
@pytest.mark.parametrize("H,G,d,dk,dims", [(4, 2, 20, 24, 12), (3, 3, 64, 64, 64), (6, 1, 100, 128, 0), (1, 1, 6, 8, 2), (2, 2, 200, 200, 100)])
def test_rotary_queries_and_keys(dtype, H, G, d, dk, dims):
    from energonai_b200.attention import attention_rotary
    B, S, base, factor, eps = 2, 9, 500.0, 3.0, 1e-3
    heads = lambda t, n: torch.nn.functional.pad(t.view(*t.shape[:-1], n, d), (0, dk - d)).reshape(*t.shape[:-1], n * dk)
    pad = lambda w: torch.nn.functional.pad(w, (0, dk - d))
    q, k = rnd(B * S, H * d, seed=1).to(dtype), rnd(B * S, G * d, seed=2).to(dtype)
    wq, wk = (1 + rnd(d, seed=3)).to(dtype), (1 + rnd(d, seed=4)).to(dtype)
    proj = torch.cat([heads(q, H), heads(k, G), rnd(B * S, 16, seed=5).to(dtype)], 1).cuda()
    freq = (base ** (-2 * torch.arange(dims // 2, dtype=torch.float64) / max(1, dims)) / factor).float().cuda()
    first = [0, 4]
    for pos, rows in ((0, 9), (0, 4), (3, 12), (100003, 5)):
        ring = torch.full((B, rows, 2 * G * dk), 9.0, dtype=dtype, device="cuda")
        kc, vc = ring[:, :, :G * dk], ring[:, :, G * dk:]
        got, keys = attention_rotary(proj, H, G, dk, d, pad(wq).cuda(), pad(wk).cuda(), eps, freq, kc, vc, S, pos_device=None if pos == 0 else i32([pos]),
                                     first=i32(first), keys=True)
        # (frequencies as the kernel has them: the angle is their 32-bit product with the position)
        tol = (3e-6 if pos < 1000 else 2e-2) if dtype == F32 else (6e-3 if pos < 1000 else 2e-2)
        for b in range(B):
            at = [pos + s - first[b] for s in range(S)]
            live = [s for s in range(S) if at[s] >= 0]
            sl = lambda t, n: t.view(B, S, n, d)[b, live].double()
            turn = lambda t: P.rotate(t, [at[s] for s in live], dims, base, factor) if dims else t
            wantq, wantk = turn(P.rms_norm(sl(q, H), wq.double(), eps)), turn(P.rms_norm(sl(k, G), wk.double(), eps))
            assert rel(got.view(B, S, H, dk)[b, live][..., :d].reshape(len(live), -1), wantq.reshape(len(live), -1)) < tol
            mine = keys.view(B, S, G, dk)[b, live]
            assert rel(mine[..., :d].reshape(len(live), -1), wantk.reshape(len(live), -1)) < tol and float(mine[..., d:].abs().sum()) == 0
            for s in range(S):
                if S - s <= rows:
                    assert torch.equal(kc[b, (pos + s) % rows], keys.view(B, S, -1)[b, s]) and torch.equal(vc[b, (pos + s) % rows].cpu(), heads(k, G).view(B, S, -1)[b, s])


def chunk_case(B, S, H, G, D, chunk, first, seed=0):
    """Random heads; the last row's query asks for the keys on both sides of its chunk's first edge, which carry large
    values, and sinks are about as large as the largest scores."""
    q, k, v = rnd(B, S, H, D, seed=seed), rnd(B, S, G, D, seed=seed + 1), rnd(B, S, G, D, seed=seed + 2)
    for b in range(B):
        f = first[b]
        edge = f + (S - 1 - f) // chunk * chunk if chunk else f
        q[b, -1] = k[b, edge].repeat_interleave(H // G, 0) * 2.0
        v[b, edge] *= 4.0
        if edge > f:
            k[b, edge - 1] = k[b, edge]
            v[b, edge - 1] *= -9.0
    return q, k, v, torch.linspace(-1.0, 6.0, H)


def chunk_want(q, k, v, scale, sinks, chunk, first):
    out = []
    for b in range(q.shape[0]):
        f, n = first[b], q.shape[1] - first[b]
        out.append(P.sink_attention(q[b, f:].double(), k[b, f:].double(), v[b, f:].double(), scale, sinks.double(), P.chunk_mask(n, chunk or None)).reshape(n, -1))
    return out


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("B,S,H,G,D,chunk", [(1, 1, 2, 1, 64, 5), (2, 130, 4, 2, 64, 0), (2, 257, 6, 2, 128, 100), (1, 700, 4, 4, 128, 256), (2, 300, 4, 1, 64, 1),
                                             (2, 520, 2, 1, 128, 129), (1, 385, 2, 2, 64, 128), (3, 400, 2, 1, 64, 37), (1, 600, 2, 1, 64, 4000)])
def test_prompt_attention_over_chunks(dtype, B, S, H, G, D, chunk):
    from energonai_b200.attention import attention_plain, attention_prefill_chunk
    first = [0, S // 3, S - 1][:B]
    q, k, v, sinks = chunk_case(B, S, H, G, D, chunk, first)
    q, k, v = (t.to(dtype) for t in (q, k, v))
    scale, fd = D ** -0.5, i32(first) if any(first) else None
    flat = lambda t: t.reshape(B, S, -1).cuda()
    got = attention_prefill_chunk(flat(q), flat(k), flat(v), D, chunk, sinks=sinks.cuda(), first=fd, scale=scale)
    plain = attention_plain(flat(q).float(), flat(k).float(), flat(v).float(), H, D, D, scale=scale, kv_heads=G, chunk=chunk, sinks=sinks.cuda(), first=fd)
    bare = attention_prefill_chunk(flat(q), flat(k), flat(v), D, chunk, first=fd, scale=scale)
    for b, w in enumerate(chunk_want(q, k, v, scale, sinks, chunk, first)):
        assert rel(plain[b, first[b]:], w) < 1e-4
        assert rel(got[b, first[b]:], w) < (2e-2 if dtype == BF16 else 3e-3)
    for b, w in enumerate(chunk_want(q, k, v, scale, torch.full((H,), -1e4), chunk, first)):
        assert rel(bare[b, first[b]:], w) < (2e-2 if dtype == BF16 else 3e-3)
    assert torch.isfinite(got).all() and torch.isfinite(bare).all()


@pytest.mark.parametrize("dtype", [BF16, F16])
@pytest.mark.parametrize("B,S,H,G,D,chunk,nsplit", [(1, 1, 1, 1, 64, 5, 1), (2, 63, 4, 2, 64, 0, 1), (3, 64, 6, 2, 128, 64, 2), (2, 65, 16, 1, 64, 64, None),
                                                    (1, 700, 40, 2, 128, 300, 3), (2, 1000, 8, 8, 128, 700, None), (2, 321, 12, 1, 64, 320, 5), (2, 200, 4, 2, 64, 1, None),
                                                    (2, 250, 4, 2, 64, 17, 2), (1, 900, 8, 2, 128, 0, 3)])
def test_step_attention_over_chunks_in_a_ring(dtype, B, S, H, G, D, chunk, nsplit):
    from energonai_b200.attention import attention_group_decode_chunk, attention_plain
    first = [0, S // 2, S - 1][:B]
    q, k, v, sinks = chunk_case(B, S, H, G, D, chunk, first, seed=7)
    q, k, v = (t.to(dtype) for t in (q, k, v))
    R = min(S + 70, chunk) if chunk else S + 70
    ring = torch.full((B, R, 2 * G * D), 3.0, dtype=dtype, device="cuda")
    for p in range(max(0, S - R), S):
        ring[:, p % R, :G * D], ring[:, p % R, G * D:] = k[:, p].reshape(B, -1).cuda(), v[:, p].reshape(B, -1).cuda()
    kc, vc, pos, fd, ql = ring[:, :, :G * D], ring[:, :, G * D:], i32([S - 1]), i32(first), q[:, -1].reshape(B, -1).cuda()
    want = chunk_want(q, k, v, 0.1, sinks, chunk, first)
    for _ in range(2):                                   # (the split counters are zero again)
        got = attention_group_decode_chunk(ql, kc, vc, D, pos, 0.1, chunk, sinks=sinks.cuda(), first=fd, nsplit=nsplit)
        for b in range(B):
            assert rel(got[b:b + 1], want[b][-1:]) < (2e-2 if dtype == BF16 else 3e-3)
    plain = attention_plain(ql.float().view(B, 1, -1), kc.float(), vc.float(), H, D, D, scale=0.1, first=fd, pos_device=pos, kv_heads=G, chunk=chunk, sinks=sinks.cuda())
    bare = attention_group_decode_chunk(ql, kc, vc, D, pos, 0.1, chunk, first=fd, nsplit=nsplit)
    free = chunk_want(q, k, v, 0.1, torch.full((H,), -1e4), chunk, first)
    for b in range(B):
        assert rel(plain[b], want[b][-1:]) < 1e-4
        assert rel(bare[b:b + 1], free[b][-1:]) < (2e-2 if dtype == BF16 else 3e-3)


def test_no_wait_ran_out():
    from energonai_b200.gemm import device_status
    assert device_status()[0] == 0
