"""Kernels of the latent-attention decoder on the GPU, each against the plain restatement."""
import pytest
import torch

import tulezen_plain as P

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


def rnd(*shape, seed=0, scale=1.0, dtype=BF):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).cuda()


def close(a, b, tol):
    a, b = a.double().cpu(), b.double().cpu()
    err, ref = (a - b).pow(2).mean().sqrt(), b.pow(2).mean().sqrt()
    assert torch.isfinite(a).all() and float(err) <= tol * float(ref) + 1e-12, (float(err), float(ref))
    assert float((a - b).abs().max()) <= 12 * tol * float(b.abs().max()) + 1e-9


def tol_of(dtype):
    return {F32: 2e-6, BF: 6e-3, torch.float16: 1e-3}[dtype]


# ---- norms -------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width,count", [(8, 8), (40, 37), (512, 512), (1032, 1030), (4096, 4096), (9000, 9000)])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_rms_norm(width, count, dtype):
    from energonai_b200.norm import rms_norm
    x, w = rnd(11, width, dtype=F32), rnd(width, seed=1, scale=0.3, dtype=dtype)
    x[:, count:] = 0
    x[3] *= 1e-3                                                   # eps matters here
    for offset in (0.0, 1.0):
        y = rms_norm(x, w, 1e-4, offset=offset, count=count)
        ref = P.rms_norm(x[:, :count].double().cpu(), w[:count].double().cpu(), 1e-4, offset == 1.0)
        close(y[:, :count], ref, tol_of(dtype))
        assert float(y[:, count:].abs().sum()) == 0


@pytest.mark.parametrize("rows,seq,pos", [(5, 3, 0), (5, 5, 0), (5, 13, 0), (5, 1, 23), (7, 2, 6)])
def test_rms_norm_ring(rows, seq, pos):
    from energonai_b200.norm import rms_norm
    B, R = 3, 64
    x, w = rnd(B * seq, 96)[:, 16:80], rnd(R, seed=1)
    ring = torch.full((B, rows, R), 7.0, dtype=BF, device="cuda")
    y = rms_norm(x, w, 1e-5, ring=ring, rows_per_batch=seq, pos_device=torch.tensor([pos], dtype=torch.int32, device="cuda"))
    want = torch.full_like(ring, 7.0)
    for s in range(max(0, seq - rows), seq):
        want[:, (pos + s) % rows] = y.view(B, seq, R)[:, s]
    assert torch.equal(ring, want)
    close(y, P.rms_norm(x.double().cpu(), w.double().cpu(), 1e-5, False), tol_of(BF))


@pytest.mark.parametrize("dtype,width,count", [(F32, 80, 76), (BF, 80, 76), (BF, 2048, 2048), (BF, 8200, 8200)])
def test_rms_residual_plain_mixed_and_with_router(dtype, width, count):
    from energonai_b200.norm import rms_residual
    T, E, top = 9, 7, 3
    y, w = rnd(T, width, dtype=dtype), rnd(width, seed=1, scale=0.3, dtype=dtype)
    y[:, count:] = 0
    w[count:] = 0
    x0 = rnd(T, width, seed=2, dtype=F32)
    x0[:, count:] = 0
    router = rnd(E, width, seed=3, scale=0.3, dtype=dtype)
    x, xt = x0.clone(), torch.empty(T, width, dtype=dtype, device="cuda")
    idx, sc = rms_residual(y, w, 1e-5, x, xt=xt, offset=1.0, count=count, router=(router, E, top))
    ref = x0.double().cpu()[:, :count] + P.rms_norm(y.double().cpu()[:, :count], w.double().cpu()[:count], 1e-5, True)
    close(x[:, :count], ref, 2e-6)
    assert torch.equal(xt, x.to(dtype)) and float(x[:, count:].abs().sum()) == 0
    ri, rw = P.router(xt.double().cpu(), router.double().cpu(), top)
    assert torch.equal(idx.cpu().long(), ri)
    close(sc, rw, 1e-5)
    # a mixture's rows, some tokens without some experts
    idx = torch.randint(0, E, (T, top), dtype=torch.int32).cuda()
    idx[2, 1] = idx[4] = -1
    rows = torch.randperm(T * top).view(T, top).to(torch.int32).cuda()
    wts, ym = torch.rand(T, top).cuda(), rnd(T * top, width, seed=5, dtype=dtype)
    ym[:, count:] = 0
    for r in (None, rows):
        x = x0.clone()
        rms_residual(ym, w, 1e-5, x, offset=1.0, count=count, mix=(idx, r, wts))
        at = (torch.arange(T * top).view(T, top) if r is None else r.cpu().long())
        ysum = (ym.double().cpu()[at] * (wts.double().cpu() * (idx.cpu() >= 0))[..., None]).sum(1)
        ref = x0.double().cpu()[:, :count] + P.rms_norm(ysum[:, :count], w.double().cpu()[:count], 1e-5, True)
        close(x[:, :count], ref, 3e-6)
        assert torch.equal(x[4], x0[4])                             # no expert at all: nothing is added


# ---- mixture of experts --------------------------------------------------------------------------------
@pytest.mark.parametrize("T,E,top", [(1, 1, 1), (5, 3, 3), (130, 8, 2), (33, 70, 40), (700, 100, 6)])
def test_route(T, E, top):
    from energonai_b200.moe import COUNT_STRIDE, new_counts, route
    g = torch.Generator().manual_seed(T)
    z = torch.randn(T, E + 5, generator=g).cuda()
    first = torch.tensor([0, 3], dtype=torch.int32, device="cuda") if T % 5 == 0 and T > 5 else None
    seq = T // 2 if first is not None else T
    counts = new_counts(E, "cuda")
    idx, w, ranks = route(z, E, top, first, seq, counts)
    pad = torch.zeros(T, dtype=torch.bool)
    if first is not None:
        pad = (torch.arange(T) % seq) < first.cpu().long()[torch.arange(T) // seq]
    s, i = torch.softmax(z[:, :E].double().cpu(), -1).topk(top, -1)
    assert torch.equal(idx.cpu().long()[~pad], i[~pad]) and (idx.cpu()[pad] == -1).all()
    close(w[~pad.cuda()], s[~pad], 1e-5)
    counts = counts[::COUNT_STRIDE].cpu()
    for e in range(E):                                              # tickets 0, 1, 2, ... of every expert
        got = ranks.cpu()[idx.cpu() == e].sort().values
        assert int(counts[e]) == got.numel() and torch.equal(got, torch.arange(got.numel(), dtype=got.dtype))


def test_route_equal_scores_take_the_lowest_index():
    from energonai_b200.moe import route
    idx, w = route(torch.zeros(2, 9, device="cuda"), 9, 4)
    assert idx.tolist() == [[0, 1, 2, 3]] * 2
    close(w, torch.full((2, 4), 1 / 9), 1e-6)


def experts_of(mlp_gate_up, mlp_down, ff):
    E, _, W = mlp_gate_up.shape
    gu = mlp_gate_up.double().cpu().view(E, -1, 2, 8, W)
    return [(gu[e, :, 0].reshape(-1, W)[:ff], gu[e, :, 1].reshape(-1, W)[:ff], mlp_down[e].double().cpu()[:, :ff]) for e in range(E)]


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("T,W,E,top,ff,limit,skew", [(1, 64, 4, 2, 24, 0.5, 0), (7, 72, 5, 1, 8, 2.0, 0), (100, 200, 3, 3, 40, 1.0, 0),
                                                     (128, 136, 9, 2, 136, 0.7, 1), (129, 72, 5, 2, 24, 0.5, 0), (300, 264, 12, 4, 72, 1.0, 1),
                                                     (400, 64, 40, 33, 16, 0.3, 0)])
def test_mixture_of_experts(dtype, T, W, E, top, ff, limit, skew):
    """Streaming and sorted paths; skew: nearly every token chooses the same expert."""
    from energonai_b200.model import MixtureOfExperts
    from energonai_b200.norm import rms_residual
    m = MixtureOfExperts(W, E, top, ff, limit, 1.702, dtype, device="cuda")
    assert m.skinny(T) == (dtype == BF and T <= 128)
    for k, (p, s) in enumerate(((m.router, 1.0), (m.gate_up, 1.0), (m.down, 1.0))):
        p.data.copy_(rnd(*p.shape, seed=10 + k, scale=s / p.shape[-1] ** 0.5, dtype=dtype))
    m.gate_up.data.view(E, -1, 2, 8, W)[:, ff // 8:] = 0 if ff % 8 else m.gate_up.data.view(E, -1, 2, 8, W)[:, ff // 8:]
    h = rnd(T, W, seed=4, dtype=dtype)
    if skew:
        h[:, 0] = 8.0
        m.router.data[1, 0] = 4.0
    for call in range(2):                                           # the row counters are ready for a second batch
        y, mix = m(h)
        x = torch.zeros(T, W, device="cuda")
        one = torch.zeros(W, dtype=dtype, device="cuda")
        rms_residual(y, one, 0.0, x, offset=1.0, mix=mix)           # the norm of the weighted sum, added to zero
        want = P.mixture(h.double().cpu(), m.router.double().cpu()[:E], experts_of(m.gate_up, m.down, ff), top, limit)
        close(x, P.rms_norm(want, torch.zeros(W), 0.0, True), 8e-3 if dtype == BF else 3e-6)


def test_mixture_leaves_padding_out():
    from energonai_b200.model import MixtureOfExperts
    m = MixtureOfExperts(64, 6, 2, 16, 1.0, 1.702, BF, device="cuda")
    for seq in (20, 150):
        first = torch.tensor([0, 7], dtype=torch.int32, device="cuda")
        h = rnd(2 * seq, 64)
        _, (idx, rows, w) = m(h, first=first, rows_per_batch=seq)
        pad = torch.arange(2 * seq, device="cuda") % seq < first.long()[torch.arange(2 * seq, device="cuda") // seq]
        assert (idx[pad] == -1).all() and (idx[~pad] >= 0).all()


@pytest.mark.parametrize("B", [1, 8, 17, 33, 70])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_per_head_product(B, dtype):
    from energonai_b200.moe import per_head
    for H, N, K in ((3, 24, 64), (2, 128, 512), (20, 512, 128), (5, 64, 264)):
        a, w = rnd(B, H * K + 16, dtype=dtype)[:, :H * K], rnd(H, N, K, seed=1, scale=K ** -0.5, dtype=dtype)
        want = torch.einsum("bhk,hnk->bhn", a.double().cpu().view(B, H, K), w.double().cpu())
        y = per_head(a, w)
        close(y, want.reshape(B, -1), tol_of(dtype) / 1.5)
        assert torch.equal(per_head(a[:1], w), y[:1])               # independent of the batch, bit for bit


def test_gemm_f32_is_true_32_bit():
    from energonai_b200.gemm import gemm_f32
    for M, N, K in ((1, 5, 7), (70, 65, 130), (300, 448, 256)):
        a, w = rnd(M, K, dtype=F32), rnd(N, K, seed=1, dtype=F32)
        close(gemm_f32(a, w), a.double().cpu() @ w.double().cpu().T, 1e-6)


# ---- windowed prompt attention ---------------------------------------------------------------------------
def plant(q, k, i, j, strength):
    """Makes key j stand out for query i: one score far above the others."""
    q[i] *= 0.1
    k[j] = q[i] / q[i].pow(2).sum(-1, keepdim=True) * strength


@pytest.mark.parametrize("D", [64, 128])
@pytest.mark.parametrize("S,window", [(1, 1), (2, 1), (100, 1), (130, 2), (300, 63), (300, 64), (300, 65), (520, 127), (520, 128), (520, 129),
                                      (700, 200), (700, 257), (640, 1000), (400, 0)])
def test_prompt_attention_window(D, S, window):
    from energonai_b200.attention import attention_plain, attention_prefill_window
    H, B, scale = 2, 2, 0.2
    q, k, v = (rnd(B, S, H, D, seed=s) for s in (0, 1, 2))
    first = [0, min(S - 1, 5)]
    if window and S > window + 140:
        for b in range(B):
            for i in (window + 3, window + 130, S - 1):
                plant(q[b], k[b], i, i - window + 1, 40.0)          # the last key inside
            plant(q[b], k[b], S - 60, S - 60 - window, 60.0)        # the first one outside
    mask = torch.zeros(B, S, dtype=BF, device="cuda")
    mask[1, :first[1]] = -10000.0
    flat = lambda t: t.reshape(B, S, H * D)
    got = attention_prefill_window(flat(q), flat(k), flat(v), D, window, mask=mask, scale=scale)
    plain = attention_plain(*(flat(t).float() for t in (q, k, v)), H, D, D, window=window, scale=scale,
                            first=torch.tensor(first, dtype=torch.int32, device="cuda"))
    for b in range(B):
        see = P.visible(S, window, first[b])
        want = P.softmax_attention(*(t[b].double().cpu() for t in (q, k, v)), scale, see).reshape(S, -1)
        close(got[b, first[b]:], want[first[b]:], 6e-3)
        close(plain[b], want, 3e-6)


def test_planted_keys_show():
    """The planted scores decide the result: leaving the window's last key out, or letting the next one
    in, changes the plain result far beyond the tolerance above."""
    S, w, H, D = 400, 65, 2, 64
    q, k, v = (rnd(S, H, D, seed=s) for s in (0, 1, 2))
    plant(q, k, w + 3, 4, 40.0)
    plant(q, k, S - 60, S - 60 - w, 60.0)
    at = lambda win: P.softmax_attention(*(t.double().cpu() for t in (q, k, v)), 0.2, P.visible(S, win))
    a, narrower, wider = at(w), at(w - 1), at(w + 1)
    assert float((a - narrower)[w + 3].abs().max()) > 0.5 and float((a - wider)[S - 60].abs().max()) > 0.5


@pytest.mark.parametrize("dk,dv", [(5, 3), (40, 72), (192, 160)])
def test_plain_attention_takes_any_head_sizes(dk, dv):
    from energonai_b200.attention import attention_plain
    S, H = 90, 3
    q, k, v = (rnd(1, S, H * d, seed=s) for s, d in ((0, dk), (1, dk), (2, dv)))
    got = attention_plain(q, k, v, H, dk, dv, window=31, scale=0.15)
    want = P.softmax_attention(*(t[0].double().cpu().view(S, H, -1) for t in (q, k, v)), 0.15, P.visible(S, 31))
    close(got[0], want.reshape(S, -1), 5e-3)


# ---- generation-step attention over the latent ring -----------------------------------------------------
@pytest.mark.parametrize("R,H", [(64, 1), (64, 20), (128, 3), (256, 16), (256, 40), (384, 17), (512, 16), (512, 33)])
@pytest.mark.parametrize("rows,window,pos", [(9, 9, 4), (9, 9, 40), (64, 64, 63), (64, 64, 64), (100, 100, 255), (130, 70, 128), (130, 70, 190),
                                             (200, 0, 150), (321, 321, 1000), (700, 640, 1234)])
def test_latent_decode(R, H, rows, window, pos):
    from energonai_b200.attention import attention_plain, latent_decode
    B, scale = 3, 0.1
    q, hist = rnd(B, H, R, seed=R + pos), rnd(B, pos + 1, R, seed=pos)
    first = [0, min(pos, 3), max(0, pos - 2)]
    lo = max(0, pos - window + 1) if window else 0
    for b in range(B):                                              # far keys: last inside, first outside, the query's own
        own = q[b, 0] / q[b, 0].float().pow(2).sum().sqrt()
        if lo > 0:
            hist[b, lo - 1] = own * 30
        hist[b, lo] = own * (12 if first[b] <= lo else 30)
        hist[b, pos] = own * 11
    ring = torch.zeros(B, rows, R, dtype=BF, device="cuda")
    for p in range(max(0, pos + 1 - rows), pos + 1):
        ring[:, p % rows] = hist[:, p]
    dev = lambda *v: torch.tensor(v, dtype=torch.int32, device="cuda")
    want = []
    for b in range(B):
        keys = hist[b, max(lo, first[b]):].double().cpu()[:, None].expand(-1, H, -1)
        want.append(P.softmax_attention(q[b:b + 1].double().cpu(), keys, keys, scale, torch.ones(1, keys.shape[0], dtype=torch.bool))[0])
    want = torch.stack(want).view(B, -1)
    one = None
    for nsplit in (1, 2, 3, 4, 9):
        got = latent_decode(q.view(B, -1), ring, R, H, window, dev(pos), scale, first=dev(*first), nsplit=nsplit)
        close(got, want, 6e-3)
        one = got if one is None else one
    alone = latent_decode(q[1:2].reshape(1, -1), ring[1:2], R, H, window, dev(pos), scale, first=dev(first[1]), nsplit=1)
    assert torch.equal(alone, one[1:2])
    plain = attention_plain(q.view(B, 1, -1).float(), ring.float(), ring.float(), H, R, R, window=window, scale=scale, first=dev(*first),
                            pos_device=dev(pos), shared_kv=True)
    close(plain.view(B, -1), want, 3e-6)


def test_no_wait_ran_out():
    from energonai_b200.gemm import device_status
    assert device_status()[0] == 0
