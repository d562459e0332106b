"""Plain, slow float64 restatement of the Moponex design, one function per mechanism, for the tests.
It shares no code with the package; sequences are processed one at a time, whole, recurrences token by
token."""
import math

import torch


def unit_rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def silu(z):
    return z * torch.sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2)))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


# ---- embedding -------------------------------------------------------------------------------------
def bigram_rows(tokens, mul_prev, mul_cur, buckets):
    """Row of the bigram table for every token; the last row for the first."""
    return [buckets if i == 0 else (tokens[i - 1] * mul_prev + t * mul_cur) % buckets for i, t in enumerate(tokens)]


# ---- selective state space --------------------------------------------------------------------------
def short_conv(x, w, b):
    """x [n, c], w [c, taps], b [c]: causal, the last column of w is the current token's."""
    n, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x) + b
    for t in range(n):
        for j in range(taps):
            s = t - (taps - 1 - j)
            if s >= 0:
                out[t] = out[t] + x[s] * w[:, j]
    return out


def ssm_scan(x, B, C, dt, a_log, d):
    """x [n, H, P], B / C [n, G, N], dt [n, H] (after softplus) -> y [n, H, P], final state [H, N, P]."""
    n, H, P = x.shape
    G, N = B.shape[1:]
    of = torch.arange(H) // (H // G)
    S = x.new_zeros(H, N, P)
    out = []
    for t in range(n):
        a = torch.exp(-torch.exp(a_log) * dt[t])
        S = a[:, None, None] * S + dt[t][:, None, None] * B[t, of][:, :, None] * x[t][:, None, :]
        out.append((S * C[t, of][:, :, None]).sum(1) + d[:, None] * x[t])
    return torch.stack(out), S


def group_norm(y, weight, groups, eps):
    """RMS norm in equal parts of the row, each by its own root mean square."""
    return unit_rms(y.view(*y.shape[:-1], groups, -1), eps).reshape(y.shape) * weight


def ssm_mixer(h, w, m, eps):
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner, n = H * P, h.shape[0]
    z, xbc, dt = (h @ w["in"].T).split([inner, inner + 2 * G * N, H], 1)
    xbc = silu(short_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc.split([inner, G * N, G * N], 1)
    dt = torch.nn.functional.softplus(dt + w["dt_bias"], threshold=1e9)
    y, _ = ssm_scan(x.view(n, H, P), B.view(n, G, N), C.view(n, G, N), dt, w["A_log"], w["D"])
    y = y.reshape(n, inner) * silu(z)
    return group_norm(y, w["norm"], m["norm_groups"], eps) @ w["o"].T


# ---- chunk-masked attention --------------------------------------------------------------------------
def rotate(x, positions, dims, base, factor):
    """x [n, H, d]: neighbouring pairs of the first `dims` dimensions turn by position * frequency."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    a = torch.as_tensor(positions, dtype=torch.float64)[:, None] * (base ** (-2 * i / dims) / factor)
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2], out[..., 1:dims:2] = u * c - v * s, v * c + u * s
    return out


def chunk_mask(n, size):
    """[n, n], True where row i sees key j; size None: every earlier key."""
    i = torch.arange(n)
    seen = i[:, None] >= i[None, :]
    return seen if size is None else seen & (i[:, None] // size == i[None, :] // size)


def sink_attention(q, k, v, scale, sink, seen):
    """q [n, H, d], k [n, G, d], v [n, G, dv], sink [H] -> [n, H, dv]."""
    H, G = q.shape[1], k.shape[1]
    share = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, share]) * scale
    s = s.masked_fill(~seen, float("-inf"))
    top = torch.maximum(s.amax(-1, keepdim=True), sink[:, None, None])
    e = torch.exp(s - top)
    p = e / (torch.exp(sink[:, None, None] - top) + e.sum(-1, keepdim=True))
    return torch.einsum("hij,jhd->ihd", p, v[:, share])


def attention_side(h, w, m, eps):
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w["q"].T + w["q.b"]).view(n, H, d)
    k = v = (h @ w["k"].T + w["k.b"]).view(n, G, d)
    q, k = rms_norm(q, w["q.norm"], eps), rms_norm(k, w["k.norm"], eps)
    rot = m.get("rot")
    if rot:
        factor = (rot.get("scaling") or {"factor": 1.0})["factor"]
        q, k = (rotate(t, range(n), rot["dims"], rot["base"], factor) for t in (q, k))
    o = sink_attention(q, k, v, m["scale"], w["sink"], chunk_mask(n, m["mask"]["size"] if m.get("mask") else None))
    return o.reshape(n, -1) @ w["o"].T


# ---- gated linear attention ---------------------------------------------------------------------------
def gla_scan(q, k, v, log_a):
    """q, k, log_a [n, H, d], v [n, H, dv] -> o [n, H, dv], final state [H, d, dv]."""
    n, H, d = q.shape
    S, out = q.new_zeros(H, d, v.shape[-1]), []
    for t in range(n):
        S = torch.exp(log_a[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def gla_side(h, w, m, eps):
    n, H, d, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(n, H, d) / math.sqrt(d)
    k, v = (h @ w["k"].T).view(n, H, d), (h @ w["v"].T).view(n, H, dv)
    z = (h @ w["a1"].T) @ w["a2"].T + w["a2.b"]
    log_a = torch.nn.functional.logsigmoid(z).view(n, H, d) / m["tau"]
    o, _ = gla_scan(q, k, v, log_a)
    o = rms_norm(o, w["norm"], eps).reshape(n, -1)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def part(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def parallel_mixer(h, w, m, eps):
    left = attention_side(h, part(w, "left."), m["left"], eps)
    right = gla_side(h, part(w, "right."), m["right"], eps)
    return (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps)) / 2


# ---- feed-forward ---------------------------------------------------------------------------------------
def dense(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def choose(z, correction, top, groups, keep):
    """Router logits [n, E] -> per token the chosen indices (best first) and their weights."""
    s = torch.softmax(z, -1)
    c = s + correction
    n, E = z.shape
    per = E // groups
    picked, weights = [], []
    for t in range(n):
        best = sorted(range(groups), key=lambda g: -float(c[t, g * per:(g + 1) * per].max()))[:keep]
        allowed = [e for g in sorted(best) for e in range(g * per, (g + 1) * per)]
        e = sorted(allowed, key=lambda e: -float(c[t, e]))[:top]
        picked.append(e)
        weights.append(s[t, e] / (s[t, e].sum() + 1e-20))
    return picked, weights


def mixture(h, w, mlp):
    r = mlp["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    picked, weights = choose(h @ w["router"].T, w["correction"], r["top"], g["count"], g["keep"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(picked[t], weights[t]):
            y = h[t] if e >= r["experts"] else gelu_erf(w[f"e{e}.up"] @ h[t]) @ w[f"e{e}.down"].T
            out[t] += a * y
    if mlp.get("shared"):
        y = gelu_erf(h @ w["shared.up"].T) @ w["shared.down"].T
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * y
    return out


def forward(cfg, tensors, tokens):
    """Logits [n, vocab] of one sequence and the residual stream behind every layer."""
    t = {k: v.double() for k, v in tensors.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    tokens = [int(x) for x in tokens]
    x = t["embed"][torch.tensor(tokens)]
    bg = cfg["embedding"].get("bigram")
    if bg:
        x = x + t["bigram"][torch.tensor(bigram_rows(tokens, bg["mul_prev"], bg["mul_cur"], bg["buckets"]))]
    streams = []
    for i, ly in enumerate(cfg["layers"]):
        w = part(t, f"l{i}.")
        mixer = {"mamba2": ssm_mixer, "parallel": parallel_mixer}[ly["type"]]
        x = x + mult * mixer(rms_norm(x, w["norm1"], eps), part(w, "mix."), ly["mixer"], eps)
        if ly["mlp"] is not None:
            h = rms_norm(x, w["norm2"], eps)
            x = x + mult * (dense(h, part(w, "mlp.")) if ly["mlp"]["kind"] == "dense" else mixture(h, part(w, "mlp."), ly["mlp"]))
        streams.append(x)
    return rms_norm(x, t["final.norm"], eps) @ t["embed"].T * cfg["logit_scale"], streams


def greedy(cfg, tensors, tokens, new):
    """-> (tokens with `new` more, smallest gap between the two best logits of the steps)."""
    tokens, gap = list(tokens), float("inf")
    for _ in range(new):
        top = forward(cfg, tensors, tokens)[0][-1].topk(2)
        gap = min(gap, float(top.values[0] - top.values[1]))
        tokens.append(int(top.indices[0]))
    return tokens, gap


# ---- small models of the tests' own ------------------------------------------------------------------
def dense_mlp(ff):
    return {"kind": "dense", "ff": ff}


def moe_mlp(experts, top, ff, identity=0, groups=None, shared=None):
    r = {"experts": experts, "top": top}
    if identity:
        r["identity"] = identity
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    out = {"kind": "moe", "router": r, "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def ssm_layer(heads, vdim, state, groups=1, conv=4, norm_groups=1, mlp=None):
    return {"type": "mamba2", "mlp": mlp,
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


def parallel_layer(left, right, mlp=None):
    """left = (heads, kv_heads, dim, scale, chunk, (rotated dims, base, factor or None) or None), right = (heads, dim, vdim,
    tau, rank)."""
    H, G, d, scale, chunk, rot = left
    a = {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "scale": scale}
    if chunk:
        a["mask"] = {"size": chunk}
    if rot:
        a["rot"] = {"dims": rot[0], "base": rot[1]}
        if rot[2]:
            a["rot"]["scaling"] = {"factor": rot[2]}
    return {"type": "parallel", "mlp": mlp, "rank": right[4],
            "mixer": {"left": a, "right": {"heads": right[0], "dim": right[1], "vdim": right[2], "tau": right[3]}}}


def make_config(layers, width, vocab, eps=2e-5, mult=0.6, logit_scale=0.3, bigram=(97, 29, 11)):
    """The ranks of the decay projections are not part of a configuration: make_tensors() takes them from `layers`,
    and `ranks` keeps them (see with_ranks)."""
    emb = {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))} if bigram else {}
    return {"architecture": "Moponex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": logit_scale,
            "embedding": emb, "layers": [{k: v for k, v in ly.items() if k != "rank"} for ly in layers], "ranks": [ly.get("rank") for ly in layers]}


def file_config(cfg):
    """What config.json holds."""
    return {k: v for k, v in cfg.items() if k != "ranks"}


def with_ranks(cfg):
    """For models built without a checkpoint: the ranks stand in the configuration."""
    out = file_config(cfg)
    out["layers"] = [dict(ly, mixer=dict(ly["mixer"], right=dict(ly["mixer"]["right"], rank=r))) if r else ly for ly, r in zip(cfg["layers"], cfg["ranks"])]
    return out


def make_tensors(cfg, seed):
    """Random bfloat16 tensors of a configuration.  Projections keep the scale of their input; decays are mostly slow,
    so that far tokens still count; sinks are about as large as scores; corrections decide choices; norm
    weights move away from one."""
    g = torch.Generator().manual_seed(seed)
    W, t = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        t[name] = (torch.randn(rows, cols, generator=g) * gain / cols ** 0.5).bfloat16()

    def vec(name, n, mean, spread=0.3):
        t[name] = (mean + spread * torch.randn(n, generator=g)).bfloat16()
    mat("embed", cfg["vocab"], W, W ** 0.5 * 0.7)
    if cfg["embedding"].get("bigram"):
        mat("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, W, W ** 0.5 * 0.5)
    vec("final.norm", W, 1.0)
    for i, (ly, rank) in enumerate(zip(cfg["layers"], cfg["ranks"])):
        p, m, f = f"l{i}.", ly["mixer"], ly["mlp"]
        vec(p + "norm1", W, 1.0)
        if ly["type"] == "mamba2":
            H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            channels = H * P + 2 * G * N
            mat(p + "mix.in", H * P + channels + H, W, 1.2)
            mat(p + "mix.conv", channels, m["conv"], 1.3)
            vec(p + "mix.conv.b", channels, 0.0)
            vec(p + "mix.dt_bias", H, -2.0, 0.7)
            vec(p + "mix.A_log", H, -2.0, 1.2)
            vec(p + "mix.D", H, 0.7)
            vec(p + "mix.norm", H * P, 1.0)
            mat(p + "mix.o", W, H * P, 1.5)
        else:
            a, r = m["left"], m["right"]
            H, G, d = a["heads"], a["kv_heads"], a["dim"]
            for name, n in (("q", H), ("k", G)):
                mat(p + "mix.left." + name, n * d, W)
                vec(p + f"mix.left.{name}.b", n * d, 0.0)
                vec(p + f"mix.left.{name}.norm", d, 1.4)
            vec(p + "mix.left.sink", H, 2.0, 1.5)
            mat(p + "mix.left.o", W, H * d)
            H, d, dv = r["heads"], r["dim"], r["vdim"]
            for name, n in (("q", d), ("k", d), ("v", dv), ("g", dv)):
                mat(p + "mix.right." + name, H * n, W, 1.2)
            mat(p + "mix.right.a1", rank, W)
            mat(p + "mix.right.a2", H * d, rank)
            vec(p + "mix.right.a2.b", H * d, 1.5, 1.5)
            vec(p + "mix.right.norm", dv, 1.0)
            mat(p + "mix.right.o", W, H * dv)
            vec(p + "mix.left.out", W, 1.0)
            vec(p + "mix.right.out", W, 0.8)
        if f is None:
            continue
        vec(p + "norm2", W, 1.0)
        if f["kind"] == "dense":
            for name, rows, cols in (("gate", f["ff"], W), ("up", f["ff"], W), ("down", W, f["ff"])):
                mat(p + "mlp." + name, rows, cols, 1.3)
            continue
        r = f["router"]
        n = r["experts"] + r.get("identity", 0)
        mat(p + "mlp.router", n, W, 2.0)
        vec(p + "mlp.correction", n, -1.0, 0.15)
        for e in range(r["experts"]):
            mat(f"{p}mlp.e{e}.up", f["expert"]["ff"], W, 1.3)
            mat(f"{p}mlp.e{e}.down", W, f["expert"]["ff"], 1.3)
        if f.get("shared"):
            mat(p + "mlp.shared.up", f["shared"]["ff"], W, 1.3)
            mat(p + "mlp.shared.down", W, f["shared"]["ff"], 1.3)
            mat(p + "mlp.shared.sg", 1, W)
    return t
