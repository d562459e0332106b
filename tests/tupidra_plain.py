"""Plain, slow float64 restatement of the Tupidra design, one function per mechanism, for the tests.
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


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(x, w):
    """x [n, c], w [c, taps]: the last column of w is the current token's, nothing lies in front of the first."""
    n, taps = x.shape[0], w.shape[1]
    out = torch.zeros_like(x)
    for t in range(n):
        for back in range(min(taps, t + 1)):
            out[t] = out[t] + x[t - back] * w[:, taps - 1 - back]
    return out


def mixed_input(h, w):
    """What a sublayer reads: the normed row plus its convolution over time."""
    return h + causal_conv(h, w)


# ---- rotations -------------------------------------------------------------------------------------
def yarn(dims, base, scaling):
    """(frequency of every pair, factor of sine and cosine)."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not scaling:
        return f, 1.0
    turns = lambda t: dims * math.log(scaling["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(scaling["fast"])), 0), min(math.ceil(turns(scaling["slow"])), dims - 1)
    out = []
    for i, v in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(v / scaling["factor"] * r + v * (1 - r))
    return out, 0.1 * math.log(scaling["factor"]) + 1


def rotate(x, positions, rot):
    """x [n, heads, d]: neighbouring pairs of the first rot.dims entries turn."""
    x = x.clone()
    freq, factor = yarn(rot["dims"], rot["base"], rot.get("scaling"))
    for row, p in enumerate(positions):
        for i, f in enumerate(freq):
            c, s = factor * math.cos(p * f), factor * math.sin(p * f)
            u, v = x[row, :, 2 * i].clone(), x[row, :, 2 * i + 1].clone()
            x[row, :, 2 * i], x[row, :, 2 * i + 1] = u * c - v * s, v * c + u * s
    return x


# ---- attention ---------------------------------------------------------------------------------------
def softmax_with_sink(s, seen, sink):
    """Weights of scores s [H, n, n]; exp(sink[h]) is in every denominator (None: it is not)."""
    s = s.masked_fill(~seen, float("-inf"))
    top = s.amax(-1, keepdim=True)
    if sink is None:
        return torch.softmax(s, -1)
    top = torch.maximum(top, sink[:, None, None])
    e = torch.exp(s - top)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink[:, None, None] - top))


def slopes(heads):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float64)


def window_mask(n, size, keep_first):
    """[n, n], True where row i sees key j; size None: every earlier key."""
    seen = torch.zeros(n, n, dtype=torch.bool)
    for i in range(n):
        for j in range(i + 1):
            seen[i, j] = size is None or i - j < size or j < keep_first
    return seen


def capped_attention(q, k, v, scale, cap, seen):
    """q [n, H, d], k [n, G, d], v [n, G, dv] -> [n, H, dv]; capped scores, distance bias, a score of 0 without a value."""
    n, H = q.shape[:2]
    share = torch.arange(H) // (H // k.shape[1])
    s = torch.einsum("ihd,jhd->hij", q, k[:, share]) * scale
    if cap:
        s = cap * torch.tanh(s / cap)
    i = torch.arange(n, dtype=torch.float64)
    s = s - slopes(H)[:, None, None] * (i[:, None] - i[None, :])
    return torch.einsum("hij,jhd->ihd", softmax_with_sink(s, seen, torch.zeros(H, dtype=torch.float64)), v[:, share])


def attention_mixer(h, w, m, eps):
    n, H, G = h.shape[0], m["heads"], m["kv_heads"]
    q = (h @ w["q"].T + w["q.b"]).view(n, H, -1)
    k = (h @ w["k"].T + w["k.b"]).view(n, G, -1)
    v = unit_rms((h @ w["v"].T + w["v.b"]).view(n, G, -1), eps)
    mask = m.get("mask") or {"size": None, "keep_first": 0}
    o = capped_attention(q, k, v, m["scale"], m.get("softcap"), window_mask(n, mask["size"], mask.get("keep_first", 0)))
    return (o.reshape(n, -1) * torch.sigmoid(h @ w["g"].T)) @ w["o"].T + w["o.b"]


def latents(h, w, m, eps):
    """(latent, rotated key part) of every position."""
    c, kr = (h @ w["dkv"].T).split([m["kv_rank"], m["rot_dim"]], 1)
    return rms_norm(c, w["dkv.norm"], eps), rotate(kr[:, None], range(h.shape[0]), m["rot"])[:, 0]


def latent_mixer(h, w, m, eps, kept):
    n, H, d = h.shape[0], m["heads"], m["dim"]
    c, kr = kept
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).view(n, H, -1)
    qr = rotate(q[:, :, d:], range(n), m["rot"])
    k, v = (c @ w["uk"].T).view(n, H, d), (c @ w["uv"].T).view(n, H, -1)
    s = (torch.einsum("ihd,jhd->hij", q[:, :, :d], k) + torch.einsum("ihd,jd->hij", qr, kr)) * m["scale"]
    p = softmax_with_sink(s, window_mask(n, None, 0), w["sink"])
    o = torch.einsum("hij,jhd->ihd", p, v).reshape(n, -1)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ---- selective scan ------------------------------------------------------------------------------------
def selective_scan(x, dt, A, B, C, D):
    """x, dt [n, c] (dt after softplus), A [c, s] (negative), B / C [n, s], D [c] -> y [n, c], state [c, s]."""
    S, out = torch.zeros_like(A), []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out.append(S @ C[t] + D * x[t])
    return torch.stack(out), S


def scan_mixer(h, w, m, eps):
    x, z = (h @ w["in"].T).split([m["inner"], m["inner"]], 1)
    x = silu(causal_conv(x, w["conv"]) + w["conv.b"])
    dt, B, C = (x @ w["x"].T).split([m["dt_rank"], m["state"], m["state"]], 1)
    dt = torch.nn.functional.softplus(dt @ w["dt"].T + w["dt.b"], threshold=1e9)
    y, _ = selective_scan(x, dt, -torch.exp(w["A_log"]), B, C, w["D"])
    return (y * silu(z)) @ w["o"].T


def dense(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def part(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens):
    """Logits [n, vocab] of one sequence and the residual stream behind every layer."""
    t = {k: v.double() for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][torch.tensor([int(v) for v in tokens])]
    streams, kept = [], {}
    for i, ly in enumerate(cfg["layers"]):
        w, m = part(t, f"l{i}."), ly["mixer"]
        mix = part(w, "mix.")
        h = mixed_input(rms_norm(x, w["norm1"], eps), w["canon1"])
        if ly["type"] == "latent_attention":
            src = m.get("kv_from")
            if src is None:
                kept[i] = latents(h, mix, m, eps)
            y = latent_mixer(h, mix, m, eps, kept[i if src is None else src])
        else:
            y = {"attention": attention_mixer, "mamba1": scan_mixer}[ly["type"]](h, mix, m, eps)
        if ly["mlp"] is not None:
            y = y + dense(mixed_input(rms_norm(x, w["norm2"], eps), w["canon2"]), part(w, "mlp."))
        x = x + y
        streams.append(x)
    return rms_norm(x, t["final.norm"], eps) @ t["head"].T, streams


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


def scan_layer(inner, state, dt_rank, conv=4, mlp=None):
    return {"type": "mamba1", "mlp": mlp, "mixer": {"inner": inner, "state": state, "dt_rank": dt_rank, "conv": conv}}


def attention_layer(heads, kv_heads, dim, vdim, scale, cap=None, mask=None, mlp=None):
    """mask = (window, kept first positions)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if cap:
        m["softcap"] = cap
    if mask:
        m["mask"] = {"size": mask[0], "keep_first": mask[1]}
    return {"type": "attention", "mlp": mlp, "mixer": m}


def latent_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, scaling=None, kv_from=None, mlp=None):
    """scaling = (factor, original, fast, slow)."""
    rot = {"dims": rot_dim, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale, "rot": rot}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": mlp, "mixer": m}


def make_config(layers, width, vocab, taps=4, eps=2e-5):
    return {"architecture": "Tupidra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "canon": {"taps": taps}, "layers": layers}


def make_tensors(cfg, seed):
    """Random bfloat16 tensors of a configuration.  Projections keep the scale of their input; decays are mostly slow, so
    that far tokens still count; sinks are about as large as scores; norm weights move away from one."""
    g = torch.Generator().manual_seed(seed)
    W, t, taps = cfg["width"], {}, cfg["canon"]["taps"]

    def mat(name, rows, cols, gain=1.0):
        t[name] = (torch.randn(rows, cols, generator=g) * gain / cols ** 0.5).bfloat16()

    def vec(name, n, mean, spread=0.3):
        t[name] = (mean + spread * torch.randn(n, generator=g)).bfloat16()
    mat("embed", cfg["vocab"], W, W ** 0.5)
    mat("head", cfg["vocab"], W)
    vec("final.norm", W, 1.0)
    for i, ly in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", ly["mixer"], ly["mlp"]
        q = p + "mix."
        vec(p + "norm1", W, 1.0)
        mat(p + "canon1", W, taps, 0.7)
        if ly["type"] == "mamba1":
            C, N, R = m["inner"], m["state"], m["dt_rank"]
            mat(q + "in", 2 * C, W, 1.2)
            mat(q + "conv", C, m["conv"], 1.3)
            vec(q + "conv.b", C, 0.0)
            mat(q + "x", R + 2 * N, C, 0.8)
            mat(q + "dt", C, R)
            vec(q + "dt.b", C, -3.0, 0.7)
            t[q + "A_log"] = (torch.randn(C, N, generator=g) - 0.5).bfloat16()
            vec(q + "D", C, 0.7)
            mat(q + "o", W, C, 0.5)
        elif ly["type"] == "attention":
            H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for name, n in (("q", H * d), ("k", G * d), ("v", G * dv)):
                mat(q + name, n, W, 1.2)
                vec(f"{q}{name}.b", n, 0.0)
            mat(q + "g", H * dv, W, 1.5)
            mat(q + "o", W, H * dv, 3.5)
            vec(q + "o.b", W, 0.0)
        else:
            H, d, r, dv, qr, kr = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "q_rank", "kv_rank"))
            mat(q + "dq", qr, W)
            vec(q + "dq.norm", qr, 1.0)
            mat(q + "uq", H * (d + r), qr, 1.2)
            if m.get("kv_from") is None:
                mat(q + "dkv", kr + r, W)
                vec(q + "dkv.norm", kr, 1.0)
            mat(q + "uk", H * d, kr, 1.2)
            mat(q + "uv", H * dv, kr, 1.2)
            vec(q + "sink", H, 1.0, 1.0)
            mat(q + "g", H * dv, W, 1.5)
            mat(q + "o", W, H * dv, 3.5)
        if f is not None:
            vec(p + "norm2", W, 1.0)
            mat(p + "canon2", W, taps, 0.7)
            for name, rows, cols in (("gate", f["ff"], W), ("up", f["ff"], W), ("down", W, f["ff"])):
                mat(p + "mlp." + name, rows, cols, 1.3)
    return t
