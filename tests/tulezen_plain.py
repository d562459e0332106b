"""Plain, slow float64 restatement of the Tulezen design, one function per mechanism, for the tests.
It shares no code with the package; sequences are processed one at a time, whole."""
import torch


def rms_norm(x, weight, eps, around_zero):
    """x / sqrt(mean(x^2) + eps), times (1 + weight) or weight."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y * (1 + weight) if around_zero else y * weight


def visible(n, window, first=0):
    """[n, n] bool: row i sees column j."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    see = (i >= j) & (j >= first)
    return see & (i - j < window) if window else see


def softmax_attention(q, k, v, scale, see):
    """q [n, H, dk], k [m, H, dk], v [m, H, dv], see [n, m] -> [n, H, dv]; a row that sees nothing is 0."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(~see, float("-inf"))
    p = torch.nan_to_num(torch.softmax(s, -1), nan=0.0)
    return torch.einsum("hij,jhd->ihd", p, v)


def latent(h, w_dkv, norm, eps):
    return rms_norm(h @ w_dkv.T, norm, eps, around_zero=False)


def latent_attention(h, c, w_q, w_uk, w_uv, w_o, heads, scale, window):
    n = h.shape[0]
    q, k, v = ((x @ w.T).view(n, heads, -1) for x, w in ((h, w_q), (c, w_uk), (c, w_uv)))
    return softmax_attention(q, k, v, scale, visible(n, window)).reshape(n, -1) @ w_o.T


def router(h, w_router, top):
    """-> (indices [n, top], scores [n, top]): softmax over all experts, best first, scores unchanged."""
    s = torch.softmax(h @ w_router.T, -1)
    w, i = s.topk(top, -1)
    return i, w


def gated(gate, up, limit):
    g, u = torch.clamp(gate, max=limit), torch.clamp(up, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def mixture(h, w_router, experts, top, limit):
    """experts: list of (gate, up, down)."""
    idx, w = router(h, w_router, top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for k in range(top):
            g, u, d = experts[int(idx[t, k])]
            out[t] += w[t, k] * (gated(g @ h[t], u @ h[t], limit) @ d.T)
    return out


def forward(cfg, tensors, tokens):
    """Logits [n, vocab] of one sequence and the residual stream behind every layer."""
    w = {k: v.double() for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    latents, streams = {}, []
    for i, ly in enumerate(cfg["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        src = m.get("kv_from")
        if src is None:
            latents[i] = latent(x, w[p + "mix.dkv"], w[p + "mix.dkv.norm"], eps)
        y = latent_attention(x, latents[i if src is None else src], w[p + "mix.q"], w[p + "mix.uk"], w[p + "mix.uv"], w[p + "mix.o"],
                             m["heads"], m["scale"], m["mask"]["size"])
        x = x + rms_norm(y, w[p + "norm1"], eps, True)
        f = ly["mlp"]
        if f is not None:
            experts = [tuple(w[f"{p}mlp.e{e}.{n}"] for n in ("gate", "up", "down")) for e in range(f["router"]["experts"])]
            x = x + rms_norm(mixture(x, w[p + "mlp.router"], experts, f["router"]["top"], f["expert"]["limit"]), w[p + "norm2"], eps, True)
        streams.append(x)
    return rms_norm(x, w["final.norm"], eps, True) @ w["head"].T, streams


def greedy(cfg, tensors, tokens, new):
    """-> (tokens with `new` more, smallest gap between the two best logits of the steps)."""
    tokens, gap = list(tokens), float("inf")
    for _ in range(new):
        top = forward(cfg, tensors, tokens)[0][-1].topk(2)
        gap = min(gap, float(top.values[0] - top.values[1]))
        tokens.append(int(top.indices[0]))
    return tokens, gap


# ---- small models of the tests' own ------------------------------------------------------------------
def make_config(layers, width, vocab, eps=3e-5):
    """layers: list of dicts with heads, dim, vdim, rank, window, scale, kv_from?, moe = (experts, top, ff, limit) or None."""
    out = []
    for ly in layers:
        m = {"heads": ly["heads"], "dim": ly["dim"], "vdim": ly["vdim"], "kv_rank": ly["rank"], "mask": {"size": ly["window"]}, "scale": ly["scale"]}
        if ly.get("kv_from") is not None:
            m["kv_from"] = ly["kv_from"]
        f = ly.get("moe")
        out.append({"type": "latent_attention", "mixer": m, "mlp": None if f is None else
                    {"kind": "moe", "router": {"experts": f[0], "top": f[1]}, "expert": {"ff": f[2], "limit": f[3]}}})
    return {"architecture": "Tulezen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": out}


def make_tensors(cfg, seed):
    """Random bfloat16 tensors of a configuration: projections keep the scale of their input, norm
    weights move away from their neutral value, the router is sharp enough for clear choices."""
    g = torch.Generator().manual_seed(seed)
    W, t = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        t[name] = (torch.randn(rows, cols, generator=g) * gain / cols ** 0.5).bfloat16()

    def vec(name, n, mean):
        t[name] = (mean + 0.3 * torch.randn(n, generator=g)).bfloat16()
    t["embed"] = torch.randn(cfg["vocab"], W, generator=g).bfloat16()
    mat("head", cfg["vocab"], W)
    vec("final.norm", W, 0.0)
    for i, ly in enumerate(cfg["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        vec(p + "norm1", W, 0.0)
        mat(p + "mix.q", m["heads"] * m["dim"], W, 1.5)
        if m.get("kv_from") is None:
            mat(p + "mix.dkv", m["kv_rank"], W)
            vec(p + "mix.dkv.norm", m["kv_rank"], 1.0)
        mat(p + "mix.uk", m["heads"] * m["dim"], m["kv_rank"], 1.5)
        mat(p + "mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
        mat(p + "mix.o", W, m["heads"] * m["vdim"])
        f = ly["mlp"]
        if f is None:
            continue
        vec(p + "norm2", W, 0.0)
        mat(p + "mlp.router", f["router"]["experts"], W, 2.0)
        for e in range(f["router"]["experts"]):
            mat(f"{p}mlp.e{e}.gate", f["expert"]["ff"], W)
            mat(f"{p}mlp.e{e}.up", f["expert"]["ff"], W)
            mat(f"{p}mlp.e{e}.down", W, f["expert"]["ff"])
    return t


def save_safetensors(path, tensors):
    import json
    import struct
    names = {torch.bfloat16: "BF16", torch.float32: "F32", torch.float16: "F16", torch.int32: "I32", torch.int64: "I64"}
    head, blobs, at = {}, [], 0
    for k, v in tensors.items():
        raw = v.contiguous().reshape(-1).view(torch.uint8).numpy().tobytes() if v.numel() else b""
        head[k] = {"dtype": names[v.dtype], "shape": list(v.shape), "data_offsets": [at, at + len(raw)]}
        blobs.append(raw)
        at += len(raw)
    text = json.dumps(head).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))
