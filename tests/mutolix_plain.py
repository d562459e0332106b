"""Plain, slow float64 restatement of the Mutolix design, one function per mechanism, for the tests.
It shares no code with the package; sequences are processed one at a time, whole, recurrences token by
token."""
import math

import torch


def unit_rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * weight


def xielu(z, p, q):
    """p, q: 0-d tensors."""
    up = torch.log1p(torch.exp(p)) * z * z + z / 2
    down = (0.5 + torch.log1p(torch.exp(q))) * (torch.exp(torch.clamp(z, max=0.0)) - 1 - z) + z / 2
    return torch.where(z > 0, up, down)


def feed_forward(h, w_up, w_down, act):
    return xielu(h @ w_up.T, act[0], act[1]) @ w_down.T


def residual_gate(y, h, w, b):
    return y * torch.sigmoid(h @ w.T + b)


# ---- matrix memory ---------------------------------------------------------------------------------
def memory_gates(h, w_i, b_i, w_f, b_f, cap):
    """-> (log input gate, log forget gate), [n, heads] each."""
    soft = lambda a: cap * torch.tanh(a / cap)
    return soft(h @ w_i.T + b_i), torch.nn.functional.logsigmoid(soft(h @ w_f.T + b_f))


def memory_scan(q, k, v, log_i, log_f):
    """The stabilised recurrence of one sequence: q, k [n, H, d], v [n, H, dv], gates [n, H] -> [n, H, dv]."""
    n, H, d = q.shape
    dv = v.shape[-1]
    S, z, m = q.new_zeros(H, d, dv), q.new_zeros(H, d), q.new_zeros(H)
    out = []
    for t in range(n):
        new = torch.maximum(log_f[t] + m, log_i[t])
        a, b = torch.exp(log_f[t] + m - new), torch.exp(log_i[t] - new)
        S = a[:, None, None] * S + b[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        z = a[:, None] * z + b[:, None] * k[t]
        m = new
        num = (S * q[t][:, :, None]).sum(1)
        den = torch.maximum((z * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(num / den[:, None])
    return torch.stack(out)


def memory_mixer(h, w, mixer, eps):
    """w: the mixer's tensors by their short names."""
    n, H, d, dv = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"]
    q = (h @ w["q"].T).view(n, H, d) / math.sqrt(d)
    k, v = (h @ w["k"].T).view(n, H, d), (h @ w["v"].T).view(n, H, dv)
    i, f = memory_gates(h, w["i"], w["i.b"], w["f"], w["f.b"], mixer["gate_cap"])
    o = unit_rms(memory_scan(q, k, v, i, f), eps).reshape(n, -1) * w["norm"]
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ---- attention -------------------------------------------------------------------------------------
def query_temperature(n, coef, every):
    return 1 + coef * torch.log(torch.tensor([(p + 1) // every + 1 for p in range(n)], dtype=torch.float64))


def distance_bias(n, r1, r2):
    """[H, n, n], to be taken off the scores (entries above the diagonal mean nothing)."""
    gap = torch.clamp(torch.arange(n)[:, None] - torch.arange(n)[None, :], min=0).double()
    return r1[:, None, None] * torch.log(1 + r2[:, None, None] * gap)


def sink_attention(q, k, v, scale, bias):
    """q [n, H, d], k [n, G, d], v [n, G, dv] -> [n, H, dv]; causal; one is added to the denominator."""
    n, H, G = q.shape[0], q.shape[1], k.shape[1]
    share = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, share]) * scale - bias
    s = s.masked_fill(~torch.tril(torch.ones(n, n, dtype=torch.bool)), float("-inf"))
    m = torch.clamp(s.amax(-1, keepdim=True), min=0.0)
    e = torch.exp(s - m)
    p = e / (torch.exp(-m) + e.sum(-1, keepdim=True))
    return torch.einsum("hij,jhd->ihd", p, v[:, share])


def attention_mixer(h, w, mixer, eps, v_first):
    """-> (output, the values this layer hands on as the first ones, or None)."""
    n, H, G, d, dv = h.shape[0], mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    q = rms_norm(h @ w["q"].T + w["q.b"], w["q.norm"], eps).view(n, H, d)
    k = rms_norm(h @ w["k"].T + w["k.b"], w["k.norm"], eps).view(n, G, d)
    v = (h @ w["v"].T + w["v.b"]).view(n, G, dv)
    qt = mixer.get("q_temp")
    if qt:
        q = q * query_temperature(n, qt["coef"], qt["every"])[:, None, None]
    mine = None
    if mixer.get("v_mix"):
        if v_first is None:
            mine = v
        else:
            v = (1 - w["vmix"]) * v + w["vmix"] * v_first
    o = sink_attention(q, k, v, mixer["scale"], distance_bias(n, w["r1"], w["r2"]))
    return o.reshape(n, -1) @ w["o"].T, mine


def forward(cfg, tensors, tokens):
    """Logits [n, vocab] of one sequence and the residual stream behind every layer."""
    t = {k: v.double() for k, v in tensors.items()}
    eps = cfg["norm"]["eps"]
    x = t["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    streams, v_first = [], None
    for i, ly in enumerate(cfg["layers"]):
        p = f"l{i}."
        mix = {k[len(p) + 4:]: v for k, v in t.items() if k.startswith(p + "mix.")}
        h = rms_norm(x, t[p + "norm1"], eps)
        if ly["type"] == "mlstm":
            y = memory_mixer(h, mix, ly["mixer"], eps)
        else:
            y, mine = attention_mixer(h, mix, ly["mixer"], eps, v_first)
            v_first = mine if mine is not None else v_first
        y = residual_gate(y, h, t[p + "rg1"], t[p + "rg1.b"])
        x = x + rms_norm(y, t[p + "norm1b"], eps) * t[p + "ls1"]
        if ly["mlp"] is not None:
            h = rms_norm(x, t[p + "norm2"], eps)
            y = feed_forward(h, t[p + "mlp.up"], t[p + "mlp.down"], t[p + "mlp.act"])
            y = residual_gate(y, h, t[p + "rg2"], t[p + "rg2.b"])
            x = x + rms_norm(y, t[p + "norm2b"], eps) * t[p + "ls2"]
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
def memory_layer(heads, dim, vdim, cap, ff=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def attention_layer(heads, kv_heads, dim, vdim, scale, coef, every, v_mix=True, ff=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale,
                                           "q_temp": {"coef": coef, "every": every}, "v_mix": v_mix},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def make_config(layers, width, vocab, eps=2e-5, embed_scale=1.7):
    return {"architecture": "Mutolix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "layers": layers}


def make_tensors(cfg, seed):
    """Random bfloat16 tensors of a configuration.  Projections keep the scale of their input; forget
    gates are mostly near one, so that far tokens still count; slopes of the distance bias differ by
    head; norm weights and gates move away from their neutral value."""
    g = torch.Generator().manual_seed(seed)
    W, t = cfg["width"], {}

    def mat(name, rows, cols, gain=1.0):
        t[name] = (torch.randn(rows, cols, generator=g) * gain / cols ** 0.5).bfloat16()

    def vec(name, n, mean, spread=0.3):
        t[name] = (mean + spread * torch.randn(n, generator=g)).bfloat16()
    mat("embed", cfg["vocab"], W, W ** 0.5 * 0.5)
    mat("head", cfg["vocab"], W)
    vec("final.norm", W, 1.0)
    for i, ly in enumerate(cfg["layers"]):
        p, m = f"l{i}.", ly["mixer"]
        H, d, dv = m["heads"], m["dim"], m["vdim"]
        for s in ("1", "2") if ly["mlp"] is not None else ("1",):
            vec(p + "norm" + s, W, 1.0)
            vec(p + f"norm{s}b", W, 1.0)
            vec(p + "ls" + s, W, 0.8)
            mat(p + "rg" + s, W, W, 1.5)
            vec(p + f"rg{s}.b", W, 1.0, 0.6)
        if ly["type"] == "mlstm":
            mat(p + "mix.q", H * d, W, 1.5)
            mat(p + "mix.k", H * d, W, 1.5)
            mat(p + "mix.v", H * dv, W)
            mat(p + "mix.g", H * dv, W, 1.5)
            mat(p + "mix.o", W, H * dv)
            vec(p + "mix.norm", H * dv, 1.0)
            mat(p + "mix.i", H, W, 1.5)
            vec(p + "mix.i.b", H, -0.5, 1.0)
            mat(p + "mix.f", H, W, 1.0)
            vec(p + "mix.f.b", H, 4.0, 1.5)
        else:
            G = m["kv_heads"]
            for name, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                mat(p + "mix." + name, rows, W)
                vec(p + f"mix.{name}.b", rows, 0.0)
            vec(p + "mix.q.norm", H * d, 1.3)
            vec(p + "mix.k.norm", G * d, 1.3)
            if m.get("v_mix"):
                t[p + "mix.vmix"] = torch.rand((), generator=g).mul(0.6).add(0.2).bfloat16()
            t[p + "mix.r1"] = torch.rand(H, generator=g).mul(2.0).bfloat16()
            t[p + "mix.r2"] = torch.rand(H, generator=g).mul(0.5).add(0.05).bfloat16()
            mat(p + "mix.o", W, H * dv)
        if ly["mlp"] is not None:
            mat(p + "mlp.up", ly["mlp"]["ff"], W)
            mat(p + "mlp.down", W, ly["mlp"]["ff"])
            t[p + "mlp.act"] = torch.tensor([0.8, -0.9]).bfloat16()
    return t
