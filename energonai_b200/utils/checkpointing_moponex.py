"""Tensors of a Moponex checkpoint -> the parameters of HybridDecoder.

Checkpoint names: 'embed' (also the head), 'bigram', 'final.norm'; per layer 'l<i>.norm1' and, with a
feed-forward, 'l<i>.norm2'; 'l<i>.mix.*' and 'l<i>.mlp.*'; weights [out, in].  The model keeps the projections of
one input stacked, heads padded with zeros, gates and ups interleaved in blocks of 8 rows, and the
weights of the parallel mixers' output norms times one half (exact in fp32)."""
import torch

from ..model.mlp import GEGLUFeedForward
from ..model.state_space import StateSpace
from .checkpointing_tulezen import _pad

__all__ = ["processing_Moponex"]


def processing_Moponex(state_dict, model):
    left = dict(state_dict)
    cfg, w, W = model.config, model.width, model.hidden_size

    def take(name, *shape):
        if name not in left:
            raise KeyError(f"checkpoint lacks {name}")
        t = left.pop(name)
        if tuple(t.shape) != shape:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration asks for {shape}")
        return t

    def heads(t, n, dim, padded):
        """[n*dim, ...] -> [n*padded, ...], every head padded on its own."""
        return _pad(t.reshape(n, dim, -1), n, padded, t.numel() // (n * dim)).reshape(n * padded, *t.shape[1:])

    def rows(t, n=None):
        return _pad(t, n or t.shape[0], W)

    def columns(t, n, dim, padded):
        """[out, n*dim] -> [W, n*padded]."""
        return _pad(t.reshape(-1, n, dim), W, n, padded).reshape(W, n * padded)

    def linear(p, name, n, dim, padded):
        return heads(rows(take(p + name, n * dim, w)), n, dim, padded)

    embed = rows(take("embed", cfg.vocab, w), model.embed.shape[0])
    out = {"embed": embed, "head": embed, "norm.weight": _pad(take("final.norm", w), W)}
    if cfg.bigram:
        out["bigram"] = rows(take("bigram", cfg.bigram.buckets + 1, w))

    def state_space(p, o, at, taps):
        H, P, G, N = at.heads, at.vdim, at.groups, at.state
        z, x, B, C, dt = take(p + "in", 2 * H * P + 2 * G * N + H, w).split([H * P, H * P, G * N, G * N, H])
        pad = lambda parts: [heads(parts[0], H, P, at.dv), heads(parts[1], G, N, at.dk), heads(parts[2], G, N, at.dk)]
        out[o + "in_proj"] = torch.cat([heads(rows(z), H, P, at.dv)] + pad([rows(t) for t in (x, B, C)]) + [rows(dt, at.in_proj.shape[0] - at.tail)])
        sizes = [H * P, G * N, G * N]
        out[o + "conv_w"] = torch.cat(pad(take(p + "conv", sum(sizes), taps).split(sizes))).t().contiguous()
        out[o + "conv_b"] = torch.cat(pad(take(p + "conv.b", sum(sizes)).split(sizes)))
        out[o + "dt_bias"], out[o + "a_log"], out[o + "skip"] = take(p + "dt_bias", H), take(p + "A_log", H), take(p + "D", H)
        out[o + "norm"] = heads(take(p + "norm", H * P), H, P, at.dv)
        out[o + "out_proj"] = columns(take(p + "o", w, H * P), H, P, at.dv)

    def parallel(p, o, at):
        a, r = at.left, at.right
        parts = [linear(p, "left.q", a.heads, a.dim, a.dk), linear(p, "left.k", a.kv_heads, a.dim, a.dk)]
        bias = [heads(take(p + "left.q.b", a.heads * a.dim), a.heads, a.dim, a.dk), heads(take(p + "left.k.b", a.kv_heads * a.dim), a.kv_heads, a.dim, a.dk)]
        for name, dim, padded in (("q", r.dim, r.dk), ("k", r.dim, r.dk), ("v", r.vdim, r.dv), ("g", r.vdim, r.dv)):
            parts.append(linear(p, "right." + name, r.heads, dim, padded))
        parts.append(rows(take(p + "right.a1", r.rank, w), r.low))
        out[o + "in_proj"] = torch.cat(parts)
        out[o + "bias"] = _pad(torch.cat(bias), at.in_proj.shape[0])
        out[o + "left.q_norm"], out[o + "left.k_norm"] = (_pad(take(f"{p}left.{n}.norm", a.dim), a.dk) for n in "qk")
        out[o + "left.sinks"] = take(p + "left.sink", a.heads)
        out[o + "left_proj"] = columns(take(p + "left.o", w, a.heads * a.dim), a.heads, a.dim, a.dk)
        a2 = take(p + "right.a2", r.heads * r.dim, r.rank)
        out[o + "right.a2"] = heads(_pad(a2, a2.shape[0], r.low), r.heads, r.dim, r.dk)
        out[o + "right.a2_bias"] = heads(take(p + "right.a2.b", r.heads * r.dim), r.heads, r.dim, r.dk)
        out[o + "right.norm"] = _pad(take(p + "right.norm", r.vdim), r.dv).repeat(r.heads)
        out[o + "right_proj"] = columns(take(p + "right.o", w, r.heads * r.vdim), r.heads, r.vdim, r.dv)
        for side in ("left", "right"):
            out[f"{o}{side}_out"] = _pad(take(f"{p}{side}.out", w).float() * 0.5, W)

    def dense(p, o, at):
        gate, up = (rows(take(p + n, at.ff, w), at.ff_padded).view(-1, 1, 8, W) for n in ("gate", "up"))
        out[o + "gate_up"] = torch.cat([gate, up], 1).reshape(2 * at.ff_padded, W)
        out[o + "down"] = _pad(take(p + "down", w, at.ff), W, at.ff_padded)

    def routed(p, o, at):
        router = [take(p + "router", at.choices, w)]
        out[o + "correction"] = take(p + "correction", at.choices)
        # filled expert by expert: a stack of every padded expert would hold them all twice
        up, down = torch.zeros(at.up.shape, dtype=model.dtype), torch.zeros(at.down.shape, dtype=model.dtype)
        for e in range(at.experts):
            up[e, :at.ff, :w] = take(f"{p}e{e}.up", at.ff, w)
            down[e, :w, :at.ff] = take(f"{p}e{e}.down", w, at.ff)
        out[o + "up"], out[o + "down"] = up, down
        if at.gated:
            router.append(take(p + "shared.sg", 1, w))
            out[o + "shared_up"] = rows(take(p + "shared.up", at.shared_ff, w), at.shared_padded)
            out[o + "shared_down"] = _pad(take(p + "shared.down", w, at.shared_ff), W, at.shared_padded)
        out[o + "router"] = rows(torch.cat(router), at.router.shape[0])

    for i, (lc, blk) in enumerate(zip(cfg.layers, model.layers)):
        p, o = f"l{i}.", f"layers.{i}."
        out[o + "norm1"] = _pad(take(p + "norm1", w), W)
        if isinstance(blk.mixer, StateSpace):
            state_space(p + "mix.", o + "mixer.", blk.mixer, lc.mixer.conv)
        else:
            parallel(p + "mix.", o + "mixer.", blk.mixer)
        if blk.mlp is not None:
            out[o + "norm2"] = _pad(take(p + "norm2", w), W)
            (dense if isinstance(blk.mlp, GEGLUFeedForward) else routed)(p + "mlp.", o + "mlp.", blk.mlp)
    if left:
        raise KeyError(f"checkpoint has tensors the configuration does not: {', '.join(sorted(left)[:8])}")
    have = model.state_dict()
    return {k: v.to(have[k].dtype) for k, v in out.items()}
