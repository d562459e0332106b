"""Tensors of a Mutolix checkpoint -> the parameters of SandwichDecoder.

Checkpoint names: 'embed', 'head', 'final.norm'; per layer 'l<i>.norm1', 'l<i>.norm1b', 'l<i>.ls1',
'l<i>.rg1', 'l<i>.rg1.b' and the same with 2 if there is a feed-forward; 'l<i>.mix.*' and
'l<i>.mlp.{up, down, act}'; weights [out, in].  The model keeps the projections of one input stacked,
heads padded with zeros, output norm and layer scale multiplied (exact in fp32 for 16-bit factors)."""
import torch

from ..gemm import xielu_params
from ..model.grouped_attention import GroupedAttention
from .checkpointing_tulezen import _pad

__all__ = ["processing_Mutolix"]


def processing_Mutolix(state_dict, model):
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

    def rows(t):
        return _pad(t, t.shape[0], W)

    def columns(t, n, dim, padded):
        """[out, n*dim] -> [W, n*padded]."""
        return _pad(t.reshape(-1, n, dim), W, n, padded).reshape(W, n * padded)

    out = {"embed": _pad(take("embed", cfg.vocab, w), cfg.vocab, W), "head": _pad(take("head", cfg.vocab, w), *model.head.shape),
           "norm.weight": _pad(take("final.norm", w), W)}

    def sublayer(p, o, s):
        """Norms of sublayer s; returns weight and bias of its residual gate."""
        out[f"{o}norm{s}"] = _pad(take(f"{p}norm{s}", w), W)
        out[f"{o}out{s}"] = _pad(take(f"{p}norm{s}b", w).float() * take(f"{p}ls{s}", w).float(), W)
        return _pad(take(f"{p}rg{s}", w, w), W, W), _pad(take(f"{p}rg{s}.b", w), W)

    def attention(p, o, m, at, gate, gate_bias):
        H, G = m.heads, m.kv_heads
        parts, bias = [], []
        for name, n, dim, padded in (("q", H, m.dim, at.dk), ("k", G, m.dim, at.dk), ("v", G, m.vdim, at.dv)):
            parts.append(heads(rows(take(p + name, n * dim, w)), n, dim, padded))
            bias.append(heads(take(f"{p}{name}.b", n * dim), n, dim, padded))
        out[o + "in_proj"], out[o + "bias"] = torch.cat(parts + [gate]), torch.cat(bias + [gate_bias])
        out[o + "q_norm"] = heads(take(p + "q.norm", H * m.dim), H, m.dim, at.dk)
        out[o + "k_norm"] = heads(take(p + "k.norm", G * m.dim), G, m.dim, at.dk)
        out[o + "r1"], out[o + "r2"] = take(p + "r1", H), take(p + "r2", H)
        if p + "vmix" in left or m.v_from is not None:        # (the first layer's is there, and unused)
            out[o + "vmix"] = take(p + "vmix").reshape(1)
        else:
            out[o + "vmix"] = torch.zeros(1)
        out[o + "out_proj"] = columns(take(p + "o", w, H * m.vdim), H, m.vdim, at.dv)

    def memory(p, o, m, at, gate, gate_bias):
        H = m.heads
        q, k = (heads(rows(take(p + n, H * m.dim, w)), H, m.dim, at.dk) for n in ("q", "k"))
        v, g = (heads(rows(take(p + n, H * m.vdim, w)), H, m.vdim, at.dv) for n in ("v", "g"))
        gates = _pad(torch.cat([take(p + "i", H, w), take(p + "f", H, w)]), at.in_proj.shape[0] - at.tail, W)
        out[o + "in_proj"] = torch.cat([q, k, v, g, gate, gates])
        out[o + "bias"] = torch.cat([gate_bias.new_zeros(at.tail - W), gate_bias, gate_bias.new_zeros(gates.shape[0])])
        out[o + "gate_bias"] = torch.stack([take(p + "i.b", H), take(p + "f.b", H)])
        out[o + "norm"] = heads(take(p + "norm", H * m.vdim), H, m.vdim, at.dv)
        out[o + "out_proj"] = columns(take(p + "o", w, H * m.vdim), H, m.vdim, at.dv)

    for i, (lc, blk) in enumerate(zip(cfg.layers, model.layers)):
        p, o = f"l{i}.", f"layers.{i}."
        fill = attention if isinstance(blk.mixer, GroupedAttention) else memory
        fill(p + "mix.", o + "mixer.", lc.mixer, blk.mixer, *sublayer(p, o, 1))
        if lc.mlp is None:
            continue
        gate, gate_bias = sublayer(p, o, 2)
        ff, ffp = lc.mlp.ff, blk.mlp.ff_padded
        out[o + "mlp.up"] = torch.cat([_pad(take(p + "mlp.up", ff, w), ffp, W), gate])
        out[o + "mlp.bias"] = torch.cat([torch.zeros(ffp, dtype=gate_bias.dtype), gate_bias])
        out[o + "mlp.down"] = _pad(take(p + "mlp.down", w, ff), W, ffp)
        out[o + "mlp.act"] = xielu_params(*take(p + "mlp.act", 2).tolist())
    if left:
        raise KeyError(f"checkpoint has tensors the configuration does not: {', '.join(sorted(left)[:8])}")
    have = model.state_dict()
    return {k: v.to(have[k].dtype) for k, v in out.items()}
