"""Tensors of a Tulezen checkpoint -> the parameters of LatentDecoder.

Checkpoint names: 'embed', 'head', 'final.norm'; per layer 'l<i>.norm1', 'l<i>.norm2',
'l<i>.mix.{q, dkv, dkv.norm, uk, uv, o}' (no dkv with kv_from), 'l<i>.mlp.router' and
'l<i>.mlp.e<j>.{gate, up, down}'; weights [out, in].  The model keeps them in the layouts its kernels
read: projections stacked, heads / latent / experts' width padded with zeros, gates and ups
interleaved in blocks of 8 rows."""
import torch

__all__ = ["processing_Tulezen"]


def _pad(t, *shape):
    out = torch.zeros(shape, dtype=t.dtype)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


def processing_Tulezen(state_dict, model):
    left = dict(state_dict)
    cfg, W, dtype = model.config, model.hidden_size, model.dtype

    def take(name, *shape):
        if name not in left:
            raise KeyError(f"checkpoint lacks {name}")
        t = left.pop(name)
        if tuple(t.shape) != shape:
            raise ValueError(f"{name}: shape {tuple(t.shape)}, the configuration asks for {shape}")
        return t

    def heads_out(t, heads, dim, padded, cols):
        """[heads*dim, in] -> [heads*padded, cols], every head padded on its own."""
        return _pad(t.reshape(heads, dim, -1), heads, padded, cols).reshape(heads * padded, cols)

    w = cfg.width
    out = {"embed": _pad(take("embed", cfg.vocab, w), cfg.vocab, W),
           "head": _pad(take("head", cfg.vocab, w), *model.head.shape),
           "norm.weight": _pad(take("final.norm", w), W)}
    for i, (lc, blk) in enumerate(zip(cfg.layers, model.layers)):
        p, o, m, at = f"l{i}.", f"layers.{i}.", lc.mixer, blk.mixer
        out[o + "norm1.weight"] = _pad(take(p + "norm1", w), W)
        q = heads_out(take(p + "mix.q", m.heads * m.dim, w), m.heads, m.dim, at.dk, W)
        if m.kv_from is None:
            q = torch.cat([q, _pad(take(p + "mix.dkv", m.kv_rank, w), at.rank, W)])
            out[o + "mixer.latent_norm.weight"] = _pad(take(p + "mix.dkv.norm", m.kv_rank), at.rank)
        out[o + "mixer.in_proj"] = q
        uk = heads_out(take(p + "mix.uk", m.heads * m.dim, m.kv_rank), m.heads, m.dim, at.dk, at.rank)
        uv = heads_out(take(p + "mix.uv", m.heads * m.vdim, m.kv_rank), m.heads, m.vdim, at.dv, at.rank)
        out[o + "mixer.kv_up"] = torch.cat([uk, uv])
        out[o + "mixer.k_absorb"] = uk.view(m.heads, at.dk, at.rank).transpose(1, 2).contiguous()
        wo = take(p + "mix.o", w, m.heads * m.vdim)
        out[o + "mixer.out_proj"] = _pad(wo.reshape(w, m.heads, m.vdim), W, m.heads, at.dv).reshape(W, m.heads * at.dv)
        if lc.mlp is None:
            continue
        E, ff, ffp = lc.mlp.experts, lc.mlp.ff, blk.mlp.ff_padded
        out[o + "norm2.weight"] = _pad(take(p + "norm2", w), W)
        out[o + "mlp.router"] = _pad(take(p + "mlp.router", E, w), *blk.mlp.router.shape)
        # filled expert by expert: a stack of every padded expert would hold them all twice
        gate_up, down = torch.zeros(E, ffp // 8, 2, 8, W, dtype=dtype), torch.zeros(E, W, ffp, dtype=dtype)
        for e in range(E):
            for k, name in enumerate(("gate", "up")):
                gate_up[e, :, k] = _pad(take(f"{p}mlp.e{e}.{name}", ff, w), ffp, W).view(ffp // 8, 8, W)
            down[e, :w, :ff] = take(f"{p}mlp.e{e}.down", w, ff)
        out[o + "mlp.gate_up"] = gate_up.view(E, 2 * ffp, W)
        out[o + "mlp.down"] = down
    if left:
        raise KeyError(f"checkpoint has tensors the configuration does not: {', '.join(sorted(left)[:8])}")
    return {k: v.to(dtype) for k, v in out.items()}
