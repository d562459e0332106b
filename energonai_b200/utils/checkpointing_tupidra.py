"""Tensors of a Tupidra checkpoint -> the parameters of ParallelDecoder.

Checkpoint names: 'embed', 'head', 'final.norm'; per layer 'l<i>.norm1', 'l<i>.canon1' and, with a feed-forward,
'l<i>.norm2', 'l<i>.canon2'; 'l<i>.mix.*' and 'l<i>.mlp.*'; weights [out, in].  The model keeps the projections of one
input stacked, the output weights of mixer and feed-forward side by side, heads and states padded with zeros, gates
and ups interleaved in blocks of 8 rows, a norm's weight times each tap in fp32, and maps of a latent row that
carry its rotated part through with ones."""
import torch

from ..model.latent_attention import RotaryLatentAttention
from ..model.selective_scan import SelectiveScan
from .checkpointing_tulezen import _pad

__all__ = ["processing_Tupidra"]


def processing_Tupidra(state_dict, model):
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

    def table(p, k):
        """norm weight * (tap, one more for the current token's), [taps, W]; shorter tables get zero rows in front."""
        taps = take(f"{p}canon{k}", w, cfg.taps).float().t().clone()
        taps[-1] += 1
        out = torch.zeros(model.taps, W)
        out[model.taps - cfg.taps:, :w] = taps * take(f"{p}norm{k}", w).float()
        return out

    def scan(p, o, m, at):
        C, N, R, inner = m.inner, m.state, m.dt_rank, at.inner
        out[o + "in_proj"] = torch.cat([rows(t, inner) for t in take(p + "in", 2 * C, w).split(C)])
        out[o + "conv_w"] = _pad(take(p + "conv", C, m.conv).t(), m.conv, inner)
        out[o + "conv_b"] = _pad(take(p + "conv.b", C), inner)
        dt, B, Cn = take(p + "x", R + 2 * N, C).split([R, N, N])
        out[o + "x_proj"] = torch.cat([_pad(dt, at.rank, inner), _pad(B, at.states, inner), _pad(Cn, at.states, inner)])
        out[o + "dt_proj"] = _pad(take(p + "dt", C, R), inner, at.rank)
        out[o + "dt_bias"], out[o + "skip"] = _pad(take(p + "dt.b", C), inner), _pad(take(p + "D", C), inner)
        out[o + "a_log"] = _pad(take(p + "A_log", C, N), inner, at.states)
        return _pad(take(p + "o", w, C), W, inner)

    def attention(p, o, m, at):
        H, G, d, dv = m.heads, m.kv_heads, m.dim, m.vdim
        parts = [("q", H, d, at.dk), ("k", G, d, at.dk), ("v", G, dv, at.dv)]
        gate = heads(rows(take(p + "g", H * dv, w)), H, dv, at.dv)
        out[o + "in_proj"] = torch.cat([heads(rows(take(p + n, k * s, w)), k, s, to) for n, k, s, to in parts] + [gate])
        out[o + "bias"] = _pad(torch.cat([heads(take(f"{p}{n}.b", k * s), k, s, to) for n, k, s, to in parts]), at.in_proj.shape[0])
        return columns(take(p + "o", w, H * dv), H, dv, at.dv)

    def latent(p, o, m, at):
        H, d, r, dv, qr, kr = m.heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank
        stacked = [rows(take(p + "dq", qr, w), at.q_cols)]
        out[o + "q_norm"] = _pad(take(p + "dq.norm", qr), at.q_cols)
        if m.kv_from is None:
            c, rot = take(p + "dkv", kr + r, w).split([kr, r])
            stacked += [rows(c, at.rot_col), rows(rot, at.rank - at.rot_col)]
            out[o + "latent_norm"] = _pad(take(p + "dkv.norm", kr), at.rot_col)
        out[o + "in_proj"] = torch.cat(stacked + [heads(rows(take(p + "g", H * dv, w)), H, dv, at.dv)])
        q = take(p + "uq", H * (d + r), qr).view(H, d + r, qr)
        q_up = torch.zeros(H, at.dk, at.q_cols, dtype=q.dtype)
        q_up[:, :d, :qr], q_up[:, at.rot_at:at.rot_at + r, :qr] = q[:, :d], q[:, d:]
        keys = _pad(take(p + "uk", H * d, kr).view(H, d, kr), H, at.dk, at.rank)
        i = torch.arange(r)
        keys[:, at.rot_at + i, at.rot_col + i] = 1                                         # the rotated part as it is
        values = _pad(take(p + "uv", H * dv, kr).view(H, dv, kr), H, at.dv, at.rank)
        out[o + "q_up"] = q_up.view(at.q_rows, at.q_cols)
        out[o + "kv_up"] = torch.cat([keys.view(at.q_rows, at.rank), values.view(at.columns, at.rank)])
        out[o + "k_absorb"] = keys.transpose(1, 2).contiguous()
        out[o + "sinks"] = take(p + "sink", H)
        return columns(take(p + "o", w, H * dv), H, dv, at.dv)

    out = {"embed": rows(take("embed", cfg.vocab, w)), "head": rows(take("head", cfg.vocab, w), model.head.shape[0]),
           "norm.weight": _pad(take("final.norm", w), W)}
    for i, (lc, blk) in enumerate(zip(cfg.layers, model.layers)):
        p, o, m, at = f"l{i}.", f"layers.{i}.", lc.mixer, blk.mixer
        kind = scan if isinstance(at, SelectiveScan) else latent if isinstance(at, RotaryLatentAttention) else attention
        out[o + "taps1"] = table(p, 1)
        weights = [kind(p + "mix.", o + "mixer.", m, at)]
        if blk.bias is not None:
            out[o + "bias"] = _pad(take(p + "mix.o.b", w), W)
        if blk.mlp is not None:
            out[o + "taps2"] = table(p, 2)
            f = blk.mlp
            gate, up = (rows(take(f"{p}mlp.{n}", f.ff, w), f.ff_padded).view(-1, 1, 8, W) for n in ("gate", "up"))
            out[o + "mlp.gate_up"] = torch.cat([gate, up], 1).reshape(2 * f.ff_padded, W)
            weights.append(_pad(take(p + "mlp.down", w, f.ff), W, f.ff_padded))
        out[o + "out_proj"] = torch.cat(weights, 1)
    if left:
        raise KeyError(f"checkpoint has tensors the configuration does not: {', '.join(sorted(left)[:8])}")
    have = model.state_dict()
    return {k: v.to(have[k].dtype) for k, v in out.items()}
