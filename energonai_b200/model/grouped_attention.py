"""Causal attention of query heads in groups that share a key / value head, without rotations: the
position enters through a bias that grows with the logarithm of the distance and through a query
temperature.  Query and key are normalised over their whole projection, the softmax has a sink (one is
added to its denominator), and the values may be mixed with those of an earlier layer.

Head sizes are padded with zeros to what the tensor-core kernels take; layers that share values share
the padding."""
import torch
from torch import nn

from ..attention import (attention_group_decode, attention_inputs, attention_plain, attention_prefill_biased, distance_bias)
from ..gemm import project
from ..nn import init_weight
from .sequence_state import RingCache, round_up

TENSOR_CORE_HEADS = (64, 128)


def padded_head(dims, dtype):
    """Head size of a group of layers that share values: 64 or 128 for the tensor-core kernels if the
    largest of `dims` fits, else None (every size rounded to 8, kernels without tensor cores)."""
    if dtype == torch.float32 or max(dims) > TENSOR_CORE_HEADS[-1]:
        return None
    return min(n for n in TENSOR_CORE_HEADS if n >= max(dims))


class GroupedAttention(nn.Module):
    def __init__(self, layer, width, cfg, head, eps, dtype, device=None):
        """cfg: GroupedAttentionConfig; head: padded head size (padded_head) or None."""
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.layer, self.width, self.eps = layer, width, eps
        self.heads, self.kv_heads, self.dim, self.vdim, self.scale = cfg.heads, cfg.kv_heads, cfg.dim, cfg.vdim, cfg.scale
        self.temp = (cfg.temp_coef, cfg.temp_every) if cfg.temp_every else None
        self.v_from = cfg.v_from
        self.tensor_core = head is not None and cfg.scale > 0
        self.dk, self.dv = (head, head) if head is not None else (round_up(cfg.dim, 8), round_up(cfg.vdim, 8))
        H, G = self.heads, self.kv_heads
        self.splits = [H * self.dk, G * self.dk, G * self.dv, width]
        self.in_proj = init_weight(sum(self.splits), width, **kw)               # q | k | v | residual gate
        self.bias = init_weight(sum(self.splits), std=0.0, **kw)
        self.q_norm = nn.Parameter(torch.ones(H * self.dk, **kw), requires_grad=False)
        self.k_norm = nn.Parameter(torch.ones(G * self.dk, **kw), requires_grad=False)
        fp32 = lambda *s: nn.Parameter(torch.zeros(*s, dtype=torch.float32, device=device), requires_grad=False)
        self.r1, self.r2, self.vmix = fp32(H), fp32(H), fp32(1)
        self.out_proj = init_weight(width, H * self.dv, **kw)

    def cache(self):
        return RingCache(self.kv_heads * (self.dk + self.dv))

    def _keys_values(self, ctx, layer):
        """Key and value views of a layer's cache (of this layer's sizes)."""
        buf = ctx.state.caches[layer].buf
        n = buf.shape[2] - self.kv_heads * self.dv
        return buf[:, :, :n], buf[:, :, n:]

    def forward(self, h, ctx):
        """h [rows, width] -> (y, pre-activation of the residual gate); keys and values are cached."""
        B, S, H, G = ctx.batch, ctx.seq, self.heads, self.kv_heads
        proj = project(h, self.in_proj, bias=self.bias)
        k, v = self._keys_values(ctx, self.layer)
        mix = self.v_from is not None
        q = attention_inputs(proj, H, G, self.dk, self.dv, self.q_norm, H * self.dim, self.k_norm, G * self.dim, self.eps, k, v, S,
                             temp=self.temp, vmix=self.vmix if mix else None, v_first=self._keys_values(ctx, self.v_from)[1] if mix else None,
                             pos_device=ctx.pos, first=ctx.first).view(B, S, -1)
        bias = (self.r1, self.r2)
        if not self.tensor_core:
            o = attention_plain(q, k, v, H, self.dk, self.dv, scale=self.scale, first=ctx.first, pos_device=ctx.pos, kv_heads=G, bias=bias,
                                sink=True)
        elif ctx.is_prompt:
            o = attention_prefill_biased(q, k[:, :S], v[:, :S], self.dk, distance_bias(*bias, S), mask=ctx.mask, scale=self.scale)
        else:
            o = attention_group_decode(q.view(B, -1), k, v, self.dk, ctx.pos, self.scale, first=ctx.first, bias=bias)
        return project(o.view(B * S, -1), self.out_proj), proj[:, proj.shape[1] - self.width:]
