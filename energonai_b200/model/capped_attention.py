"""Causal attention of query heads in groups that share a key / value head, without rotations: scores are capped by
cap * tanh(score / cap), a slope per head times the distance is taken off, one is added to the softmax denominator.
A window may keep the first positions visible; values are cached over their head's root mean square; the
concatenated heads are multiplied by the sigmoid of a gate.

One product of h gives query, key, value and gate.  The gate is applied where the attention stores its result."""
import torch
from torch import nn

from ..attention import (attention_group_decode_capped, attention_plain_capped, attention_prefill_capped, attention_values, distance_slopes, sigmoid_gate)
from ..gemm import project
from ..nn import init_weight
from .grouped_attention import padded_head
from .sequence_state import RingCache, round_up


class CappedAttention(nn.Module):
    output_bias = True

    def __init__(self, layer, width, cfg, eps, dtype, device=None):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.layer, self.eps = layer, eps
        self.heads, self.kv_heads, self.dim, self.vdim = cfg.heads, cfg.kv_heads, cfg.dim, cfg.vdim
        head = padded_head([cfg.dim, cfg.vdim], dtype)
        self.tensor_core = head is not None and cfg.scale > 0
        self.dk, self.dv = (head, head) if self.tensor_core else (round_up(cfg.dim, 8), round_up(cfg.vdim, 8))
        H, G = self.heads, self.kv_heads
        self.splits = [H * self.dk, G * self.dk, G * self.dv, H * self.dv]
        self.columns = H * self.dv                                                         # of the result
        self.in_proj = init_weight(sum(self.splits), width, **kw)                          # q | k | v | gate
        self.bias = init_weight(sum(self.splits), std=0.0, **kw)
        self.window, self.keep = cfg.window, cfg.keep_first if cfg.window else 0
        self.rule = dict(window=self.window, keep=self.keep, cap=cfg.softcap, scale=cfg.scale)
        self.register_buffer("slopes", distance_slopes(H, device), persistent=False)

    def caches(self):
        return {(self.layer, "keys"): RingCache(self.kv_heads * (self.dk + self.dv), window=self.window, keep=self.keep)}

    def forward(self, h, ctx, out):
        """h [rows, width] -> out [rows, columns]; keys and values are cached."""
        B, S, H, G = ctx.batch, ctx.seq, self.heads, self.kv_heads
        buf = ctx.state.caches[self.layer, "keys"].buf
        kc, vc = buf[:, :, :G * self.dk], buf[:, :, G * self.dk:]
        q, k, v, gate = project(h, self.in_proj, bias=self.bias).split(self.splits, 1)
        attention_values(k, v, G, self.vdim, self.eps, kc, vc, self.keep, S, pos_device=ctx.pos, first=ctx.first)
        rule = dict(self.rule, slopes=self.slopes, sink=True, first=ctx.first)
        seq = lambda t: t.view(B, S, -1)
        if not self.tensor_core:
            keys, values, kept = (seq(k), seq(v), 0) if ctx.is_prompt else (kc, vc, self.keep)
            o = attention_plain_capped(seq(q), keys, values, H, self.dk, self.dv, kept_rows=kept, pos_device=ctx.pos, kv_heads=G, **rule)
            return sigmoid_gate(o.view(B * S, -1), gate, out=out)
        if ctx.is_prompt:                # (the ring has only the last positions of a prompt)
            return attention_prefill_capped(seq(q), seq(k), seq(v), self.dk, self.dv, gate=seq(gate), out=seq(out), **rule)
        return attention_group_decode_capped(q, kc, vc, self.dk, ctx.pos, gate=gate, out=out, **rule)
