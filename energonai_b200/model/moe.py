"""Mixture-of-experts feed-forward: a softmax router over all experts, the `top` best with their
scores as they are, experts with a clamped gated unit.

Prompt-sized batches sort their rows by expert and run grouped tensor-core products; generation
steps stream the weights of the experts that were chosen.  forward() returns what the residual
kernel needs to form the weighted sum of a token's expert rows itself."""
import torch
from torch import nn

from ..gemm import project
from ..moe import SKINNY_MAX_ENTRIES, SortedRows, grouped_gemm, new_counts, route, skinny_experts
from ..nn import init_weight
from .sequence_state import round_up

SKINNY_MAX_TOKENS = 128      # up to here an expert gets a handful of rows: stream its weights instead


class MixtureOfExperts(nn.Module):
    def __init__(self, width, experts, top, ff, limit, alpha, dtype, device=None):
        super().__init__()
        if not 0 < top <= experts:
            raise ValueError(f"mixture of experts: top {top} of {experts} experts")
        self.experts, self.top, self.ff, self.gate = experts, top, ff, (limit, alpha)
        self.ff_padded = round_up(ff, 8)
        self.router = init_weight(round_up(experts, 8), width, dtype=dtype, device=device)
        self.gate_up = init_weight(experts, 2 * self.ff_padded, width, dtype=dtype, device=device)   # blocks of 8 gates, 8 ups
        self.down = init_weight(experts, width, self.ff_padded, dtype=dtype, device=device)
        self._counts = None

    def skinny(self, tokens):
        return tokens <= SKINNY_MAX_TOKENS and tokens * self.top <= SKINNY_MAX_ENTRIES and self.router.dtype != torch.float32

    def router_for_step(self, tokens):
        """(weight, experts, top) for the residual kernel to evaluate the router itself, or None."""
        return (self.router, self.experts, self.top) if self.skinny(tokens) else None

    def forward(self, h, first=None, rows_per_batch=1, routed=None):
        """h [T, width] -> (y, (idx, rows, weights)).  routed: (idx, weights) if the router has been
        evaluated already.  first: padding positions per sequence, which get no expert."""
        T = h.shape[0]
        if self.skinny(T):
            idx, w = routed if routed is not None else route(project(h, self.router, out_dtype=torch.float32),
                                                             self.experts, self.top, first, rows_per_batch)
            act = skinny_experts(h, self.gate_up, idx, self.top, gate=self.gate)
            return skinny_experts(act, self.down, idx, 1), (idx, None, w)
        if self._counts is None or self._counts.device != h.device:
            self._counts = new_counts(self.experts, h.device)
        logits = project(h, self.router, out_dtype=torch.float32)
        idx, w, ranks = route(logits, self.experts, self.top, first, rows_per_batch, counts=self._counts)
        plan = SortedRows(h, idx, ranks, self._counts)
        act = grouped_gemm(plan.x, self.gate_up, plan, gate=self.gate)
        return grouped_gemm(act, self.down, plan), (idx, plan.rows, w)
