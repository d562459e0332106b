"""Mixture-of-experts feed-forward: a softmax router over all experts, the `top` best with their
scores as they are, experts with a clamped gated unit.

Prompt-sized batches sort their rows by expert and run grouped tensor-core products; generation
steps stream the weights of the experts that were chosen.  forward() returns what the residual
kernel needs to form the weighted sum of a token's expert rows itself."""
import torch
from torch import nn

from ..gemm import project, project_unit
from ..moe import SKINNY_MAX_ENTRIES, RouterRule, SortedRows, grouped_gemm, new_counts, route, route_rule, skinny_experts
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
        """Whether this many tokens stream the chosen experts' weights."""
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


class RoutedExperts(MixtureOfExperts):
    """Mixture of experts without gates (gelu of the up projection): the choice is by score + correction among the
    best groups of neighbours, the weights are the chosen scores over their sum; the last choices
    stand for the input itself; a shared expert runs for every token, multiplied by a gate of its own,
    whose row is the router's last."""

    def __init__(self, width, cfg, dtype, device=None):
        nn.Module.__init__(self)
        kw = dict(dtype=dtype, device=device)
        self.experts, self.top, self.ff, self.shared_ff = cfg.experts, cfg.top, cfg.ff, cfg.shared_ff
        self.choices, self.groups, self.keep = cfg.experts + cfg.identity, cfg.groups, cfg.keep
        self.ff_padded, self.shared_padded = round_up(cfg.ff, 8), round_up(cfg.shared_ff, 8)
        self.gated = cfg.shared_ff > 0
        self.router = init_weight(round_up(self.choices + int(self.gated), 8), width, **kw)        # choices | shared expert's gate
        self.correction = nn.Parameter(torch.zeros(self.choices, dtype=torch.float32, device=device), requires_grad=False)
        self.up = init_weight(self.experts, self.ff_padded, width, **kw)
        self.down = init_weight(self.experts, width, self.ff_padded, **kw)
        if self.gated:
            self.shared_up = init_weight(self.shared_padded, width, **kw)
            self.shared_down = init_weight(width, self.shared_padded, **kw)
        self._counts = None

    def rule(self):
        return RouterRule(self.choices, self.experts, self.correction, self.groups, self.keep)

    def router_for_step(self, tokens):
        """What stream_add needs to evaluate the router itself, or None."""
        return (self.router, self.rule(), self.top, self.gated) if self.skinny(tokens) else None

    def forward(self, h, first=None, rows_per_batch=1, routed=None):
        """-> what stream_add adds.  routed: (idx, weights, shared gate) if the router has been evaluated already."""
        T, counts = h.shape[0], None
        skinny = self.skinny(T)
        if not skinny:
            if self._counts is None or self._counts.device != h.device:
                self._counts = new_counts(self.experts, h.device)
            counts = self._counts
        if routed is not None:
            idx, w, gate = routed
        else:
            idx, w, ranks, gate = route_rule(project(h, self.router, out_dtype=torch.float32), self.rule(), self.top, first, rows_per_batch,
                                             counts=counts, gated=self.gated)
        shared = project(project_unit(h, self.shared_up, "gelu"), self.shared_down) if self.gated else None
        if skinny:
            rows, y = None, skinny_experts(skinny_experts(h, self.up, idx, self.top, unit="gelu"), self.down, idx, 1)
        else:
            plan = SortedRows(h, idx, ranks, counts)
            rows, y = plan.rows, grouped_gemm(grouped_gemm(plan.x, self.up, plan, unit="gelu"), self.down, plan)
        return dict(y=y, mix=(idx, rows, w), ident=h, experts=self.experts, shared=shared, gate=gate)
