"""Matrix-memory mixer: per head a matrix state S with a normaliser n and a running maximum m of its log
gates, carried in fp32 from token to token (the equations are with eb_memory_scan in the header).

One product of h gives queries, keys, values, output gates, the pre-activation of the residual gate and,
in fp32, those of the two recurrence gates."""
import torch
from torch import nn

from ..gemm import project, project_parts
from ..memory import MEMORY_KEY_HEADS, head_norm_gate, memory_prompt, memory_step
from ..nn import init_weight
from .sequence_state import RecurrentState, round_up


class MatrixMemory(nn.Module):
    def __init__(self, layer, width, heads, dim, vdim, gate_cap, eps, dtype, device=None):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.layer, self.width, self.heads, self.dim, self.vdim, self.cap, self.eps = layer, width, heads, dim, vdim, gate_cap, eps
        self.scale = dim ** -0.5
        self.chunked = dtype == torch.bfloat16 and dim <= MEMORY_KEY_HEADS[-1]      # prompts on the tensor cores
        self.dk = min(n for n in MEMORY_KEY_HEADS if n >= dim) if self.chunked else round_up(dim, 8)
        self.dv = round_up(vdim, 8)
        qk, vg = heads * self.dk, heads * self.dv
        self.splits = [qk, qk, vg, vg, width]
        self.tail = sum(self.splits)
        # q | k | v | output gate | residual gate || input gates | forget gates
        self.in_proj = init_weight(self.tail + round_up(2 * heads, 8), width, **kw)
        self.bias = init_weight(self.in_proj.shape[0], std=0.0, **kw)           # (the recurrence gates' is gate_bias)
        self.gate_bias = nn.Parameter(torch.zeros(2, heads, dtype=torch.float32, device=device), requires_grad=False)
        self.norm = nn.Parameter(torch.ones(vg, dtype=dtype, device=device), requires_grad=False)
        self.out_proj = init_weight(width, vg, **kw)

    def cache(self):
        return RecurrentState([(self.heads, self.dk, self.dv), (self.heads, self.dk), (self.heads,)])

    def forward(self, h, ctx):
        """h [rows, width] -> (y, pre-activation of the residual gate); the state goes on."""
        state = ctx.state.caches[self.layer].tensors
        rows, gates = project_parts(h, self.in_proj, bias=self.bias, tail_col=self.tail)
        q, k, v, g, rg = rows.split(self.splits, 1)
        bias = self.gate_bias.unbind(0)
        if ctx.is_prompt:
            o = memory_prompt(q, k, v, gates, bias, self.cap, self.scale, state, self.heads, first=ctx.first, chunked=self.chunked)
            y = head_norm_gate(o, g, self.norm, self.heads, self.vdim, self.eps)
        else:
            y = memory_step(q, k, v, g, gates, bias, self.cap, self.scale, self.norm, self.vdim, self.eps, state, self.heads)
        return project(y, self.out_proj), rg
