"""Matrix-memory mixer: per head a matrix state S with a normaliser n and a running maximum m of its log
gates, carried in fp32 from token to token (the equations are with eb_memory_scan in the header).

One product of h gives queries, keys, values, output gates and the pre-activation of the residual gate;
the two recurrence gates are products of their own, whose results stay in fp32.  In a generation step
they come from the launch that normalised h."""
import torch
from torch import nn

from ..gemm import project
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
        self.in_proj = init_weight(sum(self.splits), width, **kw)               # q | k | v | output gate | residual gate
        self.bias = init_weight(sum(self.splits), std=0.0, **kw)
        self.gates = init_weight(round_up(2 * heads, 8), width, **kw)           # input gates | forget gates
        self.gate_bias = nn.Parameter(torch.zeros(2, heads, dtype=torch.float32, device=device), requires_grad=False)
        self.norm = nn.Parameter(torch.ones(vg, dtype=dtype, device=device), requires_grad=False)
        self.out_proj = init_weight(width, vg, **kw)

    def step_products(self):
        """Weight of the fp32 products that the launch before a generation step's mixer can take along."""
        return self.gates

    def cache(self):
        return RecurrentState([(self.heads, self.dk, self.dv), (self.heads, self.dk), (self.heads,)])

    def forward(self, h, ctx, gates=None):
        """h [rows, width] -> (y, pre-activation of the residual gate); the state goes on."""
        state = ctx.state.caches[self.layer].tensors
        q, k, v, g, rg = project(h, self.in_proj, bias=self.bias).split(self.splits, 1)
        if gates is None:
            gates = project(h, self.gates, out_dtype=torch.float32)
        bias = self.gate_bias.unbind(0)
        if ctx.is_prompt:
            o = memory_prompt(q, k, v, gates, bias, self.cap, self.scale, state, self.heads, first=ctx.first, chunked=self.chunked)
            y = head_norm_gate(o, g, self.norm, self.heads, self.vdim, self.eps)
        else:
            y = memory_step(q, k, v, g, gates, bias, self.cap, self.scale, self.norm, self.vdim, self.eps, state, self.heads)
        return project(y, self.out_proj), rg
