"""State-space mixer (Mamba-2): a causal convolution per channel in front of a recurrence whose fp32 state per head
decays by one number per token, the gate and a norm in equal parts of the row behind it (the equations are
with eb_ssm_scan in the header).

One product of h gives gate, convolution inputs and, in fp32, the step sizes.  A sequence's state is the
recurrent one and the convolution's last inputs, a ring as long as its taps."""
import torch
from torch import nn

from ..decay import PAIRED_VALUE_HEAD, chunk_heads, gate_group_norm, short_conv, ssm_prompt, ssm_step
from ..gemm import project, project_parts
from ..nn import init_weight
from .sequence_state import RecurrentState, RingCache, round_up


class StateSpace(nn.Module):
    def __init__(self, layer, width, cfg, eps, dtype, device=None):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.layer, self.eps = layer, eps
        self.heads, self.vdim, self.state, self.groups, self.norm_groups = cfg.heads, cfg.vdim, cfg.state, cfg.groups, cfg.norm_groups
        padded = chunk_heads(cfg.state, max(cfg.vdim, PAIRED_VALUE_HEAD), dtype)           # prompts on the tensor cores
        self.chunked = padded is not None
        self.dk, self.dv = padded if self.chunked else (round_up(cfg.state, 8), round_up(cfg.vdim, 8))
        self.inner = self.heads * self.dv
        self.channels = self.inner + 2 * self.groups * self.dk
        self.tail = self.inner + self.channels
        self.in_proj = init_weight(self.tail + round_up(self.heads, 8), width, **kw)       # gate | x | B | C || step sizes
        self.conv_w = init_weight(cfg.conv, self.channels, std=0.3, **kw)                  # the last row is the current token's
        self.conv_b = init_weight(self.channels, std=0.0, **kw)
        fp32 = lambda v: nn.Parameter(torch.full((self.heads,), v, dtype=torch.float32, device=device), requires_grad=False)
        self.dt_bias, self.a_log, self.skip = fp32(-2.0), fp32(-1.0), fp32(1.0)
        self.norm = nn.Parameter(torch.ones(self.inner, **kw), requires_grad=False)
        self.out_proj = init_weight(width, self.inner, **kw)

    def caches(self):
        return {(self.layer, "conv"): RingCache(self.channels, window=self.conv_w.shape[0]),
                (self.layer, "state"): RecurrentState([(self.heads, self.dk, self.dv)])}

    def forward(self, h, ctx):
        """h [rows, width] -> [rows, width]; the state goes on."""
        ring, S = ctx.state.caches[self.layer, "conv"].buf, ctx.state.caches[self.layer, "state"].tensors[0]
        rows, dt = project_parts(h, self.in_proj, tail_col=self.tail)
        z, xbc = rows.split([self.inner, self.channels], 1)
        sizes = (self.heads, self.groups, self.dk, self.dv)
        if ctx.is_prompt:
            xbc = short_conv(xbc, self.conv_w, self.conv_b, ring, ctx.batch, first=ctx.first)
            y = ssm_prompt(xbc, dt, self.dt_bias, self.a_log, self.skip, S, *sizes, first=ctx.first, chunked=self.chunked)
        else:
            y = ssm_step(xbc, self.conv_w, self.conv_b, ring, ctx.pos, dt, self.dt_bias, self.a_log, self.skip, S, *sizes, first=ctx.first)
        return project(gate_group_norm(y, z, self.norm, self.eps, self.heads, self.vdim, self.norm_groups), self.out_proj)
