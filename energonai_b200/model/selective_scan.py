"""State-space mixer with a state per channel (Mamba): a causal convolution per channel, step sizes by a low-rank projection
of its result, a recurrence in which every channel's fp32 states decay each at their own pace, a gate behind it
(the equations are with eb_selective_scan in the header).

One product of h gives the convolution's inputs and the gate, one of the convolved row the low-rank part and, in
fp32, B and C.  A sequence's state is the recurrent one and the convolution's last inputs."""
import torch
from torch import nn

from ..decay import selective_scan, selective_step, short_conv, short_conv_step
from ..gemm import project, project_parts
from ..nn import init_weight
from .sequence_state import RecurrentState, RingCache, round_up


class SelectiveScan(nn.Module):
    output_bias = False

    def __init__(self, layer, width, cfg, eps, dtype, device=None):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.layer, self.inner, self.states, self.rank = layer, round_up(cfg.inner, 8), round_up(cfg.state, 4), round_up(cfg.dt_rank, 8)
        self.columns = self.inner                                                          # of the result
        self.in_proj = init_weight(2 * self.inner, width, **kw)                            # x | gate
        self.conv_w = init_weight(cfg.conv, self.inner, std=0.3, **kw)                     # the last row is the current token's
        self.conv_b = init_weight(self.inner, std=0.0, **kw)
        self.x_proj = init_weight(self.rank + 2 * self.states, self.inner, **kw)           # low-rank step || B | C
        self.dt_proj = init_weight(self.inner, self.rank, **kw)
        fp32 = lambda v, *s: nn.Parameter(torch.full(s, v, dtype=torch.float32, device=device), requires_grad=False)
        self.dt_bias, self.a_log, self.skip = fp32(-3.0, self.inner), fp32(0.0, self.inner, self.states), fp32(1.0, self.inner)

    def caches(self):
        return {(self.layer, "conv"): RingCache(self.inner, window=self.conv_w.shape[0]),
                (self.layer, "state"): RecurrentState([(self.inner, self.states)])}

    def forward(self, h, ctx, out):
        """h [rows, width] -> out [rows, columns]; the state goes on."""
        ring, S = ctx.state.caches[self.layer, "conv"].buf, ctx.state.caches[self.layer, "state"].tensors[0]
        x, gate = project(h, self.in_proj).split([self.inner, self.inner], 1)
        if ctx.is_prompt:
            x = short_conv(x, self.conv_w, self.conv_b, ring, ctx.batch, first=ctx.first)
        else:
            x = short_conv_step(x, self.conv_w, self.conv_b, ring, ctx.pos, first=ctx.first)
        low, bc = project_parts(x, self.x_proj, tail_col=self.rank)
        rule = (self.dt_bias, self.a_log, self.skip, S)
        if ctx.is_prompt:
            return selective_scan(x, gate, project(low, self.dt_proj, out_dtype=torch.float32), bc, *rule, first=ctx.first, out=out)
        return selective_step(x, gate, low, self.dt_proj, bc, *rule, out=out)
