"""MLP1D with the reference's constructor and forward signature (energonai/model/mlp.py:8-51):
column-parallel FC1 with the activation fused into the GEMM epilogue, row-parallel FC2.
Generation steps process and return only the new position (see attention.py)."""
from typing import Callable, Optional

import torch
from torch import dtype, nn

from ..gemm import project, project_parts, project_unit, xielu_params
from ..nn import Linear1D_Col, Linear1D_Row, init_weight
from .sequence_state import round_up


def gelu_impl(x):
    """OpenAI's tanh GELU (energonai/model/model_factory.py:32-35), used as an activation tag."""
    return 0.5 * x * (1.0 + torch.tanh(0.7978845608028654 * x * (1.0 + 0.044715 * x * x)))


def activation_code(fn):
    """Maps the callables the reference passes as `activation` to an epilogue code."""
    name = getattr(fn, "__name__", str(fn))
    if fn is nn.functional.relu or name == "relu":
        return "relu"
    if name in ("gelu_impl", "gelu_tanh", "gelu_new"):
        return "gelu_tanh"
    if fn is nn.functional.gelu or name == "gelu":
        return "gelu"
    raise RuntimeError(f"MLP1D: activation {name!r} has no fused epilogue (relu, gelu, gelu_impl are supported)")


class MLP1D(nn.Module):

    def __init__(self,
                 hidden_size: int,
                 mlp_ratio: float,
                 activation: Callable,
                 dtype: dtype = torch.float16,
                 bias: bool = True,
                 disable_past_cache=False):
        super().__init__()
        self.disable_past_cache = disable_past_cache
        intermediate_dim = int(hidden_size * mlp_ratio)
        self.dense_1 = Linear1D_Col(hidden_size, intermediate_dim, bias=bias, dtype=dtype, gather_output=False)
        self.activation = activation
        self.act_code = activation_code(activation)
        self.dense_2 = Linear1D_Row(intermediate_dim, hidden_size, bias=bias, dtype=dtype, parallel_input=True)

    def forward(self, hidden_states, first_cache: Optional[bool] = True, residual=None, fold_norm=None, transient_ok=False):
        """fold_norm: see Linear1D_Col.forward (hidden_states is then the un-normalised input)."""
        if not (self.disable_past_cache or first_cache):
            hidden_states = hidden_states[:, -1:, :]
            residual = residual[:, -1:, :] if residual is not None else None
        inter = self.dense_1(hidden_states, act=self.act_code, fold_norm=fold_norm)
        return self.dense_2(inter, residual=residual, transient_ok=transient_ok)


class XIELUFeedForward(nn.Module):
    """W_down xIELU(W_up h), with the pre-activation of a residual gate, W_gate h + b, from the same
    product (the activation covers its first columns only)."""

    def __init__(self, width, ff, dtype, device=None):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.ff, self.ff_padded = ff, round_up(ff, 8)
        self.up = init_weight(self.ff_padded + width, width, **kw)              # up | residual gate
        self.bias = init_weight(self.ff_padded + width, std=0.0, **kw)
        self.act = nn.Parameter(xielu_params(0.8, 0.8).to(device), requires_grad=False)
        self.down = init_weight(width, self.ff_padded, **kw)

    def forward(self, h):
        """-> (y, pre-activation of its gate)."""
        u = project_parts(h, self.up, bias=self.bias, xielu=(self.act, self.ff_padded))
        return project(u[:, :self.ff_padded], self.down), u[:, self.ff_padded:]


class GEGLUFeedForward(nn.Module):
    """W_down (gelu_tanh(W_gate h) * (W_up h)); gates and ups interleaved in blocks of 8 rows, the unit in the epilogue
    of their product."""

    def __init__(self, width, ff, dtype, device=None, down=True):
        """down=False: the output product belongs to the block (see inner())."""
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.ff, self.ff_padded = ff, round_up(ff, 8)
        self.gate_up = init_weight(2 * self.ff_padded, width, **kw)
        self.down = init_weight(width, self.ff_padded, **kw) if down else None

    def router_for_step(self, tokens):
        return None

    def inner(self, h, out):
        """The unit's columns alone, into `out` [rows, ff_padded] (blocks that share one output product)."""
        return project_unit(h, self.gate_up, "geglu", out=out)

    def forward(self, h, first=None, rows_per_batch=1, routed=None):
        """-> what stream_add adds."""
        return dict(y=project(project_unit(h, self.gate_up, "geglu"), self.down))
