"""Two mixers side by side that read the same row: attention over chunks of the sequence, and gated linear attention
with a decaying fp32 state.  Their projections are one product; their outputs are normalised each by
itself and added in the residual step (stream_add)."""
import torch
from torch import nn

from ..attention import attention_group_decode_chunk, attention_plain, attention_prefill_chunk, attention_rotary
from ..decay import chunk_heads, gla_prompt, gla_step
from ..gemm import project
from ..memory import head_norm_gate
from ..nn import init_weight
from .grouped_attention import padded_head
from .sequence_state import RecurrentState, RingCache, round_up


class ChunkAttention(nn.Module):
    """Query heads in groups that share a key head; the values are the keys as projected.  Query and key are
    normalised head by head and rotated; a position sees its own chunk of the sequence; a number per
    head joins the softmax as a score without a value.  Reads the columns [q | k] of a projection."""

    def __init__(self, layer, cfg, eps, dtype, device=None):
        super().__init__()
        self.layer, self.eps = layer, eps
        self.heads, self.kv_heads, self.dim, self.scale, self.chunk = cfg.heads, cfg.kv_heads, cfg.dim, cfg.scale, cfg.chunk
        head = padded_head([cfg.dim], dtype)
        self.tensor_core = head is not None and cfg.scale > 0
        self.dk = head if head is not None else round_up(cfg.dim, 8)
        self.columns = (self.heads + self.kv_heads) * self.dk
        ones = lambda: nn.Parameter(torch.ones(self.dk, dtype=dtype, device=device), requires_grad=False)
        self.q_norm, self.k_norm = ones(), ones()
        self.sinks = nn.Parameter(torch.zeros(self.heads, dtype=torch.float32, device=device), requires_grad=False)
        i = torch.arange(cfg.rot_dims // 2, dtype=torch.float64)
        freq = cfg.rot_base ** (-2 * i / max(1, cfg.rot_dims)) / cfg.rot_factor
        self.register_buffer("freq", freq.to(dtype=torch.float32, device=device), persistent=False)

    def caches(self):
        return {(self.layer, "keys"): RingCache(2 * self.kv_heads * self.dk, window=self.chunk)}

    def forward(self, proj, ctx):
        """-> [rows, heads*dk]; keys and values are cached."""
        B, S, H, G, dk = ctx.batch, ctx.seq, self.heads, self.kv_heads, self.dk
        buf = ctx.state.caches[self.layer, "keys"].buf
        k, v = buf[:, :, :G * dk], buf[:, :, G * dk:]
        q, keys = attention_rotary(proj, H, G, dk, self.dim, self.q_norm, self.k_norm, self.eps, self.freq, k, v, S, pos_device=ctx.pos,
                                   first=ctx.first, keys=ctx.is_prompt)
        if ctx.is_prompt:                # (the ring has only the last positions of a prompt)
            k, v = keys.view(B, S, -1), proj[:, H * dk:self.columns].view(B, S, -1)
        if not self.tensor_core:
            return attention_plain(q.view(B, S, -1), k, v, H, dk, dk, scale=self.scale, first=ctx.first, pos_device=ctx.pos, kv_heads=G,
                                   chunk=self.chunk, sinks=self.sinks).view(B * S, -1)
        if ctx.is_prompt:
            return attention_prefill_chunk(q.view(B, S, -1), k, v, dk, self.chunk, sinks=self.sinks, first=ctx.first, scale=self.scale).view(B * S, -1)
        return attention_group_decode_chunk(q, k, v, dk, ctx.pos, self.scale, self.chunk, sinks=self.sinks, first=ctx.first)


class GatedLinearAttention(nn.Module):
    """Linear attention with a decay per key channel, sigmoid(z)^(1/tau), z a low-rank projection; the output is
    normalised head by head and gated.  Reads the columns [q | k | v | gate | low-rank part] of a projection."""

    def __init__(self, layer, cfg, eps, dtype, device=None):
        super().__init__()
        if not cfg.rank:
            raise ValueError(f"layer {layer}: the rank of the decay's projection is not known (a checkpoint's shapes or the configuration give it)")
        kw = dict(dtype=dtype, device=device)
        self.layer, self.eps, self.heads, self.dim, self.vdim, self.tau, self.rank = layer, eps, cfg.heads, cfg.dim, cfg.vdim, cfg.tau, cfg.rank
        self.scale = cfg.dim ** -0.5
        padded = chunk_heads(cfg.dim, cfg.vdim, dtype)                                     # prompts on the tensor cores
        self.chunked = padded is not None
        self.dk, self.dv = padded if self.chunked else (round_up(cfg.dim, 8), round_up(cfg.vdim, 8))
        self.low = round_up(cfg.rank, 8)
        qk, vg = self.heads * self.dk, self.heads * self.dv
        self.splits = [qk, qk, vg, vg, self.low]
        self.columns = sum(self.splits)
        self.a2 = init_weight(qk, self.low, **kw)
        self.a2_bias = init_weight(qk, std=0.0, **kw)
        self.norm = nn.Parameter(torch.ones(vg, **kw), requires_grad=False)                # (one weight per column: the heads' common one, repeated)

    def caches(self):
        return {(self.layer, "state"): RecurrentState([(self.heads, self.dk, self.dv)])}

    def forward(self, proj, ctx):
        """-> [rows, heads*dv]; the state goes on."""
        S = ctx.state.caches[self.layer, "state"].tensors[0]
        q, k, v, g, low = proj.split(self.splits, 1)
        if not ctx.is_prompt:
            return gla_step(q, k, v, g, low, self.a2, self.a2_bias, self.tau, self.scale, self.norm, self.vdim, self.eps, S, self.heads)
        z = project(low, self.a2, bias=self.a2_bias, out_dtype=torch.float32)
        o = gla_prompt(q, k, v, z, self.tau, self.scale, S, self.heads, first=ctx.first, chunked=self.chunked)
        return head_norm_gate(o, g, self.norm, self.heads, self.vdim, self.eps, silu=True)


class ParallelMixer(nn.Module):
    def __init__(self, layer, width, cfg, eps, dtype, device=None):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.left, self.right = ChunkAttention(layer, cfg.left, eps, **kw), GatedLinearAttention(layer, cfg.right, eps, **kw)
        self.in_proj = init_weight(self.left.columns + self.right.columns, width, **kw)
        self.bias = init_weight(self.in_proj.shape[0], std=0.0, **kw)
        self.left_proj = init_weight(width, self.left.heads * self.left.dk, **kw)
        self.right_proj = init_weight(width, self.right.heads * self.right.dv, **kw)
        half = lambda: nn.Parameter(torch.full((width,), 0.5, dtype=torch.float32, device=device), requires_grad=False)
        self.left_out, self.right_out = half(), half()                                     # output norms' weights, times one half

    def caches(self):
        return {**self.left.caches(), **self.right.caches()}

    def forward(self, h, ctx):
        """h [rows, width] -> what stream_add adds."""
        proj = project(h, self.in_proj, bias=self.bias)
        a = self.left(proj, ctx)
        b = self.right(proj[:, self.left.columns:], ctx)
        return dict(y=project(a, self.left_proj), w=self.left_out, y2=project(b, self.right_proj), w2=self.right_out)
