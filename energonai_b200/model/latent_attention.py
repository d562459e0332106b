"""Latent attention with a sliding window over a ring cache of latent rows.

Per token a layer keeps one latent row c = RMSNorm(W_dkv h); keys and values of every head are
linear maps of it, k = W_uk c, v = W_uv c.  Two evaluation orders give the same result:

  prompt           k and v are expanded with one GEMM and a windowed attention kernel runs on them;
  generation step  W_uk is moved onto the query and W_uv behind the attention, which then reads the
                   cached latent rows themselves, once for all heads (eb_latent_decode).

A layer may take another layer's latents instead of having its own projection (`kv_from`); it still
has its own queries, up-projections, window and scale.

Head sizes and the latent width are padded with zeros to what the tensor-core kernels take; zero
columns change no product.
"""
import torch
from torch import nn

from ..attention import (LATENT_WIDTHS, PROMPT_HEADS, attention_plain, attention_prefill_gated, attention_prefill_window, latent_decode, latent_inputs, rotate_heads,
                         sigmoid_gate, yarn_rotation)
from ..gemm import project
from ..moe import per_head
from ..nn import RMSNorm1D, init_weight
from ..norm import rms_norm
from .sequence_state import RingCache, round_up


class LatentAttention(nn.Module):
    def __init__(self, layer, width, heads, dim, vdim, kv_rank, window, scale, eps, dtype, kv_from=None, device=None):
        super().__init__()
        self.layer, self.width, self.heads, self.dim, self.vdim, self.kv_rank = layer, width, heads, dim, vdim, kv_rank
        self.window, self.scale, self.kv_from = window, scale, kv_from
        wide = max(dim, vdim)
        self.tensor_core_prompt = dtype != torch.float32 and wide <= 128 and scale > 0
        if self.tensor_core_prompt:
            self.dk = self.dv = 64 if wide <= 64 else 128
        else:
            self.dk, self.dv = round_up(dim, 8), round_up(vdim, 8)
        self.tensor_core_step = dtype != torch.float32 and kv_rank <= LATENT_WIDTHS[-1]
        self.rank = min(w for w in LATENT_WIDTHS if w >= kv_rank) if self.tensor_core_step else round_up(kv_rank, 8)
        self.q_rows = heads * self.dk
        own = kv_from is None
        self.in_proj = init_weight(self.q_rows + (self.rank if own else 0), width, dtype=dtype, device=device)   # queries | latent
        self.latent_norm = RMSNorm1D(self.rank, eps=eps, count=kv_rank, offset=0.0, dtype=dtype, device=device) if own else None
        self.kv_up = init_weight(heads * (self.dk + self.dv), self.rank, dtype=dtype, device=device)             # keys | values, head by head
        self.k_absorb = init_weight(heads, self.rank, self.dk, dtype=dtype, device=device)                       # W_uk of a head, transposed
        self.out_proj = init_weight(width, heads * self.dv, dtype=dtype, device=device)

    @property
    def source(self):
        return self.layer if self.kv_from is None else self.kv_from

    def prompt(self, h, ctx):
        """h [batch*seq, width] -> [batch*seq, width]; fills this layer's cache."""
        B, S = ctx.batch, ctx.seq
        q = project(h, self.in_proj)
        if self.kv_from is None:
            n = self.latent_norm
            ctx.latents[self.layer] = rms_norm(q[:, self.q_rows:], n.weight, n.eps, offset=n.offset, count=n.count,
                                               ring=ctx.state.caches[self.layer].buf, rows_per_batch=S)
        c = ctx.latents[self.source]
        kv = project(c, self.kv_up).view(B, S, -1)
        q3 = q.view(B, S, -1)[:, :, :self.q_rows]
        k, v = kv[:, :, :self.q_rows], kv[:, :, self.q_rows:]        # (keys have as many rows as queries)
        if self.tensor_core_prompt:
            o = attention_prefill_window(q3, k, v, self.dk, self.window, mask=ctx.mask, scale=self.scale)
        else:
            o = attention_plain(q3, k, v, self.heads, self.dk, self.dv, window=self.window, scale=self.scale, first=ctx.first)
        return project(o.view(B * S, -1), self.out_proj)

    def step(self, h, ctx):
        """h [batch, width], one new position per sequence -> [batch, width]."""
        B = ctx.batch
        q = project(h, self.in_proj)
        cache = ctx.state.caches[self.source].buf
        if self.kv_from is None:
            n = self.latent_norm
            rms_norm(q[:, self.q_rows:], n.weight, n.eps, offset=n.offset, count=n.count, write_out=False, ring=cache,
                     rows_per_batch=1, pos_device=ctx.pos)
        qa = per_head(q[:, :self.q_rows], self.k_absorb)
        if self.tensor_core_step:
            o = latent_decode(qa, cache, self.rank, self.heads, self.window, ctx.pos, self.scale, first=ctx.first)
        else:
            o = attention_plain(qa.view(B, 1, -1), cache, cache, self.heads, self.rank, self.rank, window=self.window, scale=self.scale,
                                first=ctx.first, pos_device=ctx.pos, shared_kv=True).view(B, -1)
        v = per_head(o, self.kv_up[self.q_rows:].view(self.heads, self.dv, self.rank))
        return project(v, self.out_proj)


class RotaryLatentAttention(nn.Module):
    """Latent attention whose query comes out of a latent of its own and has a rotated part; the key's rotated part is common
    to all heads and cached behind the latent, as one row.  A number per head joins the softmax as a score without
    a value, and the concatenated heads are multiplied by the sigmoid of a gate.

    The key up-projection carries the rotated part through with ones, so that a head's whole key, or the absorbed
    query, is one linear map of the cached row.  One product of h gives query latent, cached row and gate."""
    output_bias = False

    def __init__(self, layer, width, cfg, eps, dtype, device=None):
        super().__init__()
        kw = dict(dtype=dtype, device=device)
        self.layer, self.eps, self.heads, self.scale, self.kv_from = layer, eps, cfg.heads, cfg.scale, cfg.kv_from
        self.dim, self.rot_dim, self.vdim, self.q_rank, self.kv_rank = cfg.dim, cfg.rot_dim, cfg.vdim, cfg.q_rank, cfg.kv_rank
        self.rot_at, self.rot_col = round_up(cfg.dim, 8), round_up(cfg.kv_rank, 8)         # where the rotated part begins in a head, in a row
        key, row = self.rot_at + cfg.rot_dim, self.rot_col + cfg.rot_dim
        fits = [h for h in PROMPT_HEADS if h[0] >= key and h[1] >= cfg.vdim]
        self.tensor_core_prompt = dtype != torch.float32 and bool(fits) and cfg.scale > 0
        self.dk, self.dv = min(fits) if self.tensor_core_prompt else (round_up(key, 8), round_up(cfg.vdim, 8))
        self.tensor_core_step = dtype != torch.float32 and row <= LATENT_WIDTHS[-1]
        self.rank = min(w for w in LATENT_WIDTHS if w >= row) if self.tensor_core_step else round_up(row, 8)
        self.q_cols, self.q_rows, self.columns = round_up(cfg.q_rank, 8), cfg.heads * self.dk, cfg.heads * self.dv
        own = cfg.kv_from is None
        ones = lambda n: nn.Parameter(torch.ones(n, **kw), requires_grad=False)
        self.in_proj = init_weight(self.q_cols + (self.rank if own else 0) + self.columns, width, **kw)      # query latent | row | gate
        self.q_norm, self.latent_norm = ones(self.q_cols), ones(self.rot_col) if own else None
        self.q_up = init_weight(self.q_rows, self.q_cols, **kw)
        self.kv_up = init_weight(self.q_rows + self.columns, self.rank, **kw)              # keys | values, head by head
        self.k_absorb = init_weight(self.heads, self.rank, self.dk, **kw)                  # a head's key map, transposed
        self.sinks = nn.Parameter(torch.zeros(self.heads, dtype=torch.float32, device=device), requires_grad=False)
        freq, self.factor = yarn_rotation(cfg.rot_dim, cfg.rot_base, cfg.rot_scaling)
        self.register_buffer("freq", freq.to(device=device), persistent=False)

    @property
    def source(self):
        return self.layer if self.kv_from is None else self.kv_from

    def caches(self):
        return {self.layer: RingCache(self.rank)} if self.kv_from is None else {}

    def forward(self, h, ctx, out):
        """h [rows, width] -> out [rows, columns]; rows of this layer's own latents are cached."""
        B, S, H = ctx.batch, ctx.seq, self.heads
        cache, where = ctx.state.caches[self.source].buf, dict(rows_per_batch=S, pos_device=ctx.pos, first=ctx.first)
        proj = project(h, self.in_proj)
        gate, row = proj[:, proj.shape[1] - self.columns:], None
        if self.kv_from is None:
            row = dict(cols=self.rank, rot_col=self.rot_col, count=self.kv_rank, norm=self.latent_norm, freq=self.freq, factor=self.factor, ring=cache,
                       keep_rows=ctx.is_prompt)
        q, rows = latent_inputs(proj, self.q_cols, self.q_rank, self.q_norm, self.eps, row=row, **where)
        q = rotate_heads(project(q, self.q_up), H, self.dk, self.rot_at, self.freq, self.factor, **where)
        if ctx.is_prompt:
            if rows is not None:
                ctx.latents[self.layer] = rows
            kv = project(ctx.latents[self.source], self.kv_up).view(B, S, -1)
            q, k, v = q.view(B, S, -1), kv[:, :, :self.q_rows], kv[:, :, self.q_rows:]
            if self.tensor_core_prompt:
                return attention_prefill_gated(q, k, v, self.dk, self.dv, sinks=self.sinks, first=ctx.first, gate=gate.view(B, S, -1), scale=self.scale,
                                               out=out.view(B, S, -1))
            o = attention_plain(q, k, v, H, self.dk, self.dv, scale=self.scale, first=ctx.first, chunk=0, sinks=self.sinks)
            return sigmoid_gate(o.view(B * S, -1), gate, out=out)
        qa = per_head(q, self.k_absorb)
        if self.tensor_core_step:
            o = latent_decode(qa, cache, self.rank, H, 0, ctx.pos, self.scale, first=ctx.first, sinks=self.sinks)
        else:
            o = attention_plain(qa.view(B, 1, -1), cache, cache, H, self.rank, self.rank, scale=self.scale, first=ctx.first, pos_device=ctx.pos,
                                shared_kv=True, chunk=0, sinks=self.sinks).view(B, -1)
        return sigmoid_gate(per_head(o, self.kv_up[self.q_rows:].view(H, self.dv, self.rank)), gate, out=out)
