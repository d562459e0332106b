"""Decoder-only models put together from a configuration that lists their layers: a token embedding
without positions, layers whose sublayers read the residual stream itself and whose OUTPUT is
normalised before it is added (x += norm(sublayer(x))), a final norm and a head.

The residual stream is fp32 throughout; beside it travels its rounding to the operand dtype, which
is what the products read.  Served by the generation loop of every other model (GenerationModel)."""
import os

import torch
from torch import nn

from ..gemm import project
from ..nn import RMSNorm1D, init_weight
from ..norm import rms_norm, rms_residual
from ..step import greedy_step
from .generation import GenerationModel
from .latent_attention import LatentAttention, LatentCache, PromptContext, SequenceState, StepContext, round_up
from .moe import MixtureOfExperts


class OutputNormBlock(nn.Module):
    """x += norm1(mixer(x)); x += norm2(mlp(x)) (mlp may be None)."""

    def __init__(self, mixer, mlp, width, padded, eps, dtype, device=None):
        super().__init__()
        norm = lambda: RMSNorm1D(padded, eps=eps, count=width, offset=1.0, dtype=dtype, device=device)
        self.mixer, self.norm1 = mixer, norm()
        self.mlp, self.norm2 = mlp, norm() if mlp is not None else None

    @staticmethod
    def _add(y, norm, x, xt, **kw):
        # in fp32 the stream is its own operand copy
        return rms_residual(y, norm.weight, norm.eps, x, xt=None if xt is x else xt, offset=norm.offset, count=norm.count, **kw)

    def _mlp(self, x, xt, first, rows_per_batch, routed):
        y, mix = self.mlp(xt, first=first, rows_per_batch=rows_per_batch, routed=routed)
        self._add(y, self.norm2, x, xt, mix=mix)

    def prompt(self, x, xt, ctx):
        self._add(self.mixer.prompt(xt, ctx), self.norm1, x, xt)
        if self.mlp is not None:
            self._mlp(x, xt, ctx.first, ctx.seq, None)

    def step(self, x, xt, ctx):
        router = self.mlp.router_for_step(ctx.batch) if self.mlp is not None else None
        routed = self._add(self.mixer.step(xt, ctx), self.norm1, x, xt, router=router)
        if self.mlp is not None:
            self._mlp(x, xt, None, 1, routed)


class LatentDecoder(GenerationModel):
    eos_token_id = -1            # the configuration names no stop token

    def __init__(self, config, dtype=torch.bfloat16, device=None):
        super().__init__()
        from ..tp import get_tp
        if get_tp().world_size != 1:
            raise RuntimeError("LatentDecoder: one GPU per model (tensor-parallel shards of it are not implemented)")
        self.config, self.dtype = config, dtype
        W, self.vocab = config.width, config.vocab
        self.width, self.hidden_size = W, round_up(W, 8)
        Wp = self.hidden_size
        kw = dict(dtype=dtype, device=device)
        self.embed = init_weight(self.vocab, Wp, **kw)
        self.layers = nn.ModuleList()
        for i, lc in enumerate(config.layers):
            m = lc.mixer
            mixer = LatentAttention(i, Wp, m.heads, m.dim, m.vdim, m.kv_rank, m.window, m.scale, config.eps, kv_from=m.kv_from, **kw)
            mlp = None
            if lc.mlp is not None:
                mlp = MixtureOfExperts(Wp, lc.mlp.experts, lc.mlp.top, lc.mlp.ff, lc.mlp.limit, lc.mlp.alpha, **kw)
            self.layers.append(OutputNormBlock(mixer, mlp, W, Wp, config.eps, **kw))
        for blk in self.layers:
            src = blk.mixer.kv_from
            if src is not None and self.layers[src].mixer.rank != blk.mixer.rank:
                raise ValueError(f"layer {blk.mixer.layer} reads the latents of layer {src}, which have another width")
        self.norm = RMSNorm1D(Wp, eps=config.eps, count=W, offset=1.0, **kw)
        self.head = init_weight(round_up(self.vocab, 8), Wp, **kw)
        self.state = self.new_state()
        self._reserve = 0

    # ---- state ----
    def new_state(self):
        """An empty SequenceState: one ring per layer that has latents of its own, as long as the
        longest window among its readers."""
        windows = {}
        for blk in self.layers:
            windows.setdefault(blk.mixer.source, []).append(blk.mixer.window)
        return SequenceState({i: LatentCache(self.layers[i].mixer.rank, 0 if min(w) <= 0 else max(w)) for i, w in windows.items()})

    @staticmethod
    def left_padding(attention_mask):
        """Number of padding positions in front of each row of a 0/1 mask (one read of the device)."""
        m = (attention_mask != 0).to("cpu", torch.int64)
        first = m.shape[1] - m.sum(1)
        expect = (torch.arange(m.shape[1])[None, :] >= first[:, None]).to(torch.int64)
        if not torch.equal(m, expect) or int(first.max()) >= m.shape[1]:
            raise ValueError("attention_mask: left-padded prompts of at least one token are expected")
        return first.tolist()

    # ---- the two passes ----
    def _streams(self, rows):
        """Embedding rows -> (fp32 residual stream, operand copy)."""
        return (rows.clone(),) * 2 if self.dtype == torch.float32 else (rows.float(), rows)

    @torch.inference_mode()
    def prompt(self, input_ids, attention_mask=None, reserve=0, on_layer=None):
        """The prompt pass of a new batch: fills self.state and returns the final residual stream
        [batch * seq, hidden_size] fp32.  on_layer(i, x) sees the stream behind every layer."""
        B, S = input_ids.shape
        first = self.left_padding(attention_mask) if attention_mask is not None else [0] * B
        dev = input_ids.device
        self.state.begin(first, S, reserve, self.dtype, dev)
        mask = None
        if self.state.padded and self.dtype != torch.float32:
            mask = (torch.arange(S, device=dev)[None, :] < self.state.first[:, None]).to(self.dtype) * -10000.0
        ctx = PromptContext(self.state, B, S, mask)
        x, xt = self._streams(nn.functional.embedding(input_ids.reshape(-1), self.embed))
        for i, blk in enumerate(self.layers):
            blk.prompt(x, xt, ctx)
            if on_layer is not None:
                on_layer(i, x)
        return x

    def _step(self, x, xt):
        ctx = StepContext(self.state)
        for blk in self.layers:
            blk.step(x, xt, ctx)
        return self.logits(x)

    @torch.inference_mode()
    def step(self, tokens):
        """Every sequence of self.state goes on by one token; tokens [batch] -> logits [batch, vocab]."""
        if tokens.numel() != self.state.batch:
            raise ValueError(f"step: {tokens.numel()} tokens for {self.state.batch} sequences")
        self.state.ensure(self.state.length + 1)
        logits = self._step(*self._streams(nn.functional.embedding(tokens.reshape(-1), self.embed)))
        self.state.advance()
        return logits

    def logits(self, x):
        """Final norm and head of rows of the residual stream -> fp32 [rows, vocab]."""
        n = self.norm
        h = rms_norm(x, n.weight, n.eps, offset=n.offset, count=n.count)
        return project(h, self.head, out_dtype=torch.float32)[:, :self.vocab]

    # ---- what the generation loop asks for ----
    @property
    def model_dtype(self):
        return self.dtype

    def reserve_cache(self, new_tokens):
        self._reserve = max(1, int(new_tokens))

    def _cache_key(self):
        s = self.state
        return (s.padded, s.first.data_ptr(), s.kv_state.data_ptr()) + tuple(c.buf.data_ptr() for c in s.caches.values())

    def _prompt_logits(self, input_ids, attention_mask, record=None):
        x = self.prompt(input_ids, attention_mask, reserve=self._reserve)
        return self.logits(x.view(*input_ids.shape, -1)[:, -1].contiguous())

    def _check_capacity(self, tgt_len):
        cap = self.state.capacity()
        if cap is not None and cap < tgt_len:
            raise RuntimeError(f"latent cache holds {cap} positions, {tgt_len} needed")

    def _new_step_state(self, batch_size, tgt_len, model_dtype, dev, ids_dtype):
        if ids_dtype != torch.int64:
            raise RuntimeError("token ids must be int64")
        return {"kv_state": self.state.kv_state, "hidden": torch.empty((batch_size, self.hidden_size), dtype=model_dtype, device=dev),
                "step_counter": torch.zeros(1, dtype=torch.int32, device=dev)}

    def _seed_steps(self, st, tok, cur_len):
        st["hidden"].copy_(nn.functional.embedding(tok, self.embed))

    def _static_step(self, st):
        logits = self._step(*self._streams(st["hidden"]))
        greedy_step(logits, st["out_ids"], st["tok"], st["kv_state"], st["step_counter"], word_emb=self.embed,
                    hidden_out=st["hidden"], add_pos=False)

    def _eager_step(self, st, tok, pos, record=None):
        return self.step(tok)

    def _end_generation(self, produced):
        self.state.set_length(produced - 1)
