"""The decoder of state-space layers and of attention beside gated linear attention: a norm in front of every sublayer,

    x += m * sublayer(norm(x)),

feed-forwards dense or routed, embeddings to which a row per pair of neighbouring tokens is added, the embedding
table as head.  Everything between two sublayers is one launch (stream_add): residual sum, the norm of
the next sublayer and, in generation steps, the router of the mixture behind it."""
import torch
from torch import nn

from ..nn import init_weight
from ..norm import stream_add
from ..step import greedy_step
from .config import DenseConfig, StateSpaceConfig
from .layered_decoder import LayeredDecoder
from .mlp import GEGLUFeedForward
from .moe import RoutedExperts
from .parallel_mixer import ParallelMixer
from .sequence_state import RecurrentState
from .state_space import StateSpace

LAST_TOKEN = "last token"        # what a sequence's next bigram row depends on


class PreNormBlock(nn.Module):
    def __init__(self, mixer, mlp, padded, dtype, device=None):
        super().__init__()
        ones = lambda: nn.Parameter(torch.ones(padded, dtype=dtype, device=device), requires_grad=False)
        self.mixer, self.norm1 = mixer, ones()
        self.mlp, self.norm2 = mlp, ones() if mlp is not None else None


class HybridDecoder(LayeredDecoder):
    tied = True

    def build_layers(self, config, **kw):
        Wp, eps = self.hidden_size, config.eps
        self.bigram = init_weight(config.bigram.buckets + 1, Wp, **kw) if config.bigram else None
        for i, lc in enumerate(config.layers):
            mixer = (StateSpace if isinstance(lc.mixer, StateSpaceConfig) else ParallelMixer)(i, Wp, lc.mixer, eps, **kw)
            mlp = None
            if isinstance(lc.mlp, DenseConfig):
                mlp = GEGLUFeedForward(Wp, lc.mlp.ff, **kw)
            elif lc.mlp is not None:
                mlp = RoutedExperts(Wp, lc.mlp, **kw)
            self.layers.append(PreNormBlock(mixer, mlp, Wp, **kw))

    def caches(self):
        out = {}
        for blk in self.layers:
            out.update(blk.mixer.caches())
        if self.bigram is not None:
            out[LAST_TOKEN] = RecurrentState([()], dtype=torch.int64)
        return out

    # ---- embedding ----
    def _pair_rows(self, prev, tokens):
        b = self.config.bigram
        return (prev * b.mul_prev + tokens * b.mul_cur) % b.buckets

    def _last_token(self):
        return self.state.caches[LAST_TOKEN].tensors[0]

    def embed_prompt(self, input_ids):
        rows = super().embed_prompt(input_ids)
        if self.bigram is None:
            return rows, None
        prev = torch.nn.functional.pad(input_ids[:, :-1], (1, 0))
        start = torch.arange(input_ids.shape[1], device=input_ids.device)[None, :] <= self.state.first[:, None]
        pair = self._pair_rows(prev, input_ids).masked_fill(start, self.config.bigram.buckets)
        self._last_token().copy_(input_ids[:, -1])
        return rows, nn.functional.embedding(pair.reshape(-1), self.bigram)

    def embed_step(self, tokens):
        rows = super().embed_step(tokens)
        if self.bigram is None:
            return rows, None
        last = self._last_token()
        pair = nn.functional.embedding(self._pair_rows(last, tokens.reshape(-1)), self.bigram)
        last.copy_(tokens.reshape(-1))
        return rows, pair

    # ---- layers ----
    def run(self, rows, ctx, on_layer=None):
        eps, count, m = self.config.eps, self.width, self.config.residual_mult
        x = torch.empty(rows[0].shape, dtype=torch.float32, device=rows[0].device)
        # behind the last layer: the final norm of a step (of a prompt only some rows go on to the head)
        into = [dict(w_next=blk.norm1) for blk in self.layers]
        into.append({} if ctx.is_prompt else dict(w_next=self.norm.weight, next_scale=self.config.logit_scale))
        h = stream_add(x, eps, count, src=rows[0], src2=rows[1], **into[0])
        for i, blk in enumerate(self.layers):
            y = blk.mixer(h, ctx)
            y = y if isinstance(y, dict) else dict(y=y)
            if blk.mlp is not None:
                router = blk.mlp.router_for_step(ctx.batch) if not ctx.is_prompt else None
                h = stream_add(x, eps, count, **y, scale=m, w_next=blk.norm2, router=router)
                h, routed = h if router is not None else (h, None)
                y = blk.mlp(h, first=ctx.first if ctx.is_prompt else None, rows_per_batch=ctx.seq, routed=routed)
            h = stream_add(x, eps, count, **y, scale=m, **into[i + 1])
            if on_layer is not None:
                on_layer(i, x)
        return x, h

    def logits(self, x):
        return self.head_logits(stream_add(x, self.config.eps, self.width, w_next=self.norm.weight, next_scale=self.config.logit_scale))

    # ---- what the generation loop asks for ----
    def _new_step_state(self, batch_size, tgt_len, model_dtype, dev, ids_dtype):
        st = super()._new_step_state(batch_size, tgt_len, model_dtype, dev, ids_dtype)
        st["pair"] = torch.empty_like(st["hidden"]) if self.bigram is not None else None
        return st

    def _seed_steps(self, st, tok, cur_len):
        super()._seed_steps(st, tok, cur_len)
        if self.bigram is not None:
            st["pair"].copy_(nn.functional.embedding(self._pair_rows(self._last_token(), tok), self.bigram))

    def _static_step(self, st):
        logits = self._step((st["hidden"], st["pair"]))
        b = self.config.bigram
        greedy_step(logits, st["out_ids"], st["tok"], st["kv_state"], st["step_counter"], word_emb=self.embed, hidden_out=st["hidden"], add_pos=False,
                    bigram=(self.bigram, b.mul_prev, b.mul_cur, b.buckets, st["pair"]) if b else None)

    def _end_generation(self, produced):
        super()._end_generation(produced)
        if self.bigram is not None:
            self._last_token().copy_(self._decode_state["out_ids"][:, produced - 2])
