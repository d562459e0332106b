"""Decoder-only models put together from a configuration that lists their layers: a token embedding
without positions, the layers, a final norm and a head.  The residual stream is fp32 throughout.

LayeredDecoder is what they share: the batch's state, the prompt pass, the step, and what the
generation loop of every other model (GenerationModel) asks for.  A subclass builds its layers and says
how the stream runs through them."""
import torch
from torch import nn

from ..gemm import project
from ..nn import RMSNorm1D, init_weight
from ..norm import rms_norm
from ..step import greedy_step
from .generation import GenerationModel
from .sequence_state import PromptContext, SequenceState, StepContext, round_up


class LayeredDecoder(GenerationModel):
    """A subclass fills self.layers in build_layers() and supplies
      caches()                    {layer: RingCache or RecurrentState} of an empty state
      run(rows, ctx, on_layer)    embedding rows (operand dtype) through all layers -> (x, h): the fp32
                                  stream, and its final norm if it is at hand (else None)
    and, where the rows are more than the tokens' own,
      embed_prompt(input_ids), embed_step(tokens)    what run() takes as rows"""
    eos_token_id = -1            # the configurations name no stop token
    norm_offset = 0.0            # 1.0: norm weights are stored around zero
    tied = False                 # the head is the embedding table

    def __init__(self, config, dtype=torch.bfloat16, device=None):
        super().__init__()
        from ..tp import get_tp
        if get_tp().world_size != 1:
            raise RuntimeError(f"{type(self).__name__}: one GPU per model (tensor-parallel shards of it are not implemented)")
        self.config, self.dtype = config, dtype
        self.vocab, self.width, self.hidden_size = config.vocab, config.width, round_up(config.width, 8)
        kw = dict(dtype=dtype, device=device)
        self.embed = init_weight(round_up(self.vocab, 8) if self.tied else self.vocab, self.hidden_size, **kw)
        self.layers = nn.ModuleList()
        self.build_layers(config, **kw)
        self.norm = RMSNorm1D(self.hidden_size, eps=config.eps, count=self.width, offset=self.norm_offset, **kw)
        self.head = self.embed if self.tied else init_weight(round_up(self.vocab, 8), self.hidden_size, **kw)
        self.state = self.new_state()
        self._reserve = 0

    def new_state(self):
        return SequenceState(self.caches())

    @staticmethod
    def left_padding(attention_mask):
        """Number of padding positions in front of each row of a 0/1 mask (one read of the device)."""
        m = (attention_mask != 0).to("cpu", torch.int64)
        first = m.shape[1] - m.sum(1)
        expect = (torch.arange(m.shape[1])[None, :] >= first[:, None]).to(torch.int64)
        if not torch.equal(m, expect) or int(first.max()) >= m.shape[1]:
            raise ValueError("attention_mask: left-padded prompts of at least one token are expected")
        return first.tolist()

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
        return self.run(self.embed_prompt(input_ids), ctx, on_layer)[0]

    def embed_prompt(self, input_ids):
        return nn.functional.embedding(input_ids.reshape(-1), self.embed)

    def embed_step(self, tokens):
        return nn.functional.embedding(tokens.reshape(-1), self.embed)

    def _step(self, rows):
        x, h = self.run(rows, StepContext(self.state))
        return self.logits(x) if h is None else self.head_logits(h)

    @torch.inference_mode()
    def step(self, tokens):
        """Every sequence of self.state goes on by one token; tokens [batch] -> logits [batch, vocab]."""
        if tokens.numel() != self.state.batch:
            raise ValueError(f"step: {tokens.numel()} tokens for {self.state.batch} sequences")
        self.state.ensure(self.state.length + 1)
        logits = self._step(self.embed_step(tokens))
        self.state.advance()
        return logits

    def logits(self, x):
        """Final norm and head of rows of the residual stream -> fp32 [rows, vocab]."""
        n = self.norm
        return self.head_logits(rms_norm(x, n.weight, n.eps, offset=n.offset, count=n.count))

    def head_logits(self, h):
        return project(h, self.head, out_dtype=torch.float32)[:, :self.vocab]

    # ---- what the generation loop asks for ----
    @property
    def model_dtype(self):
        return self.dtype

    def reserve_cache(self, new_tokens):
        self._reserve = max(1, int(new_tokens))

    def _cache_key(self):
        s = self.state
        return (s.padded, s.first.data_ptr(), s.kv_state.data_ptr()) + tuple(p for c in s.caches.values() for p in c.pointers())

    def _prompt_logits(self, input_ids, attention_mask, record=None):
        x = self.prompt(input_ids, attention_mask, reserve=self._reserve)
        return self.logits(x.view(*input_ids.shape, -1)[:, -1].contiguous())

    def _check_capacity(self, tgt_len):
        cap = self.state.capacity()
        if cap is not None and cap < tgt_len:
            raise RuntimeError(f"the caches hold {cap} positions, {tgt_len} needed")

    def _new_step_state(self, batch_size, tgt_len, model_dtype, dev, ids_dtype):
        if ids_dtype != torch.int64:
            raise RuntimeError("token ids must be int64")
        return {"kv_state": self.state.kv_state, "hidden": torch.empty((batch_size, self.hidden_size), dtype=model_dtype, device=dev),
                "step_counter": torch.zeros(1, dtype=torch.int32, device=dev)}

    def _seed_steps(self, st, tok, cur_len):
        st["hidden"].copy_(nn.functional.embedding(tok, self.embed))

    def _static_step(self, st):
        logits = self._step(st["hidden"])
        greedy_step(logits, st["out_ids"], st["tok"], st["kv_state"], st["step_counter"], word_emb=self.embed,
                    hidden_out=st["hidden"], add_pos=False)

    def _eager_step(self, st, tok, pos, record=None):
        return self.step(tok)

    def _end_generation(self, produced):
        self.state.set_length(produced - 1)
