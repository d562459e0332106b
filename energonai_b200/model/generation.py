"""The generation loop every decoder of this package is served with.

It keeps the reference's interface (input_ids / attention_mask in, token ids extended to max_tokens
out; sampling through the same logits warpers; greedy = top_k 1; energonai/model/model_factory.py:
103-159) but does the work once: the prompt is run through the model a single time, every later
step runs only the new token against the caches, and the final norm + LM head see only the last
position (the reference re-embeds the whole sequence and runs the head on every position each step,
model_factory.py:112-131, with the same result for the sampled token).  Greedy steps are captured
in a CUDA graph once and replayed.

A model supplies:
  model_dtype                      the operand dtype
  reserve_cache(new_tokens)        announces how many steps will follow the prompt
  _prompt_logits(ids, mask, record)  the prompt pass; logits of the last position [batch, vocab]
  _check_capacity(tgt_len)         raises unless the caches hold the whole call
  _cache_key()                     identity of the cache memory (a captured step is tied to it)
  _new_step_state(...)             the fixed buffers of a generation step, among them "kv_state", a
                                   device int32 pair (position of the token to process, its successor)
  _seed_steps(st, tok, cur_len)    fills them for a new call
  _static_step(st)                 one greedy step driven by device-side positions (captured)
  _eager_step(st, tok, pos, record)  one step; logits [batch, vocab]
  _end_generation(produced)        host bookkeeping
"""
from typing import Optional

import torch
from torch import nn


class GenerationModel(nn.Module):
    eos_token_id = 50256          # the reference hard-codes this stop id (model_factory.py:133)
    use_cuda_graph = True         # greedy generation steps are captured once and replayed
    stop_check_every = 16         # replayed steps between two host reads of the stop condition

    def _graph_state(self, batch_size, tgt_len, model_dtype, dev, ids_dtype):
        key = (batch_size, tgt_len, model_dtype, ids_dtype, self._cache_key())
        st = getattr(self, "_decode_state", None)
        if st is None or st["key"] != key:
            st = {"key": key, "graph": None, "out_ids": torch.empty((batch_size, tgt_len), dtype=ids_dtype, device=dev),
                  "tok": torch.empty((batch_size,), dtype=ids_dtype, device=dev)}
            st.update(self._new_step_state(batch_size, tgt_len, model_dtype, dev, ids_dtype))
            self._decode_state = st
        return st

    @torch.inference_mode()
    def forward(self, hidden_states=None, input_ids=None, attention_mask=None, seq_lens=None,
                max_tokens: Optional[int] = None, top_k: Optional[int] = None, top_p: Optional[float] = None,
                temperature: Optional[float] = None, record=None):
        batch_size, cur_len = input_ids.shape
        tgt_len = cur_len + 1 if not max_tokens else max_tokens
        if cur_len >= tgt_len:
            return input_ids
        if attention_mask is None:
            attention_mask = torch.ones_like(input_ids)
        dev = input_ids.device
        model_dtype = self.model_dtype
        self.reserve_cache(tgt_len - cur_len)
        greedy = top_k == 1 and (temperature is None or temperature > 0)
        step_times = record.setdefault("step_events", []) if record is not None else None
        from .. import _lib
        launches0, replayed = _lib.launch_count, 0

        def mark():
            if step_times is not None:
                ev = torch.cuda.Event(enable_timing=True)
                ev.record()
                step_times.append(ev)

        # ---- prompt pass ----
        mark()
        logits = self._prompt_logits(input_ids, attention_mask, record)
        if record is not None:
            record.setdefault("logits", []).append(logits.clone())
        tok = logits.argmax(-1) if greedy else self.generate(input_ids, logits, top_k=top_k, top_p=top_p,
                                                             temperature=temperature)
        mark()
        if not max_tokens:
            return tok
        if torch.all(tok == self.eos_token_id):
            return input_ids

        # ---- generation steps ----
        self._check_capacity(tgt_len)
        st = self._graph_state(batch_size, tgt_len, model_dtype, dev, input_ids.dtype)
        out_ids = st["out_ids"]
        out_ids[:, :cur_len] = input_ids
        out_ids[:, cur_len] = tok
        st["tok"].copy_(tok)
        st["kv_state"].copy_(torch.tensor([cur_len, cur_len + 1], dtype=torch.int32), non_blocking=False)
        self._seed_steps(st, tok, cur_len)
        use_graph = greedy and self.use_cuda_graph and (record is None or record.get("allow_graph", False))
        produced = cur_len + 1
        checked = cur_len + 1                                  # columns of out_ids already tested for the stop condition
        for pos in range(cur_len + 1, tgt_len):
            if use_graph:
                if st["graph"] is None and pos == cur_len + 1:
                    before = _lib.launch_count
                    self._static_step(st)                      # eager once: also warms every kernel up
                    st["launches"] = _lib.launch_count - before
                elif st["graph"] is None:
                    g = torch.cuda.CUDAGraph()
                    before = _lib.launch_count
                    with torch.cuda.graph(g):
                        self._static_step(st)
                    launches0 += _lib.launch_count - before    # captured, not executed
                    st["graph"] = g
                    g.replay()
                    replayed += st["launches"]
                else:
                    st["graph"].replay()
                    replayed += st["launches"]
                mark()
                # The reference stops when every sequence has just produced the stop token
                # (model_factory.py:133-134).  Asking after every step would make the host wait for
                # the device once per token; replays are queued ahead instead and the question is
                # asked for a window of steps at a time.  Steps queued beyond the stopping point
                # only wrote cache rows and columns that are cut off below.
                if (pos - cur_len) % self.stop_check_every == 0 or pos == tgt_len - 1:
                    hit = (out_ids[:, checked:pos + 1] == self.eos_token_id).all(0).nonzero()
                    if hit.numel():
                        produced = checked + int(hit[0])
                        break
                    checked = pos + 1
                produced = pos + 1
                continue
            logits = self._eager_step(st, tok, pos, record)
            if record is not None:
                record.setdefault("logits", []).append(logits.clone())
            tok = logits.argmax(-1) if greedy else self.generate(out_ids[:, :pos], logits, top_k=top_k, top_p=top_p,
                                                                 temperature=temperature)
            out_ids[:, pos] = tok
            mark()
            if torch.all(tok == self.eos_token_id):
                break
            produced = pos + 1
        self._end_generation(produced)
        self.launches_last_call = _lib.launch_count - launches0 + replayed   # kernels of this library executed
        return out_ids[:, :produced].clone()

    def get_logits_processor(self, top_k=None, top_p=None, temperature=None):
        from transformers.generation import (LogitsProcessorList, TemperatureLogitsWarper, TopKLogitsWarper,
                                             TopPLogitsWarper)
        processor_list = LogitsProcessorList()
        if temperature is not None and temperature != 1.0:
            processor_list.append(TemperatureLogitsWarper(temperature))
        if top_k is not None and top_k != 0:
            processor_list.append(TopKLogitsWarper(top_k))
        if top_p is not None and top_p < 1.0:
            processor_list.append(TopPLogitsWarper(top_p))
        return processor_list

    def generate(self, input_ids, logits, top_k=None, top_p=None, temperature=None):
        """model_factory.py:153-159 on last-position logits [batch, vocab]."""
        logits = self.get_logits_processor(top_k, top_p, temperature)(input_ids, logits)
        probs = torch.softmax(logits, -1, dtype=torch.float)
        return torch.multinomial(probs, num_samples=1).squeeze(1)
