"""Replays a trace: given token ids go through a model step by step, the wanted logits are written.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

The model is the one a server would load from DIR (registry.load_model); its prompt pass, its step
function and its caches do the work.  Steps come on standard input, one JSON object a line:

    {"step": 7, "entries": [{"id": "u1", "tokens": [40, 2], "want": [1]}, {"id": "u2", ...}], "end": ["u2"]}

The entries of a step are one batch: all begin (prompts, left-padded to the longest) or all go on by
one token.  Requests named in "end" are finished; their cache memory is given back.  The logits at
the places in "want" go to OUT/<step>.f32 (fp32, [wanted, vocab]); after every step "done <step>" is
printed."""
import argparse
import json
import os
import sys

import torch


class TraceSession:
    """Requests by name on top of a model's prompt() / step() and its SequenceState.  Batches that
    were started separately live side by side, each with a state of its own."""

    def __init__(self, model, device):
        self.model, self.device = model, device
        self.batches = []                      # [names, SequenceState]

    def _check(self, entries):
        names = [e["id"] for e in entries]
        if len(set(names)) != len(names):
            raise ValueError("a request occurs twice in a step")
        for e in entries:
            toks = e["tokens"]
            if not toks or min(toks) < 0 or max(toks) >= self.model.vocab:
                raise ValueError(f"request {e['id']}: a token is outside the vocabulary, or there is none")
            if any(not 0 <= k < len(toks) for k in e.get("want", [])):
                raise ValueError(f"request {e['id']}: a wanted place is outside its tokens")
        return names

    @torch.inference_mode()
    def run(self, entries, end=()):
        """One step; fp32 logits [wanted, vocab] in the order of the entries, or None."""
        out = None
        if entries:
            names = self._check(entries)
            live = [n for b in self.batches for n in b[0]]
            known = [n in live for n in names]
            if not any(known):
                out = self._start(names, entries)
            elif all(known):
                out = self._go_on(names, entries)
            else:
                raise ValueError("a running batch takes no new requests")
        for name in end:
            self._finish(name)
        return out

    def _start(self, names, entries):
        S = max(len(e["tokens"]) for e in entries)
        ids = torch.zeros(len(entries), S, dtype=torch.long)
        mask = torch.zeros(len(entries), S, dtype=torch.long)
        rows = []
        for r, e in enumerate(entries):
            n = len(e["tokens"])
            ids[r, S - n:] = torch.tensor(e["tokens"], dtype=torch.long)
            mask[r, S - n:] = 1
            rows += [r * S + S - n + k for k in e.get("want", [])]
        self.model.state = state = self.model.new_state()
        x = self.model.prompt(ids.to(self.device), mask, reserve=64)
        self.batches.append([list(names), state])
        if not rows:
            return None
        return self.model.logits(x.index_select(0, torch.tensor(rows, device=self.device)))

    def _go_on(self, names, entries):
        if any(len(e["tokens"]) != 1 for e in entries):
            raise ValueError("a running request goes on by one token at a time")
        got = {}
        for batch in list(self.batches):
            here = [n for n in batch[0] if n in names]
            if not here:
                continue
            if len(here) < len(batch[0]):            # the others stay where they are: two batches from now on
                at = [batch[0].index(n) for n in here]
                rest = [i for i in range(len(batch[0])) if i not in at]
                mine = [here, batch[1].fork(at)]
                batch[1].keep(rest)
                batch[0] = [batch[0][i] for i in rest]
                self.batches.append(mine)
                batch = mine
            by = {e["id"]: e["tokens"][0] for e in entries}
            self.model.state = batch[1]
            logits = self.model.step(torch.tensor([by[n] for n in batch[0]], dtype=torch.long, device=self.device))
            got.update({n: logits[i] for i, n in enumerate(batch[0])})
        rows = [got[e["id"]] for e in entries for _ in e.get("want", [])]
        return torch.stack(rows) if rows else None

    def _finish(self, name):
        for batch in self.batches:
            if name in batch[0]:
                keep = [i for i, n in enumerate(batch[0]) if n != name]
                if keep:
                    batch[1].keep(keep)
                    batch[0] = [batch[0][i] for i in keep]
                else:
                    self.batches.remove(batch)
                    if self.model.state is batch[1]:
                        self.model.state = self.model.new_state()
                return
        raise ValueError(f"request {name} is not running")


def main(argv=None):
    ap = argparse.ArgumentParser(description="Feeds given token ids through a model, step by step, and writes logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens live requests hold at any time (the caches grow as needed)")
    args = ap.parse_args(argv)
    from .build import build
    build()                                          # nothing to do when the library is up to date
    from .gemm import device_status
    from .registry import load_model
    device = torch.device("cuda", torch.cuda.current_device())
    model = load_model(args.model, dtype=args.dtype, device=device)
    session = TraceSession(model, device)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = session.run(step.get("entries", []), step.get("end", []))
        if logits is not None:
            data = logits.float().cpu().numpy().astype("<f4").tobytes()
            status = device_status()
            if status[0] != 0:
                raise RuntimeError(f"a bounded device-side wait ran out: {status}")
            path = os.path.join(args.out, f"{step['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(data)
            os.replace(path + ".part", path)
        print(f"done {step['step']}", flush=True)
    return 0
