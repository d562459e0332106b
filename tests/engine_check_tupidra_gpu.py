"""One engine life cycle with a latent-attention, selective-scan and capped-attention decoder, in a fresh process:

    python tests/engine_check_tupidra_gpu.py FOLDER

The worker loads the model of FOLDER through the registry; BatchManagerForGeneration merges requests
of unequal lengths into left-padded batches; every answer must be the plain restatement's greedy
continuation of that request alone.  Exit code 0 on success."""
import json
import os
import socket
import sys

import torch

import tupidra_plain as P
from energonai_b200 import BatchManagerForGeneration, launch_engine
from energonai_b200.utils import load_safetensors


def load(folder=None):
    from energonai_b200.registry import load_model
    return load_model(folder, dtype="float32")


def free_port():
    with socket.socket() as s:
        s.bind(("127.0.0.1", 0))
        return s.getsockname()[1]


def main(folder):
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    tensors = load_safetensors(os.path.join(folder, "model.safetensors"))
    g = torch.Generator().manual_seed(3)
    prompts = {uid: torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for uid, n in enumerate((5, 17, 1, 9, 30, 12))}
    new = {uid: 16 - uid for uid in prompts}
    engine = launch_engine(1, 1, "127.0.0.1", free_port(), free_port(), load, batch_manager=BatchManagerForGeneration(max_batch_size=3),
                           folder=folder)
    try:
        for uid, p in prompts.items():
            engine.submit(uid, dict(input_ids=p, attention_mask=[1] * len(p), max_tokens=new[uid], top_k=1, top_p=None, temperature=None))
        got = {uid: engine.get(uid) for uid in prompts}
    finally:
        engine.shutdown()
    for uid, p in prompts.items():
        want, gap = P.greedy(cfg, tensors, p, new[uid])
        assert gap > 1e-5, (uid, gap)
        assert got[uid][-len(want):].tolist() == want, (uid, got[uid], want)
    print("engine tupidra ok", flush=True)


if __name__ == "__main__":
    main(sys.argv[1])
