"""Which model a name or a model folder stands for.

`build_model(name, **kwargs)` runs a registered factory (the opt_*, gpt2_*, bert_* factories of
energonai/model/model_factory.py:228-354 under their names, and the architectures below).
`load_model(folder)` reads folder/config.json, picks the architecture by its "architecture" key,
builds it and loads folder/model.safetensors (or every *.safetensors file of the folder)."""
import json
import os

import torch

_ARCHITECTURES, _FACTORIES = {}, {}

DTYPES = {"float32": torch.float32, "float16": torch.float16, "bfloat16": torch.bfloat16}


class Architecture:
    """config: class with from_dict() and, where only a checkpoint's shapes give some size, with_shapes();
    model: class taking (config, dtype, device); convert(state, model): checkpoint tensors -> the model's
    parameters."""

    def __init__(self, name, config, model, convert):
        self.name, self.config, self.model, self.convert = name, config, model, convert


def register_architecture(name, config, model, convert):
    _ARCHITECTURES[name] = Architecture(name, config, model, convert)
    _FACTORIES[name] = lambda config_dict=None, dtype=torch.bfloat16, device=None, **kw: model(
        config.from_dict(config_dict if config_dict is not None else kw), dtype=dtype, device=device)


def register_factory(name, fn):
    _FACTORIES[name] = fn


def architectures():
    _populate()
    return sorted(_ARCHITECTURES)


def models():
    _populate()
    return sorted(_FACTORIES)


def build_model(name, **kwargs):
    _populate()
    if name not in _FACTORIES:
        raise KeyError(f"unknown model {name!r}; known: {', '.join(sorted(_FACTORIES))}")
    return _FACTORIES[name](**kwargs)


def read_config(folder):
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def load_model(folder, dtype="bfloat16", device=None):
    """The model of a folder, its weights loaded, on `device` (default: the current GPU)."""
    from .utils import load_checkpoint, load_state_dict
    _populate()
    config = read_config(folder)
    name = config.get("architecture")
    if name not in _ARCHITECTURES:
        raise ValueError(f"{folder}: architecture {name!r} is not registered (known: {', '.join(sorted(_ARCHITECTURES))})")
    arch = _ARCHITECTURES[name]
    dtype = DTYPES[dtype] if isinstance(dtype, str) else dtype
    weights = os.path.join(folder, "model.safetensors")
    weights = weights if os.path.exists(weights) else folder
    sizes = arch.config.from_dict(config)
    if hasattr(sizes, "with_shapes"):
        sizes = sizes.with_shapes({k: tuple(v.shape) for k, v in load_state_dict(weights).items()})
    model = arch.model(sizes, dtype=dtype)
    load_checkpoint(weights, model, preprocess_fn=lambda state: arch.convert(state, model))
    return model.to(device if device is not None else torch.device("cuda", torch.cuda.current_device())).eval()


_done = False


def _populate():
    global _done
    if _done:
        return
    _done = True
    from . import model as M
    from .model.config import HybridDecoderConfig, LatentDecoderConfig, ParallelDecoderConfig, SandwichDecoderConfig
    from .model.hybrid_decoder import HybridDecoder
    from .model.latent_decoder import LatentDecoder
    from .model.parallel_decoder import ParallelDecoder
    from .model.sandwich_decoder import SandwichDecoder
    from .utils.checkpointing_moponex import processing_Moponex
    from .utils.checkpointing_mutolix import processing_Mutolix
    from .utils.checkpointing_tulezen import processing_Tulezen
    from .utils.checkpointing_tupidra import processing_Tupidra
    for name in ("opt_125M", "opt_6B", "opt_13B", "opt_30B", "opt_66B", "opt_175B", "gpt2_small", "gpt2_large", "gpt2_8B", "gpt3",
                 "hf_gpt2", "bert_small", "bert_large", "bert_8B", "bert_175B"):
        register_factory(name, getattr(M, name))
    register_architecture("Tulezen", LatentDecoderConfig, LatentDecoder, processing_Tulezen)
    register_architecture("Mutolix", SandwichDecoderConfig, SandwichDecoder, processing_Mutolix)
    register_architecture("Moponex", HybridDecoderConfig, HybridDecoder, processing_Moponex)
    register_architecture("Tupidra", ParallelDecoderConfig, ParallelDecoder, processing_Tupidra)
