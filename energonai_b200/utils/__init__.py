"""Checkpoint loading into tensor-parallel shards (energonai/utils/checkpointing*.py)."""
from .checkpointing import load_checkpoint, load_state_dict, remove_prefix  # noqa: F401
from .checkpointing_hf_gpt2 import processing_HF_GPT  # noqa: F401
from .checkpointing_moponex import processing_Moponex  # noqa: F401
from .checkpointing_mutolix import processing_Mutolix  # noqa: F401
from .checkpointing_opt import load_175b, preprocess_175b, processing_OPT  # noqa: F401
from .checkpointing_tulezen import processing_Tulezen  # noqa: F401
from .checkpointing_tupidra import processing_Tupidra  # noqa: F401
from .safetensors_io import load_safetensors  # noqa: F401
