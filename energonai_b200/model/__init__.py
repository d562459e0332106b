"""Layer modules and model factories with the interfaces of the reference's `energonai.model`."""
from .attention import MultiHeadAttention1D
from .mlp import GEGLUFeedForward, MLP1D, XIELUFeedForward, gelu_impl
from .endecoder import Block1D
from .embedding import Embedding1D
from .downstream import LMHead1D
from .generation import GenerationModel
from .config import HybridDecoderConfig, LatentDecoderConfig, ParallelDecoderConfig, SandwichDecoderConfig
from .sequence_state import RecurrentState, RingCache, SequenceState
from .latent_attention import LatentAttention, RotaryLatentAttention
from .moe import MixtureOfExperts, RoutedExperts
from .layered_decoder import LayeredDecoder
from .latent_decoder import LatentDecoder, OutputNormBlock
from .grouped_attention import GroupedAttention
from .matrix_memory import MatrixMemory
from .sandwich_decoder import SandwichBlock, SandwichDecoder
from .state_space import StateSpace
from .parallel_mixer import ChunkAttention, GatedLinearAttention, ParallelMixer
from .hybrid_decoder import HybridDecoder, PreNormBlock
from .capped_attention import CappedAttention
from .selective_scan import SelectiveScan
from .parallel_decoder import ParallelBlock, ParallelDecoder
from .model_factory import (PipelineModel, create_pipeline_model, gpt2_small, gpt2_large, gpt2_8B, gpt3, hf_gpt2,
                            bert_small, bert_large, bert_8B, bert_175B, opt_125M, opt_6B, opt_13B, opt_30B, opt_66B,
                            opt_175B)

__all__ = ["MultiHeadAttention1D", "MLP1D", "Block1D", "Embedding1D", "LMHead1D", "PipelineModel", "gelu_impl",
           "create_pipeline_model", "gpt2_small", "gpt2_large", "gpt2_8B", "gpt3", "hf_gpt2", "bert_small",
           "bert_large", "bert_8B", "bert_175B", "opt_125M", "opt_6B", "opt_13B", "opt_30B", "opt_66B", "opt_175B",
           "GenerationModel", "LatentDecoderConfig", "LatentDecoder", "LatentAttention", "RingCache", "RecurrentState",
           "SequenceState", "MixtureOfExperts", "OutputNormBlock", "LayeredDecoder", "GroupedAttention", "MatrixMemory", "SandwichBlock",
           "SandwichDecoder", "SandwichDecoderConfig", "XIELUFeedForward", "HybridDecoder", "HybridDecoderConfig", "PreNormBlock", "StateSpace",
           "ChunkAttention", "GatedLinearAttention", "ParallelMixer", "RoutedExperts", "GEGLUFeedForward", "ParallelDecoder",
           "ParallelDecoderConfig", "ParallelBlock", "RotaryLatentAttention", "CappedAttention", "SelectiveScan"]
