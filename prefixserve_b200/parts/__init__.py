from . import attention, biased_attention, combined, delta, embedding, ffn, gate, head_norm_attention, latent_attention, linear_attention, matrix_memory, min_gru, moe, norm, normed_attention, position, recurrent, stream  # noqa: F401  (registers the built-in kinds)
from .base import (CacheNeed, CacheView, FeedForward, FixedState, Gate, ItemView, Mixer, Norm, PagedKV, ParamSpec, Part,
                   PositionEncoding, StepContext)
from .block import Block, register_arrangement
from .model import DecoderModel, build_model
from .registry import (kinds, make, register_embedding, register_ffn, register_gate, register_head, register_mixer, register_norm,
                       register_position, register_stream)

__all__ = [
    "Block", "CacheNeed", "CacheView", "DecoderModel", "FeedForward", "FixedState", "Gate", "ItemView", "Mixer", "Norm",
    "PagedKV", "ParamSpec", "Part", "PositionEncoding", "StepContext", "build_model", "kinds", "make",
    "register_arrangement", "register_embedding", "register_ffn", "register_gate", "register_head", "register_mixer", "register_norm", "register_position", "register_stream",
]
