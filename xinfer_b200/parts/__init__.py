"""The parts a decoder block is put together from, and their registries."""
from .base import (CacheTensor, FeedForward, LayerCache, Mixer, Norm, PagedCacheNeed, Part, PositionEncoding,
                   StepContext, Workspace, build_part, part_class, register_feed_forward,
                   register_mixer, register_norm, register_position_encoding, unregister)
from . import (norm, rope, attention, swiglu, talking_attention, min_gru, parallel, polynorm_mlp,  # noqa: F401
               table_experts, latent_attention, selective_state, gated_delta, token_side, routed_experts, gated_linear_attention,
               input_conv, matrix_memory)                                                           # (register the built-in kinds)
from .block import Block

__all__ = [
    "CacheTensor", "FeedForward", "LayerCache", "Mixer", "Norm", "PagedCacheNeed", "Part", "PositionEncoding",
    "StepContext", "Workspace", "build_part", "part_class", "register_feed_forward",
    "register_mixer", "register_norm", "register_position_encoding", "unregister", "Block",
]
