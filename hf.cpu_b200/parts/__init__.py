from .base import (Block, CacheSpec, FeedForward, Mixer, Norm, Part, PositionEncoding, StateSpec, Transition,
                   make_part, register_part, unregister_part)
from . import attention, block, embedding, ffn, latent_attention, moe, norm, parallel, recurrent, rotary, transition  # noqa: F401  (register the built-in parts)

__all__ = ["Part", "Norm", "PositionEncoding", "Mixer", "FeedForward", "Block", "CacheSpec", "StateSpec", "Transition",
           "make_part", "register_part", "unregister_part"]
