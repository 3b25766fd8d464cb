"""The parts a model is put together from, and their registry."""
from . import (attention, block, delta_rule, embedding, feedforward, latent_attention, lightning_attention,
               linear_attention, mapped_attention, matrix_lstm, moe, norm, parallel, position, selective_scan, sink_attention,
               state_space)  # noqa: F401  (they register themselves)
from .base import (Arrangement, CompositeCacheSpec, Embedding, FeedForward, FreeSize, Head, KVCacheSpec, Mixer, Norm, Part,
                   PositionEncoding, RowCacheSpec, StateCacheSpec, TensorSpec, build_part, known_parts, register_part)
from .linear import Linear

__all__ = ["Arrangement", "CompositeCacheSpec", "Embedding", "FeedForward", "FreeSize", "Head", "KVCacheSpec", "Linear", "Mixer", "Norm",
           "Part", "PositionEncoding", "RowCacheSpec", "StateCacheSpec", "TensorSpec", "build_part", "known_parts",
           "register_part"]
