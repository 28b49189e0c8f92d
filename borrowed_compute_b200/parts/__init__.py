from . import (attention, attention_kv, block, channel_delta, delta_rule, diff_attention, distance_bias, embedding, latent_attention, linear_recurrence, mlp, moe, norm, polynorm, reentry, rope,  # noqa: F401
               short_conv, side_by_side, sinusoidal, streams, talking_attention)      # (importing registers the built-in parts)
from .base import (BLOCKS, CONNECTIONS, CONVOLUTIONS, EMBEDDINGS, FEED_FORWARDS, HEADS, JUNCTIONS, MIXERS, NORMS, POSITION_ENCODINGS, SCALES, Block, CacheNeed, Embedding,
                   FeedForward, Head, Junction, LayerSpec, Mixer, ModelSpec, Norm, Part, PartSpec, PositionEncoding, Registry, RotaryTable,
                   RunMemory, RunSpec, Runtime, ShortConvolution, StateNeed, StepContext, TensorSpec)

__all__ = [
    "BLOCKS", "CONNECTIONS", "CONVOLUTIONS", "EMBEDDINGS", "FEED_FORWARDS", "HEADS", "JUNCTIONS", "MIXERS", "NORMS", "POSITION_ENCODINGS", "SCALES", "Block", "CacheNeed", "Embedding",
    "FeedForward", "Head", "Junction", "LayerSpec", "Mixer", "ModelSpec", "Norm", "Part", "PartSpec", "PositionEncoding", "Registry",
    "RotaryTable", "RunMemory", "RunSpec", "Runtime", "ShortConvolution", "StateNeed", "StepContext", "TensorSpec",
]
