from .base import (BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, POSITION_ENCODINGS, BuildContext,
                   CacheNeed, FeedForward, Mixer, Norm, ParamSpec, Part, PositionEncoding, Registry, RESIDUAL_GATES, RESIDUAL_SCALES, STREAM_VECTORS, StateNeed,
                   TOKEN_FILTERS, TOKEN_SIDES,                   TokenFilter)
from . import (attention, block, decay_memory, dense_ffn, dyt, embedding, group_rmsnorm, head_memory, latent_attention, layernorm, mlstm, moe, parallel, pool_attention, residual_gate, residual_scale, rmsnorm, rope,  # noqa: F401
               selective_scan, short_conv, sink_attention, stream_vectors, swiglu, token_side)  # noqa: F401  (register the built-in parts)
from .block import Block

__all__ = ["Block", "BLOCKS", "EMBEDDINGS", "FEED_FORWARDS", "HEADS", "MIXERS", "NORMS", "POSITION_ENCODINGS",
           "BuildContext", "CacheNeed", "FeedForward", "Mixer", "Norm", "ParamSpec", "Part", "PositionEncoding",
           "Registry", "RESIDUAL_GATES", "RESIDUAL_SCALES", "STREAM_VECTORS", "StateNeed", "TOKEN_FILTERS", "TOKEN_SIDES", "TokenFilter"]
