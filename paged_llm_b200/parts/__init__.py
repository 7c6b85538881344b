"""Parts a model is assembled from.  Importing the package registers the
built-in ones."""

from .base import (BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, POSITION_ENCODINGS, Block, Embedding, FeedForward, FixedState,
                   Head, LayerSpec, LazyLinear, LazyNormed, materialize, Mixer, ModelSpec, Norm, PagedKV, Part, PartSpec, PositionEncoding, ScheduleEntry,
                   StreamBranch, TensorSpec, cache_leaves, make_part, register_block, register_embedding, register_feed_forward, register_head, register_mixer, register_norm,
                   register_position_encoding)
from . import (attention, block, convolved_attention, delta_rule, embedding, general_delta, input_conv, latent_attention, linear_attention, mlp, norm,  # noqa: F401
               parallel, recurrent, rope, routed_mlp, ssm, stream_join)  # noqa: F401  (registration)

__all__ = [
    "BLOCKS", "EMBEDDINGS", "FEED_FORWARDS", "HEADS", "MIXERS", "NORMS", "POSITION_ENCODINGS", "Block", "Embedding", "FeedForward", "FixedState",
    "Head", "LayerSpec", "LazyLinear", "LazyNormed", "materialize", "Mixer", "ModelSpec", "Norm", "PagedKV", "Part", "PartSpec", "PositionEncoding", "ScheduleEntry",
    "StreamBranch", "TensorSpec", "cache_leaves", "make_part", "register_block", "register_embedding", "register_feed_forward", "register_head", "register_mixer", "register_norm",
    "register_position_encoding",
]
