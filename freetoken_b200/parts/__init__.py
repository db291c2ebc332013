"""Parts a decoder layer is assembled from (see :mod:`.base` for the interfaces)."""

from . import (attention, block, composite, embedding, key_attention, mlp, moe, norm, position,  # noqa: F401
               recurrent, stream_map)  # (registers the kinds)
from .base import (BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, POSITIONS, STREAM_MAPS, Block,
                   CacheView, Embedding, FeedForward, Head, Mixer, Norm, Part, Position, Segment,
                   StepContext, StepPlan, StepShape, StreamMap, Workspace, register_block, register_embedding,
                   register_feed_forward, register_head, register_mixer, register_norm,
                   register_position, register_stream_map)

__all__ = [
    "BLOCKS", "EMBEDDINGS", "FEED_FORWARDS", "HEADS", "MIXERS", "NORMS", "POSITIONS", "STREAM_MAPS", "Block",
    "CacheView", "Embedding", "FeedForward", "Head", "Mixer", "Norm", "Part", "Position",
    "Segment", "StepContext", "StepPlan", "StepShape", "StreamMap", "Workspace", "register_block", "register_embedding",
    "register_feed_forward", "register_head", "register_mixer", "register_norm",
    "register_position", "register_stream_map",
]
