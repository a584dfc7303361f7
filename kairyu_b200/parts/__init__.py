"""Model parts and their registries.  Importing this package registers the
built-in parts; more can be registered from outside with the same decorators."""

from kairyu_b200.parts import (  # noqa: F401  (registration)
    attention, block, delta_rule, diff_attention, embedding, ffn, gated_attention, latent_attention, learned_positions, moe, norm, rglru, rope, side_by_side, state_space, stream_map,
    talking_attention,
)
from kairyu_b200.parts.base import (
    BLOCKS,
    EMBEDDINGS,
    FEED_FORWARDS,
    HEADS,
    MIXERS,
    NORMS,
    POSITION_ENCODINGS,
    STREAM_MAPS,
    Block,
    CacheView,
    FeedForward,
    LayerCall,
    LayerSpec,
    Mixer,
    ModelSpec,
    Norm,
    PagedKVSpec,
    Part,
    PartSpec,
    PositionEncoding,
    StateSpec,
    StepContext,
    StreamMap,
    TensorSpec,
)

__all__ = [
    "BLOCKS", "EMBEDDINGS", "FEED_FORWARDS", "HEADS", "MIXERS", "NORMS", "POSITION_ENCODINGS", "STREAM_MAPS",
    "Block", "CacheView", "FeedForward", "LayerCall", "LayerSpec", "Mixer", "ModelSpec", "Norm",
    "PagedKVSpec", "Part", "PartSpec", "PositionEncoding", "StateSpec", "StepContext", "StreamMap", "TensorSpec",
]
