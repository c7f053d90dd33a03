"""Parts of a layer: norms, position encodings, mixers, feed-forwards, blocks."""

from . import (  # noqa: F401  (registers the kinds)
    attention,
    block,
    delta_rule,
    ffn,
    gated_recurrence,
    latent_attention,
    linear_recurrence,
    matrix_memory,
    moe,
    norms,
    positions,
    side_by_side,
    wkv,
)
from .base import (
    BuildContext,
    CacheView,
    FeedForward,
    Mixer,
    Norm,
    Part,
    PositionEncoding,
    WeightInfo,
    arrangement_class,
    build_part,
    part_class,
    register_arrangement,
    register_part,
)

__all__ = [
    "BuildContext",
    "CacheView",
    "FeedForward",
    "Mixer",
    "Norm",
    "Part",
    "PositionEncoding",
    "WeightInfo",
    "arrangement_class",
    "build_part",
    "part_class",
    "register_arrangement",
    "register_part",
]
