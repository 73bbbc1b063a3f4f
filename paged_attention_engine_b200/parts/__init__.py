from .base import (
    BLOCKS, CONNECTIONS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, POSITION_ENCODINGS,
    REGISTRIES, Block, CacheNeed, EntryCache, Part, ProjectedMixer, Registry, Runtime, StateNeed, TensorSpec,
    layer_part_specs, with_sub_parts,
)
from . import (attention, blocks, connections, delta_rule, feed_forward, gated_attention, gated_delta, heads, latent_attention, matrix_memory, norms,
               retention, rotary, scored_attention, side_by_side, state_space)  # noqa: F401  (registration)

__all__ = [
    "BLOCKS", "CONNECTIONS", "EMBEDDINGS", "FEED_FORWARDS", "HEADS", "MIXERS", "NORMS", "POSITION_ENCODINGS",
    "REGISTRIES", "Block", "CacheNeed", "EntryCache", "Part", "ProjectedMixer", "Registry", "Runtime", "StateNeed", "TensorSpec",
    "layer_part_specs", "with_sub_parts",
]
