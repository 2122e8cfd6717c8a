"""Parts a model is assembled from. Importing this package registers the built-in kinds."""

from matricxon_b200.parts import (  # noqa: F401  (registration)
    attention, block, delta, latent_attention, linear_attention, mlp, norm, parallel, pass_input, recurrent, rotary, routed,
    selective, side_input)
from matricxon_b200.parts.base import (
    Block,
    BranchMixer,
    CacheBinding,
    FeedForward,
    KVCacheRequest,
    Mixer,
    Norm,
    Part,
    PositionEncoding,
    Runtime,
    StateRequest,
    build_part,
    part_class,
    register_part,
)

__all__ = ["Block", "BranchMixer", "CacheBinding", "FeedForward", "KVCacheRequest", "Mixer", "Norm", "Part",
           "PositionEncoding", "Runtime", "StateRequest", "build_part", "part_class",
           "register_part"]
