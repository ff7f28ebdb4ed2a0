from .base import (NO_ROTATION, Block, CachePlane, CacheSpec, Embedding, FeedForward, Mixer, Norm, Part, PartSpec, PositionEncoding,
                   RotationRule, StateSpec, Workspace, build_part, known_parts, register_part)
from . import (attention, block, capped_attention, conv_attention, delta, latent_attention, linear_attention, mlp, moe,  # noqa: F401
               norm, normed_attention, pair_embedding, parallel, pre_norm_stream, recurrent, rope, sandwich, side_by_side,  # noqa: F401
               streams)  # noqa: F401  (register the built-in parts)
from .linear import linear

__all__ = ["NO_ROTATION", "Block", "CachePlane", "CacheSpec", "Embedding", "FeedForward", "Mixer", "Norm", "Part", "PartSpec",
           "PositionEncoding", "RotationRule", "StateSpec", "Workspace", "build_part", "known_parts", "register_part",
           "linear"]
