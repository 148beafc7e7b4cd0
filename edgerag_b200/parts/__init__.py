"""Parts a decoder is assembled from.  Importing the package registers the built-in kinds."""

from .base import (Block, DepthUpdate, FeedForward, LayerCall, LayerSpec, Mixer, ModelPlan, Norm, NormedUpdate, Part, PartSpec,
                   PositionEncoding, ScaledUpdate, StreamCall, StreamOp, SumUpdate, WeightSpec, build_part, register_part,
                   registered, settle_update)
from . import (attention, block, delta, depth, diff_attention, embedding, glu, latent_attention, layernorm, mlp, moe,  # noqa: F401
               reentry, rmsnorm, rope, ssd, swiglu)                                                                       # (registration)

__all__ = ["Block", "DepthUpdate", "FeedForward", "LayerCall", "LayerSpec", "Mixer", "ModelPlan", "Norm", "NormedUpdate", "Part",
           "PartSpec", "PositionEncoding", "ScaledUpdate", "StreamCall", "StreamOp", "SumUpdate", "WeightSpec", "build_part", "register_part",
           "registered", "settle_update"]
