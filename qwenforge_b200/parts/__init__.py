from .base import FeedForward, Mixer, Norm, Part, PositionEncoding, TensorSpec
from .registry import build_block, build_part, register_part, registered_parts
from . import attention, block, differential, embedding, experts, gated_ff, latent_attention, mlp, norm, recurrent, rotary, side_by_side, stream, swiglu  # noqa: F401  (registers the built-in parts)

__all__ = ["FeedForward", "Mixer", "Norm", "Part", "PositionEncoding", "TensorSpec", "build_part", "register_part",
           "registered_parts", "build_block"]
