"""Parts a model is put together from; importing the package registers the built-in ones."""
from . import (attention, block, conv_attention, delta_rule, differential_attention, embedding, gla, latent_attention, lightning,
               mixed_attention, mlp, moe, norm, pooled_attention, recurrent, rglru, rope, side_by_side, sink_attention, ssm, summed_mixers, token_shifted)  # noqa: F401
from .base import FeedForward, Mixer, Norm, Part, PositionEncoding, Runtime, Workspace
from .registry import build, lookup, register
from .spec import CacheNeed, LayerSpec, ModelSpec, ParamSpec, PartSpec, RunEntry

__all__ = [
    "CacheNeed", "FeedForward", "LayerSpec", "Mixer", "ModelSpec", "Norm", "ParamSpec", "Part",
    "PartSpec", "PositionEncoding", "RunEntry", "Runtime", "Workspace", "build", "lookup", "register",
]
