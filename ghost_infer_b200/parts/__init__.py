from . import (attention, block, differential_attention, embedding, head_normed_attention, hyper, injection, latent_attention, linear_state, mamba2, mlp, mlstm, moe, norm,
               normed_attention, parallel, rope, sink_attention, token_side)  # noqa: F401  (registers the built-in parts)
from .base import Block, Embedding, FeedForward, Injection, Mixer, Norm, Part, PositionEncoding, RowRead, Runtime, StreamRead, WeightSpec
from .registry import lookup, register, registered, unregister
from .spec import ExtraPart, LayerSpec, ModelSpec, PartSpec, ScheduleEntry, looped_schedule

__all__ = ["Block", "Embedding", "FeedForward", "Injection", "Mixer", "Norm", "Part", "PositionEncoding", "RowRead", "Runtime", "StreamRead", "WeightSpec",
           "lookup", "register", "registered", "unregister", "ExtraPart", "LayerSpec", "ModelSpec", "PartSpec", "ScheduleEntry", "looped_schedule"]
