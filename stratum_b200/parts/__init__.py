from . import (attention, block, conv_attention, delta_rule, differential_attention, embedding, latent_attention, linear_attention,  # noqa: F401
               linear_recurrence, mixer_mean, mlp, moe, norm, reentry, retention, rope, sink_attention, state_space)  # noqa: F401  (registers the built-in parts)
from .base import (Arrangement, Embedding, FeedForward, Head, Mixer, Norm, Part, PositionEncoding,
                   RotaryTable, Runtime)
from .registry import find_part, register_part, registered
from .spec import LayerSpec, ModelSpec, PartSpec, ScheduleEntry, TensorSpec

__all__ = ["Arrangement", "Embedding", "FeedForward", "Head", "Mixer", "Norm", "Part", "PositionEncoding",
           "RotaryTable", "Runtime", "find_part", "register_part", "registered", "LayerSpec", "ModelSpec",
           "PartSpec", "ScheduleEntry", "TensorSpec"]
