"""Parts a layer is put together from; importing this package registers them."""
from . import (attention, block, delta_rule, distance_attention, embedding, gating, general_attention, latent_attention,  # noqa: F401
               linear_attention, matrix_memory, mlp, norm, recurrent, rotary, routed_mlp, talking_attention)
from .base import Part, Runtime
from .linear import Linear

__all__ = ["Part", "Runtime", "Linear"]
