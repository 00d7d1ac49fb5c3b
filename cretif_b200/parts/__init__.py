"""Parts a model is put together from: embedding, norms, mixers, feed-forwards,
position encodings, heads, and the arrangements that wire them into a block."""
from .base import (LayerCache, Part, StepContext, build_part, lookup_part, register_part,
                   registered_parts)
from . import (attention, block, delta_rule, embedding, experts, latent_attention,  # noqa: F401
               matrix_memory, merge, mlp, norm, parallel, position, retention, shift, state_space,
               token_side)
# (importing registers the parts)

__all__ = ["LayerCache", "Part", "StepContext", "build_part", "lookup_part", "register_part",
           "registered_parts"]
