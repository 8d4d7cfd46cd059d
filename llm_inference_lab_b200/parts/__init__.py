"""Parts a model is put together from.  Importing the package registers the built-in kinds."""
from . import (attention, block, delta, diff_attention, embedding, hyper, latent, linear_state,  # noqa: F401
               matrix_memory, mlp, moe, norm, norm_attention, reentry, rope, selective_state,          # (registration)
               token_gate, window_attention)
from .base import (BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, POSITIONS, Block, CacheView, Embedding,
                   FeedForward, GroupView, Head, Mixer, Norm, Part, PositionEncoding, StepContext, lookup,
                   register_part)
from .spec import (CacheParts, FixedState, LayerCall, LayerSpec, ModelBlueprint, PagedKV, PagedLatent, PartSpec, Reentry,
                   TensorSpec)

__all__ = ["BLOCKS", "EMBEDDINGS", "FEED_FORWARDS", "HEADS", "MIXERS", "NORMS", "POSITIONS", "Block", "CacheView",
           "Embedding", "FeedForward", "GroupView", "Head", "Mixer", "Norm", "Part", "PositionEncoding",
           "StepContext", "lookup", "register_part", "CacheParts", "FixedState", "LayerCall", "LayerSpec", "ModelBlueprint",
           "PagedKV", "PagedLatent", "PartSpec", "Reentry", "TensorSpec"]
