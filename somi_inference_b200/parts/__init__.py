"""Parts of a decoder layer, their registries, and the generic decoder built from them."""

from . import (block, conv_attention, differential_attention, embedding, extras,  # noqa: F401
               feedforward, latent, mamba2, matrix_state, mixer, moe, norm, normed_attention,  # (register kinds)
               position, side_by_side)
from .base import (BranchSum, BuildContext, CacheNeeds, GatedDelta, NormedDelta, PagedKVNeeds,
                   ScaledBranches, StateNeeds, TensorDecl)
from .model import Decoder, declared_tensors
from .registry import (ARRANGEMENTS, EMBEDDINGS, FEED_FORWARDS, HEADS, LAYER_EXTRAS, MIXERS, NORMS,
                       POSITION_ENCODINGS, STREAM_PARTS)

__all__ = ["BranchSum", "STREAM_PARTS", "BuildContext", "CacheNeeds", "GatedDelta", "NormedDelta", "PagedKVNeeds", "ScaledBranches", "StateNeeds", "TensorDecl", "Decoder",
           "declared_tensors", "ARRANGEMENTS", "EMBEDDINGS", "FEED_FORWARDS", "HEADS", "LAYER_EXTRAS", "MIXERS",
           "NORMS", "POSITION_ENCODINGS"]
