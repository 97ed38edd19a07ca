from .base import (BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, POSITIONS, BiasedBranch, BranchSum, CacheRef, KVNeed, MeanOfNormed,
                   NormedBranch, ParamSpec, PartSpec, Partials, Residual, StateNeed, as_branch, branch_pair, spec)
from .plan import LayerRun, ModelPlan
from . import (norm, position, attention, linear_attention, state_space, latent_attention, time_mixing, gated_recurrence, feed_forward, embedding, block,  # noqa: F401  (register the built-in parts)
               hyper_connections, experts)

__all__ = ["BLOCKS", "EMBEDDINGS", "HEADS", "FEED_FORWARDS", "MIXERS", "NORMS", "POSITIONS", "CacheRef", "KVNeed", "ParamSpec", "PartSpec",
           "Residual", "Partials", "MeanOfNormed", "BranchSum", "BiasedBranch", "NormedBranch", "as_branch", "branch_pair", "StateNeed", "spec", "LayerRun", "ModelPlan"]
