"""Parts a layer is put together from.  Importing the package registers the
built-in kinds."""
from . import (attention, block, channel_delta, gated_block, hyper_block, latent_attention, lightning, linear_state, mingru, mlp, mlstm, norm,  # noqa: F401  (registration)
               parallel, rotary, routed_experts, selective_scan, state_space)
from .base import (FeedForward, KVCacheView, Mixer, Norm, Part, PositionEncoding, StateCacheView,
                   StepContext)
from .registry import (BLOCKS, FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, build_part,
                       register_part)
from .spec import KVPagesNeed, LayerSpec, ModelSpec, PartSpec, Run, StateNeed, TensorSpec

__all__ = ["FeedForward", "KVCacheView", "Mixer", "Norm", "Part", "PositionEncoding", "StateCacheView",
           "StepContext", "BLOCKS", "FEED_FORWARDS", "MIXERS", "NORMS", "POSITION_ENCODINGS",
           "build_part", "register_part", "KVPagesNeed", "LayerSpec", "ModelSpec", "PartSpec", "Run",
           "StateNeed", "TensorSpec"]
