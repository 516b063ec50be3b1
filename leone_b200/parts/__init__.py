"""Parts a layer is built from.  Importing this package registers the built-in kinds."""
from . import (attention, block, embedding, experts, gated_delta, gated_linear_attention, head, injection,  # noqa: F401
               latent_attention, layer_norm, linear_attention, mamba2, min_gru, mlp, pooled_attention, rms_norm, rotary, short_conv, side_by_side, swiglu,
               token_gate)
from .base import (Block, Embedding, FeedForward, FixedState, Head, Mixer, Norm, PagedCacheView, PagedKV, Part,
                   PositionEncoding, Runtime, StateView, WeightSpec)
from .spec import LayerSpec, ModelSpec, PartSpec

__all__ = ["Block", "Embedding", "FeedForward", "FixedState", "Head", "Mixer", "Norm", "PagedCacheView", "PagedKV",
           "Part", "PositionEncoding", "Runtime", "StateView", "WeightSpec", "LayerSpec",
           "ModelSpec", "PartSpec"]
