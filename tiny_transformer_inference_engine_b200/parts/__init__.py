"""Parts a model is assembled from.  Importing this package registers the built-in kinds."""
from .base import (PartSpec, ParamSpec, LayerSpec, RunEntry, ModelSpec, PagedKVNeed, FixedStateNeed,
                   PagedKVView, FixedStateView, StepContext, ResidualStream, Part, Norm, PositionEncoding,
                   Mixer, FeedForward, Embedding, Head, Block)
from . import norm, rope, attention, latent_attention, rglru, wkv, mlstm, retention, selective_scan, ffn, moe, embedding, block  # noqa: F401  (registration)
