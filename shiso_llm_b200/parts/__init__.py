"""Model parts: plan data, interfaces, registries and the built-in parts."""

from .plan import LayerSpec, ModelPlan, PartSpec, RunEntry, sequential_order
from .base import (
    BLOCKS, EMBEDDINGS, FEED_FORWARDS, HEADS, MIXERS, NORMS, POSITION_ENCODINGS, SIDES,
    Block, BuildEnv, DeferredLinear, Embedding, FeedForward, FixedState, Head, Mixer, Norm, NormedOutput, NormedPair, PagedKV,
    Part, PositionEncoding, Registry, SideInput, Stream,
)
from . import norm, position, attention, short_conv, feed_forward, block, embedding  # register built-ins
from . import hyper, wkv, retention, pooled_attention, parallel  # noqa: F401  (more built-ins)
from . import lightning, mamba2, latent_attention, masked_attention, gated_delta  # noqa: F401  (more built-ins)
from . import differential_attention, matrix_memory, token_side  # noqa: F401  (more built-ins)
from .model import Model

__all__ = [
    "BLOCKS", "EMBEDDINGS", "FEED_FORWARDS", "HEADS", "MIXERS", "NORMS", "POSITION_ENCODINGS", "SIDES",
    "Block", "BuildEnv", "DeferredLinear", "Embedding", "FeedForward", "FixedState", "Head", "LayerSpec", "Mixer",
    "Model", "ModelPlan", "Norm", "NormedOutput", "NormedPair", "PagedKV", "Part", "PartSpec", "PositionEncoding", "Registry",
    "RunEntry", "SideInput", "Stream", "sequential_order",
]
