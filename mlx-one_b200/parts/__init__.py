from . import blocks, embeddings, feed_forwards, mixers, norms, positions  # register the built-in kinds
from .base import (Block, Embedding, FeedForward, FixedState, Mixer, Norm, NormedInput, NormedUpdate, PagedKeyValues,
                   PagedView, Part, PositionEncoding, Runtime, StateView, StepContext, StreamUpdate)
from .model import Model, cache_entries, expected_tensors
from .registry import BLOCKS, EMBEDDINGS, FEED_FORWARDS, MIXERS, NORMS, POSITIONS
from .spec import FreeSize, Injection, LayerCall, LayerSpec, ModelSpec, PartSpec, TensorSpec

__all__ = ["Block", "Embedding", "FeedForward", "FixedState", "Mixer", "Norm", "NormedInput", "NormedUpdate",
           "PagedKeyValues", "PagedView", "Part", "PositionEncoding", "Runtime", "StateView", "StepContext",
           "StreamUpdate", "Model", "cache_entries", "expected_tensors", "BLOCKS", "EMBEDDINGS", "FEED_FORWARDS", "MIXERS",
           "NORMS", "POSITIONS", "FreeSize", "Injection", "LayerCall", "LayerSpec", "ModelSpec", "PartSpec",
           "TensorSpec"]
