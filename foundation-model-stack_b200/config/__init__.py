from .model_config import ModelConfig
from .specs import (BlockSpec, DecoderSpec, EmbeddingSpec, FeedForwardSpec, LayerCall, MixerSpec, NormSpec,
                    PositionSpec, TokenSideSpec)

__all__ = ["ModelConfig", "BlockSpec", "DecoderSpec", "EmbeddingSpec", "FeedForwardSpec", "LayerCall", "MixerSpec",
           "NormSpec", "PositionSpec", "TokenSideSpec"]
