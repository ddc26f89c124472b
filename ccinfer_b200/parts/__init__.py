from .attention import GroupedQueryAttention
from .base import (Block, CachedTensor, CacheNeed, FeedForward, Mixer, Norm, Part, PositionEncoding, Residual, StateNeed,
                   TensorSpec)
from .block import LayerScaleBlock, PostNormBlock, PreNormBlock, SandwichNormBlock
from .delta import ChannelGatedDelta, HeadGatedDelta
from .embedding import LoopInput, OutputHead, TokenEmbedding, TokenSideInput
from .feedforward import ClampedGLU, GeluGLU, SquaredReLU, SwiGLU
from .latent import LatentAttention
from .linear_attention import GatedLinearAttention
from .matrix_memory import ExponentialGateMemory, Retention
from .moe import MixtureOfExperts
from .norm import LayerNorm, RMSNorm, StreamRows
from .parallel import ParallelMixers
from .position import NoPosition, QueryTemperature, RotaryHalf
from .ssm import SelectiveStateSpace
from .streams import HyperConnectionBlock, StreamsConnection, StreamsNorm

__all__ = ["Block", "CachedTensor", "CacheNeed", "ChannelGatedDelta", "ClampedGLU", "ExponentialGateMemory",
           "FeedForward", "GatedLinearAttention", "GeluGLU", "GroupedQueryAttention", "HeadGatedDelta",
           "HyperConnectionBlock", "LatentAttention", "LayerNorm", "LayerScaleBlock", "LoopInput", "Mixer",
           "MixtureOfExperts", "NoPosition", "Norm", "OutputHead", "ParallelMixers", "Part", "PositionEncoding",
           "PostNormBlock", "PreNormBlock", "QueryTemperature", "RMSNorm", "Residual", "Retention", "RotaryHalf", "SandwichNormBlock", "SelectiveStateSpace",
           "SquaredReLU", "StateNeed", "StreamRows",
           "StreamsConnection", "StreamsNorm", "SwiGLU", "TensorSpec", "TokenEmbedding", "TokenSideInput"]
