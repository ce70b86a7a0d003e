from .base import (BuildContext, ParamSpec, Part, PartSpec, ProductChoice, build_part,
                   known_parts, register_part, unregister_part)
from .block import Block, HyperPreNormBlock, ParallelBlock, PostNormBlock, PreNormBlock, SandwichBlock
from .feedforward import FeedForward, GatedMLP, ReluSquaredMLP, RoutedExperts, SwiGLU
from .io import Embedding, Head, LinearHead, TokenEmbedding, TokenPositionalEmbedding
from .linear import Linear
from .mixer import DifferentialAttention, GQAAttention, LatentAttention, Mixer, SideBySide
from .recurrent import (ChannelDelta, ForgetGateAttention, GatedDelta, GatedLinearRecurrence, LightningAttention,
                        Retention)
from .norm import Averaged, Contribution, DynamicTanh, HyperConnected, LayerNorm, Norm, RMSNorm, residual_add, stream_add
from .plan import LayerPlan, ModelPlan, ScheduleEntry
from .position import NoPosition, PositionEncoding, RotaryHalfSplit, RotaryTable

__all__ = ["BuildContext", "ParamSpec", "Part", "PartSpec", "ProductChoice", "build_part", "known_parts",
           "register_part", "unregister_part", "Block", "HyperPreNormBlock", "HyperConnected", "ChannelDelta", "PostNormBlock", "PreNormBlock", "SandwichBlock", "FeedForward", "ReluSquaredMLP", "SwiGLU", "GatedMLP", "RoutedExperts", "GatedDelta", "LightningAttention", "DifferentialAttention", "DynamicTanh", "TokenPositionalEmbedding", "stream_add",
           "Contribution", "LayerNorm",
           "Embedding", "Head", "LinearHead", "TokenEmbedding", "Linear", "GQAAttention", "Mixer",
           "Norm", "RMSNorm", "residual_add", "LayerPlan", "ModelPlan", "ScheduleEntry",
           "NoPosition", "PositionEncoding", "RotaryHalfSplit", "RotaryTable"]
