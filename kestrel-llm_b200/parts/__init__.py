from .base import (Block, CacheSpec, CombinedSpec, FeedForward, FixedStateSpec, Mixer, Norm, PagedKVSpec, Part,
                   PositionEncoding, Rotation, WeightSlot)
from .linear import Linear
from .norm import RMSNorm
from .rotary import FrequencyScaling, RampScaling, NoPositionEncoding, RotaryHalf, RotaryInterleaved, SinusoidalPositions
from .attention import GroupedQueryAttention
from .mlp import DenseMLP, GatedMLP
from .attention_gated import GatedWindowAttention
from .attention_latent import LatentAttention
from .attention_differential import DifferentialAttention
from .delta import ChannelDeltaMixer, HeadDeltaMixer
from .recurrence import ForgetGateRecurrence, RemovalDeltaMixer
from .retention import RetentionMixer
from .parallel import JoinedMixers, ParallelMixers
from .ssm import StateSpaceMixer
from .time_mix import TimeMixRecurrence
from .moe import GroupRoutedExperts, RoutedExperts, SoftmaxRoutedExperts
from .rglru import GatedDiagonalRecurrence
from .side_input import TokenSideInput, TokenTable
from .block import ParallelBlock, PostNormBlock, PreNormBlock, SandwichBlock
from .embedding import LMHead, StreamRows, TokenEmbedding

__all__ = ["Block", "CacheSpec", "FeedForward", "FixedStateSpec", "Mixer", "Norm", "PagedKVSpec", "Part",
           "PositionEncoding", "Rotation", "WeightSlot", "Linear", "RMSNorm", "NoPositionEncoding", "RotaryHalf", "RotaryInterleaved",
           "GroupedQueryAttention", "GatedMLP", "PreNormBlock", "LMHead", "TokenEmbedding", "SinusoidalPositions",
           "GatedWindowAttention", "LatentAttention", "ChannelDeltaMixer", "RoutedExperts", "TokenSideInput", "TokenTable", "ParallelBlock",
           "CombinedSpec", "FrequencyScaling", "DenseMLP", "ForgetGateRecurrence", "RemovalDeltaMixer", "ParallelMixers", "SandwichBlock",
           "RampScaling", "GroupRoutedExperts", "GatedDiagonalRecurrence", "StreamRows", "DifferentialAttention",
           "RetentionMixer", "SoftmaxRoutedExperts", "PostNormBlock", "HeadDeltaMixer", "JoinedMixers", "StateSpaceMixer", "TimeMixRecurrence"]
