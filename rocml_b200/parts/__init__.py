"""Parts a layer is put together from: mixers, feed-forwards, norms, position encodings,
and their arrangement in a block.  Importing this package registers the built-in kinds."""
from .base import (
    BuildEnv, DeferredNorm, FeedForward, Mixer, Norm, Part, PositionEncoding, ResidualSink, build_block,
    build_feed_forward,
    build_mixer, build_norm, build_position, register_arrangement, register_feed_forward,
    register_mixer, register_norm, register_position, registered,
)
from .linear import Linear
from .norm import LayerNorm, RMSNorm
from .position import LearnedPosition, NoPosition, RotaryNeox, RotaryPairs, SinusoidPosition
from .attention import Attention
from .mlp import DenseMLP, GatedMLP
from .latent_attention import LatentAttention
from .routed_mlp import RoutedMLP
from .linear_attention import LinearAttention
from .state_space import StateSpace
from .gated_delta import GatedDelta
from .mlstm import MatrixLSTM
from .rglru import RealGatedLRU
from .side_by_side import SideBySide
from .block import OutputNormBlock, ParallelBlock, PostNormBlock, PreNormBlock, SandwichNormBlock

__all__ = [
    "BuildEnv", "DeferredNorm", "ResidualSink", "FeedForward", "Mixer", "Norm", "Part", "PositionEncoding", "build_block",
    "build_feed_forward", "build_mixer", "build_norm", "build_position", "register_arrangement",
    "register_feed_forward", "register_mixer", "register_norm", "register_position", "registered",
    "Linear", "RMSNorm", "NoPosition", "RotaryNeox", "Attention", "GatedMLP", "PreNormBlock", "LatentAttention", "RoutedMLP", "SandwichNormBlock", "SinusoidPosition", "RotaryPairs", "LinearAttention", "ParallelBlock", "StateSpace", "PostNormBlock", "LayerNorm",
    "LearnedPosition", "GatedDelta", "SideBySide", "OutputNormBlock",
    "DenseMLP", "MatrixLSTM", "RealGatedLRU",
]
