from .block import HyperConnectionBlock, ParallelSublayersBlock, PreNormBlock, SublayerNormBlock
from .context import StepContext, Workspace
from .embedding import LMHead, TokenEmbedding
from .feed_forward import DenseMLP, GatedMLP
from .latent_attention import LatentAttention
from .matrix_state import DecayedMemory, DeltaMemory, FixedMemory, StabilizedMemory
from .mingru import MinGRUMixer
from .mixer import CausalSelfAttention
from .moe import RoutedExperts
from .norm import GroupRMSNorm, LayerNorm, ShiftedRMSNorm, StreamSumRMSNorm
from .parallel import ParallelMixer
from .position import LearnedAbsolutePositions, RotaryPositions, SinusoidalPositions
from .state_space import StateSpaceMixer
from .window_attention import WindowAttention
from .registry import get_part, part_names, register_part, unregister_part

__all__ = ["DecayedMemory", "DeltaMemory", "FixedMemory", "StabilizedMemory", "ParallelSublayersBlock", "SinusoidalPositions", "MinGRUMixer", "ShiftedRMSNorm", "HyperConnectionBlock", "GatedMLP", "StreamSumRMSNorm", "ParallelMixer", "StateSpaceMixer", "WindowAttention", "PreNormBlock", "SublayerNormBlock", "LatentAttention", "RoutedExperts", "GroupRMSNorm", "RotaryPositions", "StepContext", "Workspace", "LMHead", "TokenEmbedding", "DenseMLP",
           "CausalSelfAttention", "LayerNorm", "LearnedAbsolutePositions", "get_part", "part_names",
           "register_part", "unregister_part"]
