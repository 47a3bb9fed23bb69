from .attention import Attention
from .base import KINDS, Part, make_part, register_part, registered
from .block import ParallelBlock, PreNormBlock, SandwichBlock
from .embedding import LMHead, TokenEmbedding
from .delta import ChannelDelta, HeadDelta
from .diff_attention import DifferentialAttention
from .latent_attention import LatentAttention
from .mingru import MinGRU
from .rglru import RealGatedLRU
from .table_experts import TableExperts, TableRouting
from .token_mix import InputConv, PassInput, TokenShift, TokenSide
from .moe import RoutedExperts
from .mlp import ClampedGLU, DenseMLP, GatedMLP, PolyNormMLP
from .norm import DynamicTanh, LayerNorm, PendingDelta, RMSNorm, ScaledTerms, UnitMix
from .parallel import ConvAttention, MatrixMemory, NormedAttention, ParallelMixer, StateSpaceDual, SummedMixers
from .sink_attention import SinkAttention
from .streams import HyperBlock, PendingStreams, ResultGate, StreamNorm
from .rope import NoPosition, Rope, RotaryPosition, frequency_factors, store_kv

__all__ = ["Attention", "KINDS", "Part", "make_part", "register_part", "registered", "PreNormBlock", "LMHead",
           "TokenEmbedding", "GatedMLP", "DenseMLP", "ClampedGLU", "RoutedExperts", "ChannelDelta", "HeadDelta", "SinkAttention", "DifferentialAttention", "LatentAttention", "MinGRU", "RealGatedLRU", "TableExperts", "TableRouting", "PassInput", "ParallelBlock", "ScaledTerms", "TokenShift", "TokenSide", "RMSNorm", "DynamicTanh", "LayerNorm", "PendingDelta", "UnitMix", "SandwichBlock", "InputConv", "PolyNormMLP", "ConvAttention", "ParallelMixer", "StateSpaceDual", "NormedAttention", "MatrixMemory", "SummedMixers", "HyperBlock", "PendingStreams", "ResultGate", "StreamNorm", "NoPosition", "Rope", "RotaryPosition", "frequency_factors", "store_kv"]
