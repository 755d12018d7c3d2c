from .attention import DifferentialAttention, GQAAttention
from .base import (KVCacheSpec, MATRIX, ParamSpec, Part, Precision, StateSpec, StepTables, TABLE, VECTOR, part_class,
                   register_part)
from .block import ParallelBlock, PostNormBlock, PreNormBlock, SandwichNormBlock
from .embedding import OutputHead, TokenEmbedding
from .feed_forward import PolyNormFeedForward, RoutedFeedForward, SquaredReLUFeedForward, SwiGLUFeedForward
from .latent_attention import LatentAttention
from .norm import LayerNorm, RMSNorm
from .parallel import ParallelMixer
from .position import RopeScaling, RotaryEmbedding
from .recurrent import GatedDeltaRule, GatedLinearAttention, GeneralDeltaRule, MLSTM, MinGRU, Retention, ShortConvolution, StateSpace
from .side_input import TokenSideInput

__all__ = [
    "DifferentialAttention", "GQAAttention", "GatedDeltaRule", "GatedLinearAttention", "LayerNorm", "Retention", "ShortConvolution", "GeneralDeltaRule", "MLSTM", "ParallelBlock", "ParallelMixer", "SquaredReLUFeedForward", "StateSpace", "TokenSideInput", "KVCacheSpec", "LatentAttention", "MinGRU", "PostNormBlock", "PolyNormFeedForward", "RoutedFeedForward", "SandwichNormBlock", "MATRIX", "OutputHead", "ParamSpec", "Part", "Precision", "PreNormBlock",
    "RMSNorm", "RopeScaling", "RotaryEmbedding", "StateSpec", "StepTables", "SwiGLUFeedForward", "TABLE", "TokenEmbedding", "VECTOR",
    "part_class", "register_part",
]
