from .attention import Attention
from .base import (Block, BuildOptions, FeedForward, HalfSum, KVSpec, Mixer, Norm, Part, PositionEncoding, StateSpec)
from .block import HiddenStream, ParallelBlock, PostNormBlock, PreNormBlock, SandwichBlock
from .embedding import PairTable, PositionTable, TokenEmbedding, VocabHead
from .experts import RoutedExperts, ScoredExperts, TableExperts
from .feedforward import PlainFeedForward, SwiGLU
from .gated_recurrence import GatedDeltaRule, GatedLinearAttention
from .layer_norm import LayerNorm
from .latent_attention import LatentAttention
from .linear import Linear
from .linear_attention import DecayLinearAttention
from .maps_attention import MapsAttention, alibi_slopes
from .mlstm import MatrixMemory
from .norm import RMSNorm
from .side_by_side import SideBySide
from .state_space import StateSpaceMixer
from .position import RotaryEncoding, scaled_inv_freq
from .stream import DepthAverage, InputConv, PassOffset, TokenSide, TokenTable

__all__ = ["GatedDeltaRule", "GatedLinearAttention", "LayerNorm", "PairTable", "HalfSum", "SandwichBlock", "SideBySide", "Attention", "Block", "BuildOptions", "FeedForward", "KVSpec", "Mixer", "Norm", "Part", "PositionEncoding",
           "StateSpec", "HiddenStream", "PreNormBlock", "ParallelBlock", "RoutedExperts", "LatentAttention", "MatrixMemory", "TokenEmbedding", "VocabHead", "SwiGLU", "Linear",
           "RMSNorm", "RotaryEncoding", "scaled_inv_freq", "DecayLinearAttention", "MapsAttention", "PassOffset", "TokenSide",
           "TokenTable", "DepthAverage", "InputConv", "PlainFeedForward", "PositionTable", "PostNormBlock", "TableExperts",
           "ScoredExperts", "StateSpaceMixer", "alibi_slopes"]
