from .attention import PagedAttention
from .attention_biased import BiasedAttention
from .attention_latent import LatentAttention
from .attention_masked import MaskedAttention
from .base import (ANY, INIT_EYE, INIT_NORM, INIT_NORMAL, INIT_ONES, INIT_SHARE, INIT_SMALL, MATRIX, TABLE, VECTOR, FeedForward, Mixer, Norm, ParamSpec, Part,
                   PositionEncoding, Source, walk)
from .block import ParallelBlock, PostNormBlock, PreNormBlock, SandwichBlock
from .embedding import BigramEmbedding, OutputHead, PositionedEmbedding, TokenEmbedding
from .hyper import HyperConnection, HyperConnectionBlock, ResidualStreams
from .mlp import ClampedGLU, DenseMLP, GatedMLP, GatedUnit, RoutedExperts
from .norm import DynamicTanh, LayerNorm, RMSNorm
from .recurrent import DecayedLinearAttention, GatedDeltaMixer, HeadDecayDeltaMixer, MatrixMemoryMixer, ParallelMixer, SelectiveScanMixer, StateSpaceMixer
from .rotary import LinearRotary, RampedRotary, RotaryEncoding

__all__ = ["DecayedLinearAttention", "PositionedEmbedding", "PostNormBlock", "BigramEmbedding", "DynamicTanh", "LinearRotary", "MatrixMemoryMixer", "MaskedAttention", "SandwichBlock", "ParallelBlock", "GatedUnit", "RoutedExperts", "HeadDecayDeltaMixer", "SelectiveScanMixer", "ClampedGLU", "LayerNorm", "GatedDeltaMixer", "ParallelMixer", "StateSpaceMixer", "RampedRotary",
           "PagedAttention", "BiasedAttention", "LatentAttention", "HyperConnection", "HyperConnectionBlock", "ResidualStreams", "DenseMLP", "FeedForward", "Mixer", "Norm", "ParamSpec", "Part", "PositionEncoding", "Source", "walk",
           "PreNormBlock", "OutputHead", "TokenEmbedding", "GatedMLP", "RMSNorm", "RotaryEncoding",
           "ANY", "INIT_EYE", "INIT_NORM", "INIT_NORMAL", "INIT_ONES", "INIT_SHARE", "INIT_SMALL", "MATRIX", "TABLE", "VECTOR"]
