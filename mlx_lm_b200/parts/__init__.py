from .base import (INT_TABLE, MATRIX, VECTOR, Block, FeedForward, Init, Mixer, Norm, PagedKVSpec, ParamSpec, Part,
                   PositionEncoding, RowChoice, StateSpec, Summands, make_part, register_part, registered_parts)
from .block import HyperBlock, OutputNormBlock, ParallelBlock, PreNormBlock, SandwichBlock, StreamBlock
from .feed_forward import MLP, ExpertsMLP, GatedMLP, LearnedActMLP
from .linear import FusedLinear, Linear
from .mixers import (Attention, DifferentialAttention, LatentAttention, ParallelMixer, SinkAttention,
                     TalkingHeadsAttention)
from .model import (EMBEDDING_CACHE, LoopInput, Model, ModelDescription, OutputHead, Reentry, RunEntry, TokenEmbedding,
                    TokenPairEmbedding)
from .norms import DynamicTanh, LayerNorm, RMSNorm, StreamsNorm
from .recurrent import GatedDeltaMixer, Mamba2Mixer, MLSTMMixer, RetentionMixer, RGLRUMixer, WKVMixer
from .side import TokenSideInput
from .positions import LearnedAbsolute, NoPosition, Sinusoidal, rotation_frequencies

__all__ = ["INT_TABLE", "MATRIX", "VECTOR", "Block", "FeedForward", "Init", "Mixer", "Norm", "PagedKVSpec",
           "ParamSpec", "Part", "PositionEncoding", "StateSpec", "make_part", "register_part", "registered_parts",
           "PreNormBlock", "MLP", "Linear", "Attention", "Model", "ModelDescription", "OutputHead", "RunEntry",
           "TokenEmbedding", "LayerNorm", "LearnedAbsolute", "NoPosition", "StreamBlock", "GatedMLP", "FusedLinear",
           "ParallelMixer", "SinkAttention", "LoopInput", "Reentry", "RMSNorm", "GatedDeltaMixer", "Mamba2Mixer",
           "TokenSideInput", "LearnedActMLP", "LatentAttention", "TalkingHeadsAttention", "WKVMixer", "DynamicTanh",
           "ExpertsMLP", "SandwichBlock", "Sinusoidal", "ParallelBlock", "DifferentialAttention", "rotation_frequencies",
           "EMBEDDING_CACHE", "HyperBlock", "RetentionMixer", "RGLRUMixer", "StreamsNorm", "TokenPairEmbedding",
           "MLSTMMixer", "OutputNormBlock", "RowChoice", "Summands"]
