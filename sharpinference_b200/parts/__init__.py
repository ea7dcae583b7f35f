"""Parts that layers are put together from: norms, position encodings, mixers, feed-forwards, blocks."""
from .base import (Block, CacheSpec, ColumnMixer, FeedForward, LayerSlot, Mixer, Norm, Part, PositionEncoding, StateSpec,
                   StepContext, StreamOp, make_part, part_kinds, register_part)
from .linear import GroupedLinear, Linear
from .norm import DynamicTanh, L2Norm, LayerNorm, NormedUpdate, RMSNorm
from .position import (NoPositionEncoding, RotaryEncoding, leading_rotary_inv_freq, leading_rotary_inv_freq_parts,
                       partial_rotary_inv_freq, rotary_inv_freq, yarn_inv_freq)
from .attention import PagedAttention, distance_bias_table, distance_bucket
from .latent import LatentAttention
from .mlstm import MLSTMMixer, fused_mlstm_columns
from .feedforward import DenseMLP, DenseSwiGLU, MoESigmoidTop1, MoESigmoidTopK, MoESigmoidTopKGated, MoESoftmaxGroups, MoESigmoidGroups
from .block import ParallelBlock, ParallelPairBlock, PreNormBlock, SandwichBlock
from .stream import AddInput, ReinjectInput
from .hyper import GroupRMSNorm, HyperBlock, PairEmbedding
from .wkv import WKVMixer
from .mamba import BranchPair, SelectiveScanMixer, StateSpaceDualityMixer, ssd_projection_order
from .conv_attention import ConvAttention, conv_attention_columns
from .lightning import LightningAttention, LightningPlanner, lightning_columns
from .delta import ChannelDelta, DeltaPlanner, delta_columns
from .token_side import TableWithPositions, TokenSide
from .branches import ScaledBranches

__all__ = ["Block", "CacheSpec", "FeedForward", "LayerSlot", "Mixer", "Norm", "Part", "PositionEncoding",
           "StateSpec", "StepContext", "make_part", "part_kinds", "register_part", "GroupedLinear", "Linear",
           "L2Norm", "RMSNorm", "NoPositionEncoding", "RotaryEncoding", "rotary_inv_freq", "PagedAttention",
           "DenseSwiGLU", "MoESigmoidTop1", "PreNormBlock", "StreamOp", "partial_rotary_inv_freq", "MLSTMMixer",
           "fused_mlstm_columns", "DenseMLP", "MoESigmoidTopK", "ParallelBlock", "ReinjectInput", "GroupRMSNorm",
           "HyperBlock", "PairEmbedding", "WKVMixer", "BranchPair", "SelectiveScanMixer", "leading_rotary_inv_freq", "DynamicTanh", "LatentAttention", "MoESigmoidTopKGated", "StateSpaceDualityMixer",
           "ssd_projection_order", "distance_bias_table", "distance_bucket", "LayerNorm", "yarn_inv_freq",
           "ColumnMixer", "ConvAttention", "conv_attention_columns", "LightningAttention", "LightningPlanner", "lightning_columns",
           "ChannelDelta", "DeltaPlanner", "delta_columns", "TableWithPositions", "TokenSide", "NormedUpdate", "SandwichBlock",
           "MoESigmoidGroups", "ScaledBranches", "ParallelPairBlock", "AddInput", "MoESoftmaxGroups", "leading_rotary_inv_freq_parts"]
