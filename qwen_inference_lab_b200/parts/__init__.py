"""Model parts: each owns its sizes, constants and parameters, none knows its model."""
from .base import (FeedForward, KVCacheSpec, Mixer, Norm, Param, Part, PlanView, PositionEncoding, Segments,
                   StateSpec, StepContext, StepPlanner)
from .linear import JointProjection, Linear, StackedLinear
from .norm import ExactRMSNorm, LayerNorm, RMSNorm, ScalarRMSNorm, TanhNorm
from .rotary import RotaryEmbedding, RotaryFrequencies, rotary_table
from .attention import GroupedQueryAttention
from .feed_forward import GatedMLP, PlainMLP
from .experts import RoutedExperts
from .linear_attention import DecayLinearAttention, GatedLinearAttention, MatrixMemory, TiedGateLinearAttention
from .matrix_state import GatedDeltaRule, Retention
from .latent_attention import LatentAttention
from .parallel import ParallelMixers
from .block import DeferredPreNormBlock, ParallelBlock, PostNormBlock, PreNormBlock, SandwichNormBlock
from .side_input import TokenSideInput
from .decoder import DecoderModel, LayerCall, TokenEmbedding
