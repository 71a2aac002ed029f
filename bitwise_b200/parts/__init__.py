from .attention import GQAAttention
from .base import (FEED_FORWARDS, MIXERS, NORMS, POSITION_ENCODINGS, FeedForward, Mixer, Norm, PagedKVNeed,
                   PagedKVView, PagedLatentNeed, PagedLatentView, Part, PositionEncoding, SlotStateNeed, SlotStateView, StepContext, Workspace,
                   register_feed_forward, register_mixer, register_norm, register_position_encoding)
from .block import DepthMix, ParallelBlock, PostNormBlock, PreNormBlock, SandwichBlock, ScaledResidualBlock
from .token_side import TokenSide, TokenSideTable
from .embedding import OutputHead, TokenEmbedding
from .mlp import DenseFFN, SwiGLU
from .latent_attention import LatentAttention
from .linear_recurrence import GatedLinearAttention
from .paired import PairedMixer
from .state_recurrence import ChannelDelta, MatrixMemory, ShiftedRecurrence, StateSpace
from .norm import LayerNorm, RMSNorm, TanhNorm
from .rope import (HalfRotaryEncoding, LinearScaling, PairRotaryEncoding, RampScaling, RotaryEncoding, WavelengthScaling,
                   inverse_frequencies)
from .routed_ffn import ClampedGLU, RoutedFFN
from .scored_attention import SEQUENCE_TILE, ScoredAttention, distance_slopes
