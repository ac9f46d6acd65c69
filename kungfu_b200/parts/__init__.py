"""Parts a model is composed of: norms, position encodings, mixers, feed-forwards, blocks."""
from .base import (Block, FeedForward, FixedState, Mixer, Norm, PagedKV, Part, PositionEncoding, StateBundle, StateNeed,
                   known, make, register_block, register_feed_forward, register_mixer, register_norm,
                   register_position)
from .norm import GroupRmsNorm, NoNorm, RmsNorm, StreamsNorm
from .rope import Rope
from .conv import InputConv, ShortConv
from .attention import ConvGatedAttention, PagedAttention, RowNormAttention, TalkingAttention
from .differential import DifferentialAttention
from .ssm import Mamba2Mixer
from .latent import LatentAttention
from .delta import GatedDeltaMixer
from .lightning import LightningAttention
from .mlstm import MatrixMemory, SideBySide
from .moe import RoutedExperts
from .side import TokenSide
from .ffn import DenseFfn, GatedFfn, PolyNormFfn
from .embedding import Embedding, LmHead, PairEmbedding, StreamsEmbedding
from .block import ParallelBlock, SandwichBlock, ScaledBlock, StreamsBlock, StreamsMix
from .model import DecoderModel, LayerCall, default_schedule
