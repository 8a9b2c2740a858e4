from .base import (Arena, Block, FeedForward, GroupStepView, Mixer, Norm, Part, PartSpec,
                   PositionEncoding, StepContext, register, NORMS, POSITION_ENCODINGS, MIXERS,
                   FEED_FORWARDS, BLOCKS)
from .norm import GroupRMSNorm, RMSNorm
from .rope import NeoxRope, ScaledRope
from .attention import GQAAttention
from .linear_attention import DecayedLinearAttention, GatedLinearAttention
from .latent_attention import LatentAttention
from .delta_rule import GatedDeltaRule
from .moe import RoutedExperts
from .state_space import StateSpace
from .matrix_memory import MatrixMemory
from .parallel import ParallelMixers
from .mlp import MLP, SwiGLU
from .block import PreNormBlock
from .gated_post_norm import GatedPostNormBlock
from .sandwich_norm import SandwichNormBlock
from .post_norm import PostNormBlock
from .side_by_side import SideBySideBlock

__all__ = ["Arena", "Block", "FeedForward", "GroupStepView", "Mixer", "Norm", "Part", "PartSpec",
           "PositionEncoding", "StepContext", "register", "NORMS", "POSITION_ENCODINGS", "MIXERS",
           "FEED_FORWARDS", "BLOCKS", "RMSNorm", "GroupRMSNorm", "NeoxRope", "ScaledRope", "GQAAttention", "GatedLinearAttention", "DecayedLinearAttention", "LatentAttention", "GatedDeltaRule", "RoutedExperts", "ParallelMixers", "SwiGLU", "MLP",
           "PreNormBlock", "GatedPostNormBlock", "SandwichNormBlock", "PostNormBlock", "StateSpace", "MatrixMemory", "SideBySideBlock"]
