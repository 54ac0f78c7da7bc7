"""The parts a model is put together from. Importing the package registers the built-in kinds."""
from .base import (Block, FeedForward, Mixer, Norm, Part, PositionEncoding, RunCache, Runtime, part_class,
                   register_block, register_feed_forward, register_mixer, register_norm, register_position_encoding)
from .linear import Linear
from .norm import DynamicTanh, LayerNorm, RmsNorm
from .rope import RotaryTable
from .attention import GqaAttention
from .mlp import DenseGlu, DenseMlp
from .linear_attention import FixedDecayLinearAttention, GatedLinearAttention
from .state_space import SelectiveStateSpace
from .matrix_memory import MatrixMemory
from .delta_rule import GeneralDelta
from .parallel import ParallelMixers
from .latent_attention import LatentAttention
from .experts import RoutedExperts
from .block import ParallelResidualBlock, PostNormBlock, PreNormBlock, SandwichNormBlock
