from .attention import HeadNormAttention, RadixAttention, RotaryAttention, RowNormAttention
from .embedding import VocabParallelEmbedding
from .linear import ColumnParallelLinear, Linear, MergedLinear, RowParallelLinear
from .lightning import LightningAttention
from .mlp import MLP, ParallelMLP, SquaredReluMLP
from .latent_attention import LatentAttention, latent_plan
from .norm import DynamicTanh, GemmaRMSNorm, LayerNorm, OutputRMSNorm, PostRMSNorm, RMSNorm
from .parallel_mixer import NormedParallelMixer, ParallelMixer
from .state_space import StateSpace
from .quantize_base import LinearMethodBase, QuantizeMethodBase, UnquantizedLinearMethod, set_weight_attrs
