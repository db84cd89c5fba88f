from .attention import HeadNormAttention, RadixAttention, RowNormAttention
from .embedding import VocabParallelEmbedding
from .linear import ColumnParallelLinear, Linear, MergedLinear, RowParallelLinear
from .lightning import LightningAttention
from .mlp import MLP, ParallelMLP, SquaredReluMLP
from .latent_attention import LatentAttention, latent_plan
from .norm import DynamicTanh, GemmaRMSNorm, LayerNorm, OutputRMSNorm, PostRMSNorm, RMSNorm
from .parallel_mixer import ParallelMixer
from .quantize_base import LinearMethodBase, QuantizeMethodBase, UnquantizedLinearMethod, set_weight_attrs
