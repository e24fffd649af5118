"""Model families: multi-exit MoE ``TriuneTransformer``, dense ``UniversalTransformer`` and ``HybridTransformer`` with
layers that differ (``Bubitar``, ``Famalorn``)."""

from .attention import HybridAttention, SoftmaxAttention, VectorisedGLA
from .block import DenseFFN, TransformerBlock
from .bubitar import Bubitar
from .famalorn import Famalorn
from .hybrid import HybridTransformer
from .moe import MoE_FFN, RoutingResult
from .norms import RMSNorm
from .rotary import RotaryEmbedding
from .router import GumbelSoftmaxRouter
from .transformer import TriuneTransformer

__all__ = [
    "Bubitar", "Famalorn", "HybridTransformer", "HybridAttention", "SoftmaxAttention", "VectorisedGLA", "DenseFFN", "TransformerBlock", "MoE_FFN",
    "RoutingResult", "RMSNorm", "RotaryEmbedding", "GumbelSoftmaxRouter", "TriuneTransformer",
]
