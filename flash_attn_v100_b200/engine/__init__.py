"""Decoder engine on the library's operators: a tensor-parallel Qwen3-shaped decoder and the hybrid decoders."""
from .config import HybridConfig, ModelConfig, qwen3_8b_shaped, tiny_config  # noqa: F401
from .weights import hybrid_weights, make_rank_weights, random_hybrid_tensors  # noqa: F401
from .model import TPDecoder  # noqa: F401
from .hybrid import HybridDecoder  # noqa: F401
from .registry import load_model  # noqa: F401
from .runner import GenerationRunner  # noqa: F401
