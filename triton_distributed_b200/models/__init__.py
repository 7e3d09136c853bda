"""Models and engine (exports follow ``python/triton_dist/models/__init__.py:32-56``)."""
from .auto import AutoLLM, AutoTokenizer
from .config import ARCHS, ArchConfig, LikosunConfig, ModelConfig
from .engine import Engine
from .kv_cache import KV_Cache, LatentCache
from .likosun import Likosun
from .qwen import Qwen3
from .utils import logger, sample_token, seed_everything


__all__ = ["ARCHS", "ArchConfig", "LikosunConfig", "ModelConfig", "AutoLLM", "AutoTokenizer", "Qwen3", "Likosun", "KV_Cache", "LatentCache",
           "Engine",
           "sample_token", "seed_everything", "logger"]
