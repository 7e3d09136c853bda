"""Models and engine (exports follow ``python/triton_dist/models/__init__.py:32-56``)."""
from .auto import AutoLLM, AutoTokenizer
from .config import ARCHS, ArchConfig, LikosunConfig, ModelConfig, SizilornConfig
from .engine import Engine
from .kv_cache import HybridCache, KV_Cache, LatentCache
from .likosun import Likosun
from .qwen import Qwen3
from .sizilorn import Sizilorn
from .utils import logger, sample_token, seed_everything


__all__ = ["ARCHS", "ArchConfig", "LikosunConfig", "SizilornConfig", "ModelConfig", "AutoLLM", "AutoTokenizer", "Qwen3", "Likosun",
           "Sizilorn", "KV_Cache", "LatentCache", "HybridCache", "Engine",
           "sample_token", "seed_everything", "logger"]
