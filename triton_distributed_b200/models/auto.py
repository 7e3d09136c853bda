"""Model classes by architecture: what ``AutoLLM``, ``Engine`` and the command-line programs use to pick one."""
from __future__ import annotations

from .config import ModelConfig


class AutoLLM:
    """``AutoLLM.from_pretrained(config, group)``: pick the model class for ``config`` (a name in ``ARCHS`` or the config.json of a
    checkpoint directory)."""

    @staticmethod
    def model_class(config: ModelConfig):
        arch = config.arch()
        design = getattr(arch, "architecture", None)
        if design == "Likosun":
            from .likosun import Likosun
            return Likosun
        if design == "Sizilorn":
            from .sizilorn import Sizilorn
            return Sizilorn
        if arch.num_experts:
            from .qwen_moe import Qwen3MoE
            return Qwen3MoE
        from .qwen import Qwen3
        return Qwen3

    @staticmethod
    def from_pretrained(config: ModelConfig, group=None):
        cls = AutoLLM.model_class(config)
        if config.dtype not in cls.dtypes:
            raise UnsupportedDtype(f"{cls.__name__} runs in {', '.join(str(d) for d in cls.dtypes)}, not {config.dtype}")
        return cls(config, group)


class UnsupportedDtype(ValueError):
    """The model class has no kernels for the storage type that was asked for."""


class AutoTokenizer:
    """Tokenizers come from Hugging Face files; without a local copy there is nothing to load offline."""

    @staticmethod
    def from_pretrained(config: ModelConfig):
        import transformers
        path = config.checkpoint_dir or config.model_name
        return transformers.AutoTokenizer.from_pretrained(path, local_files_only=True)
