"""Model configuration.

``ModelConfig`` keeps the fields of the reference (``python/triton_dist/models/config.py:30-37``). The
architecture tables replace the Hugging Face hub lookup, which needs a network: they carry exactly the
numbers of the published ``config.json`` files of the Qwen3 dense family, plus a tiny shape for tests.
"""
from __future__ import annotations

import dataclasses
import typing

import torch


@dataclasses.dataclass
class ArchConfig:
    hidden_size: int
    intermediate_size: int
    num_hidden_layers: int
    num_attention_heads: int
    num_key_value_heads: int
    head_dim: int = 128
    vocab_size: int = 151936
    rms_norm_eps: float = 1e-6
    rope_theta: float = 1e6
    tie_word_embeddings: bool = False
    # MoE (0 experts = dense)
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True


@dataclasses.dataclass(frozen=True)
class LatentAttentionSpec:
    """Latent attention without positions: `heads` query heads of `dim`, values of `vdim`, one cached latent of `kv_rank`
    per token, scores multiplied by `scale`, one sink logit per head."""
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float

    kind = "latent_attention"


@dataclasses.dataclass(frozen=True)
class DenseMlpSpec:
    """``down(relu(up(h)) ** 2)`` with `ff` inner columns."""
    ff: int

    kind = "dense"


@dataclasses.dataclass(frozen=True)
class WkvSpec:
    """Decayed outer-product memory per head (`dim` x `dim`), with token-shifted inputs and a low-rank decay whose rank a
    checkpoint gives by the shape of its matrices; `decay_rank` is for random weights."""
    heads: int
    dim: int
    decay_rank: int = dataclasses.field(default=64, compare=False, metadata={"in_config": False})

    kind = "wkv"


@dataclasses.dataclass(frozen=True)
class RotaryScaling:
    """Wavelengths above original / low are stretched by `factor`, those below original / high kept, a linear passage between."""
    factor: float
    low: float
    high: float
    original: float


@dataclasses.dataclass(frozen=True)
class RotarySpec:
    """Rotary positions on the first `dims` dimensions of a head, with frequencies base ** (-2 i / dims)."""
    dims: int
    base: float
    scaling: RotaryScaling | None = None


@dataclasses.dataclass(frozen=True)
class GatedAttentionSpec:
    """Grouped-query attention with normed and rotated q and k, scores multiplied by `scale`, a sigmoid gate per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: RotarySpec


@dataclasses.dataclass(frozen=True)
class GatedDeltaSpec:
    """Gated delta rule, memory `dim` x `vdim` per head, a causal convolution over `conv` tokens on q, k and v."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclasses.dataclass(frozen=True)
class ParallelSpec:
    """Two mixers side by side on one input."""
    left: GatedAttentionSpec
    right: GatedDeltaSpec

    kind = "parallel"


@dataclasses.dataclass(frozen=True)
class SwigluMlpSpec:
    """``down(silu(gate(h)) * up(h))`` with `ff` inner columns."""
    ff: int

    kind = "dense"


@dataclasses.dataclass(frozen=True)
class LayerSpec:
    mixer: LatentAttentionSpec | WkvSpec | ParallelSpec
    mlp: DenseMlpSpec | SwigluMlpSpec | None


def _spec_from_dict(cls, sizes: dict):
    """An instance of a spec class from its part of config.json: numbers, nested specs, None where the class allows it."""
    out = {}
    for name, hint in typing.get_type_hints(cls).items():
        field = cls.__dataclass_fields__[name]
        if not field.metadata.get("in_config", True):
            continue
        options = [t for t in typing.get_args(hint) if t is not type(None)] or [hint]
        value = sizes.get(name) if field.default is None else sizes[name]
        if value is not None:
            value = _spec_from_dict(options[0], value) if dataclasses.is_dataclass(options[0]) else options[0](value)
        out[name] = value
    return cls(**out)


def _spec_to_dict(spec) -> dict:
    out = {}
    for f in dataclasses.fields(spec):
        if f.metadata.get("in_config", True):
            value = getattr(spec, f.name)
            out[f.name] = _spec_to_dict(value) if dataclasses.is_dataclass(value) else value
    return out


def _layers_from_config(entries: list[dict], mixers: tuple, mlps: tuple) -> tuple[LayerSpec, ...]:
    """The `layers` list of a config.json whose entries give 'type', 'mixer' and 'mlp'; `mixers` and `mlps` are what the design has."""
    def pick(classes: tuple, kind: str, sizes: dict, what: str):
        table = {c.kind: c for c in classes}
        if kind not in table:
            raise ValueError(f"unknown {what} {kind!r}; known: {sorted(table)}")
        return _spec_from_dict(table[kind], sizes)
    return tuple(LayerSpec(pick(mixers, e["type"], e["mixer"], "mixer"),
                           None if e.get("mlp") is None else pick(mlps, e["mlp"]["kind"], e["mlp"], "feed-forward")) for e in entries)


def _layers_to_config(layers: tuple[LayerSpec, ...]) -> list[dict]:
    return [{"type": layer.mixer.kind, "mixer": _spec_to_dict(layer.mixer),
             "mlp": None if layer.mlp is None else {"kind": layer.mlp.kind, **_spec_to_dict(layer.mlp)}} for layer in layers]


@dataclasses.dataclass(frozen=True)
class LikosunConfig:
    """Likosun: a parallel decoder (mixer and feed-forward read one layer norm) with gated sublayers, an fp32 residual stream
    averaged over depth after every layer, and latent attention. Every layer states its own kinds and sizes."""
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    norm_eps: float
    embedding_scale: float
    residual_mult: float

    architecture = "Likosun"
    num_experts = 0

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def with_layers(self, n: int) -> "LikosunConfig":
        return dataclasses.replace(self, layers=self.layers[:n])

    @staticmethod
    def from_dict(c: dict) -> "LikosunConfig":
        layers = _layers_from_config(c["layers"], (LatentAttentionSpec,), (DenseMlpSpec,))
        return LikosunConfig(vocab_size=int(c["vocab"]), hidden_size=int(c["width"]), layers=layers,
                             norm_eps=float(c["norm"]["eps"]), embedding_scale=float(c["embedding"]["scale"]),
                             residual_mult=float(c["residual_mult"]))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "layers": _layers_to_config(self.layers),
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult}


@dataclasses.dataclass(frozen=True)
class SizilornConfig:
    """Sizilorn: a sequential pre-norm decoder with tanh norms, recurrent mixers (decayed outer products) and layers that run gated
    attention and a gated delta rule side by side, and a per-layer input from the token's own embedding."""
    vocab_size: int
    hidden_size: int
    layers: tuple[LayerSpec, ...]
    norm_eps: float
    side_dim: int

    architecture = "Sizilorn"
    num_experts = 0

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def with_layers(self, n: int) -> "SizilornConfig":
        return dataclasses.replace(self, layers=self.layers[:n])

    @staticmethod
    def from_dict(c: dict) -> "SizilornConfig":
        return SizilornConfig(vocab_size=int(c["vocab"]), hidden_size=int(c["width"]),
                              layers=_layers_from_config(c["layers"], (WkvSpec, ParallelSpec), (SwigluMlpSpec,)),
                              norm_eps=float(c["norm"]["eps"]), side_dim=int(c["token_side"]["dim"]))

    def to_dict(self) -> dict:
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "layers": _layers_to_config(self.layers),
                "norm": {"eps": self.norm_eps}, "token_side": {"dim": self.side_dim}}


# the designs that read 'architecture' from config.json
DESIGNS = {c.architecture: c for c in (LikosunConfig, SizilornConfig)}
Arch = typing.Union[ArchConfig, LikosunConfig, SizilornConfig]


def _sizilorn(vocab: int, width: int, n_layers: int, heads: int, ff: int, side: int) -> SizilornConfig:
    """Blocks of one parallel layer behind three recurrent ones; attention and delta heads of 128, recurrent heads of 64."""
    kv = max(1, heads // 4)
    recurrent = LayerSpec(WkvSpec(width // 64, 64), SwigluMlpSpec(ff))
    parallel = LayerSpec(ParallelSpec(GatedAttentionSpec(heads, kv, 128, 128, 128 ** -0.5, RotarySpec(128, 5e5, RotaryScaling(8.0, 1.0, 4.0, 8192))),
                                      GatedDeltaSpec(heads, heads // 2, 128, 128, 4)), SwigluMlpSpec(ff))
    return SizilornConfig(vocab, width, tuple(parallel if i % 4 == 3 else recurrent for i in range(n_layers)), 1e-6, side)


def _likosun(vocab: int, width: int, n_layers: int, heads: int, dim: int, vdim: int, kv_rank: int, ff: int) -> LikosunConfig:
    layer = LayerSpec(LatentAttentionSpec(heads, dim, vdim, kv_rank, dim ** -0.5), DenseMlpSpec(ff))
    return LikosunConfig(vocab, width, (layer,) * n_layers, 1e-6, width ** 0.5, 0.5)


ARCHS: dict[str, Arch] = {
    "Qwen/Qwen3-8B": ArchConfig(4096, 12288, 36, 32, 8),
    "Qwen/Qwen3-14B": ArchConfig(5120, 17408, 40, 40, 8),
    "Qwen/Qwen3-32B": ArchConfig(5120, 25600, 64, 64, 8),
    "Qwen/Qwen3-30B-A3B": ArchConfig(2048, 6144, 48, 32, 4, num_experts=128, num_experts_per_tok=8,
                                     moe_intermediate_size=768),
    "Qwen/Qwen3-235B-A22B": ArchConfig(4096, 12288, 94, 64, 4, num_experts=128, num_experts_per_tok=8,
                                       moe_intermediate_size=1536),
    # what ONE rank of a tensor-parallel Qwen3-32B computes at TP = 8 (heads, KV heads and intermediate size divided by
    # eight, vocabulary shard): a single-GPU stand-in for tuning the per-rank kernel chain without the collectives
    "Qwen3-32B-tp8-shard": ArchConfig(5120, 3200, 64, 8, 1, vocab_size=18992),
    # test shapes: same structure, divisible by 8 ranks
    "tiny-qwen3": ArchConfig(512, 1024, 2, 8, 8, vocab_size=1024),
    "tiny-qwen3-gqa": ArchConfig(1024, 2048, 3, 16, 8, vocab_size=2048),
    "tiny-qwen3-moe": ArchConfig(512, 1024, 2, 8, 8, vocab_size=1024, num_experts=16, num_experts_per_tok=4,
                                 moe_intermediate_size=256),
    "tiny-likosun": LikosunConfig(1000, 264, (
        LayerSpec(LatentAttentionSpec(4, 40, 24, 72, 0.2), DenseMlpSpec(520)),
        LayerSpec(LatentAttentionSpec(8, 32, 48, 56, 0.15), None),
        LayerSpec(LatentAttentionSpec(2, 72, 136, 96, 0.1), DenseMlpSpec(200))), 1e-5, 12.0, 0.4),
    # shapes of real layers (random weights; benchmarks): a small, a middle and a large model
    "likosun-1b": _likosun(32768, 2048, 24, 16, 128, 128, 512, 8192),
    "likosun-7b": _likosun(65536, 4096, 32, 32, 128, 128, 512, 16384),
    "likosun-20b": _likosun(65536, 5120, 48, 64, 128, 128, 512, 25600),
    "tiny-sizilorn": SizilornConfig(1000, 264, (
        LayerSpec(WkvSpec(5, 40, 24), None),
        LayerSpec(ParallelSpec(GatedAttentionSpec(4, 2, 56, 72, 0.15, RotarySpec(40, 1e4, RotaryScaling(4.0, 1.0, 4.0, 64))),
                               GatedDeltaSpec(6, 2, 48, 24, 3)), SwigluMlpSpec(520)),
        LayerSpec(WkvSpec(3, 72, 16), SwigluMlpSpec(200))), 1e-5, 20),
    "sizilorn-1b": _sizilorn(32768, 2048, 24, 16, 5632, 128),
    "sizilorn-7b": _sizilorn(65536, 4096, 32, 32, 11008, 256),
}


@dataclasses.dataclass
class ModelConfig:
    model_name: str = "Qwen/Qwen3-32B"
    max_length: int = 4096
    dtype: torch.dtype = torch.bfloat16
    local_only: bool = False
    rank: int = 0
    world_size: int = 8
    # extensions: a directory with HF-layout safetensors (config.json + shards); None = random initialisation
    checkpoint_dir: str | None = None
    seed: int = 0
    num_layers_override: int | None = None  # build fewer layers (tests only)

    def arch(self) -> Arch:
        if self.checkpoint_dir is not None:
            from .weights import read_arch_from_checkpoint
            a = read_arch_from_checkpoint(self.checkpoint_dir)
        elif self.model_name in ARCHS:
            a = ARCHS[self.model_name]
        else:
            raise ValueError(f"unknown model {self.model_name!r}; known: {sorted(ARCHS)} (or pass checkpoint_dir)")
        if self.num_layers_override is not None:
            n = self.num_layers_override
            a = dataclasses.replace(a, num_hidden_layers=n) if isinstance(a, ArchConfig) else a.with_layers(n)
        return a
