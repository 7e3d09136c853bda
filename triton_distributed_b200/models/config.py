"""Model configuration.

``ModelConfig`` keeps the fields of the reference (``python/triton_dist/models/config.py:30-37``). The
architecture tables replace the Hugging Face hub lookup, which needs a network: they carry exactly the
numbers of the published ``config.json`` files of the Qwen3 dense family, plus a tiny shape for tests.
"""
from __future__ import annotations

import dataclasses

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
class LayerSpec:
    mixer: LatentAttentionSpec
    mlp: DenseMlpSpec | None


_MIXERS = {c.kind: c for c in (LatentAttentionSpec,)}
_MLPS = {c.kind: c for c in (DenseMlpSpec,)}


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
        def pick(table: dict, kind: str, sizes: dict, what: str):
            if kind not in table:
                raise ValueError(f"unknown {what} {kind!r}; known: {sorted(table)}")
            return table[kind](**{f.name: (float if f.type == "float" else int)(sizes[f.name]) for f in dataclasses.fields(table[kind])})
        layers = []
        for entry in c["layers"]:
            mlp = entry.get("mlp")
            layers.append(LayerSpec(pick(_MIXERS, entry["type"], entry["mixer"], "mixer"),
                                    None if mlp is None else pick(_MLPS, mlp["kind"], mlp, "feed-forward")))
        return LikosunConfig(vocab_size=int(c["vocab"]), hidden_size=int(c["width"]), layers=tuple(layers),
                             norm_eps=float(c["norm"]["eps"]), embedding_scale=float(c["embedding"]["scale"]),
                             residual_mult=float(c["residual_mult"]))

    def to_dict(self) -> dict:
        layers = [{"type": layer.mixer.kind, "mixer": dataclasses.asdict(layer.mixer),
                   "mlp": None if layer.mlp is None else {"kind": layer.mlp.kind, **dataclasses.asdict(layer.mlp)}} for layer in self.layers]
        return {"architecture": self.architecture, "vocab": self.vocab_size, "width": self.hidden_size, "layers": layers,
                "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult}


def _likosun(vocab: int, width: int, n_layers: int, heads: int, dim: int, vdim: int, kv_rank: int, ff: int) -> LikosunConfig:
    layer = LayerSpec(LatentAttentionSpec(heads, dim, vdim, kv_rank, dim ** -0.5), DenseMlpSpec(ff))
    return LikosunConfig(vocab, width, (layer,) * n_layers, 1e-6, width ** 0.5, 0.5)


ARCHS: dict[str, ArchConfig | LikosunConfig] = {
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

    def arch(self) -> ArchConfig | LikosunConfig:
        if self.checkpoint_dir is not None:
            from .weights import read_arch_from_checkpoint
            a = read_arch_from_checkpoint(self.checkpoint_dir)
        elif self.model_name in ARCHS:
            a = ARCHS[self.model_name]
        else:
            raise ValueError(f"unknown model {self.model_name!r}; known: {sorted(ARCHS)} (or pass checkpoint_dir)")
        if self.num_layers_override is not None:
            n = self.num_layers_override
            a = a.with_layers(n) if isinstance(a, LikosunConfig) else dataclasses.replace(a, num_hidden_layers=n)
        return a
