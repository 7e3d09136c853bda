"""Sizilorn decoder: sequential pre-norm layers with tanh norms, recurrent or two-sided mixers, and a per-layer token input.

Layer i, on the fp32 stream x:

    x += mixer(norm1(x))             "wkv": decayed outer products;  "parallel": half the sum of gated attention and the gated delta
                                     rule, each RMS-normed over the width
    x += swiglu(norm2(x))            where the layer has a feed-forward
    x += rms(proj (gelu(gate x) * e)) * gain      e: this layer's part of the token's side embedding

A "parallel" layer has one input GEMM for both sides, [q | k | v | gates | q k v | b | a | gate]; a "wkv" layer multiplies its five
token-shifted mixes in one launch in decode. Everything between two GEMMs on the stream (post norms, residual, the next norm) is
one launch. The stream and all states stay fp32.

The interface is that of ``Qwen3`` (``set_fwd``, ``init_triton_dist_AR_ctx``, ``inference``, ``finalize``), so ``Engine`` serves both.
Forward mode: ``triton_dist_AR`` (native kernels, replicated activations, one all-reduce per sublayer). Storage types: bf16 / f16, or
fp32 with every product in true fp32.
"""
from __future__ import annotations

import functools

import torch

from .. import ops
from ..kernels.allreduce import AllReduceMethod
from ..layers.nvidia.gated_attn import GatedAttention
from ..layers.nvidia.latent_attn import pad_matrix, pad_up, pad_vector, shard_local
from ..layers.nvidia.recurrent import GatedDelta, WkvMixer
from ..layers.nvidia.tp_mlp import TP_MLP
from .config import LayerSpec, ModelConfig, ParallelSpec, SizilornConfig
from .kv_cache import HybridCache
from .weights import RandomSource, SafetensorsSource, WeightSource


class StreamNorm:
    """A tanh norm's weights, as keyword arguments of the residual-stream ops."""

    def __init__(self, src: WeightSource, name: str, width_pad: int):
        self.gain, self.bias = pad_vector(src.get(name), width_pad), pad_vector(src.get(name + ".b"), width_pad)
        self.kind = ops.TanhNorm(float(src.get(name + ".alpha")))

    @property
    def kw(self) -> dict:
        return {"gain": self.gain, "bias": self.bias, "center": self.kind}


class SizilornLayer:

    def __init__(self, layer_idx: int, rank: int, world_size: int, group):
        self.layer_idx, self.rank, self.world_size, self.group = layer_idx, rank, world_size, group

    def _get(self, src: WeightSource, prefix: str, name: str, rows: int | None = None, cols: int | None = None) -> torch.Tensor:
        """This rank's `rows` / `cols` of a tensor (None: the whole dimension)."""
        part = [None if n is None else slice(self.rank * n, (self.rank + 1) * n) for n in (rows, cols)]
        return src.get(prefix + name, rows=part[0], cols=part[1])

    def load(self, src: WeightSource, arch: SizilornConfig, spec: LayerSpec, dtype: torch.dtype, positions: int) -> None:
        p, m, w, eps = f"l{self.layer_idx}.", spec.mixer, self.world_size, arch.norm_eps
        P = pad_up(arch.hidden_size)
        self.norm1 = StreamNorm(src, p + "norm1", P)
        self.parallel = isinstance(m, ParallelSpec)
        if self.parallel:
            left, right = (functools.partial(self._get, src, f"{p}mix.{side}.") for side in ("left", "right"))
            self.left, self.right = GatedAttention(m.left, eps, w, dtype), GatedDelta(m.right, eps, w)
            self.left._init_parameters(left, P, positions)
            self.right._init_parameters(right, P)
            rows = self.left.input_rows(left, P), self.right.input_rows(right, P)
            self.n_left = len(rows[0])
            self.splits = [r.shape[0] for side in rows for r in side]
            self.w_in = torch.cat([r for side in rows for r in side]).contiguous()
            self.left_gain, self.right_gain = pad_vector(src.get(p + "mix.left.out"), P), pad_vector(src.get(p + "mix.right.out"), P)
        else:
            self.mixer = WkvMixer(m, eps, w)
            self.mixer._init_parameters(functools.partial(self._get, src, p + "mix."), P)
        self.mlp = None
        if spec.mlp is not None:
            fs = shard_local(spec.mlp.ff, w, self.rank)
            F = pad_up(spec.mlp.ff // w)
            self.norm2 = StreamNorm(src, p + "norm2", P)
            self.mlp = TP_MLP(self.rank, w, self.group)
            self.mlp._init_parameters(gate=pad_matrix(src.get(p + "mlp.gate", rows=fs), F, P), up=pad_matrix(src.get(p + "mlp.up", rows=fs), F, P),
                                      down=pad_matrix(src.get(p + "mlp.down", cols=fs), P, F))
        D = pad_up(arch.side_dim)
        self.side_gate = pad_matrix(src.get(p + "side.gate"), D, P)
        self.side_proj = pad_matrix(src.get(p + "side.proj"), P, D)
        self.side_gain = pad_vector(src.get(p + "side.norm"), P)

    def cache_layer(self, dtype: torch.dtype) -> HybridCache.Layer:
        if self.parallel:
            return HybridCache.Layer(pages=self.left.cache_pages(), states=self.right.cache_states(dtype))
        return HybridCache.Layer(states=self.mixer.cache_states(dtype))

    def mix(self, h: torch.Tensor, cache: HybridCache, step: dict) -> torch.Tensor:
        """h [T, P] -> partial sums of the mixer's sides [2 or 1, T, P]."""
        out = torch.empty((2 if self.parallel else 1, *h.shape), dtype=h.dtype, device=h.device)
        if not self.parallel:
            self.mixer.partial_fwd(h, cache, self.layer_idx, out[0])
            return out
        parts = ops.linear(h, self.w_in).split(self.splits, dim=1)
        self.left.partial_fwd(parts[: self.n_left], cache, self.layer_idx, step, out[0])
        self.right.partial_fwd(parts[self.n_left:], cache, self.layer_idx, out[1])
        return out


class Sizilorn:

    dtypes = (torch.bfloat16, torch.float16, torch.float32)
    library_subset = "sizilorn"   # the native kernels that one GPU needs (``build.SUBSETS``)

    def __init__(self, model_config: ModelConfig, group=None, source: WeightSource | None = None):
        self.model_config, self.group = model_config, group
        self.rank, self.world_size = model_config.rank, model_config.world_size
        self.dtype = model_config.dtype
        self.arch = model_config.arch()
        if not isinstance(self.arch, SizilornConfig):
            raise ValueError(f"{model_config.model_name} is not a Sizilorn model")
        for spec in self.arch.layers:
            m = spec.mixer
            counts = [m.left.heads, m.left.kv_heads, m.right.heads, m.right.kv_heads] if isinstance(m, ParallelSpec) else [m.heads]
            if any(n % self.world_size for n in counts + ([spec.mlp.ff] if spec.mlp is not None else [])):
                raise ValueError("heads and feed-forward sizes must be divisible by the world size")
        self.device = "cuda" if torch.cuda.is_available() else "cpu"
        self.mode = "triton_dist_AR"
        self.ar_ctx, self.ar_method = None, None
        self.max_length = model_config.max_length
        self.layer_taps: list[torch.Tensor] | None = None  # set to a list to collect the fp32 stream after every layer
        self.init_parameters(source)

    # ------------------------------------------------------------------ weights
    def init_parameters(self, source: WeightSource | None = None) -> None:
        cfg, a = self.model_config, self.arch
        if source is None:
            if cfg.checkpoint_dir:
                source = SafetensorsSource(cfg.checkpoint_dir, self.device, self.dtype)
            else:
                big = a.hidden_size ** 2 * a.num_hidden_layers > 5e7
                source = RandomSource(a, self.dtype, cfg.seed, self.device, consistent=not big)
        P = pad_up(a.hidden_size)
        self.pitch = P
        self.embed = pad_matrix(source.get("embed"), a.vocab_size, P)
        self.side_embed = source.get("side.embed").contiguous()
        self.head = pad_matrix(source.get("head"), pad_up(a.vocab_size), P)
        self.final_norm = StreamNorm(source, "final.norm", P)
        self.layers = []
        for i, spec in enumerate(a.layers):
            layer = SizilornLayer(i, self.rank, self.world_size, self.group)
            layer.load(source, a, spec, self.dtype, self.max_length)
            self.layers.append(layer)
        self.num_layers = a.num_hidden_layers

    def make_cache(self, batch_size: int, max_length: int | None = None) -> HybridCache:
        return HybridCache([layer.cache_layer(self.dtype) for layer in self.layers], batch_size, max_length or self.max_length, self.dtype,
                           device=self.device)

    # ------------------------------------------------------------------ modes and contexts
    def set_fwd(self, mode: str = "triton_dist_AR") -> None:
        if mode != "triton_dist_AR":
            raise ValueError(f"Sizilorn runs in mode 'triton_dist_AR' (native kernels, replicated activations), not {mode!r}")
        self.mode = mode

    def init_triton_dist_AR_ctx(self, max_M: int, ar_method: AllReduceMethod | None = None) -> None:
        self.ar_method = ar_method
        if self.world_size > 1 and self.ar_ctx is None:
            from ..kernels.nvidia import create_allreduce_ctx
            self.ar_ctx = create_allreduce_ctx(64 << 20, self.rank, self.world_size, self.world_size)
        # pre-size the split-K scratch so that nothing allocates inside a CUDA graph capture
        widest = max([self.head.shape[0]] + [layer.w_in.shape[0] if layer.parallel else layer.mixer.w_in.shape[0] for layer in self.layers]
                     + [layer.mlp.gate_up_proj.shape[0] for layer in self.layers if layer.mlp is not None])
        ops.reserve_skinny_scratch(torch.device("cuda", torch.cuda.current_device()),
                                   pad_up(min(max_M, 256), 16) * pad_up(widest, 128), pad_up(widest, 128) // 128)

    def finalize(self) -> None:
        if self.ar_ctx:
            self.ar_ctx.finalize()
        self.ar_ctx = None

    def _reduced(self, t: torch.Tensor) -> torch.Tensor:
        """The sum over ranks of partial sums [..., T, P]."""
        if self.world_size == 1:
            return t
        from ..kernels.nvidia import all_reduce
        return all_reduce(t.view(-1, self.pitch), None, self.ar_method, self.ar_ctx).view(t.shape)

    # ------------------------------------------------------------------ forward
    @torch.no_grad()
    def inference(self, input_ids: torch.Tensor, position_ids: torch.Tensor, kv_cache: HybridCache, wo_lm_head: bool = False,
                  kv_len: int | None = None) -> torch.Tensor:
        """input_ids / position_ids [B, S]: the next S tokens of every sequence, at consecutive positions. Returns fp32 logits
        [B, 1, V] of the last position, or the normed hidden states [B, S, P] with ``wo_lm_head`` (see ``lm_logits``). `kv_len`:
        the longest sequence after this step, when the host knows it (read from the device otherwise; one-token steps do not
        need it and never synchronise)."""
        bsz, S = input_ids.shape
        a, W = self.arch, self.arch.hidden_size
        if S > 1 and kv_len is None:
            kv_len = int(position_ids.max()) + 1
        ids = input_ids.reshape(-1).contiguous()
        step = {"bsz": bsz, "seqlen": S, "kv_len": kv_len if S > 1 else None, "slots": kv_cache.slots(position_ids),
                "positions": position_ids.reshape(-1).to(torch.int32), "kv_lens": (position_ids[:, -1] + 1).to(torch.int32)}
        first = self.layers[0].norm1
        x, h = ops.embed_norm(ids, self.embed, 1.0, W, first.gain, first.bias, 0.0, first.kind)
        for i, layer in enumerate(self.layers):
            out = self._reduced(layer.mix(h, kv_cache, step))
            then = layer.norm2.kw if layer.mlp is not None else {"center": ops.COPY}
            if layer.parallel:
                h = ops.residual_post(x, W, 0.5, out[0], layer.left_gain, out[1], layer.right_gain, a.norm_eps, **then)
            else:
                h = ops.residual_norm(x, W, 1.0, out[0], **then)
            if layer.mlp is not None:
                h = ops.residual_norm(x, W, 1.0, self._reduced(layer.mlp.partial_fwd(h)), center=ops.COPY)
            act = ops.token_side(ops.linear(h, layer.side_gate), ids, self.side_embed, i * a.side_dim, a.side_dim)
            y = ops.linear(act, layer.side_proj)
            norm = self.final_norm if i + 1 == self.num_layers else self.layers[i + 1].norm1
            h = ops.residual_post(x, W, 1.0, y, layer.side_gain, post_eps=a.norm_eps, **norm.kw)
            if self.layer_taps is not None:
                self.layer_taps.append(x[:, :W].clone())
        hidden = h.view(bsz, S, self.pitch)
        return hidden if wo_lm_head else self.lm_logits(hidden[:, -1:, :])

    def lm_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits [B, n, V] of normed hidden states [B, n, P]. (The head is replicated over ranks.)"""
        rows = hidden.reshape(-1, self.pitch).contiguous()
        logits = ops.linear(rows, self.head)[:, : self.arch.vocab_size]
        return logits.float().view(*hidden.shape[:-1], -1)
