"""Likosun decoder: parallel layers with gated sublayers, latent attention, squared-relu feed-forward and a depth average.

Layer i, on the fp32 stream x (X_0 = embedding, scaled):

    h       = layernorm(x; norm1)
    X_{i+1} = x + m * ( sigmoid(rg1 h + rg1.b) * attention(h)  +  sigmoid(rg2 h + rg2.b) * feedforward(h) )
    x       = sum_{j <= i+1} dwa[j] * X_j

All matrices that read h form ONE GEMM per layer: [q | latent | up | rg1 | rg2]. After it: one launch for the latent norm, the
cache write and the activation; attention; the two output projections; and one launch for everything between the last GEMM
of a layer and the first of the next (gates, residual, depth average, layer norm). The stream and the states X_j stay fp32.

The interface is that of ``Qwen3`` (``set_fwd``, ``init_triton_dist_AR_ctx``, ``inference``, ``finalize``), so ``Engine`` serves both.
Forward mode: ``triton_dist_AR`` (native kernels, replicated activations, one all-reduce per layer over both sublayers' partial
sums). Storage types: bf16 / f16, or fp32 with every product in true fp32.
"""
from __future__ import annotations

import torch

from .. import ops
from ..kernels.allreduce import AllReduceMethod
from ..layers.nvidia.latent_attn import LatentAttention, pad_matrix, pad_up, pad_vector, shard_local
from .config import LayerSpec, LikosunConfig, ModelConfig
from .kv_cache import LatentCache
from .weights import RandomSource, SafetensorsSource, WeightSource


class LikosunLayer:

    def __init__(self, layer_idx: int, rank: int, world_size: int, group):
        self.layer_idx, self.rank, self.world_size = layer_idx, rank, world_size
        self.attn = LatentAttention(rank, world_size, group)

    def load(self, src: WeightSource, arch: LikosunConfig, spec: LayerSpec) -> None:
        p, m, w = f"l{self.layer_idx}.", spec.mixer, self.world_size
        P = pad_up(arch.hidden_size)
        heads = m.heads // w
        qs, vs = shard_local(m.heads * m.dim, w, self.rank), shard_local(m.heads * m.vdim, w, self.rank)
        self.attn._init_parameters(
            uk=src.get(p + "mix.uk", rows=qs), uv=src.get(p + "mix.uv", rows=vs), o=src.get(p + "mix.o", cols=vs),
            latent_norm=src.get(p + "mix.dkv.norm"), sink=src.get(p + "mix.sink", rows=shard_local(m.heads, w, self.rank)),
            heads=heads, dim=m.dim, vdim=m.vdim, kv_rank=m.kv_rank, scale=m.scale, eps=arch.norm_eps, width_pad=P)
        rows = self.attn.input_rows(src.get(p + "mix.q", rows=qs), src.get(p + "mix.dkv"), P)
        self.inter = self.inter_pad = 0
        self.down = self.gate2_b = None
        if spec.mlp is not None:
            fs = shard_local(spec.mlp.ff, w, self.rank)
            self.inter = spec.mlp.ff // w
            self.inter_pad = pad_up(self.inter)
            rows.append(pad_matrix(src.get(p + "mlp.up", rows=fs), self.inter_pad, P))
            self.down = pad_matrix(src.get(p + "mlp.down", cols=fs), P, self.inter_pad)
        rows.append(pad_matrix(src.get(p + "rg1"), P, P))
        self.gate1_b = pad_vector(src.get(p + "rg1.b"), P)
        if spec.mlp is not None:
            rows.append(pad_matrix(src.get(p + "rg2"), P, P))
            self.gate2_b = pad_vector(src.get(p + "rg2.b"), P)
        self.w_in = torch.cat(rows, dim=0).contiguous()
        self.splits = [r.shape[0] for r in rows]
        self.norm_w, self.norm_b = pad_vector(src.get(p + "norm1"), P), pad_vector(src.get(p + "norm1.b"), P)
        self.depth_weights = src.get(p + "dwa").to(torch.float32).contiguous()

    def sublayers(self, h: torch.Tensor, kv_cache: LatentCache, step: dict):
        """h [T, P] -> (partial sums [2 or 1, T, P] of the sublayers, gate logits of the mixer, of the feed-forward or None)."""
        proj = ops.linear(h, self.w_in)
        parts = proj.split(self.splits, dim=1)
        q, latent, gate1 = parts[0], parts[1], parts[-1] if self.down is None else parts[-2]
        up, gate2 = (None, None) if self.down is None else (parts[2], parts[-1])
        act = ops.latent_prep(latent, self.attn.latent_norm, kv_cache.layer(self.layer_idx), step["slots"], self.attn.kv_rank,
                              self.attn.eps, up)
        out = torch.empty((1 if self.down is None else 2, *h.shape), dtype=h.dtype, device=h.device)
        self.attn.partial_fwd(q, kv_cache, self.layer_idx, step, out=out[0])
        if self.down is not None:
            ops.linear(act, self.down, out=out[1])
        return out, gate1, gate2


class Likosun:

    dtypes = (torch.bfloat16, torch.float16, torch.float32)
    library_subset = "likosun"   # the native kernels that one GPU needs (``build.SUBSETS``)

    def __init__(self, model_config: ModelConfig, group=None, source: WeightSource | None = None):
        self.model_config, self.group = model_config, group
        self.rank, self.world_size = model_config.rank, model_config.world_size
        self.dtype = model_config.dtype
        self.arch = model_config.arch()
        if not isinstance(self.arch, LikosunConfig):
            raise ValueError(f"{model_config.model_name} is not a Likosun model")
        for spec in self.arch.layers:
            if spec.mixer.heads % self.world_size or (spec.mlp is not None and spec.mlp.ff % self.world_size):
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
        self.head = pad_matrix(source.get("head"), pad_up(a.vocab_size), P)
        self.norm_w, self.norm_b = pad_vector(source.get("final.norm"), P), pad_vector(source.get("final.norm.b"), P)
        self.layers = []
        for i, spec in enumerate(a.layers):
            layer = LikosunLayer(i, self.rank, self.world_size, self.group)
            layer.load(source, a, spec)
            self.layers.append(layer)
        self.num_layers = a.num_hidden_layers

    def make_cache(self, batch_size: int, max_length: int | None = None) -> LatentCache:
        return LatentCache([layer.attn.pitch for layer in self.layers], batch_size, max_length or self.max_length, self.dtype,
                           device=self.device)

    # ------------------------------------------------------------------ modes and contexts
    def set_fwd(self, mode: str = "triton_dist_AR") -> None:
        if mode != "triton_dist_AR":
            raise ValueError(f"Likosun runs in mode 'triton_dist_AR' (native kernels, replicated activations), not {mode!r}")
        self.mode = mode

    def init_triton_dist_AR_ctx(self, max_M: int, ar_method: AllReduceMethod | None = None) -> None:
        self.ar_method = ar_method
        if self.world_size > 1 and self.ar_ctx is None:
            from ..kernels.nvidia import create_allreduce_ctx
            self.ar_ctx = create_allreduce_ctx(64 << 20, self.rank, self.world_size, self.world_size)
        # pre-size the split-K scratch so that nothing allocates inside a CUDA graph capture
        widest = max([self.head.shape[0]] + [layer.w_in.shape[0] for layer in self.layers])
        ops.reserve_skinny_scratch(torch.device("cuda", torch.cuda.current_device()),
                                   pad_up(min(max_M, 256), 16) * pad_up(widest, 128), pad_up(widest, 128) // 128)

    def finalize(self) -> None:
        if self.ar_ctx:
            self.ar_ctx.finalize()
        self.ar_ctx = None

    # ------------------------------------------------------------------ forward
    @torch.no_grad()
    def inference(self, input_ids: torch.Tensor, position_ids: torch.Tensor, kv_cache: LatentCache, wo_lm_head: bool = False,
                  kv_len: int | None = None) -> torch.Tensor:
        """input_ids / position_ids [B, S]: the next S tokens of every sequence, at consecutive positions. Returns fp32 logits
        [B, 1, V] of the last position, or the normed hidden states [B, S, P] with ``wo_lm_head`` (see ``lm_logits``). `kv_len`:
        the longest sequence after this step, when the host knows it (read from the device otherwise; one-token steps do not
        need it and never synchronise)."""
        bsz, S = input_ids.shape
        a = self.arch
        if S > 1 and kv_len is None:
            kv_len = int(position_ids.max()) + 1
        step = {"bsz": bsz, "seqlen": S, "kv_len": kv_len if S > 1 else None, "slots": kv_cache.slots(position_ids),
                "kv_lens": (position_ids[:, -1] + 1).to(torch.int32)}
        T = bsz * S
        states = torch.empty((max(self.num_layers, 1), T, self.pitch), dtype=torch.float32, device=self.device)
        first = self.layers[0]
        x, h = ops.embed_norm(input_ids, self.embed, a.embedding_scale, a.hidden_size, first.norm_w, first.norm_b, a.norm_eps, True,
                              state0=states[0])
        for i, layer in enumerate(self.layers):
            out, gate1, gate2 = layer.sublayers(h, kv_cache, step)
            if self.world_size > 1:
                from ..kernels.nvidia import all_reduce
                out = all_reduce(out.view(-1, self.pitch), None, self.ar_method, self.ar_ctx).view(out.shape)
            last = i + 1 == self.num_layers
            gain, bias = (self.norm_w, self.norm_b) if last else (self.layers[i + 1].norm_w, self.layers[i + 1].norm_b)
            h = ops.residual_norm(x, a.hidden_size, a.residual_mult, out[0], gate1, layer.gate1_b,
                                  out[1] if gate2 is not None else None, gate2, layer.gate2_b, states=states,
                                  weights=layer.depth_weights, keep=not last, gain=gain, bias=bias, eps=a.norm_eps, center=True)
            if self.layer_taps is not None:
                self.layer_taps.append(x[:, : a.hidden_size].clone())
        hidden = h.view(bsz, S, self.pitch)
        return hidden if wo_lm_head else self.lm_logits(hidden[:, -1:, :])

    def lm_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        """fp32 logits [B, n, V] of normed hidden states [B, n, P]. (The head is replicated over ranks.)"""
        rows = hidden.reshape(-1, self.pitch).contiguous()
        logits = ops.linear(rows, self.head)[:, : self.arch.vocab_size]
        return logits.float().view(*hidden.shape[:-1], -1)
