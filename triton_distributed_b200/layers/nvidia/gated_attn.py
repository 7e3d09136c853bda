"""Grouped-query attention with any head size, normed and partially rotated queries and keys, and a sigmoid gate per head.

It stands beside ``TP_Attn`` (128-wide heads, neox rotation, no gate). Heads are sharded over ranks (q, k, v, g by rows, o by
columns). Kernels by storage type and head size:

  one token per sequence    the 128-wide split-KV decode kernel, the gate in its merge; smaller heads are padded to 128 in the cache
  several                   the tcgen05 prefill attention on the cached keys and values (keys up to 256 wide), gate in its epilogue
  otherwise, and fp32       one warp per row (``ops.gqa_attention_plain``)
"""
from __future__ import annotations

import math
from typing import TYPE_CHECKING

import torch

from ... import ops
from .latent_attn import pad_heads, pad_matrix, pad_up

if TYPE_CHECKING:
    from ...models.config import GatedAttentionSpec, RotarySpec
    from ...models.kv_cache import HybridCache

DECODE_HEAD = 128  # head size of the decode kernel


def rotation_frequencies(rot: RotarySpec) -> torch.Tensor:
    """fp64 [dims / 2]: base ** (-2 i / dims), long wavelengths stretched as the scaling says."""
    f = float(rot.base) ** (-torch.arange(0, rot.dims, 2, dtype=torch.float64) / max(rot.dims, 1))
    sc = rot.scaling
    if sc is None:
        return f
    length = 2 * math.pi / f
    share = (sc.original / length - sc.low) / (sc.high - sc.low)
    mixed = (1 - share) * f / sc.factor + share * f
    return torch.where(length < sc.original / sc.high, f, torch.where(length > sc.original / sc.low, f / sc.factor, mixed))


def rotation_table(rot: RotarySpec, positions: int, device) -> torch.Tensor:
    """fp32 [positions, dims] with (cos, sin) of pair 0, of pair 1, ..."""
    angle = torch.arange(positions, dtype=torch.float64)[:, None] * rotation_frequencies(rot)[None]
    return torch.stack([torch.cos(angle), torch.sin(angle)], dim=-1).reshape(positions, rot.dims).to(torch.float32).to(device).contiguous()


class GatedAttention:

    def __init__(self, spec: GatedAttentionSpec, eps: float, world_size: int, dtype: torch.dtype):
        self.spec, self.eps = spec, eps
        self.heads, self.kv_heads = spec.heads // world_size, spec.kv_heads // world_size
        self.qk_in, self.v_in = pad_up(spec.dim), pad_up(spec.vdim)
        self.fast_decode = dtype != torch.float32 and max(self.qk_in, self.v_in) <= DECODE_HEAD
        self.fast_prefill = dtype != torch.float32 and self.qk_in <= 256
        self.dim, self.vdim = (DECODE_HEAD, DECODE_HEAD) if self.fast_decode else (self.qk_in, self.v_in)  # as cached
        self._ws: dict = {}

    def _init_parameters(self, get, width_pad: int, positions: int) -> None:
        """``get(name, rows=, cols=)`` returns this rank's part of a tensor of the mixer; `positions`: the longest sequence."""
        self.q_gain, self.k_gain = get("q.norm").contiguous(), get("k.norm").contiguous()
        o = get("o", cols=self.heads * self.spec.vdim)
        self.wo = pad_heads(o.t().contiguous(), self.heads, self.vdim, width_pad).t().contiguous()   # [width, heads * vdim]
        self.cos_sin = rotation_table(self.spec.rot, positions, o.device)

    def input_rows(self, get, width_pad: int) -> list[torch.Tensor]:
        """Rows of the fused input projection: q, k, v, gate logits."""
        H, G, s = self.heads, self.kv_heads, self.spec
        return [pad_heads(get("q", rows=H * s.dim), H, self.qk_in, width_pad), pad_heads(get("k", rows=G * s.dim), G, self.qk_in, width_pad),
                pad_heads(get("v", rows=G * s.vdim), G, self.v_in, width_pad), pad_matrix(get("g", rows=H), pad_up(H), width_pad)]

    def cache_pages(self) -> dict:
        return {"k": (self.kv_heads, self.dim), "v": (self.kv_heads, self.vdim)}

    @torch.no_grad()
    def partial_fwd(self, parts, cache: HybridCache, layer_idx: int, step: dict, out: torch.Tensor) -> torch.Tensor:
        """`parts`: this block's slices of the fused projection; `out` [B * S, width] receives this rank's partial sum. `step` carries
        ``bsz``, ``seqlen``, ``positions`` int32, ``slots``, ``kv_lens`` int32 [B] and ``kv_len`` (host: longest sequence after this step)."""
        q, k, v, gate = parts
        gate = gate[:, : self.heads]
        B, S = step["bsz"], step["seqlen"]
        kp, vp = cache.pages(layer_idx, "k"), cache.pages(layer_idx, "v")
        # the score scale goes into q while it is fp32
        q = ops.head_norm_rope(q, k, v, self.heads, self.kv_heads, self.spec.dim, self.q_gain, self.k_gain, self.eps, self.cos_sin,
                               step["positions"], step["slots"], kp, vp, q_scale=self.spec.scale)
        if S == 1 and self.fast_decode:
            splits = ops.choose_kv_splits(B, self.kv_heads, self.heads // self.kv_heads, cache.max_length)
            o = ops.decode_attention(q, kp, vp, step["kv_lens"], cache.block_table, 1.0, 0.0, splits, workspace=self._ws, gate=gate)
        elif S > 1 and self.fast_prefill:
            L = cache.blocks_per_seq * cache.page_size
            if "cu_q" not in step:  # the same for every layer of the step
                step["cu_q"] = torch.arange(0, (B + 1) * S, S, dtype=torch.int32, device=q.device)
                step["cu_k"] = torch.arange(0, (B + 1) * L, L, dtype=torch.int32, device=q.device)
            o = ops.prefill_attention(q, kp.view(-1, self.kv_heads, self.dim), vp.view(-1, self.kv_heads, self.vdim), step["cu_q"],
                                      step["cu_k"], S, step["kv_len"], 1.0, True, seqlens_k=step["kv_lens"], gate=gate)
        else:
            o = ops.gqa_attention_plain(q, kp, vp, step["kv_lens"], cache.block_table, S, 1.0, gate=gate)
        return ops.linear(o.view(B * S, -1), self.wo, out=out)
