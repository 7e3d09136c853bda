"""Latent attention block: keys and values of all heads are linear images of one cached vector per token.

The reference has no such layer; it stands beside ``TP_Attn`` and offers the same split into parameters, a native
``partial_fwd`` without the final reduction, and per-step tensors prepared by the model. Heads are sharded over ranks
(``q``, ``uk``, ``uv`` by rows, ``o`` by columns); the latent projection and its cache are replicated.

Two forms of the same product, chosen by how many tokens a sequence brings:
  absorbed   the products with the key and value maps are taken on the query side, the kernel attends the latents
             themselves (decode, short portions, the 32-bit mode)
  expanded   keys and transposed values of the whole prefix are computed from the cached latents with the tiled GEMM, then
             the tcgen05 prefill attention runs on them (prompts)

Sizes need no alignment in a checkpoint: the loader pads every row that a kernel reads with 16-byte accesses to a multiple of
eight elements; padding weights are zero, so padding columns carry zeros.
"""
from __future__ import annotations

import torch

from ... import ops
from .tp_mlp import shard_local


def pad_up(n: int, to: int = 8) -> int:
    return (n + to - 1) // to * to


def pad_matrix(w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    """`w` [r, c] in the top left corner of a zero matrix [rows, cols]."""
    if w.shape == (rows, cols):
        return w.contiguous()
    out = torch.zeros((rows, cols), dtype=w.dtype, device=w.device)
    out[: w.shape[0], : w.shape[1]] = w
    return out


def pad_vector(v: torch.Tensor, n: int) -> torch.Tensor:
    return pad_matrix(v[None, :], 1, n)[0].contiguous()


def pad_heads(w: torch.Tensor, heads: int, size: int, cols: int) -> torch.Tensor:
    """[heads * d, c] laid out head by head -> [heads * size, cols], every head padded to `size` rows."""
    d = w.shape[0] // heads
    out = torch.zeros((heads, size, cols), dtype=w.dtype, device=w.device)
    out[:, :d, : w.shape[1]] = w.view(heads, d, -1)
    return out.view(heads * size, cols)


class LatentAttention:

    # a sequence that brings at least this many tokens is attended in expanded form: expanding costs
    # kv * rank * (dim + vdim) per head once, the absorbed form reads latents of `rank` columns for every query token
    EXPAND_TOKENS = 32

    def __init__(self, rank: int = 0, world_size: int = 1, group=None):
        self.rank, self.world_size, self.group = rank, world_size, group

    def _init_parameters(self, *, uk, uv, o, latent_norm, sink, heads: int, dim: int, vdim: int, kv_rank: int, scale: float,
                         eps: float, width_pad: int):
        """From this rank's shards: uk [heads * dim, kv_rank], uv [heads * vdim, kv_rank], o [width, heads * vdim], sink [heads];
        `heads` counts the local heads. The query and latent projections belong to the layer's fused input projection
        (``input_rows``)."""
        self.heads, self.kv_rank, self.scale, self.eps = heads, kv_rank, float(scale), float(eps)
        self.dim, self.vdim, self.pitch = pad_up(dim), pad_up(vdim), pad_up(kv_rank)
        self.uk = pad_heads(uk, heads, self.dim, self.pitch)                         # [heads * dim, pitch]
        self.uk_t = self.uk.view(heads, self.dim, self.pitch).transpose(1, 2).contiguous()  # [heads, pitch, dim]
        self.uv = pad_heads(uv, heads, self.vdim, self.pitch)                        # [heads * vdim, pitch]
        self.wo = pad_heads(o.t().contiguous(), heads, self.vdim, width_pad).t().contiguous()  # [width, heads * vdim]
        self.latent_norm = pad_vector(latent_norm, self.pitch)
        self.sink = sink.to(torch.float32).contiguous()

    def input_rows(self, q: torch.Tensor, dkv: torch.Tensor, width_pad: int) -> list[torch.Tensor]:
        """Rows of the fused input projection that this block reads: queries, then the latent."""
        return [pad_heads(q, self.heads, self.dim, width_pad), pad_matrix(dkv, self.pitch, width_pad)]

    @torch.no_grad()
    def attend(self, q, kv_cache, layer_idx: int, step) -> torch.Tensor:
        """q [B * S, heads * dim] (column slice of the fused projection); the latents of these tokens are in the cache already.
        Returns [B * S, heads * vdim]. `step` carries ``bsz``, ``seqlen``, ``kv_lens`` int32 [B] and ``kv_len`` (host: longest
        sequence after this step, None inside a captured decode step)."""
        q3 = q.unflatten(1, (self.heads, self.dim))
        if self.expands(step["seqlen"], step["kv_len"], q.dtype):
            out = self._attend_expanded(q3, kv_cache, layer_idx, step)
        else:
            out = self._attend_absorbed(q3, kv_cache, layer_idx, step)
        return out.view(out.shape[0], -1)

    def expands(self, seqlen: int, kv_len: int | None, dtype: torch.dtype) -> bool:
        return seqlen >= self.EXPAND_TOKENS and kv_len is not None and dtype != torch.float32 and self.dim <= 256

    def _attend_absorbed(self, q3, kv_cache, layer_idx, step):
        cache = kv_cache.layer(layer_idx)
        qc = ops.head_linear(q3, self.uk_t)
        splits, rows = ops.choose_latent_splits(step["bsz"], step["seqlen"] * self.heads, step["kv_len"] or kv_cache.max_length)
        ctx = ops.latent_attention(qc, cache, step["kv_lens"], kv_cache.block_table, step["seqlen"], self.scale, self.sink, splits, rows)
        return ops.head_linear(ctx, self.uv.view(self.heads, self.vdim, self.pitch))

    def _attend_expanded(self, q3, kv_cache, layer_idx, step):
        B, S, kv = step["bsz"], step["seqlen"], step["kv_len"]
        kv8 = pad_up(kv)
        kv_cache.blank(layer_idx, kv, kv8)  # the rows in between are unused slots: masked, and must be finite
        c = kv_cache.rows(layer_idx, kv8)   # [B * kv8, pitch]
        k = ops.linear(c, self.uk)
        vt = ops.linear(self.uv, c)         # values already transposed: [heads * vdim, B * kv8]
        if "cu_q" not in step:  # the same for every layer of the step
            step["cu_q"] = torch.arange(0, (B + 1) * S, S, dtype=torch.int32, device=q3.device)
            step["cu_k"] = torch.arange(0, (B + 1) * kv8, kv8, dtype=torch.int32, device=q3.device)
        return ops.prefill_attention_vt(q3, k.view(B * kv8, self.heads, self.dim), vt.view(self.heads, self.vdim, B * kv8), step["cu_q"],
                                        step["cu_k"], step["kv_lens"], S, self.scale, True, self.sink)

    @torch.no_grad()
    def partial_fwd(self, q, kv_cache, layer_idx: int, step, out: torch.Tensor | None = None) -> torch.Tensor:
        """Attention and output projection without the reduction over ranks."""
        return ops.linear(self.attend(q, kv_cache, layer_idx, step), self.wo, out=out)


__all__ = ["LatentAttention", "pad_heads", "pad_matrix", "pad_up", "pad_vector", "shard_local"]
