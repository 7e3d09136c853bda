"""Mixers with a matrix-valued memory per head: decayed outer products (``WkvMixer``) and the gated delta rule (``GatedDelta``).

Heads are sharded over ranks; what a sequence carries from call to call (the memory in fp32, the previous token, the last inputs of
the convolution) lives in the cache's states. The same kernels serve prompts, portions and single tokens. Heads are padded to
multiples of eight channels with zero weights.
"""
from __future__ import annotations

from typing import TYPE_CHECKING

import torch

from ... import ops
from .latent_attn import pad_heads, pad_matrix, pad_up, pad_vector

if TYPE_CHECKING:
    from ...models.config import GatedDeltaSpec, WkvSpec
    from ...models.kv_cache import HybridCache


def _head_vector(v: torch.Tensor, heads: int, size: int) -> torch.Tensor:
    """[heads * d] (or [heads, d]) -> fp32 [heads * size], every head padded with zeros."""
    return pad_matrix(v.reshape(heads, -1).to(torch.float32), heads, size).reshape(-1).contiguous()


class WkvMixer:

    INPUTS = "rkvgw"   # the token-shifted mixes, in the order of the fused projection

    def __init__(self, spec: WkvSpec, eps: float, world_size: int):
        self.spec, self.eps = spec, eps
        self.heads, self.dim = spec.heads // world_size, pad_up(spec.dim)

    def _init_parameters(self, get, width_pad: int) -> None:
        """``get(name, rows=, cols=)`` returns this rank's part of a tensor of the mixer."""
        H, D, N = self.heads, self.dim, self.heads * self.spec.dim
        self.mu = torch.stack([pad_vector(get(f"mu.{s}"), width_pad) for s in self.INPUTS]).contiguous()
        w1 = get("w1")
        self.rank = pad_up(w1.shape[0])
        mats = [pad_heads(get(s, rows=N), H, D, width_pad) for s in "rkvg"] + [w1]
        mats = [pad_matrix(m, pad_up(m.shape[0], 128), width_pad) for m in mats]
        self.rows = [m.shape[0] for m in mats]
        self.w_in = torch.cat(mats).contiguous()
        self.w2 = pad_heads(get("w2", rows=N), H, D, self.rank)   # [heads * dim, rank]
        self.w0, self.gain = _head_vector(get("w0", rows=N), H, D), _head_vector(get("norm", rows=N), H, D)
        self.u = _head_vector(get("u", rows=H), H, D)
        self.wo = pad_heads(get("o", cols=N).t().contiguous(), H, D, width_pad).t().contiguous()

    def cache_states(self, dtype: torch.dtype) -> dict:
        return {"last": ((self.mu.shape[1],), dtype), "memory": ((self.heads, self.dim, self.dim), torch.float32)}

    @torch.no_grad()
    def partial_fwd(self, h: torch.Tensor, cache: HybridCache, layer_idx: int, out: torch.Tensor) -> torch.Tensor:
        """h [B * S, width] -> this rank's partial sum in `out`."""
        mixes = ops.token_mix(h, self.mu, cache.state(layer_idx, "last"))
        r, k, v, gate, low = ops.linear_groups(mixes, self.w_in, self.rows).split(self.rows, dim=1)
        N = self.heads * self.dim
        z = ops.tanh_linear(low[:, : self.rank], self.w2)
        o = ops.wkv(r[:, :N], k[:, :N], v[:, :N], z, gate[:, :N], self.w0, self.u, self.gain, cache.state(layer_idx, "memory"), self.spec.dim,
                    self.spec.dim, self.eps)
        return ops.linear(o, self.wo, out=out)


class GatedDelta:

    def __init__(self, spec: GatedDeltaSpec, eps: float, world_size: int):
        self.spec, self.eps = spec, eps
        self.heads, self.kv_heads = spec.heads // world_size, spec.kv_heads // world_size
        self.dim, self.vdim = pad_up(spec.dim), pad_up(spec.vdim)

    def _init_parameters(self, get, width_pad: int) -> None:
        H, G, s = self.heads, self.kv_heads, self.spec
        taps = [pad_heads(get("q.conv", rows=G * s.dim), G, self.dim, s.conv), pad_heads(get("k.conv", rows=G * s.dim), G, self.dim, s.conv),
                pad_heads(get("v.conv", rows=H * s.vdim), H, self.vdim, s.conv)]
        self.sizes = [t.shape[0] for t in taps]                                 # channels of q, k, v
        self.taps = torch.cat(taps).to(torch.float32).t().contiguous()          # [conv, channels]
        self.a_log, self.dt_bias = (get(n, rows=H).to(torch.float32).contiguous() for n in ("A_log", "dt_bias"))
        self.gain = pad_vector(get("norm").to(torch.float32), self.vdim)
        o = get("o", cols=H * s.vdim)
        self.wo = pad_heads(o.t().contiguous(), H, self.vdim, width_pad).t().contiguous()

    def input_rows(self, get, width_pad: int) -> list[torch.Tensor]:
        """Rows of the fused input projection: [q | k | v] (one convolution), step-size logits, decay logits, gate."""
        H, G, s = self.heads, self.kv_heads, self.spec
        qkv = torch.cat([pad_heads(get("q", rows=G * s.dim), G, self.dim, width_pad), pad_heads(get("k", rows=G * s.dim), G, self.dim, width_pad),
                         pad_heads(get("v", rows=H * s.vdim), H, self.vdim, width_pad)])
        return [qkv, pad_matrix(get("b", rows=H), pad_up(H), width_pad), pad_matrix(get("a", rows=H), pad_up(H), width_pad),
                pad_heads(get("g", rows=H * s.vdim), H, self.vdim, width_pad)]

    def cache_states(self, dtype: torch.dtype) -> dict:
        return {"inputs": ((self.spec.conv - 1, sum(self.sizes)), dtype), "memory": ((self.heads, self.dim, self.vdim), torch.float32)}

    @torch.no_grad()
    def partial_fwd(self, parts, cache: HybridCache, layer_idx: int, out: torch.Tensor) -> torch.Tensor:
        """`parts`: this block's slices of the fused projection; `out` receives this rank's partial sum."""
        qkv, b, a, gate = parts
        q, k, v = ops.short_conv(qkv, self.taps, cache.state(layer_idx, "inputs")).split(self.sizes, dim=1)
        o = ops.gated_delta(q, k, v, a[:, : self.heads], b[:, : self.heads], gate, self.a_log, self.dt_bias, self.gain,
                            cache.state(layer_idx, "memory"), self.spec.dim, self.spec.vdim, self.eps)
        return ops.linear(o, self.wo, out=out)
