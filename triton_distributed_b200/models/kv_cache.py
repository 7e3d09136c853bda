"""Paged caches: keys and values head-sharded over the tensor-parallel ranks, one latent row per token and layer, or pages and
recurrent states side by side.

Same interface as the reference's dense cache (``python/triton_dist/models/kv_cache.py:29-66``:
``update_kv_cache``, ``rand_fill_kv_cache``, ``inc_offset``, ``clear``, ``get_kv_len``) but stored as pages
``[layers, num_blocks, page, kv_heads / world, head_dim]`` with a block table, which is the layout the
decode-attention kernel reads. Sequence b owns blocks ``b * blocks_per_seq ...`` so the table is static
and a decode step can be captured in a CUDA graph. ``PagedCache`` owns the pages' bookkeeping (slots, block table,
offsets), the subclasses own what a page holds.
"""
from __future__ import annotations

import dataclasses

import torch


class PagedCache:

    def __init__(self, num_layers: int, batch_size: int, max_length: int, dtype, page_size: int = 64, device="cuda") -> None:
        self.num_layers, self.batch_size, self.max_length = num_layers, batch_size, max_length
        self.dtype, self.page_size = dtype, page_size
        self.blocks_per_seq = (max_length + page_size - 1) // page_size
        self.num_blocks = batch_size * self.blocks_per_seq
        self.kv_offset = torch.zeros(batch_size, dtype=torch.int32, device=device)
        self.block_table = torch.arange(self.num_blocks, dtype=torch.int32, device=device).view(batch_size, self.blocks_per_seq)

    def slots(self, positions: torch.Tensor) -> torch.Tensor:
        """Flat slot index (block * page + offset) of token position [B, S] of every sequence -> int64 [B*S]."""
        B, S = positions.shape
        base = torch.arange(B, device=positions.device, dtype=torch.int64)[:, None] * (self.blocks_per_seq * self.page_size)
        return (base + positions.to(torch.int64)).reshape(-1)

    def inc_offset(self, n: int = 1) -> None:
        self.kv_offset += n

    def clear(self) -> None:
        self.kv_offset.zero_()

    def save_state(self):
        """What a decode step changes beyond the slots it writes (running a step again would change it again); None here: pages
        are written at their slot, whatever was there."""
        return None

    def restore_state(self, saved) -> None:
        """Back to ``save_state``'s result, in place."""

    def get_kv_len(self) -> torch.Tensor:
        return self.kv_offset


class KV_Cache(PagedCache):

    def __init__(self, num_layers: int = 32, batch_size: int = 1, max_length: int = 32 * 1024, kv_heads: int = 8,
                 head_dim: int = 128, dtype=torch.bfloat16, world_size: int = 8, page_size: int = 64,
                 device="cuda") -> None:
        super().__init__(num_layers, batch_size, max_length, dtype, page_size, device)
        self.kv_heads, self.head_dim, self.world_size = kv_heads, head_dim, world_size
        self.local_kv_heads = max(1, kv_heads // world_size)
        shape = (num_layers, self.num_blocks, page_size, self.local_kv_heads, head_dim)
        self.k_cache = torch.zeros(shape, device=device, dtype=dtype)
        self.v_cache = torch.zeros(shape, device=device, dtype=dtype)

    def layer(self, layer_idx: int):
        """(k pages, v pages) of one layer: [num_blocks, page, kv_heads_local, head_dim]."""
        return self.k_cache[layer_idx], self.v_cache[layer_idx]

    def update_kv_cache(self, new_k: torch.Tensor, new_v: torch.Tensor, layer_idx: int):
        """Append [B, S, kv_heads_local, D] at the current offsets (the fused rope kernel normally does this)."""
        B, S = new_k.shape[:2]
        pos = self.kv_offset[:, None].to(torch.int64) + torch.arange(S, device=new_k.device)[None, :]
        sl = self.slots(pos)
        self.k_cache[layer_idx].view(-1, self.local_kv_heads, self.head_dim)[sl] = new_k.reshape(-1, self.local_kv_heads, self.head_dim)
        self.v_cache[layer_idx].view(-1, self.local_kv_heads, self.head_dim)[sl] = new_v.reshape(-1, self.local_kv_heads, self.head_dim)
        return self.k_cache[layer_idx], self.v_cache[layer_idx], self.kv_offset

    def rand_fill_kv_cache(self, offset: int) -> None:
        self.k_cache.copy_(torch.rand_like(self.k_cache) / 10)
        self.v_cache.copy_(torch.rand_like(self.v_cache) / 10)
        self.kv_offset.fill_(offset)


class LatentCache(PagedCache):
    """Latent attention's cache: layer i keeps one row of ``widths[i]`` elements per token (shared by all heads, so it is
    replicated over tensor-parallel ranks), as pages ``[num_blocks, page, widths[i]]``."""

    def __init__(self, widths: list[int], batch_size: int, max_length: int, dtype=torch.bfloat16, page_size: int = 64,
                 device="cuda") -> None:
        super().__init__(len(widths), batch_size, max_length, dtype, page_size, device)
        self.c_cache = [torch.zeros((self.num_blocks, page_size, w), device=device, dtype=dtype) for w in widths]

    def layer(self, layer_idx: int) -> torch.Tensor:
        """Pages of one layer: [num_blocks, page, width]."""
        return self.c_cache[layer_idx]

    def rows(self, layer_idx: int, count: int) -> torch.Tensor:
        """The first `count` latent rows of every sequence as one matrix [batch * count, width] (a sequence's pages are
        consecutive; a view where the rows of the batch are, else a copy)."""
        c = self.c_cache[layer_idx].view(self.batch_size, self.blocks_per_seq * self.page_size, -1)[:, :count]
        return c.reshape(self.batch_size * count, -1)

    def blank(self, layer_idx: int, start: int, stop: int) -> None:
        """Zero the unused rows [start, stop) of every sequence."""
        if stop > start:
            self.c_cache[layer_idx].view(self.batch_size, self.blocks_per_seq * self.page_size, -1)[:, start:stop].zero_()


class HybridCache(PagedCache):
    """Layers of different kinds: some keep rows per token in pages, some a state of fixed size per sequence, some both.

    ``layers[i]`` maps names to shapes: ``pages`` name -> the shape of a token's row, stored ``[num_blocks, page, *row]`` in the
    cache's type; ``states`` name -> (shape, type), stored ``[batch, *shape]``. States start at zero: ``clear`` zeroes them (pages need
    not be), in place, so that a captured decode step keeps its addresses."""

    @dataclasses.dataclass
    class Layer:
        pages: dict[str, tuple[int, ...]] = dataclasses.field(default_factory=dict)
        states: dict[str, tuple[tuple[int, ...], torch.dtype]] = dataclasses.field(default_factory=dict)

    def __init__(self, layers: list["HybridCache.Layer"], batch_size: int, max_length: int, dtype=torch.bfloat16, page_size: int = 64,
                 device="cuda") -> None:
        super().__init__(len(layers), batch_size, max_length, dtype, page_size, device)
        self._pages = [{n: torch.zeros((self.num_blocks, page_size, *row), device=device, dtype=dtype) for n, row in layer.pages.items()}
                       for layer in layers]
        self._states = [{n: torch.zeros((batch_size, *shape), device=device, dtype=dt) for n, (shape, dt) in layer.states.items()}
                        for layer in layers]

    def pages(self, layer_idx: int, name: str) -> torch.Tensor:
        return self._pages[layer_idx][name]

    def state(self, layer_idx: int, name: str) -> torch.Tensor:
        return self._states[layer_idx][name]

    def _all_states(self) -> list[torch.Tensor]:
        return [t for layer in self._states for t in layer.values()]

    def clear(self) -> None:
        super().clear()
        for t in self._all_states():
            t.zero_()

    def save_state(self):
        return [t.clone() for t in self._all_states()]

    def restore_state(self, saved) -> None:
        for t, old in zip(self._all_states(), saved):
            t.copy_(old)
