"""Single-GPU hot ops backed by the sm_100a kernels in ``csrc/kernels``.

Every function here launches native code on the current CUDA stream and fails loudly when the
native library or a GPU is missing: there is no silent PyTorch fallback (the CPU reference
semantics live in :mod:`triton_distributed_b200.ref`).

Replaces in the reference: cuBLAS ``F.linear``, ``flashinfer.norm.rmsnorm``,
``flashinfer.apply_rope_with_cos_sin_cache_inplace``, ``act_fn(gate) * up`` and the softmax/topk router
(``layers/nvidia/tp_mlp.py:159-186``, ``tp_attn.py:60-75,159-195``, ``kernels/nvidia/moe_reduce_rs.py:172-189``).
"""
from __future__ import annotations

import ctypes
import dataclasses
import functools
import os

import torch

from . import _lib
from ._lib import c_float, dtype_code, ptr, stream_ptr

# number of native kernel launches issued through this module (bench.py reports it)
launch_count = 0


def _count(n: int = 1) -> None:
    global launch_count
    launch_count += n


def _check_2d(t: torch.Tensor, name: str) -> None:
    if t.dim() != 2 or t.stride(1) != 1:
        raise ValueError(f"{name} must be a 2-D tensor with unit inner stride, got shape {tuple(t.shape)} stride {t.stride()}")


def gemm(a: torch.Tensor, b: torch.Tensor, out: torch.Tensor | None = None, max_ctas: int = 0) -> torch.Tensor:
    """``a[M,K] @ b[N,K].T`` on the persistent tcgen05 kernel (128x256x64 tiles, fp32 accumulation)."""
    _lib.require_cuda()
    _check_2d(a, "a"), _check_2d(b, "b")
    M, K = a.shape
    N = b.shape[0]
    if b.shape[1] != K or a.dtype != b.dtype:
        raise ValueError("gemm: shape/dtype mismatch")
    if out is None:
        out = torch.empty((M, N), dtype=a.dtype, device=a.device)
    _lib.call("b200_gemm", ptr(a), ptr(b), ptr(out), M, N, K, a.stride(0), b.stride(0), out.stride(0),
              dtype_code(a.dtype), max_ctas, stream_ptr())
    _count()
    return out


class _SkinnyScratch:
    """Per-device split-K scratch shared by all skinny GEMM calls of a stream (each call re-zeroes it). Buffers that were
    outgrown stay allocated: a captured CUDA graph may hold their addresses."""

    def __init__(self):
        self.bufs: dict[int, tuple[torch.Tensor, torch.Tensor]] = {}
        self.outgrown: list[tuple[torch.Tensor, torch.Tensor]] = []

    def get(self, device: torch.device, floats: int, tiles: int):
        key = device.index if device.index is not None else torch.cuda.current_device()
        cur = self.bufs.get(key)
        if cur is None or cur[0].numel() < floats or cur[1].numel() < tiles:
            if cur is not None:
                torch.cuda.synchronize()
                self.outgrown.append(cur)
            nf = max(floats, 4 << 20, 0 if cur is None else cur[0].numel())
            nt = max(tiles, 4096, 0 if cur is None else cur[1].numel())
            cur = (torch.zeros(nf, dtype=torch.float32, device=device), torch.zeros(nt, dtype=torch.int32, device=device))
            self.bufs[key] = cur
        return cur


_skinny_scratch = _SkinnyScratch()


def reserve_skinny_scratch(device, floats: int, tiles: int) -> None:
    """Pre-size the split-K scratch (call before CUDA-graph capture so no allocation happens inside)."""
    _skinny_scratch.get(torch.device(device), floats, tiles)


class SkinnyEpilogue(ctypes.Structure):
    """Mirror of ``b200::SkinnyEpilogue`` (csrc/kernels/gemm_skinny_sm100.cu): what the decode GEMM does with a
    finished tile besides storing it. Build one with ``skinny_row_scale``, ``skinny_qkv_heads`` or ``skinny_residual``."""
    _fields_ = [("kind", ctypes.c_int), ("sumsq_in", ctypes.c_void_p), ("scale_dim", ctypes.c_float), ("eps", ctypes.c_float),
                ("Hq", ctypes.c_int), ("Hkv", ctypes.c_int), ("positions", ctypes.c_void_p), ("slots", ctypes.c_void_p),
                ("cos_sin", ctypes.c_void_p), ("q_gamma", ctypes.c_void_p), ("k_gamma", ctypes.c_void_p),
                ("q_out", ctypes.c_void_p), ("k_cache", ctypes.c_void_p), ("v_cache", ctypes.c_void_p),
                ("head_eps", ctypes.c_float), ("residual_in", ctypes.c_void_p), ("residual_out", ctypes.c_void_p),
                ("next_gamma", ctypes.c_void_p), ("scaled_out", ctypes.c_void_p), ("sumsq_out", ctypes.c_void_p)]

    def __init__(self, **kw):
        super().__init__()
        self._keep = []  # tensors referenced by raw pointers stay alive as long as the description does
        for k, v in kw.items():
            if isinstance(v, torch.Tensor):
                self._keep.append(v)
                v = v.data_ptr()
            setattr(self, k, v)


def _dptr(t: torch.Tensor | None):
    return None if t is None else t.data_ptr()


def skinny_row_scale(sumsq: torch.Tensor, dim: int, eps: float, base: SkinnyEpilogue | None = None) -> SkinnyEpilogue:
    """Epilogue ``out[m, :] *= rsqrt(sumsq[m] / dim + eps)``: the RMSNorm of the GEMM's input when its producer already
    applied the gain. `sumsq` fp32 [>= M]. Combines with another epilogue when `base` is given."""
    ep = base if base is not None else SkinnyEpilogue(kind=0)
    ep.sumsq_in, ep.scale_dim, ep.eps = sumsq.data_ptr(), float(dim), float(eps)
    ep._keep.append(sumsq)
    return ep


def skinny_qkv_heads(positions: torch.Tensor, slots: torch.Tensor | None, cos_sin: torch.Tensor, num_q_heads: int,
                     num_kv_heads: int, q_out: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                     q_gamma: torch.Tensor | None, k_gamma: torch.Tensor | None, eps: float) -> SkinnyEpilogue:
    """Epilogue of the fused qkv projection (head dim 128): per-head RMSNorm of q / k, neox RoPE, q to ``q_out``
    [M, Hq, 128] and k / v into the caches viewed as [slots, Hkv, 128] at ``slots`` (int64 [M], None = identity)."""
    if positions.dtype != torch.int32 or cos_sin.dtype != torch.float32 or (slots is not None and slots.dtype != torch.int64):
        raise ValueError("positions must be int32, slots int64 and cos_sin float32")
    ep = SkinnyEpilogue(kind=1, Hq=num_q_heads, Hkv=num_kv_heads, positions=positions, cos_sin=cos_sin, q_out=q_out,
                        k_cache=k_cache, v_cache=v_cache, head_eps=float(eps))
    for name, t in (("slots", slots), ("q_gamma", q_gamma), ("k_gamma", k_gamma)):
        if t is not None:
            setattr(ep, name, t.data_ptr())
            ep._keep.append(t)
    return ep


def skinny_residual(residual: torch.Tensor, sumsq_out: torch.Tensor | None, next_gamma: torch.Tensor | None = None,
                    scaled_out: torch.Tensor | None = None, residual_out: torch.Tensor | None = None) -> SkinnyEpilogue:
    """Epilogue ``h = out + residual``: writes h to ``residual_out`` (default: in place), ``h * next_gamma`` to
    ``scaled_out`` and adds ``sum(h^2)`` per token to ``sumsq_out`` (fp32, zeroed by the caller once per step)."""
    ro = residual if residual_out is None else residual_out
    ep = SkinnyEpilogue(kind=2, residual_in=residual, residual_out=ro)
    for name, t in (("sumsq_out", sumsq_out), ("next_gamma", next_gamma), ("scaled_out", scaled_out)):
        if t is not None:
            setattr(ep, name, t.data_ptr())
            ep._keep.append(t)
    return ep


def gemm_skinny(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor | None = None, swiglu: bool = False,
                splits: int = 0, epilogue: SkinnyEpilogue | None = None) -> torch.Tensor | None:
    """Decode GEMM for ``M <= 256`` tokens: ``x[M,K] @ w[N,K].T`` with the weights streamed once.

    With ``swiglu=True``, ``w`` is ``[gate; up]`` (2*I rows) and the result is ``silu(x gate^T) * (x up^T)`` [M, I].
    With ``epilogue`` (M <= 16) the finished tiles go through a fused epilogue instead of (or before) the plain store;
    the qkv-heads and residual kinds write their own outputs and return None unless ``out`` is given. The models do
    not use the epilogues: a decode step chained through them (5 launches per layer instead of 9) measured 15.6 ms
    against 13.8 ms on one B200 (Qwen3-32B, batch 8), because the epilogue runs on the one CTA that finishes each tile,
    on the critical path, while the separate small kernels spread over the machine and start early under programmatic
    dependent launch. They remain available for callers whose chain is launch-bound (no PDL, no graph).
    """
    _lib.require_cuda()
    _check_2d(x, "x"), _check_2d(w, "w")
    M, K = x.shape
    n_rows = w.shape[0]
    N = n_rows // 2 if swiglu else n_rows
    own_output = epilogue is not None and epilogue.kind in (1, 2)
    if out is None and not own_output:
        out = torch.empty((M, N), dtype=x.dtype, device=x.device)
    lib = _lib.load()
    lib.b200_gemm_skinny_scratch_floats.restype = ctypes.c_longlong
    floats = lib.b200_gemm_skinny_scratch_floats(M, N, 1 if swiglu else 0)
    tiles = (N + 127) // 128
    scratch, tickets = _skinny_scratch.get(x.device, floats, tiles)
    ldc = out.stride(0) if out is not None else (epilogue._keep[0].stride(0) if epilogue.kind == 2 else N)
    if epilogue is None:
        _lib.call("b200_gemm_skinny", ptr(x), ptr(w), ptr(out), M, N, K, x.stride(0), w.stride(0), ldc,
                  1 if swiglu else 0, dtype_code(x.dtype), ptr(scratch), ptr(tickets), splits, stream_ptr())
    else:
        if ctypes.sizeof(SkinnyEpilogue) != lib.b200_gemm_skinny_epilogue_bytes():
            raise RuntimeError("SkinnyEpilogue layout differs between the Python binding and the native library")
        _lib.call("b200_gemm_skinny_fused", ptr(x), ptr(w), ptr(out), M, N, K, x.stride(0), w.stride(0), ldc,
                  1 if swiglu else 0, dtype_code(x.dtype), ptr(scratch), ptr(tickets), ctypes.byref(epilogue), stream_ptr())
    _count()
    return out


def linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``x @ w.T`` for any leading shape: the skinny kernel for <= 256 rows, else the tiled one; fp32 has its own kernel."""
    lead = x.shape[:-1]
    x2 = x.reshape(-1, x.shape[-1])
    o2 = out.reshape(-1, w.shape[0]) if out is not None else None
    if x2.dtype == torch.float32:
        y = gemm_f32(x2, w, o2)
    else:
        y = gemm_skinny(x2, w, o2) if x2.shape[0] <= 256 else gemm(x2, w, o2)
    return y.reshape(*lead, w.shape[0])


_GROUP_TILE = 128  # rows of a decode-GEMM tile


def linear_groups(x: torch.Tensor, w: torch.Tensor, rows: list[int]) -> torch.Tensor:
    """Several inputs, each with its own rows of one weight matrix: x [T, G, K], w [sum(rows), K] with ``rows[g]`` rows (multiples
    of 128) for input g; returns ``[x_0 @ w_0.T | x_1 @ w_1.T | ...]`` [T, sum(rows)]. Up to 256 tokens are one launch."""
    _lib.require_cuda()
    T, G, K = x.shape
    if not x.is_contiguous() or w.shape != (sum(rows), K) or w.stride(1) != 1 or len(rows) != G or any(r % _GROUP_TILE for r in rows):
        raise ValueError("linear_groups: shape/layout mismatch")
    out = torch.empty((T, w.shape[0]), dtype=x.dtype, device=x.device)
    if T <= 256 and x.dtype != torch.float32:
        lib = _lib.load()
        lib.b200_gemm_skinny_scratch_floats.restype = ctypes.c_longlong
        scratch, tickets = _skinny_scratch.get(x.device, lib.b200_gemm_skinny_scratch_floats(T, w.shape[0], 0), w.shape[0] // _GROUP_TILE)
        tiles = (ctypes.c_int * G)(*[r // _GROUP_TILE for r in rows])
        _lib.call("b200_gemm_skinny_groups", ptr(x), ptr(w), ptr(out), T, K, G, tiles, G * K, w.stride(0), out.stride(0),
                  dtype_code(x.dtype), ptr(scratch), ptr(tickets), stream_ptr())
        _count()
        return out
    at = 0
    for g, r in enumerate(rows):
        (gemm_f32 if x.dtype == torch.float32 else gemm)(x[:, g], w[at:at + r], out[:, at:at + r])
        at += r
    return out


def gemm_f32(a: torch.Tensor, b: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``a[M,K] @ b[N,K].T`` in true fp32 (no TF32), for the models' 32-bit mode."""
    _lib.require_cuda()
    _check_2d(a, "a"), _check_2d(b, "b")
    M, K = a.shape
    N = b.shape[0]
    if b.shape[1] != K or a.dtype != torch.float32 or b.dtype != torch.float32:
        raise ValueError("gemm_f32: shape/dtype mismatch")
    if out is None:
        out = torch.empty((M, N), dtype=a.dtype, device=a.device)
    _lib.call("b200_gemm_f32", ptr(a), ptr(b), ptr(out), M, N, K, a.stride(0), b.stride(0), out.stride(0), stream_ptr())
    _count()
    return out


def rmsnorm(x: torch.Tensor, gamma: torch.Tensor, eps: float, residual: torch.Tensor | None = None,
            out: torch.Tensor | None = None) -> torch.Tensor:
    """RMSNorm over the last dim. With `residual`, computes ``residual += x`` in place first and normalises the sum.

    ``gamma`` is treated as a weight: the kernel fetches it before it waits for the kernel launched just before it
    (programmatic dependent launch), so it must not be an output of that kernel. The same holds for the gains of
    ``qk_norm_rope`` and of the fused all-reduce + RMSNorm."""
    _lib.require_cuda()
    hidden = x.shape[-1]
    x2 = x.reshape(-1, hidden)
    if not x2.is_contiguous():
        x2 = x2.contiguous()
    if out is None:
        out = torch.empty_like(x2)
    o2 = out.reshape(-1, hidden)
    r2 = residual.reshape(-1, hidden) if residual is not None else None
    _lib.call("b200_rmsnorm", ptr(x2), ptr(r2), ptr(r2), ptr(gamma), ptr(o2), x2.shape[0], hidden, c_float(eps),
              dtype_code(x.dtype), stream_ptr())
    _count()
    return o2.reshape(x.shape)


def qk_norm_rope(qkv: torch.Tensor, positions: torch.Tensor, cos_sin: torch.Tensor, num_q_heads: int,
                 num_kv_heads: int, k_cache: torch.Tensor, v_cache: torch.Tensor, slots: torch.Tensor | None,
                 q_gamma: torch.Tensor | None, k_gamma: torch.Tensor | None, eps: float = 1e-6,
                 q_out: torch.Tensor | None = None) -> torch.Tensor:
    """Per-head RMSNorm of q/k, neox RoPE, and the write of k/v into the KV cache at `slots`, in one kernel.

    qkv: [T, (Hq + 2 Hkv) * 128]; positions: int32 [T]; cos_sin: fp32 [max_pos, 128] (cos | sin);
    caches: [num_slots, Hkv, 128] (any view whose first dim is the slot); slots: int64 [T] (None = identity).
    Returns q [T, Hq, 128].
    """
    _lib.require_cuda()
    T = qkv.shape[0]
    D = 128
    if qkv.shape[1] != (num_q_heads + 2 * num_kv_heads) * D or not qkv.is_contiguous():
        raise ValueError("qkv must be contiguous [T, (Hq + 2*Hkv) * 128]")
    if positions.dtype != torch.int32 or cos_sin.dtype != torch.float32:
        raise ValueError("positions must be int32 and cos_sin float32")
    if q_out is None:
        q_out = torch.empty((T, num_q_heads, D), dtype=qkv.dtype, device=qkv.device)
    _lib.call("b200_qk_norm_rope", ptr(qkv), ptr(positions), ptr(slots), ptr(q_gamma), ptr(k_gamma), ptr(cos_sin),
              ptr(q_out), ptr(k_cache), ptr(v_cache), T, num_q_heads, num_kv_heads, D, c_float(eps),
              dtype_code(qkv.dtype), stream_ptr())
    _count()
    return q_out


def embedding(ids: torch.Tensor, table: torch.Tensor, out: torch.Tensor | None = None, gamma: torch.Tensor | None = None,
              scaled_out: torch.Tensor | None = None, sumsq_out: torch.Tensor | None = None) -> torch.Tensor:
    """``table[ids]`` for int64 ids of any shape -> [*ids.shape, H] (ids outside the table give zero rows).

    For a following RMSNorm folded into the consumer GEMM: ``sumsq_out`` (fp32 [T]) receives every row's sum of
    squares and ``scaled_out`` ([T, H]) the row times ``gamma``."""
    _lib.require_cuda()
    if not table.is_contiguous() or table.dim() != 2:
        raise ValueError("embedding table must be a contiguous [V, H] tensor")
    flat = ids.reshape(-1).to(torch.int64).contiguous()
    V, H = table.shape
    if out is None:
        out = torch.empty((flat.numel(), H), dtype=table.dtype, device=table.device)
    _lib.call("b200_embedding", ptr(flat), ptr(table), ptr(out), flat.numel(), ctypes.c_longlong(V), H, dtype_code(table.dtype),
              ptr(gamma), ptr(scaled_out), ptr(sumsq_out), stream_ptr())
    _count()
    return out.reshape(*ids.shape, H)


def silu_mul(x: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
    """``silu(x[..., :I]) * x[..., I:]`` for the fused [gate | up] projection."""
    _lib.require_cuda()
    inter = x.shape[-1] // 2
    x2 = x.reshape(-1, x.shape[-1])
    _check_2d(x2, "x")
    if out is None:
        out = torch.empty((x2.shape[0], inter), dtype=x.dtype, device=x.device)
    _lib.call("b200_silu_mul", ptr(x2), ptr(out), x2.shape[0], inter, x2.stride(0), dtype_code(x.dtype), stream_ptr())
    _count()
    return out.reshape(*x.shape[:-1], inter)


def silu_mul_fp8(x: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
    """SwiGLU gate fused with block quantisation: x [T, 2 * I] (gate | up, I % 128 == 0) -> (e4m3 [T, I], fp32 scales
    [T, I / 128]) with scale = amax / 448 per 128 channels, the activation format of ``grouped_gemm_fp8``."""
    _lib.require_cuda()
    x2 = x.reshape(-1, x.shape[-1])
    _check_2d(x2, "x")
    inter = x2.shape[1] // 2
    out8 = torch.empty((x2.shape[0], inter), dtype=torch.float8_e4m3fn, device=x.device)
    scale = torch.empty((x2.shape[0], inter // 128), dtype=torch.float32, device=x.device)
    _lib.call("b200_silu_mul_fp8", ptr(x2), ptr(out8), ptr(scale), x2.shape[0], inter, x2.stride(0), dtype_code(x.dtype),
              stream_ptr())
    _count()
    return out8, scale


def topk_softmax(logits: torch.Tensor, k: int, renormalize: bool = False):
    """Router: softmax over experts then top-k. Returns (ids int32 [T,k], weights fp32 [T,k])."""
    _lib.require_cuda()
    T, E = logits.shape
    logits = logits.contiguous()
    ids = torch.empty((T, k), dtype=torch.int32, device=logits.device)
    w = torch.empty((T, k), dtype=torch.float32, device=logits.device)
    _lib.call("b200_topk_softmax", ptr(logits), dtype_code(logits.dtype), T, E, k, ptr(ids), ptr(w),
              1 if renormalize else 0, stream_ptr())
    _count()
    return ids, w


def top_p_sample(logits: torch.Tensor, temperature: float, top_p: float, uniform: torch.Tensor | None = None) -> torch.Tensor:
    """Nucleus sampling without a sort. logits fp32 [B, V]; returns int64 token ids [B, 1]."""
    _lib.require_cuda()
    if logits.dtype != torch.float32 or logits.stride(-1) != 1:
        logits = logits.float().contiguous()
    B, V = logits.shape
    if uniform is None:
        uniform = torch.rand(B, dtype=torch.float32, device=logits.device)
    out = torch.empty((B, 1), dtype=torch.int64, device=logits.device)
    _lib.call("b200_top_p_sample", ptr(logits), logits.stride(0), B, V, c_float(temperature), c_float(top_p),
              ptr(uniform), ptr(out), stream_ptr())
    _count()
    return out


_attn_tickets: dict = {}


def choose_kv_splits(batch: int, num_kv_heads: int, group: int, max_kv_len: int, sm_count: int = 148) -> int:
    """Split count for the decode kernel: one wave of CTAs at two per SM (the per-warp-ring kernel keeps 96 KB of
    shared memory per CTA) and at least 128 tokens (two 64-token tiles) per split. With few (batch, KV head) groups,
    as under tensor parallelism, the kernel is bound by the latency of its serial tile loop, not by bytes: measured on
    the per-rank shapes of an 8-way split (batch 8, one KV head, 2 K tokens) 16 splits beat 4 by 0.42 ms per 64-layer
    step. ``B200DIST_KV_SPLITS`` forces a value (for experiments)."""
    forced = os.environ.get("B200DIST_KV_SPLITS")
    if forced:
        return max(1, int(forced))
    ctas = batch * num_kv_heads * ((group + 15) // 16)
    by_machine = max(1, (2 * sm_count) // max(ctas, 1))
    by_len = max(1, max_kv_len // 128)
    return int(max(1, min(by_machine, by_len, 64)))


# measured on the end-to-end decode step (one GPU, CUDA graph): the in-kernel merge costs 0.3 ms per step more than the
# separate combine launch, whose start overlaps the split kernel under programmatic dependent launch
_FUSED_COMBINE_DEFAULT = os.environ.get("B200DIST_ATTN_FUSED_COMBINE", "0") == "1"


def decode_attention(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, kv_lens: torch.Tensor,
                     block_table: torch.Tensor, scale: float, soft_cap: float = 0.0, num_splits: int = 1,
                     out: torch.Tensor | None = None, return_lse: bool = False, workspace: dict | None = None,
                     fused_combine: bool | None = None, ring: int = -1, gate: torch.Tensor | None = None):
    """Paged GQA decode attention. q [B,Hq,128]; caches [num_blocks, page, Hkv, 128]; kv_lens int32 [B];
    block_table int32 [B, max_blocks]. Returns out [B,Hq,128] (and natural-log LSE fp32 [B,Hq]).

    With ``num_splits > 1`` the last CTA of every (batch, head group) merges the split partials inside the same
    launch (``fused_combine=False`` runs the separate combine kernel instead). ``ring`` selects the K/V pipeline:
    0 = two-stage CTA-wide, 3 / 6 = per-warp rings of that depth, -1 = the library default. ``gate`` [B, Hq] (unit inner
    stride): every head's output is multiplied by its sigmoid, in the combine launch."""
    _lib.require_cuda()
    B, Hq, D = q.shape
    page, Hkv = k_cache.shape[1], k_cache.shape[2]
    if not (q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous() and block_table.stride(1) == 1):
        raise ValueError("decode_attention needs contiguous q / caches and a row-major block table")
    if out is None:
        out = torch.empty_like(q)
    if gate is not None and (gate.shape != (B, Hq) or gate.stride(1) != 1 or gate.dtype != q.dtype or return_lse):
        raise ValueError("decode_attention: the gate is [B, Hq] in the type of q, without a log-sum-exp")
    if fused_combine is None:
        fused_combine = _FUSED_COMBINE_DEFAULT
    fused_combine = fused_combine and gate is None
    lse = torch.empty((B, Hq), dtype=torch.float32, device=q.device) if return_lse else None
    tickets = None
    if num_splits > 1 or gate is not None:
        if workspace is not None and "o_part" in workspace and workspace["o_part"].numel() >= B * Hq * num_splits * D:
            o_part, lse_part = workspace["o_part"], workspace["lse_part"]
        else:
            o_part = torch.empty(B * Hq * num_splits * D, dtype=torch.float32, device=q.device)
            lse_part = torch.empty(B * Hq * num_splits, dtype=torch.float32, device=q.device)
            if workspace is not None:
                workspace["o_part"], workspace["lse_part"] = o_part, lse_part
        if fused_combine:
            n_groups = B * Hkv * ((Hq // Hkv + 15) // 16)
            holder = workspace if workspace is not None else _attn_tickets.setdefault(q.device, {})
            tickets = holder.get("tickets")
            if tickets is None or tickets.numel() < n_groups or tickets.device != q.device:
                tickets = torch.zeros(max(n_groups, 1024), dtype=torch.int32, device=q.device)
                holder["tickets"] = tickets
    else:
        o_part = lse_part = None
    _lib.call("b200_decode_attn", ptr(q), ptr(k_cache), ptr(v_cache), ptr(block_table), block_table.stride(0),
              ptr(kv_lens), B, Hq, Hkv, D, page, c_float(scale), c_float(soft_cap), num_splits, ptr(o_part),
              ptr(lse_part), ptr(tickets), ptr(None if gate is not None else out), ptr(lse), dtype_code(q.dtype), ring, stream_ptr())
    _count()
    if gate is not None:
        _lib.call("b200_decode_combine_gated", ptr(o_part), ptr(lse_part), B, Hq, num_splits, ptr(gate), gate.stride(0), ptr(out),
                  dtype_code(q.dtype), stream_ptr())
        _count()
    elif num_splits > 1 and tickets is None:
        _lib.call("b200_decode_combine", ptr(o_part), ptr(lse_part), ctypes.c_longlong(num_splits * D),
                  ctypes.c_longlong(D), ctypes.c_longlong(num_splits), ctypes.c_longlong(1), B * Hq, num_splits,
                  ptr(out), None, ptr(lse), dtype_code(q.dtype), stream_ptr())
        _count()
    return (out, lse) if return_lse else out


_pipe_status: dict = {}


def _pipeline_status(device: torch.device) -> torch.Tensor:
    """One int32 word per device that single-GPU pipeline kernels raise when an internal wait expires."""
    key = device.index if device.index is not None else torch.cuda.current_device()
    st = _pipe_status.get(key)
    if st is None:
        st = _pipe_status[key] = torch.zeros(1, dtype=torch.int32, device=device)
    return st


def check_pipeline_status(device=None) -> None:
    """Synchronise and raise if a pipeline kernel of this device gave up on an internal wait since the last check."""
    dev = torch.device("cuda", torch.cuda.current_device()) if device is None else torch.device(device)
    key = dev.index if dev.index is not None else torch.cuda.current_device()
    st = _pipe_status.get(key)
    if st is None:
        return
    code = int(st.item())
    if code != 0:
        st.zero_()
        raise RuntimeError(f"a pipeline kernel on {dev} gave up on an internal wait (status {code}); its output is incomplete")


def prefill_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_seqlens_q: torch.Tensor,
                      cu_seqlens_k: torch.Tensor, max_seqlen_q: int, max_seqlen_k: int, scale: float,
                      causal: bool = True, out: torch.Tensor | None = None,
                      seqlens_k: torch.Tensor | None = None, gate: torch.Tensor | None = None) -> torch.Tensor:
    """Variable-length attention on the tcgen05 prefill kernel. q [total_q, Hq, dk]; k [total_k, Hkv, dk], v [total_k, Hkv, dv]
    (sizes in multiples of 8, dk <= 256); cu_seqlens_* int32 [B + 1] on the device. ``gate`` [total_q, Hq] (unit inner stride):
    every head's output is multiplied by its sigmoid. With ``causal`` query i of a sequence attends keys <= i + (k_len - q_len).

    Packed sequences: leave ``seqlens_k`` None (lengths are differences of ``cu_seqlens_k``). Keys in place: give
    ``seqlens_k`` int32 [B]; sequence b then reads rows ``cu_seqlens_k[b] ... + seqlens_k[b]`` of k / v, which may be the
    slot view of a paged KV cache whose sequences own contiguous runs of slots. Returns [total_q, Hq, dv]."""
    _lib.require_cuda()
    total_q, Hq, D = q.shape
    total_k, Hkv, _ = k.shape
    dv = v.shape[2]
    if not (q.is_contiguous() and k.is_contiguous() and v.is_contiguous()) or k.shape[:2] != v.shape[:2] or k.shape[2] != D:
        raise ValueError("prefill_attention needs contiguous q / k / v of matching shapes")
    if gate is not None and (gate.shape != (total_q, Hq) or gate.stride(1) != 1 or gate.dtype != q.dtype):
        raise ValueError("prefill_attention: the gate is [total_q, Hq] in the type of q")
    if q.dtype not in (torch.bfloat16, torch.float16) or k.dtype != q.dtype or v.dtype != q.dtype:
        raise TypeError("prefill_attention handles bf16 / f16")
    B = cu_seqlens_q.numel() - 1
    cu_q = cu_seqlens_q.to(device=q.device, dtype=torch.int32).contiguous()
    cu_k = cu_seqlens_k.to(device=q.device, dtype=torch.int32).contiguous()
    k_lens = seqlens_k.to(device=q.device, dtype=torch.int32).contiguous() if seqlens_k is not None else None
    lib = _lib.load()
    lib.b200_prefill_attention_scratch_bytes.restype = ctypes.c_longlong
    nbytes = int(lib.b200_prefill_attention_scratch_bytes(B, Hkv, dv, int(max_seqlen_k)))
    scratch = torch.empty(nbytes, dtype=torch.uint8, device=q.device)
    if out is None:
        out = torch.empty((total_q, Hq, dv), dtype=q.dtype, device=q.device)
    _lib.call("b200_prefill_attention", ptr(q), ptr(k), ptr(v), ptr(cu_q), ptr(cu_k), ptr(k_lens), B, total_q, total_k,
              int(max_seqlen_q), int(max_seqlen_k), Hq, Hkv, D, dv, c_float(scale), 1 if causal else 0, ptr(gate),
              gate.stride(0) if gate is not None else 0, ptr(scratch), ptr(out),
              dtype_code(q.dtype), ptr(_pipeline_status(q.device)), stream_ptr())
    _count(2)
    return out


def combine_partials(o_part: torch.Tensor, lse_part: torch.Tensor, out_dtype: torch.dtype) -> torch.Tensor:
    """Merge attention partials over dim 0: o_part fp32 [R, BH, 128], lse_part fp32 [R, BH] -> [BH, 128]."""
    _lib.require_cuda()
    R, BH, D = o_part.shape
    out = torch.empty((BH, D), dtype=out_dtype, device=o_part.device)
    _lib.call("b200_decode_combine", ptr(o_part), ptr(lse_part), ctypes.c_longlong(o_part.stride(1)),
              ctypes.c_longlong(o_part.stride(0)), ctypes.c_longlong(lse_part.stride(1)),
              ctypes.c_longlong(lse_part.stride(0)), BH, R, ptr(out), None, None, dtype_code(out_dtype), stream_ptr())
    _count()
    return out


# ---- fp32 residual stream (csrc/kernels/residual.cu) ------------------------------------------
@dataclasses.dataclass(frozen=True)
class TanhNorm:
    """``tanh(alpha x) * gain + bias`` in place of a norm with statistics (``center`` argument of the ops below)."""
    alpha: float


COPY = "copy"  # as ``center``: no norm, the stream in the storage type


def _norm_args(width, gain, bias, eps, center, h):
    """`center`: True = layer norm, False = RMS norm, a ``TanhNorm``, or ``COPY``."""
    if isinstance(center, TanhNorm):
        kind, factor = 2, center.alpha
    else:
        kind, factor = (3, 0.0) if center == COPY else (1 if center else 0, eps)
    return ptr(gain), ptr(bias), c_float(factor), kind, ptr(h)


def embed_norm(ids: torch.Tensor, table: torch.Tensor, scale: float, width: int, gain: torch.Tensor, bias: torch.Tensor | None,
               eps: float, center: bool | TanhNorm, state0: torch.Tensor | None = None) -> tuple[torch.Tensor, torch.Tensor]:
    """``x = table[ids] * scale`` in fp32 and ``h = norm(x)`` in the table's type, one kernel. ids int64 [T]; table [V, P]
    with P >= width columns (padding columns zero). ``center``: layer norm, else RMS norm, or a ``TanhNorm``. ``state0`` fp32 [T, P]
    receives a copy of x. Returns (x fp32 [T, P], h [T, P])."""
    _lib.require_cuda()
    flat = ids.reshape(-1).to(torch.int64).contiguous()
    T, P = flat.numel(), table.shape[1]
    x = torch.empty((T, P), dtype=torch.float32, device=table.device)
    h = torch.empty((T, P), dtype=table.dtype, device=table.device)
    _lib.call("b200_embed_norm", ptr(flat), ptr(table), T, ctypes.c_longlong(table.shape[0]), width, P, c_float(scale), ptr(x),
              ptr(state0), *_norm_args(width, gain, bias, eps, center, h), dtype_code(table.dtype), stream_ptr())
    _count()
    return x, h


def residual_norm(x: torch.Tensor, width: int, mult: float, a: torch.Tensor, gate_a: torch.Tensor | None = None,
                  bias_a: torch.Tensor | None = None, b: torch.Tensor | None = None, gate_b: torch.Tensor | None = None,
                  bias_b: torch.Tensor | None = None, states: torch.Tensor | None = None, weights: torch.Tensor | None = None,
                  keep: bool = False, gain: torch.Tensor | None = None, bias: torch.Tensor | None = None, eps: float = 0.0,
                  center: bool | TanhNorm | str = True) -> torch.Tensor | None:
    """One pass over the fp32 residual stream ``x`` [T, P] (updated in place):
    ``s = x + mult * (sigmoid(gate_a + bias_a) * a + sigmoid(gate_b + bias_b) * b)``; with ``weights`` (fp32 [n + 1])
    ``x = sum_j weights[j] * states[j] + weights[n] * s`` over the n earlier states (``states`` fp32 [>= n, T, P]; s is stored
    as state n with ``keep``), else ``x = s``; returns ``norm(x)`` when ``gain`` is given (see ``_norm_args`` for ``center``; ``COPY``
    returns x in the type of a and takes no gain). a, b [T, P]; the gate logits may be
    column slices of a wider GEMM output (same row pitch)."""
    _lib.require_cuda()
    T, P = x.shape
    if x.dtype != torch.float32 or a.shape != x.shape or not a.is_contiguous() or (b is not None and (b.shape != x.shape or not b.is_contiguous())):
        raise ValueError("residual_norm: x must be fp32 [T, P] and the sublayer results contiguous [T, P]")
    ldg = gate_a.stride(0) if gate_a is not None else 0
    if gate_b is not None and gate_a is not None and gate_b.stride(0) != ldg:
        raise ValueError("residual_norm: the gates need one row pitch")
    if gate_b is not None and gate_a is None:
        ldg = gate_b.stride(0)
    n = weights.numel() - 1 if weights is not None else 0
    if weights is not None and (weights.dtype != torch.float32 or states is None or states.shape[0] < n + (1 if keep else 0)
                                or states.shape[1:] != x.shape or not states.is_contiguous()):
        raise ValueError("residual_norm: weights fp32 [n + 1] need contiguous fp32 states [>= n, T, P]")
    h = torch.empty((T, P), dtype=a.dtype, device=a.device) if gain is not None or center == COPY else None
    _lib.call("b200_residual_norm", ptr(a), ptr(gate_a), ptr(bias_a), ptr(b), ptr(gate_b), ptr(bias_b), ldg, c_float(mult), ptr(x),
              ptr(states), ctypes.c_longlong(T * P), ptr(weights), n, 1 if keep else 0, T, width, P,
              *_norm_args(width, gain, bias, eps, center, h), dtype_code(a.dtype), stream_ptr())
    _count()
    return h


def residual_post(x: torch.Tensor, width: int, mult: float, a: torch.Tensor, gain_a: torch.Tensor, b: torch.Tensor | None = None,
                  gain_b: torch.Tensor | None = None, post_eps: float = 0.0, gain: torch.Tensor | None = None,
                  bias: torch.Tensor | None = None, eps: float = 0.0, center: bool | TanhNorm | str = True) -> torch.Tensor | None:
    """``x += mult * (rms(a) * gain_a + rms(b) * gain_b)`` on the fp32 stream x [T, P] (in place; b optional): sublayer results [T, P]
    that are RMS-normed over the width on their way in. Returns ``norm(x)`` as ``residual_norm`` does."""
    _lib.require_cuda()
    T, P = x.shape
    if x.dtype != torch.float32 or a.shape != x.shape or not a.is_contiguous() or (b is not None and (b.shape != x.shape or not b.is_contiguous())):
        raise ValueError("residual_post: x must be fp32 [T, P] and the sublayer results contiguous [T, P]")
    h = torch.empty((T, P), dtype=a.dtype, device=a.device) if gain is not None or center == COPY else None
    _lib.call("b200_residual_post", ptr(a), ptr(gain_a), ptr(b), ptr(gain_b), c_float(post_eps), c_float(mult), ptr(x), T, width, P,
              *_norm_args(width, gain, bias, eps, center, h), dtype_code(a.dtype), stream_ptr())
    _count()
    return h


def token_side(g: torch.Tensor, ids: torch.Tensor, table: torch.Tensor, offset: int, dim: int) -> torch.Tensor:
    """``gelu(g) * table[ids, offset : offset + dim]`` (tanh form of gelu). g [T, P] contiguous, P >= dim; ids int64 [T]; returns [T, P],
    zeros behind `dim`."""
    _lib.require_cuda()
    if not g.is_contiguous() or not table.is_contiguous() or table.dtype != g.dtype or ids.dtype != torch.int64 or ids.numel() != g.shape[0]:
        raise ValueError("token_side: shape/layout mismatch")
    act = torch.empty_like(g)
    _lib.call("b200_token_side", ptr(g), ptr(ids), ptr(table), ptr(act), g.shape[0], ctypes.c_longlong(table.shape[0]), dim, g.shape[1],
              table.shape[1], offset, dtype_code(g.dtype), stream_ptr())
    _count()
    return act


# ---- recurrent mixers (csrc/kernels/recurrent.cu) ---------------------------------------------
def token_mix(h: torch.Tensor, mu: torch.Tensor, last: torch.Tensor) -> torch.Tensor:
    """``h_t + (h_{t-1} - h_t) * mu_g`` for every row of mu [G, P]: h [B * S, P] -> [B * S, G, P]. ``last`` [B, P] is the token before
    the call and is replaced by the call's last one."""
    _lib.require_cuda()
    T, P = h.shape
    B, G = last.shape[0], mu.shape[0]
    if not (h.is_contiguous() and mu.is_contiguous() and last.is_contiguous()) or T % B or mu.shape[1] != P or last.shape[1] != P:
        raise ValueError("token_mix: shape/layout mismatch")
    out = torch.empty((T, G, P), dtype=h.dtype, device=h.device)
    _lib.call("b200_token_mix", ptr(h), ptr(mu), ptr(last), ptr(out), B, T // B, G, P, dtype_code(h.dtype), stream_ptr())
    _count()
    return out


def tanh_linear(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``tanh(x) @ w.T``, the second half of a low-rank map: x [T, K] (rows may be strided), w [N, K]. One launch for few tokens, tanh
    and the tiled GEMM for many."""
    if x.shape[0] <= 256:
        return head_linear(x[:, None], w[None], tanh=True)[:, 0]
    _check_2d(x, "x")
    act = torch.empty(x.shape, dtype=x.dtype, device=x.device)
    _lib.call("b200_tanh_rows", ptr(x), ptr(act), x.shape[0], x.shape[1], x.stride(0), dtype_code(x.dtype), stream_ptr())
    _count()
    return linear(act, w)


def short_conv(x: torch.Tensor, taps: torch.Tensor, last: torch.Tensor) -> torch.Tensor:
    """Causal convolution per channel, then silu: x [B * S, C] (rows may be strided), taps fp32 [n, C] (the last weighs the current
    token), ``last`` [B, n - 1, C] the inputs before the call, replaced by the last ones of the call. Returns [B * S, C]."""
    _lib.require_cuda()
    T, C = x.shape
    n, B = taps.shape[0], last.shape[0]
    if x.stride(1) != 1 or taps.dtype != torch.float32 or not (taps.is_contiguous() and last.is_contiguous()) or taps.shape[1] != C \
            or last.shape[1:] != (n - 1, C) or last.dtype != x.dtype or T % B:
        raise ValueError("short_conv: shape/layout mismatch")
    out = torch.empty((T, C), dtype=x.dtype, device=x.device)
    _lib.call("b200_short_conv", ptr(x), ptr(taps), ptr(last), ptr(out), B, T // B, C, n, x.stride(0), dtype_code(x.dtype), stream_ptr())
    _count()
    return out


def _check_recurrent(state, rows, fp32, name):
    if state.dtype != torch.float32 or not state.is_contiguous() or any(t.dtype != torch.float32 or not t.is_contiguous() for t in fp32):
        raise ValueError(f"{name}: the state and the per-channel constants must be contiguous fp32")
    if any(t.stride(1) != 1 or t.dtype != rows[0].dtype or t.shape[0] != rows[0].shape[0] for t in rows):
        raise ValueError(f"{name}: the inputs must be rows of one type with unit inner stride")


def wkv(r: torch.Tensor, k: torch.Tensor, v: torch.Tensor, z: torch.Tensor, gate: torch.Tensor, w0: torch.Tensor, u: torch.Tensor,
        gain: torch.Tensor, state: torch.Tensor, dim: int, vdim: int, eps: float, plain: bool = False) -> torch.Tensor:
    """Decayed outer-product memory with a bonus ``u`` for the current token and decays ``exp(-exp(z + w0))`` per key channel, then
    the RMS norm of every head, ``gain`` and ``silu(gate)``. r, k, z [B * S, H * D], v, gate [B * S, H * E] (rows may be strided);
    w0, u [H * D], gain [H * E]; ``state`` [B, H, D, E] is updated. D and E are multiples of 8, ``dim`` / ``vdim`` the true sizes.
    Returns [B * S, H * E]."""
    _lib.require_cuda()
    B, H, D, E = state.shape
    _check_recurrent(state, (r, k, v, z, gate), (w0, u, gain), "wkv")
    T = r.shape[0]
    if T % B or r.shape[1] != H * D or k.shape != r.shape or z.shape != r.shape or v.shape[1] != H * E or gate.shape != v.shape \
            or w0.numel() != H * D or u.numel() != H * D or gain.numel() != H * E:
        raise ValueError("wkv: shape mismatch")
    out = torch.empty((T, H * E), dtype=r.dtype, device=r.device)
    _lib.call("b200_wkv", ptr(r), r.stride(0), ptr(k), k.stride(0), ptr(v), v.stride(0), ptr(z), z.stride(0), ptr(gate), gate.stride(0),
              ptr(w0), ptr(u), ptr(gain), c_float(eps), ptr(state), ptr(out), B, T // B, H, dim, D, vdim, E, int(plain),
              dtype_code(r.dtype), stream_ptr())
    _count()
    return out


def gated_delta(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, a: torch.Tensor, b: torch.Tensor, gate: torch.Tensor,
                a_log: torch.Tensor, dt_bias: torch.Tensor, gain: torch.Tensor, state: torch.Tensor, dim: int, vdim: int, eps: float,
                plain: bool = False) -> torch.Tensor:
    """Gated delta rule on unit-length q (times dim ** -0.5) and k, then the RMS norm of every head, ``gain`` and ``silu(gate)``. q, k
    [B * S, G * D], v, gate [B * S, H * E], a (decay) and b (step size) logits [B * S, H] (rows may be strided; a and b with one
    pitch); a_log, dt_bias [H], gain [E]; ``state`` [B, H, D, E] is updated. Returns [B * S, H * E]."""
    _lib.require_cuda()
    B, H, D, E = state.shape
    _check_recurrent(state, (q, k, v, a, b, gate), (a_log, dt_bias, gain), "gated_delta")
    T, G = q.shape[0], q.shape[1] // D
    if T % B or q.shape[1] != G * D or k.shape != q.shape or v.shape[1] != H * E or gate.shape != v.shape or a.shape[1] != H \
            or b.shape != a.shape or a.stride(0) != b.stride(0) or a_log.numel() != H or dt_bias.numel() != H or gain.numel() != E:
        raise ValueError("gated_delta: shape mismatch")
    out = torch.empty((T, H * E), dtype=q.dtype, device=q.device)
    _lib.call("b200_gated_delta", ptr(q), q.stride(0), ptr(k), k.stride(0), ptr(v), v.stride(0), ptr(a), ptr(b), a.stride(0), ptr(gate),
              gate.stride(0), ptr(a_log), ptr(dt_bias), ptr(gain), c_float(eps), ptr(state), ptr(out), B, T // B, H, G, dim, D, vdim, E,
              int(plain), dtype_code(q.dtype), stream_ptr())
    _count()
    return out


# ---- grouped-query attention of any head size (csrc/kernels/gqa_attn.cu) ----------------------
def head_norm_rope(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, heads: int, kv_heads: int, dim: int, gain_q: torch.Tensor | None,
                   gain_k: torch.Tensor | None, eps: float, cos_sin: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor,
                   k_cache: torch.Tensor, v_cache: torch.Tensor, q_scale: float = 1.0) -> torch.Tensor:
    """Per-head RMS norm of q and k, interleaved rotary positions on their first ``cos_sin.shape[1]`` dimensions, ``q_scale`` on q, and
    the write of k and v to ``slots``, in one kernel. q, k, v: column slices of one GEMM output, heads of equal (padded) size;
    caches [..., kv_heads, D'] with D' at least that size (zeros behind). cos_sin fp32 [positions, rot]: (cos, sin) of pair 0, 1, ...
    Returns q [T, heads, D']."""
    _lib.require_cuda()
    T, ld = q.shape[0], q.stride(0)
    qk_in, v_in, qk_out, v_out = q.shape[1] // heads, v.shape[1] // kv_heads, k_cache.shape[-1], v_cache.shape[-1]
    if k.shape[1] != kv_heads * qk_in or k.stride(0) != ld or v.stride(0) != ld or positions.dtype != torch.int32 \
            or cos_sin.dtype != torch.float32 or not cos_sin.is_contiguous() or slots.dtype != torch.int64 \
            or not (k_cache.is_contiguous() and v_cache.is_contiguous()) or k_cache.shape[-2] != kv_heads:
        raise ValueError("head_norm_rope: shape/layout mismatch")
    out = torch.empty((T, heads, qk_out), dtype=q.dtype, device=q.device)
    _lib.call("b200_head_norm_rope", ptr(q), ptr(k), ptr(v), ld, ptr(gain_q), ptr(gain_k), ptr(cos_sin), ptr(positions), ptr(slots),
              ptr(out), ptr(k_cache), ptr(v_cache), T, heads, kv_heads, dim, cos_sin.shape[1], qk_in, qk_out, v_in, v_out, c_float(eps),
              c_float(q_scale), dtype_code(q.dtype), stream_ptr())
    _count()
    return out


def gqa_attention_plain(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, kv_lens: torch.Tensor, block_table: torch.Tensor,
                        tokens: int, scale: float, gate: torch.Tensor | None = None) -> torch.Tensor:
    """Causal attention of the last `tokens` tokens of every sequence over paged keys, any head sizes (multiples of 4) and storage
    type: q [B * tokens, H, dk], caches [blocks, page, G, dk] / [..., dv], kv_lens int32 [B] with the new tokens. ``gate``
    [B * tokens, H]: every head's output times its sigmoid. Returns [B * tokens, H, dv]."""
    _lib.require_cuda()
    T, H, dk = q.shape
    B, page, G, dv = kv_lens.numel(), k_cache.shape[1], k_cache.shape[2], v_cache.shape[3]
    if T != B * tokens or k_cache.shape[3] != dk or not (q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous()) \
            or block_table.stride(1) != 1 or (gate is not None and (gate.shape != (T, H) or gate.stride(1) != 1 or gate.dtype != q.dtype)):
        raise ValueError("gqa_attention_plain: shape/layout mismatch")
    out = torch.empty((T, H, dv), dtype=q.dtype, device=q.device)
    _lib.call("b200_gqa_attention_plain", ptr(q), ptr(k_cache), ptr(v_cache), ptr(block_table), block_table.stride(0), ptr(kv_lens), B,
              tokens, H, G, dk, dv, page, c_float(scale), ptr(gate), gate.stride(0) if gate is not None else 0, ptr(out),
              dtype_code(q.dtype), stream_ptr())
    _count()
    return out


# ---- latent attention (csrc/kernels/latent_attn.cu, prefill_attn_sm100.cu) --------------------
def latent_prep(latent_in: torch.Tensor | None, gain: torch.Tensor | None, cache: torch.Tensor | None, slots: torch.Tensor | None,
                rank: int, eps: float, up: torch.Tensor | None = None) -> torch.Tensor | None:
    """RMS norm of ``latent_in`` [T, >= rank] into rows ``slots`` (int64 [T]) of ``cache`` [..., P], and squared relu of ``up``
    [T, I] (returned), in one launch. Both inputs may be column slices of the same GEMM output."""
    _lib.require_cuda()
    src = latent_in if latent_in is not None else up
    T, ld = src.shape[0], src.stride(0)
    if latent_in is not None and up is not None and up.stride(0) != ld:
        raise ValueError("latent_prep: both inputs need one row pitch")
    inter = up.shape[1] if up is not None else 0
    act = torch.empty((T, inter), dtype=up.dtype, device=up.device) if up is not None else None
    pitch = cache.shape[-1] if cache is not None else 0
    _lib.call("b200_latent_prep", ptr(latent_in), ptr(gain), ptr(cache), ptr(slots), rank, pitch, c_float(eps), ptr(up), ptr(act),
              inter, ld, T, dtype_code(src.dtype), stream_ptr())
    _count()
    return act


def head_linear(x: torch.Tensor, w: torch.Tensor, tanh: bool = False) -> torch.Tensor:
    """Per-head GEMM ``y[t, h, :] = w[h] @ x[t, h, :]``: x [T, H, K] (unit inner stride), w [H, N, K] -> y [T, H, N]. With ``tanh`` of
    tanh(x)."""
    _lib.require_cuda()
    T, H, K = x.shape
    N = w.shape[1]
    if w.shape != (H, N, K) or not w.is_contiguous() or x.stride(2) != 1 or x.dtype != w.dtype:
        raise ValueError("head_linear: shape/layout mismatch")
    y = torch.empty((T, H, N), dtype=x.dtype, device=x.device)
    ll = ctypes.c_longlong
    _lib.call("b200_head_linear", ptr(x), ptr(w), ptr(y), T, H, N, K, ll(x.stride(0)), ll(x.stride(1)), ll(y.stride(0)),
              ll(y.stride(1)), int(tanh), dtype_code(x.dtype), stream_ptr())
    _count()
    return y


@functools.lru_cache(maxsize=None)
def choose_latent_splits(batch: int, rows: int, max_kv_len: int, sm_count: int = 148) -> tuple[int, int]:
    """(splits, query rows per CTA) of the absorbed latent attention, for `rows` query rows of each of `batch` sequences: the
    least estimated time, from what a 64-key tile takes by rows per CTA (measured; a CTA has an SM to itself) and what writing
    and merging the partial results of one more split costs."""
    n_tiles = max(1, (max_kv_len + 63) // 64)
    best = (float("inf"), 1, 16)
    for per_cta, tile_us in ((16, 1.2), (32, 1.25), (64, 1.4)):
        if per_cta > 16 and rows <= per_cta // 2:
            continue
        ctas = batch * ((rows + per_cta - 1) // per_cta)
        for splits in range(1, min(64, n_tiles) + 1):
            tiles = -(-n_tiles // splits)
            cost = -(-ctas * splits // sm_count) * tiles * tile_us + 7e-4 * batch * rows * splits
            if cost < best[0]:
                best = (cost, -(-n_tiles // tiles), per_cta)
    return best[1], best[2]


def latent_attention(q: torch.Tensor, cache: torch.Tensor, kv_lens: torch.Tensor, block_table: torch.Tensor, tokens: int,
                     scale: float, sink: torch.Tensor | None = None, num_splits: int = 1, rows_per_cta: int = 0,
                     variant: str | None = None) -> torch.Tensor:
    """Attention of absorbed queries over paged latents that are both keys and values. q [B * tokens, H, P]; cache
    [blocks, page, P]; kv_lens int32 [B] (the new tokens included); block_table int32 [B, *]; query token i of a sequence attends
    keys j <= kv_len - tokens + i. ``sink`` fp32 [H]. Returns [B * tokens, H, P].

    ``variant``: "tc" (tcgen05 tiles; 16-bit, ranks up to 512) or "plain" (one warp per row, any type and rank); None picks the
    first that handles the operands."""
    _lib.require_cuda()
    T, H, P = q.shape
    B = kv_lens.numel()
    if T != B * tokens or cache.shape[-1] != P or not (q.is_contiguous() and cache.is_contiguous()) or block_table.stride(1) != 1:
        raise ValueError("latent_attention: shape/layout mismatch")
    if sink is not None and (sink.dtype != torch.float32 or sink.numel() != H):
        raise ValueError("latent_attention: sink must be fp32 [H]")
    page = cache.shape[1]
    out = torch.empty_like(q)
    if variant is None:
        variant = "plain" if q.dtype == torch.float32 or P > 512 or page % 64 != 0 else "tc"
    shape = (ptr(block_table), block_table.stride(0), ptr(kv_lens), B, tokens, H, P, page, c_float(scale))
    if variant == "plain":
        _lib.call("b200_latent_attention_plain", ptr(q), ptr(cache), *shape, ptr(sink), ptr(out), dtype_code(q.dtype), stream_ptr())
        _count()
        return out
    o_part = torch.empty((T * H, num_splits, P), dtype=torch.float32, device=q.device)
    lse_part = torch.empty((T * H, num_splits), dtype=torch.float32, device=q.device)
    per_cta = rows_per_cta or (16 if tokens * H <= 16 else 32 if tokens * H <= 32 else 64)
    _lib.call("b200_latent_decode", ptr(q), ptr(cache), ctypes.c_longlong(cache.shape[0] * page), *shape, num_splits, per_cta,
              ptr(o_part), ptr(lse_part), dtype_code(q.dtype), ptr(_pipeline_status(q.device)), stream_ptr())
    _lib.call("b200_latent_combine", ptr(o_part), ptr(lse_part), ptr(sink), T * H, H, num_splits, P, ptr(out), dtype_code(q.dtype),
              stream_ptr())
    _count(2)
    return out


def prefill_attention_vt(q: torch.Tensor, k: torch.Tensor, vt: torch.Tensor, cu_seqlens_q: torch.Tensor, cu_seqlens_k: torch.Tensor,
                         seqlens_k: torch.Tensor, max_seqlen_q: int, scale: float, causal: bool = True,
                         sink: torch.Tensor | None = None) -> torch.Tensor:
    """``prefill_attention`` for other head sizes, transposed values and an optional sink logit per head. q [total_q, Hq, dk]
    (rows may be strided), k [total_k, Hkv, dk], vt [Hkv, dv, total_k]: the keys of a sequence are rows ``cu_seqlens_k[b]`` ... of k and
    the same columns of vt (``seqlens_k[b]`` of them; multiples of 8 apart; what lies between must be finite). sink fp32 [Hq] or
    None; dk <= 256, dk, dv and total_k multiples of 8. Returns [total_q, Hq, dv]."""
    _lib.require_cuda()
    total_q, Hq, dk = q.shape
    total_k, Hkv, _ = k.shape
    B, dv = seqlens_k.numel(), vt.shape[1]
    if q.stride(2) != 1 or q.stride(1) != dk or not (k.is_contiguous() and vt.is_contiguous()) or vt.shape != (Hkv, dv, total_k):
        raise ValueError("prefill_attention_vt: shape/layout mismatch")
    out = torch.empty((total_q, Hq, dv), dtype=q.dtype, device=q.device)
    _lib.call("b200_prefill_attention_vt", ptr(q), ctypes.c_longlong(q.stride(0)), ptr(k), ptr(vt), ptr(cu_seqlens_q),
              ptr(cu_seqlens_k), ptr(seqlens_k), B, total_q, total_k, int(max_seqlen_q), Hq, Hkv, dk, dv, c_float(scale),
              1 if causal else 0, ptr(sink), ptr(out), dtype_code(q.dtype), ptr(_pipeline_status(q.device)), stream_ptr())
    _count()
    return out
