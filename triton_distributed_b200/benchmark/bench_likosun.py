"""Likosun next to the framework's closest model: prefill and decode throughput at equal size, and every new kernel's distance
from its roofline beside the like kernel of a Qwen3 layer. One GPU, random weights.

``python bench.py --workload likosun [--likosun-models likosun-1b likosun-7b]`` prints one JSON line with what ``run`` returns.
The Qwen3 partner has the same width, depth and heads (four query heads per KV head) and the inner size that makes the parameter
count equal. Kernel rows: device time of one cold call (L2 flushed, minimum over calls); ``roofline_us`` is the larger of bytes
over the measured copy bandwidth and FLOPs over the measured cuBLAS rate, counted from the operands.
"""
from __future__ import annotations

import gc
import json
import statistics
from pathlib import Path

import torch

from .. import ops, utils
from ..models import ARCHS, ArchConfig, Engine, LikosunConfig, ModelConfig


def peaks() -> tuple[float, float, str]:
    """(copy bytes/s, bf16 FLOP/s, where from)."""
    f = Path(__file__).resolve().parents[2] / "MEASURED_PEAKS.json"
    if f.exists():
        p = json.loads(f.read_text())
        return p["hbm_gbs"] * 1e9, p["bf16_tflops"] * 1e12, "measured"
    return 6.65e12, 1.59e15, "fallback"


def layer_params(a: LikosunConfig) -> int:
    m, W = a.layers[0].mixer, a.hidden_size
    return W * (m.heads * m.dim + m.kv_rank + m.heads * m.vdim + 2 * a.layers[0].mlp.ff + 2 * W) + m.kv_rank * m.heads * (m.dim + m.vdim)


def partner(name: str) -> str:
    """Registers and names the Qwen3 architecture of equal size."""
    a = ARCHS[name]
    H, W = a.layers[0].mixer.heads, a.hidden_size
    kv = max(1, H // 4)
    ff = (layer_params(a) - W * 128 * (2 * H + 2 * kv)) // (3 * W) // 128 * 128
    ARCHS[f"qwen3-shape-of-{name}"] = ArchConfig(W, ff, a.num_hidden_layers, H, kv, vocab_size=a.vocab_size)
    return f"qwen3-shape-of-{name}"


def throughput(name: str, batch: int, prompt: int, steps: int, warmup: int, group=None) -> dict:
    cfg = ModelConfig(model_name=name, max_length=(prompt + steps + warmup + 80) // 64 * 64, rank=0, world_size=1)
    eng = Engine(cfg, temperature=0.0, group=group)
    ids = torch.randint(0, eng.model.arch.vocab_size, (batch, prompt), device="cuda")

    def timed(fn, n):
        torch.cuda.synchronize()
        marks = [torch.cuda.Event(enable_timing=True) for _ in range(n + 1)]
        marks[0].record()
        for i in range(n):
            fn()
            marks[i + 1].record()
        torch.cuda.synchronize()
        return [marks[i].elapsed_time(marks[i + 1]) for i in range(n)]

    pre = timed(lambda: eng.prefill(ids), 5)[2:]
    first = eng.prefill(ids)
    launches = ops.launch_count
    eng.prepare_decode(first)
    launches = (ops.launch_count - launches) // 4      # three warm-up steps and the captured one
    for _ in range(max(3, warmup)):
        eng.decode_one()
    dec = timed(eng.decode_one, steps)
    ops.check_pipeline_status()
    params = sum(t.numel() for t in _tensors(eng.model))
    out = {"model": name, "parameters": params, "prefill_ms": min(pre), "prefill_tokens_per_s": batch * prompt / min(pre) * 1e3,
           "decode_ms": statistics.mean(dec), "decode_ms_min": min(dec), "decode_tokens_per_s": batch / statistics.mean(dec) * 1e3,
           "weight_read_bound_ms": 2 * params / peaks()[0] * 1e3, "launches_per_step": launches}
    eng.graph.reset()
    eng.graph = None
    del eng
    gc.collect()
    torch.cuda.empty_cache()
    return out


def _tensors(model):
    """Weight matrices a forward pass reads (not the embedding, of which a step reads a few rows, nor second layouts)."""
    yield getattr(model, "head", None) if hasattr(model, "head") else model.lm_head
    for layer in model.layers:
        if hasattr(layer, "side_proj"):     # Sizilorn
            yield from (layer.w_in, layer.left.wo, layer.right.wo) if layer.parallel else (layer.mixer.w_in, layer.mixer.w2, layer.mixer.wo)
            yield from (layer.mlp.gate_up_proj, layer.mlp.down_proj, layer.side_gate, layer.side_proj)
        elif hasattr(layer, "w_in"):
            yield from (layer.w_in, layer.attn.uk, layer.attn.uv, layer.attn.wo, layer.down)
        else:
            yield from (layer.attn.wqkv, layer.attn.wo, layer.mlp.gate_up_proj, layer.mlp.down_proj)


def _row(name: str, fn, nbytes: float, flops: float = 0.0, iters: int = 12) -> dict:
    hbm, tc, _ = peaks()
    _, _, times = utils.perf_func_cold(fn, iters, 3)
    us = min(times) * 1e3
    roof = max(nbytes / hbm, flops / tc) * 1e6
    return {"kernel": name, "us": round(us, 2), "roofline_us": float(f"{roof:.3g}"), "of_roofline": float(f"{roof / us:.3g}")}


def kernels(name: str, batch: int = 8, prompt: int = 2048) -> list[dict]:
    """Pairs of (new kernel, like kernel of the partner model); ``ratio`` = of_roofline of the new one over the like one."""
    a, q = ARCHS[name], ARCHS[partner(name)]
    m, W, L = a.layers[0].mixer, a.hidden_size, a.num_hidden_layers
    H, d, v, r, ff, Hkv = m.heads, m.dim, m.vdim, m.kv_rank, a.layers[0].mlp.ff, q.num_key_value_heads
    dev, bf = "cuda", torch.bfloat16

    def rnd(*s, dt=bf):
        return torch.randn(*s, device=dev, dtype=torch.float32).to(dt)

    pairs = []

    def pair(new: dict, like: dict):
        pairs.append({**new, "like": like, "ratio": round(new["of_roofline"] / like["of_roofline"], 2)})

    for kv in (prompt, 8 * prompt):                                                  # ---- decode attention
        lens = torch.full((batch,), kv, dtype=torch.int32, device=dev)
        pages = batch * kv // 64
        table = torch.arange(pages, dtype=torch.int32, device=dev).view(batch, -1)
        cache, qc, sink = rnd(pages, 64, r), rnd(batch, H, r), torch.zeros(H, device=dev)
        splits, rows = ops.choose_latent_splits(batch, H, kv)
        new = _row(f"latent attention + combine, kv {kv}", lambda: ops.latent_attention(qc, cache, lens, table, 1, 0.1, sink, splits, rows),
                   2.0 * batch * kv * r, 4.0 * batch * H * kv * r)
        kc, vc, qq = rnd(pages, 64, Hkv, 128), rnd(pages, 64, Hkv, 128), rnd(batch, H, 128)
        ws: dict = {}
        sp = ops.choose_kv_splits(batch, Hkv, H // Hkv, kv)
        pair(new, _row(f"decode attention + combine, kv {kv}",
                       lambda: ops.decode_attention(qq, kc, vc, lens, table, 0.1, 0.0, sp, workspace=ws),
                       4.0 * batch * kv * Hkv * 128, 4.0 * batch * H * kv * 128))
        del cache, kc, vc
    x = rnd(batch, W)
    # ---- per-head products
    for label, N, K in (("absorb queries", r, d), ("values from latents", v, r)):
        xh, wh = rnd(batch, H, K), rnd(H, N, K)
        wl = rnd(H * N * K // W // 128 * 128, W)   # a decode GEMM of as many weight bytes
        pair(_row(f"head_linear, {label}, {batch} tokens", lambda: ops.head_linear(xh, wh), 2.0 * H * N * K),
             _row("gemm_skinny of equal bytes", lambda: ops.gemm_skinny(x, wl), 2.0 * wl.numel()))
    for T in (batch, batch * prompt):                                                 # ---- row-wise kernels
        cols = H * d + r + ff + 2 * W
        proj, gain = rnd(T, cols), rnd(r)
        cache, slots = torch.zeros(T // 64 + 1, 64, r, device=dev, dtype=bf), torch.arange(T, device=dev)
        lat, up = proj[:, H * d:H * d + r], proj[:, H * d + r:H * d + r + ff]
        new = _row(f"latent_prep, {T} tokens", lambda: ops.latent_prep(lat, gain, cache, slots, r, 1e-6, up), 4.0 * T * (r + ff))
        gu = rnd(T, 2 * q.intermediate_size)
        pair(new, _row(f"silu_mul, {T} tokens", lambda: ops.silu_mul(gu), 6.0 * T * q.intermediate_size))
        del gu
        ga, gb = proj[:, -2 * W:-W], proj[:, -W:]
        xs, s1, s2, g, b = rnd(T, W, dt=torch.float32), rnd(T, W), rnd(T, W), rnd(W), rnd(W)
        n = L // 2
        states, wts = torch.zeros(n + 1, T, W, device=dev), torch.ones(n + 1, device=dev)
        new = _row(f"residual_norm with {n} earlier states, {T} tokens",
                   lambda: ops.residual_norm(xs, W, 0.5, s1, ga, b, s2, gb, b, states=states, weights=wts, keep=True, gain=g, bias=b, eps=1e-6),
                   T * W * (8 + 8 + 4 + 4 * n + 4 + 2.0))
        res = rnd(T, W)
        pair(new, _row(f"rmsnorm with residual, {T} tokens", lambda: ops.rmsnorm(s1, g, 1e-6, residual=res), 8.0 * T * W))
        del states, proj
        ids, tab = torch.randint(0, a.vocab_size, (T,), device=dev), rnd(a.vocab_size, W)
        st0 = torch.empty(T, W, device=dev)
        new = _row(f"embed_norm, {T} tokens", lambda: ops.embed_norm(ids, tab, 2.0, W, g, b, 1e-6, True, state0=st0), T * W * 12.0)
        pair(new, _row(f"embedding, {T} tokens", lambda: ops.embedding(ids, tab), 4.0 * T * W))
    S, B = prompt, batch                                                              # ---- prompts
    R = B * S
    c, uk, uv = rnd(R, r), rnd(H * d, r), rnd(H * v, r)
    xp = rnd(R, W)
    w_like = rnd(H * 128, W)
    like = _row(f"gemm {R} x {H * 128} x {W}", lambda: ops.linear(xp, w_like),
                2.0 * (R * W + R * H * 128 + H * 128 * W), 2.0 * R * H * 128 * W)
    pair(_row(f"expand keys: gemm {R} x {H * d} x {r}", lambda: ops.linear(c, uk), 2.0 * (R * r + H * d * r + R * H * d), 2.0 * R * H * d * r), like)
    pair(_row(f"expand values: gemm {H * v} x {R} x {r}", lambda: ops.linear(uv, c), 2.0 * (R * r + H * v * r + R * H * v), 2.0 * R * H * v * r), like)
    qp, kp, vt = rnd(B * S, H, d), rnd(B * S, H, d), rnd(H, v, B * S)
    cu = torch.arange(0, (B + 1) * S, S, dtype=torch.int32, device=dev)
    lens = torch.full((B,), S, dtype=torch.int32, device=dev)
    sink = torch.zeros(H, device=dev)
    new = _row(f"prefill attention with sink, {B} x {S}", lambda: ops.prefill_attention_vt(qp, kp, vt, cu, cu, lens, S, 0.1, True, sink),
               2.0 * B * S * H * (2 * d + 2 * v), B * H * S * S * (d + v) * 1.0, iters=6)
    kg, vg = rnd(B * S, Hkv, 128), rnd(B * S, Hkv, 128)
    pair(new, _row(f"prefill attention, {B} x {S}", lambda: ops.prefill_attention(qp, kg, vg, cu, cu, S, S, 0.1),
                   2.0 * B * S * 128 * (2 * H + 2 * Hkv), B * H * S * S * 256.0, iters=6))
    ops.check_pipeline_status()
    torch.cuda.empty_cache()
    return pairs


def run(models: list[str], batch: int, prompt: int, steps: int, warmup: int, with_kernels: bool = True, group=None) -> dict:
    torch.manual_seed(0)
    out = {"workload": "likosun", "batch": batch, "prompt": prompt, "steps": steps, "dtype": "bf16", "data": "synthetic, random weights",
           "peaks": peaks()[2], "l2": "weights exceed the L2; kernel rows flush it before every call", "models": [], "kernels": {}}
    for name in models:
        new = throughput(name, batch, prompt, steps, warmup, group)
        like = throughput(partner(name), batch, prompt, steps, warmup, group)
        out["models"].append({"likosun": new, "qwen3": like})
    if with_kernels:
        for name in models:
            out["kernels"][name] = kernels(name, batch, prompt)
    return out
