"""Sizilorn next to the framework's closest model: prefill and decode throughput at equal size, and every new kernel's distance
from its roofline beside the like kernel of a Qwen3 layer. One GPU, random weights.

``python bench.py --workload sizilorn [--sizilorn-models sizilorn-1b sizilorn-7b]`` prints one JSON line with what ``run`` returns.
The Qwen3 partner has the same width, depth and number of attention heads and the inner size that makes the parameter count equal.
Kernel rows as in ``bench_likosun``: ``roofline_us`` is the larger of bytes over the measured copy bandwidth and FLOPs over the rate of
the unit that has to do them: the measured cuBLAS rate for matrix products on 16-bit operands, the nominal fp32 rate (128 fused
multiply-adds per SM and clock) for the recurrences, whose state and inputs are 32-bit by design.
"""
from __future__ import annotations

import torch

from .. import ops
from ..models import ARCHS, ArchConfig, SizilornConfig
from .bench_likosun import _row, peaks, throughput

FP32_FLOPS = 148 * 128 * 2 * 1.965e9


def layer_params(a: SizilornConfig) -> float:
    """Matrix elements a forward pass reads per layer, averaged over the layers."""
    W, total = a.hidden_size, 0
    for layer in a.layers:
        m = layer.mixer
        if m.kind == "wkv":
            total += 5 * W * m.heads * m.dim + m.decay_rank * (W + m.heads * m.dim)
        else:
            p, q = m.left, m.right
            total += W * (p.heads * (p.dim + p.vdim) + p.kv_heads * (p.dim + p.vdim) + 2 * q.kv_heads * q.dim + 3 * q.heads * q.vdim)
        total += 3 * W * layer.mlp.ff + 2 * W * a.side_dim
    return total / a.num_hidden_layers


def partner(name: str) -> str:
    """Registers and names the Qwen3 architecture of equal size."""
    a = ARCHS[name]
    W = a.hidden_size
    H = next(layer.mixer.left.heads for layer in a.layers if layer.mixer.kind == "parallel")
    kv = max(1, H // 4)
    ff = int(layer_params(a) - W * 128 * (2 * H + 2 * kv)) // (3 * W) // 128 * 128
    ARCHS[f"qwen3-shape-of-{name}"] = ArchConfig(W, ff, a.num_hidden_layers, H, kv, vocab_size=a.vocab_size)
    return f"qwen3-shape-of-{name}"


def kernels(name: str, batch: int = 8, prompt: int = 2048) -> list[dict]:
    """Pairs of (new kernel, like kernel of the partner model); ``ratio`` = of_roofline of the new one over the like one."""
    a, q3 = ARCHS[name], ARCHS[partner(name)]
    W, side = a.hidden_size, a.side_dim
    m = next(layer.mixer for layer in a.layers if layer.mixer.kind == "wkv")
    par = next(layer.mixer for layer in a.layers if layer.mixer.kind == "parallel")
    at, de = par.left, par.right
    Hkv, hbm, tc = q3.num_key_value_heads, *peaks()[:2]
    dev, bf = "cuda", torch.bfloat16
    pairs: list[dict] = []

    def rnd(*s, dt=bf):
        return torch.randn(*s, device=dev, dtype=torch.float32).to(dt)

    def fp32(flops: float) -> float:
        return flops * tc / FP32_FLOPS        # as the FLOPs of the 16-bit rate that take as long

    def pair(new: dict, like: dict):
        pairs.append({**new, "like": like, "ratio": round(new["of_roofline"] / like["of_roofline"], 2)})

    def attention(kv: int, gate: bool):
        lens = torch.full((batch,), kv, dtype=torch.int32, device=dev)
        table = torch.arange(batch * kv // 64, dtype=torch.int32, device=dev).view(batch, -1)
        kc, vc, q = rnd(batch * kv // 64, 64, Hkv, 128), rnd(batch * kv // 64, 64, Hkv, 128), rnd(batch, at.heads, 128)
        g, ws = (rnd(batch, at.heads) if gate else None), {}
        splits = ops.choose_kv_splits(batch, Hkv, at.heads // Hkv, kv)
        return _row(f"decode attention + combine{', gated' if gate else ''}, kv {kv}",
                    lambda: ops.decode_attention(q, kc, vc, lens, table, 0.1, 0.0, splits, workspace=ws, gate=g), 4.0 * batch * kv * Hkv * 128,
                    4.0 * batch * at.heads * kv * 128)

    decode_like = attention(prompt, False)
    pair(attention(prompt, True), decode_like)
    S = prompt
    cu = torch.arange(0, (batch + 1) * S, S, dtype=torch.int32, device=dev)
    qp, kg, vg = rnd(batch * S, at.heads, 128), rnd(batch * S, Hkv, 128), rnd(batch * S, Hkv, 128)
    gate = rnd(batch * S, at.heads)

    def prefill(g):
        return _row(f"prefill attention{', gated' if g is not None else ''}, {batch} x {S}", lambda: ops.prefill_attention(qp, kg, vg, cu, cu, S, S, 0.1, gate=g),
                    2.0 * batch * S * 128 * (2 * at.heads + 2 * Hkv), batch * at.heads * S * S * 256.0, iters=6)

    prefill_like = prefill(None)
    pair(prefill(gate), prefill_like)
    del qp, kg, vg
    for T in (batch, batch * prompt):
        tag = f"{T} tokens"
        tokens = T // batch
        # ---- recurrences (the attention of equal batch and length is the like kernel)
        N = m.heads * m.dim
        rows = [rnd(T, N) for _ in range(5)]
        st, c = torch.zeros(batch, m.heads, m.dim, m.dim, device=dev), torch.ones(N, device=dev)
        pair(_row(f"wkv, {m.heads} heads of {m.dim}, {tag}", lambda: ops.wkv(*rows, c, c, c, st, m.dim, m.dim, 1e-6),
                  12.0 * T * N + 8.0 * st.numel(), fp32(5.0 * T * N * m.dim), iters=6), decode_like if tokens == 1 else prefill_like)
        qk, E = de.kv_heads * de.dim, de.heads * de.vdim
        rows, ab = [rnd(T, qk), rnd(T, qk), rnd(T, E), rnd(T, E)], rnd(T, 2 * de.heads)
        st, c = torch.zeros(batch, de.heads, de.dim, de.vdim, device=dev), torch.ones(max(de.heads, de.vdim), device=dev)
        pair(_row(f"gated_delta, {de.heads} heads of {de.dim}, {tag}",
                  lambda: ops.gated_delta(rows[0], rows[1], rows[2], ab[:, : de.heads], ab[:, de.heads:], rows[3], c[: de.heads], c[: de.heads], c[: de.vdim],
                                          st, de.dim, de.vdim, 1e-6),
                  2.0 * T * (2 * qk + 3 * E) + 8.0 * st.numel(), fp32(7.0 * T * E * de.dim), iters=6), decode_like if tokens == 1 else prefill_like)
        del rows, ab, st
        # ---- row-wise kernels
        gu = rnd(T, 2 * q3.intermediate_size)
        glu = _row(f"silu_mul, {tag}", lambda: ops.silu_mul(gu), 6.0 * T * q3.intermediate_size)
        del gu
        g, b, s1, s2, res = rnd(W), rnd(W), rnd(T, W), rnd(T, W), rnd(T, W)
        norm = _row(f"rmsnorm with residual, {tag}", lambda: ops.rmsnorm(s1, g, 1e-6, residual=res), 8.0 * T * W)
        xs, tanh = rnd(T, W, dt=torch.float32), ops.TanhNorm(0.5)
        pair(_row(f"residual_norm, tanh, {tag}", lambda: ops.residual_norm(xs, W, 1.0, s1, gain=g, bias=b, center=tanh), 12.0 * T * W), norm)
        pair(_row(f"residual_post of one, tanh, {tag}", lambda: ops.residual_post(xs, W, 1.0, s1, g, post_eps=1e-6, gain=g, bias=b, center=tanh), 12.0 * T * W), norm)
        pair(_row(f"residual_post of two, tanh, {tag}", lambda: ops.residual_post(xs, W, 0.5, s1, g, s2, g, 1e-6, gain=g, bias=b, center=tanh), 14.0 * T * W), norm)
        mu, last = rnd(5, W), rnd(batch, W)
        pair(_row(f"token_mix, {tag}", lambda: ops.token_mix(s1, mu, last), 12.0 * T * W), glu)
        C = 2 * qk + E
        wide, taps, hist = rnd(T, C + 8), rnd(de.conv, C, dt=torch.float32), rnd(batch, de.conv - 1, C)
        pair(_row(f"short_conv, {tag}", lambda: ops.short_conv(wide[:, :C], taps, hist), 4.0 * T * C), glu)
        del wide
        ids, tab, gs = torch.randint(0, a.vocab_size, (T,), device=dev), rnd(a.vocab_size, side * 4), rnd(T, side)
        emb_table = rnd(a.vocab_size, side)
        emb = _row(f"embedding of {side} columns, {tag}", lambda: ops.embedding(ids, emb_table), 4.0 * T * side)
        pair(_row(f"token_side, {tag}", lambda: ops.token_side(gs, ids, tab, side, side), 6.0 * T * side), emb)
        cols = (at.heads + 2 * Hkv) * 128
        proj, pos = rnd(T, cols), torch.arange(T, dtype=torch.int32, device=dev) % prompt
        kc, vc, slots = rnd(T, 1, Hkv, 128), rnd(T, 1, Hkv, 128), torch.arange(T, device=dev)
        cs, gq = torch.randn(prompt, 128, device=dev), rnd(128)
        pq, pk, pv = proj.split([at.heads * 128, Hkv * 128, Hkv * 128], dim=1)
        pair(_row(f"head_norm_rope, {tag}", lambda: ops.head_norm_rope(pq, pk, pv, at.heads, Hkv, 128, gq, gq, 1e-6, cs, pos, slots, kc, vc), 4.0 * T * cols),
             _row(f"qk_norm_rope, {tag}", lambda: ops.qk_norm_rope(proj, pos, cs, at.heads, Hkv, kc.view(T, Hkv, 128), vc.view(T, Hkv, 128), slots, gq, gq),
                  4.0 * T * cols))
        del proj, kc, vc
        # ---- products of another form than the partner's
        x, w = rnd(T, 5, W), rnd(4 * N + 128, W)
        xl = rnd(T, W)
        new = _row(f"linear_groups, five inputs, {tag}", lambda: ops.linear_groups(x, w, [N] * 4 + [128]), 2.0 * (w.numel() + x.numel() + T * w.shape[0]),
                   2.0 * T * w.numel())
        big = _row(f"linear of equal size, {tag}", lambda: ops.linear(xl, w), 2.0 * (w.numel() + xl.numel() + T * w.shape[0]), 2.0 * T * w.numel())
        pair(new, big)
        low, w2 = rnd(T, m.decay_rank), rnd(N, m.decay_rank)
        pair(_row(f"tanh_linear, rank {m.decay_rank}, {tag}", lambda: ops.tanh_linear(low, w2),
                  2.0 * (low.numel() + w2.numel() + T * N), 2.0 * T * w2.numel()),
             _row(f"linear of equal size, {tag}", lambda: ops.linear(low, w2), 2.0 * (low.numel() + w2.numel() + T * N), 2.0 * T * w2.numel()))
        del x
    ops.check_pipeline_status()
    torch.cuda.empty_cache()
    return pairs


def run(models: list[str], batch: int, prompt: int, steps: int, warmup: int, with_kernels: bool = True, group=None) -> dict:
    torch.manual_seed(0)
    out = {"workload": "sizilorn", "batch": batch, "prompt": prompt, "steps": steps, "dtype": "bf16", "data": "synthetic, random weights",
           "peaks": peaks()[2], "l2": "weights exceed the L2; kernel rows flush it before every call", "models": [], "kernels": {}}
    for name in models:
        new = throughput(name, batch, prompt, steps, warmup, group)
        like = throughput(partner(name), batch, prompt, steps, warmup, group)
        out["models"].append({"sizilorn": new, "qwen3": like})
    if with_kernels:
        for name in models:
            out["kernels"][name] = kernels(name, batch, prompt)
    return out
