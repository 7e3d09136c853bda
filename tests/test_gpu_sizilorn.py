"""Sizilorn on one GPU: every mechanism's kernel and the whole model against the plain implementation in ``ref/sizilorn.py``."""
import json
import os
import subprocess
import sys

import pytest
import torch

import sizilorn_cases as sc
from triton_distributed_b200 import ref

pytestmark = pytest.mark.gpu

TOL = {torch.float32: 2e-4, torch.bfloat16: 0.06, torch.float16: 0.01}
DTYPES = [torch.float32, torch.bfloat16, torch.float16]


def _close(got, want, dtype, factor=1.0):
    d = (got.double().cpu() - want.double().cpu()).pow(2).mean().sqrt()
    assert torch.isfinite(got).all()
    assert d <= factor * {torch.float32: 2e-6, torch.bfloat16: 6e-3, torch.float16: 8e-4}[dtype] * want.double().pow(2).mean().sqrt(), d


@pytest.fixture(autouse=True)
def _own_random_numbers():
    """The tests here draw from a fixed stream and leave the global ones as they found them."""
    with torch.random.fork_rng(devices=[0]):
        torch.manual_seed(11)
        yield


def _d(t):
    return t.double().cpu()


# ------------------------------------------------------------------------------------------------ the stream between two GEMMs
def _rows(T, width, dtype, scale=1.0):
    t = torch.zeros(T, (width + 7) // 8 * 8, device="cuda", dtype=dtype)
    t[:, :width] = torch.randn(T, width) * scale
    return t


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,width", [(5, 75), (3, 2048), (200, 1100), (30, 5120), (2, 9001)])
@pytest.mark.parametrize("two", [False, True])
def test_residual_post(dtype, T, width, two):
    from triton_distributed_b200 import ops
    x, a, b = _rows(T, width, torch.float32), _rows(T, width, dtype, 3.0), _rows(T, width, dtype, 0.01)
    ga, gb, gain, bias = (_rows(1, width, dtype)[0] for _ in range(4))
    x0 = x.clone()
    for kind in (ops.TanhNorm(0.8), ops.COPY, True, None):
        x.copy_(x0)
        kw = {} if kind is None else {"center": kind} if kind == ops.COPY else {"center": kind, "gain": gain, "bias": bias, "eps": 1e-4}
        h = ops.residual_post(x, width, 0.5, a, ga, b if two else None, gb if two else None, 1e-5, **kw)
        want = _d(x0)[:, :width] + 0.5 * ref.unit_rms_ref(_d(a)[:, :width], 1e-5) * _d(ga)[:width]
        if two:
            want = want + 0.5 * ref.unit_rms_ref(_d(b)[:, :width], 1e-5) * _d(gb)[:width]
        _close(x[:, :width], want, torch.float32)
        assert torch.all(x[:, width:] == 0)
        if kind is None:
            assert h is None
            continue
        if kind == ops.COPY:
            assert torch.equal(h, x.to(dtype))
            continue
        g, c = _d(gain)[:width], _d(bias)[:width]
        _close(h[:, :width], ref.layer_norm_ref(want, g, c, 1e-4) if kind is True else ref.tanh_norm_ref(want, 0.8, g, c), dtype)
        assert torch.all(h[:, width:] == 0)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,width", [(4, 75), (3, 2048), (170, 1030)])
def test_tanh_norm_of_embedding_and_residual(dtype, T, width):
    from triton_distributed_b200 import ops
    table, gain, bias = _rows(30, width, dtype, 2.0), _rows(1, width, dtype)[0], _rows(1, width, dtype)[0]
    ids = torch.randint(0, 30, (T,), device="cuda")
    x, h = ops.embed_norm(ids, table, 1.0, width, gain, bias, 0.0, ops.TanhNorm(0.6))
    assert torch.equal(x, table[ids].float())
    g, c = _d(gain)[:width], _d(bias)[:width]
    _close(h[:, :width], ref.tanh_norm_ref(_d(x)[:, :width], 0.6, g, c), dtype)
    a = _rows(T, width, dtype)
    want = _d(x) + _d(a)
    h = ops.residual_norm(x, width, 1.0, a, gain=gain, bias=bias, center=ops.TanhNorm(1.3))
    _close(x, want, torch.float32)
    _close(h[:, :width], ref.tanh_norm_ref(want[:, :width], 1.3, g, c), dtype)
    h = ops.residual_norm(x, width, 1.0, a, center=ops.COPY)
    assert torch.equal(h, x.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,dim,layer", [(1, 7, 2), (50, 16, 0), (9, 130, 3)])
def test_token_side(dtype, T, dim, layer):
    from triton_distributed_b200 import ops
    P, V = (dim + 7) // 8 * 8, 40
    table, g = torch.randn(V, 4 * dim, device="cuda").to(dtype), (2 * torch.randn(T, P, device="cuda")).to(dtype)
    ids = torch.randint(0, V, (T,), device="cuda")
    act = ops.token_side(g, ids, table, layer * dim, dim)
    want = ref.gelu_tanh_ref(_d(g)[:, :dim]) * _d(table)[ids.cpu()][:, layer * dim:(layer + 1) * dim]
    _close(act[:, :dim], want, dtype)
    assert torch.all(act[:, dim:] == 0)
    ids[0] = V                                      # outside the table: zeros
    assert torch.all(ops.token_side(g, ids, table, layer * dim, dim)[0] == 0)


# ------------------------------------------------------------------------------------------------ projections
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,K,rows", [(1, 8, [128, 256]), (7, 72, [384, 128, 128, 256, 128]), (40, 520, [128, 640, 128]), (300, 64, [256, 128])])
def test_linear_groups(dtype, T, K, rows):
    """Every group of rows multiplies its own input, also when the row length is not a whole number of k-blocks."""
    from triton_distributed_b200 import ops
    G = len(rows)
    x, w = torch.randn(T, G, K, device="cuda").to(dtype), torch.randn(sum(rows), K, device="cuda").to(dtype)
    got = ops.linear_groups(x, w, rows).split(rows, dim=1)
    for g, part in enumerate(w.split(rows)):
        _close(got[g], _d(x[:, g]) @ _d(part).t(), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,N,K", [(1, 40, 8), (33, 264, 64), (300, 128, 136), (5, 72, 264)])
def test_tanh_linear(dtype, T, N, K):
    from triton_distributed_b200 import ops
    wide = torch.randn(T, K + 16, device="cuda").to(dtype)
    w = torch.randn(N, K, device="cuda").to(dtype)
    want = torch.tanh(_d(wide[:, 8:8 + K])) @ _d(w).t()
    _close(ops.tanh_linear(wide[:, 8:8 + K], w), want, dtype, factor=1.5)
    _close(ops.head_linear(wide[:, None, 8:8 + K], w[None], tanh=True)[:, 0], want, dtype, factor=1.5)


# ------------------------------------------------------------------------------------------------ carried inputs
def _cuts(S):
    return [[S], [1] * S, [2] * (S // 2) + [1] * (S % 2), [1, S - 1], [S - 2, 1, 1], [3, 16, 2, S - 21]]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("P,G", [(8, 1), (80, 5), (1032, 8)])
def test_token_mix(dtype, P, G):
    from triton_distributed_b200 import ops
    S, B = 37, 3
    h, mu = torch.randn(B, S, P, device="cuda").to(dtype), torch.rand(G, P, device="cuda").to(dtype)
    want = torch.stack([torch.stack([ref.token_mix_ref(_d(h[b]), _d(mu[g])) for g in range(G)], 1) for b in range(B)])
    for cut in _cuts(S):
        last, out, at = torch.zeros(B, P, device="cuda", dtype=dtype), [], 0
        for n in cut:
            out.append(ops.token_mix(h[:, at:at + n].reshape(B * n, P).contiguous(), mu, last).view(B, n, G, P))
            at += n
        _close(torch.cat(out, 1), want, dtype)
        assert torch.equal(last, h[:, -1])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("C,taps", [(8, 1), (24, 2), (520, 3), (72, 4), (16, 5), (8, 9)])
def test_short_conv(dtype, C, taps):
    from triton_distributed_b200 import ops
    S, B = 37, 2
    wide = torch.randn(B, S, C + 16, device="cuda").to(dtype)
    x, w = wide[..., 8:8 + C], torch.randn(C, taps, device="cuda")
    want = torch.stack([ref.swish_ref(ref.short_conv_ref(_d(x[b]), _d(w))) for b in range(B)])
    first = None
    for cut in _cuts(S):
        last, out, at = torch.zeros(B, taps - 1, C, device="cuda", dtype=dtype), [], 0
        for n in cut:
            part = wide[:, at:at + n].reshape(B * n, C + 16).contiguous()[:, 8:8 + C]
            out.append(ops.short_conv(part, w.t().contiguous(), last).view(B, n, C))
            at += n
        out = torch.cat(out, 1)
        _close(out, want, dtype)
        assert torch.equal(last, x[:, S - taps + 1:])
        first = out if first is None else first
        assert torch.equal(out, first)


# ------------------------------------------------------------------------------------------------ recurrences
def _pad_heads(x, size):
    out = torch.zeros(*x.shape[:-1], size, dtype=x.dtype, device=x.device)
    out[..., : x.shape[-1]] = x
    return out.flatten(-2)


def _wkv_case(B, S, H, D, E, dtype):
    Dp, Ep = (D + 7) // 8 * 8, (E + 7) // 8 * 8
    r, k, z = (torch.randn(B * S, H, D, device="cuda").to(dtype) for _ in range(3))
    v, gate = (torch.randn(B * S, H, E, device="cuda").to(dtype) for _ in range(2))
    w0 = torch.empty(H, D, device="cuda").uniform_(-7.0, 0.5)
    u, gain = torch.randn(H, D, device="cuda"), torch.randn(H, E, device="cuda")
    state = torch.randn(B, H, D, E, device="cuda")

    def run(plain, cut):
        st = torch.zeros(B, H, Dp, Ep, device="cuda")
        st[:, :, :D, :E] = state
        from triton_distributed_b200 import ops
        out, at = [], 0
        for n in cut:
            rows = [_pad_heads(t.view(B, S, *t.shape[1:])[:, at:at + n].reshape(B * n, *t.shape[1:]), p)
                    for t, p in ((r, Dp), (k, Dp), (v, Ep), (z, Dp), (gate, Ep))]
            wide = torch.cat([rows[0], rows[1]], 1)            # column slices of a wider output
            rows[0], rows[1] = wide[:, : H * Dp], wide[:, H * Dp:]
            o = ops.wkv(*rows, _pad_heads(w0, Dp), _pad_heads(u, Dp), _pad_heads(gain, Ep), st, D, E, 1e-3, plain=plain)
            assert torch.all(o.view(-1, H, Ep)[..., E:] == 0)
            out.append(o.view(B, n, H, Ep)[..., :E])
            at += n
        assert torch.all(st[:, :, D:] == 0) and torch.all(st[..., E:] == 0)
        return torch.cat(out, 1), st[:, :, :D, :E]

    def oracle():
        outs, states = [], []
        for b in range(B):
            sl = slice(b * S, (b + 1) * S)
            w = torch.exp(-torch.exp(_d(z[sl]) + _d(w0)))
            o, st = ref.decayed_outer_ref(_d(r[sl]), _d(k[sl]), _d(v[sl]), w, _d(u), _d(state[b]))
            outs.append(ref.unit_rms_ref(o, 1e-3) * _d(gain) * ref.swish_ref(_d(gate[sl])))
            states.append(st)
        return torch.stack(outs), torch.stack(states)
    return run, oracle


def _delta_case(B, S, H, D, E, dtype):
    G = max(1, H // 2)
    Dp, Ep, Hp = (D + 7) // 8 * 8, (E + 7) // 8 * 8, (H + 7) // 8 * 8
    q, k = (torch.randn(B * S, G, D, device="cuda").to(dtype) for _ in range(2))
    v, gate = (torch.randn(B * S, H, E, device="cuda").to(dtype) for _ in range(2))
    ab = torch.randn(B * S, 2 * Hp, device="cuda").to(dtype)
    a_log, dt, gain = torch.randn(H, device="cuda") - 1, torch.randn(H, device="cuda") - 2, torch.randn(E, device="cuda")
    state = torch.randn(B, H, D, E, device="cuda")

    def run(plain, cut):
        from triton_distributed_b200 import ops
        st = torch.zeros(B, H, Dp, Ep, device="cuda")
        st[:, :, :D, :E] = state
        out, at = [], 0
        for n in cut:
            def part(t):
                return t.view(B, S, *t.shape[1:])[:, at:at + n].reshape(B * n, *t.shape[1:])
            pab = part(ab)
            o = ops.gated_delta(_pad_heads(part(q), Dp), _pad_heads(part(k), Dp), _pad_heads(part(v), Ep), pab[:, :H], pab[:, Hp:Hp + H],
                                _pad_heads(part(gate), Ep), a_log, dt, torch.nn.functional.pad(gain, (0, Ep - E)), st, D, E, 1e-3, plain=plain)
            assert torch.all(o.view(-1, H, Ep)[..., E:] == 0)
            out.append(o.view(B, n, H, Ep)[..., :E])
            at += n
        assert torch.all(st[:, :, D:] == 0) and torch.all(st[..., E:] == 0)
        return torch.cat(out, 1), st[:, :, :D, :E]

    def oracle():
        outs, states = [], []
        for b in range(B):
            sl = slice(b * S, (b + 1) * S)
            g = torch.exp(-torch.exp(_d(a_log)) * ref.softplus_ref(_d(ab[sl, :H]) + _d(dt)))
            o, st = ref.gated_delta_ref(ref.unit_vector_ref(_d(q[sl])) * D ** -0.5, ref.unit_vector_ref(_d(k[sl])), _d(v[sl]), g,
                                        ref.sigmoid_ref(_d(ab[sl, Hp:Hp + H])), _d(state[b]))
            outs.append(ref.unit_rms_ref(o, 1e-3) * _d(gain) * ref.swish_ref(_d(gate[sl])))
            states.append(st)
        return torch.stack(outs), torch.stack(states)
    return run, oracle


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("case", [_wkv_case, _delta_case], ids=["wkv", "delta"])
@pytest.mark.parametrize("B,S,H,D,E", [(1, 35, 2, 8, 8), (2, 24, 4, 64, 64), (1, 33, 2, 20, 13), (1, 23, 2, 65, 128), (2, 25, 2, 128, 72), (1, 24, 1, 136, 24),
                                       (37, 21, 4, 24, 16), (37, 21, 4, 72, 100)])
def test_recurrences(case, dtype, B, S, H, D, E):
    run, oracle = case(B, S, H, D, E, dtype)
    want, state = oracle()
    for plain in (False, True):
        got, st = run(plain, [S])
        _close(got, want, dtype, factor=3.0)
        _close(st, state, torch.float32, factor=3.0)
        for cut in _cuts(S)[1:]:
            o2, st2 = run(plain, cut)
            _close(o2, got, dtype, factor=0.2 if plain else 1.0)
            _close(st2, st, torch.float32, factor=0.1 if plain else 1.0)


@pytest.mark.parametrize("plain", [False, True])
@pytest.mark.parametrize("place", [0, 15, 16, 17, 100])
def test_a_far_token_is_remembered(plain, place):
    """One token writes far more than the others and is read, almost undecayed, a few hundred tokens later, and not before it."""
    from triton_distributed_b200 import ops
    S, H, D = 300, 2, 24
    k, r = 0.01 * torch.randn(S, H, D, device="cuda"), 0.01 * torch.randn(S, H, D, device="cuda")
    v = torch.randn(S, H, D, device="cuda")
    k[place, :, 3], r[:, :, 3] = 50.0, 1.0
    zero, gate = torch.zeros(S, H * D, device="cuda"), torch.full((S, H * D), 20.0, device="cuda")
    one = torch.ones(H * D, device="cuda")
    st = torch.zeros(1, H, D, D, device="cuda")
    out = ops.wkv(r.flatten(1), k.flatten(1), v.flatten(1), zero, gate, -14.0 * one, one, one, st, D, D, 1e-9, plain=plain).view(S, H, D).cpu()
    want = ref.unit_rms_ref(v[place].double().cpu(), 1e-9)
    for t in (place, place + 1, place + 16, 299):
        assert (out[t] / 20 - want).abs().max() < 0.1, t
    if place:
        assert (out[place - 1] / 20 - want).abs().max() > 0.5
    # the delta rule: with a full step the memory gives back what was stored under this key, until it is overwritten
    ab = torch.full((S, 2 * 8), -30.0, device="cuda")
    ab[place, 8:] = 30.0                                     # step size 1 at the place, 0 elsewhere; no decay
    st = torch.zeros(1, H, D, D, device="cuda")
    kk = torch.randn(S, H, D, device="cuda")
    kk[-1] = kk[place]
    out = ops.gated_delta(kk.flatten(1), kk.flatten(1), v.flatten(1), ab[:, :H], ab[:, 8:8 + H], gate, torch.zeros(H, device="cuda"),
                          torch.zeros(H, device="cuda"), one[:D], st, D, D, 1e-9, plain=plain).view(S, H, D).cpu()
    assert (out[-1] / 20 - want).abs().max() < 1e-3 and (out[place] / 20 - want).abs().max() < 1e-3
    if place:
        assert out[place - 1].abs().max() < 1e-3


# ------------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,E,rot,Dc,Ec,norm", [(4, 2, 18, 13, 10, 128, 128, True), (3, 3, 64, 64, 64, 64, 64, True), (2, 1, 200, 136, 100, 200, 136, True),
                                                    (8, 1, 128, 96, 0, 128, 128, True), (2, 2, 26, 30, 26, 32, 32, False)])
def test_head_norm_rope(dtype, H, G, D, E, rot, Dc, Ec, norm):
    from triton_distributed_b200 import ops
    from triton_distributed_b200.layers.nvidia.gated_attn import rotation_table
    from triton_distributed_b200.models.config import RotarySpec
    T, Di, Ei = 6, (D + 7) // 8 * 8, (E + 7) // 8 * 8
    q, k, v = (torch.randn(T, n, s, device="cuda").to(dtype) for n, s in ((H, D), (G, D), (G, E)))
    proj = torch.cat([_pad_heads(q, Di), _pad_heads(k, Di), _pad_heads(v, Ei), torch.randn(T, 8, device="cuda").to(dtype)], 1)
    qs, ks, vs = proj[:, : H * Di], proj[:, H * Di:(H + G) * Di], proj[:, (H + G) * Di:(H + G) * Di + G * Ei]
    gq, gk = (torch.randn(D, device="cuda").to(dtype) for _ in range(2))
    pos = [0, 1, 63, 64, 500, 77]
    slots = torch.tensor([5, 0, 63, 64, -1, 127], device="cuda")
    kc, vc = torch.full((2, 64, G, Dc), 9.0, device="cuda", dtype=dtype), torch.full((2, 64, G, Ec), 9.0, device="cuda", dtype=dtype)
    table = rotation_table(RotarySpec(rot, 700.0), 501, "cuda")
    out = ops.head_norm_rope(qs, ks, vs, H, G, D, gq if norm else None, gk if norm else None, 1e-3, table,
                             torch.tensor(pos, dtype=torch.int32, device="cuda"), slots, kc, vc, q_scale=0.3)
    wq = sc.rotation(ref.unit_rms_ref(_d(q), 1e-3) * _d(gq) if norm else _d(q), pos, rot, 700.0) * 0.3
    wk = sc.rotation(ref.unit_rms_ref(_d(k), 1e-3) * _d(gk) if norm else _d(k), pos, rot, 700.0)
    _close(out[..., :D], wq, dtype)
    assert torch.all(out[..., D:] == 0)
    keep = slots >= 0
    flat_k, flat_v = kc.view(128, G, Dc), vc.view(128, G, Ec)
    _close(flat_k[slots[keep]][..., :D], wk[keep.cpu()], dtype)
    assert torch.equal(flat_v[slots[keep]][..., :E], v[keep]) and torch.all(flat_k[slots[keep]][..., D:] == 0) and torch.all(flat_v[slots[keep]][..., E:] == 0)
    untouched = torch.ones(128, dtype=torch.bool)
    untouched[slots[keep].cpu()] = False
    assert torch.all(flat_k.cpu()[untouched] == 9.0) and torch.all(flat_v.cpu()[untouched] == 9.0)


def _attend(kind, q, kc, vc, lens, S, gate):
    """q [B * S, H, D]; caches [blocks, page, G, *] with every sequence's pages in a row."""
    from triton_distributed_b200 import ops
    B, page = len(lens), kc.shape[1]
    per = kc.shape[0] // B
    kv = torch.tensor(lens, dtype=torch.int32, device="cuda")
    table = torch.arange(kc.shape[0], dtype=torch.int32, device="cuda").view(B, per)
    if kind == "plain":
        return ops.gqa_attention_plain(q, kc, vc, kv, table, S, 1.0, gate=gate)
    if kind == "decode":
        return torch.stack([ops.decode_attention(q, kc, vc, kv, table, 1.0, 0.0, n, gate=gate) for n in (1, 3, 8)])
    cu_q = torch.arange(0, (B + 1) * S, S, dtype=torch.int32, device="cuda")
    cu_k = torch.arange(0, (B + 1) * per * page, per * page, dtype=torch.int32, device="cuda")
    return ops.prefill_attention(q, kc.view(-1, *kc.shape[2:]), vc.view(-1, *vc.shape[2:]), cu_q, cu_k, S, max(lens), 1.0, True, seqlens_k=kv, gate=gate)


@pytest.mark.parametrize("kind,dtype,H,G,D,E,S,lens", [
    ("plain", torch.float32, 4, 2, 20, 12, 3, [3, 130, 64]), ("plain", torch.bfloat16, 2, 1, 264, 40, 1, [65, 1]),
    ("plain", torch.float16, 6, 6, 8, 136, 9, [200, 9]), ("decode", torch.bfloat16, 8, 2, 128, 128, 1, [1, 64, 65, 300]),
    ("decode", torch.float16, 20, 1, 128, 128, 1, [129, 700]), ("prefill", torch.bfloat16, 4, 2, 40, 24, 150, [150, 215]),
    ("prefill", torch.float16, 2, 2, 200, 136, 2, [130, 2]), ("prefill", torch.bfloat16, 8, 1, 128, 128, 130, [257]),
    ("prefill", torch.bfloat16, 2, 1, 256, 264, 33, [100])])
def test_gated_attention_kernels(kind, dtype, H, G, D, E, S, lens):
    B, page = len(lens), 64
    per = (max(lens) + page - 1) // page
    kc, vc = torch.randn(B * per, page, G, D, device="cuda").to(dtype), torch.randn(B * per, page, G, E, device="cuda").to(dtype)
    q = (torch.randn(B * S, H, D, device="cuda") * 2 / D ** 0.5).to(dtype)
    wide = torch.randn(B * S, H + 12, device="cuda").to(dtype)
    gate = wide[:, 4:4 + H]
    got = _attend(kind, q, kc, vc, lens, S, gate)
    for b, n in enumerate(lens):
        rows = slice(b * S, (b + 1) * S)
        k, v = (_d(c.view(B, per * page, G, -1)[b, :n]) for c in (kc, vc))
        want = ref.grouped_attention_ref(_d(q[rows]), k, v, 1.0, n - S) * ref.sigmoid_ref(_d(gate[rows]))[:, :, None]
        for o in (got if kind == "decode" else [got]):
            _close(o[rows], want, dtype, factor=2.0)
    bare = _attend(kind, q, kc, vc, lens, S, None)
    _close((bare * torch.sigmoid(gate.float())[:, :, None].to(dtype)), got, dtype, factor=2.0)


@pytest.mark.parametrize("kind,n,S", [("plain", 70, 3), ("plain", 321, 1), ("decode", 1, 1), ("decode", 65, 1), ("decode", 321, 1), ("prefill", 265, 150),
                                      ("prefill", 130, 2)])
def test_attention_sees_exactly_the_keys_up_to_its_own(kind, n, S):
    """One key at a time dwarfs the others: rows at or after it return its value, rows before it must not notice it."""
    H, D, page = 2, 128, 64
    per = (n + page - 1) // page
    q = torch.zeros(S, H, D, device="cuda", dtype=torch.bfloat16)
    q[..., 0] = 8.0
    gate = torch.full((S, H), 20.0, device="cuda", dtype=torch.bfloat16)
    for j in sorted({0, 1, 63, 64, 65, 127, 128, n - S - 1, n - S, n - 2, n - 1} & set(range(n))):
        kc, vc = (torch.randn(per, page, H, D, device="cuda") * 0.05).bfloat16(), torch.zeros(per, page, H, D, device="cuda", dtype=torch.bfloat16)
        kc[..., 0] = 0.0
        kc.view(-1, H, D)[j, :, 0], vc.view(-1, H, D)[j] = 8.0, 1.0
        if n % page:
            kc.view(-1, H, D)[n:, :, 0], vc.view(-1, H, D)[n:] = 30.0, 5.0     # slots that hold no token of the sequence
        got = _attend(kind, q, kc, vc, [n], S, gate)
        seen = (torch.arange(S) + n - S >= j).float()
        for o in (got if kind == "decode" else [got]):
            assert (o[:, :, 7].float().cpu() - seen[:, None]).abs().max() < 0.02, j


# ------------------------------------------------------------------------------------------------ the model
_refs = {}


def _case(name, n=170, seed=0):
    """(config, weights, tokens, oracle logits and streams); computed once per module."""
    key = (name, n, seed)
    if key not in _refs:
        cfg, w = sc.named(name)
        toks = sc.tokens_for(cfg, n, seed)
        _refs[key] = (cfg, w, toks, ref.sizilorn_ref(toks, cfg, w))
    return _refs[key]


def _engine(tmp_path, name, dtype, max_length=256):
    from triton_distributed_b200.models import Engine, ModelConfig
    cfg, w = sc.named(name)
    path = sc.save(tmp_path / name, cfg, w)
    return Engine(ModelConfig(model_name=name, checkpoint_dir=path, max_length=max_length, dtype=dtype, rank=0, world_size=1), temperature=0.0)


def _run(eng, toks, cuts):
    """Feed one sequence (or several of equal length: toks [bsz][n]) in portions; logits of every position."""
    from triton_distributed_b200 import ops
    rows = toks if isinstance(toks[0], list) else [toks]
    ids = torch.tensor(rows, device="cuda")
    eng.start(ids.shape[0])
    out, at, i = [], 0, 0
    while at < ids.shape[1]:
        n = min(cuts[min(i, len(cuts) - 1)], ids.shape[1] - at)
        i += 1
        out.append(eng.extend(ids[:, at:at + n], want=list(range(n))).cpu().clone())
        at += n
    ops.check_pipeline_status()
    return torch.cat(out, 1)


MODES = [("odd", torch.float32), ("odd", torch.bfloat16), ("odd", torch.float16), ("equal", torch.float32), ("equal", torch.bfloat16),
         ("wide", torch.float32), ("wide", torch.bfloat16), ("large", torch.float32), ("large", torch.bfloat16)]


@pytest.mark.parametrize("name,dtype", MODES)
def test_whole_prompt_and_stream_after_every_layer(tmp_path, name, dtype):
    cfg, w, toks, (want, after) = _case(name)
    eng = _engine(tmp_path, name, dtype)
    eng.model.layer_taps = []
    got = _run(eng, toks, [len(toks)])[0]
    assert got.shape == want.shape
    assert sc.rms_error(got, want).max() < TOL[dtype]
    for i, x in enumerate(eng.model.layer_taps):
        _close(x, after[i], dtype, factor=8.0)
    assert len(eng.model.layer_taps) == len(cfg["layers"])


@pytest.mark.parametrize("name,dtype", [("odd", torch.float32), ("odd", torch.bfloat16), ("wide", torch.bfloat16), ("large", torch.bfloat16),
                                        ("equal", torch.float32)])
@pytest.mark.parametrize("cuts", [[1], [2], [17], [3, 40, 1, 2, 64, 5, 1], [63, 1, 64, 1, 33, 8], [15, 2, 16, 1], [168, 1]])
def test_portions_do_not_change_the_logits(tmp_path, name, dtype, cuts):
    _, _, toks, (want, _) = _case(name)
    got = _run(_engine(tmp_path, name, dtype), toks, cuts)[0]
    assert sc.rms_error(got, want).max() < TOL[dtype]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_slots_and_states_are_reused_without_a_trace(tmp_path, dtype):
    """A long request, then others in the same slots and states: as if the engine were new."""
    cfg, w, toks, (want, _) = _case("odd")
    eng = _engine(tmp_path, "odd", dtype)
    _run(eng, sc.tokens_for(cfg, 250, 9), [120, 1, 2, 90, 1])
    for cuts in ([170], [1, 2, 30, 1, 70, 1]):
        assert sc.rms_error(_run(eng, toks, cuts)[0], want).max() < TOL[dtype]
    one = _run(eng, toks[:1], [1])[0]
    assert sc.rms_error(one, want[:1]).max() < TOL[dtype]


@pytest.mark.parametrize("name,dtype", [("odd", torch.float32), ("wide", torch.bfloat16)])
def test_batches_against_each_alone(tmp_path, name, dtype):
    cfg, w = sc.named(name)
    rows = [sc.tokens_for(cfg, 100, s) for s in (3, 4, 5)]
    wants = [ref.sizilorn_ref(r, cfg, w)[0] for r in rows]
    eng = _engine(tmp_path, name, dtype)
    for cuts in ([100], [40, 2, 1, 1, 37, 3]):
        together = _run(eng, rows, cuts)
        for b, r in enumerate(rows):
            assert sc.rms_error(together[b], wants[b]).max() < TOL[dtype]
            alone = _run(eng, r, cuts)[0]
            assert sc.rms_error(together[b], alone).max() < TOL[dtype]


def test_long_decoding(tmp_path):
    _, _, toks, (want, _) = _case("odd", 420)
    for dtype in (torch.float32, torch.bfloat16):
        got = _run(_engine(tmp_path, "odd", dtype, max_length=420), toks, [20] + [1] * 400)[0]
        assert sc.rms_error(got, want).max() < TOL[dtype]


def test_greedy_generation_through_the_engine(tmp_path):
    cfg, w = sc.named("odd")
    prompts = [sc.tokens_for(cfg, 40, s) for s in (21, 24)]
    wanted = [ref.sizilorn_greedy_ref(p, 16, cfg, w) for p in prompts]

    def agrees(out, least_margin, at_least):
        for b, (want, margins) in enumerate(wanted):
            n = next((i for i, m in enumerate(margins) if m < least_margin), 16)   # a near tie may fall either way
            assert n >= at_least and out[b, : 40 + n].tolist() == prompts[b] + want[:n]

    ids = torch.tensor(prompts, device="cuda")
    agrees(_engine(tmp_path, "odd", torch.float32).serve(ids, gen_len=16).cpu(), 2e-3, 13)
    for no_graph in (False, True):
        e = _engine(tmp_path, "odd", torch.bfloat16)
        e.no_graph = no_graph
        agrees(e.serve(ids, gen_len=16).cpu(), 0.2, 4)
        again = e.serve(ids, gen_len=16).cpu()               # the same engine, the captured step used again
        agrees(again, 0.2, 4)
    e.temperature = 0.8                                   # top-p sampling takes the same logits
    s = e.serve(ids, gen_len=5)
    assert s.shape == (2, 45) and int(s.max()) < cfg["vocab"]


def test_named_architecture_runs():
    from triton_distributed_b200.models import Engine, ModelConfig
    eng = Engine(ModelConfig(model_name="tiny-sizilorn", max_length=128, rank=0, world_size=1), temperature=0.0)
    out = eng.serve(torch.randint(0, 1000, (2, 50), device="cuda"), gen_len=6)
    assert out.shape == (2, 56)
    with pytest.raises(ValueError, match="triton_dist_AR"):
        eng.model.set_fwd("torch")


def test_trace_replay(tmp_path):
    cfg, w, toks, (want, _) = _case("odd")
    path = sc.save(tmp_path / "m", cfg, w)
    other = sc.tokens_for(cfg, 50, 8)
    want2, _ = ref.sizilorn_ref(other, cfg, w)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:60], "want": [59, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[60:61], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[61:63], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": toks[63:], "want": [0, 1, 106]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": other, "want": [0, 49]}], "end": ["b"]}]
    places = {0: (want, [59, 3]), 1: (want, [60]), 3: (want, [63, 64, 169]), 4: (want2, [0, 49])}
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    for dtype in (torch.float32, torch.bfloat16):
        out = tmp_path / str(dtype)
        r = subprocess.run([sys.executable, exe, "--model", path, "--dtype", str(dtype).split(".")[1], "--out", str(out), "--max-tokens", "170"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
        assert sorted(os.listdir(out)) == ["0.f32", "1.f32", "3.f32", "4.f32"]
        for i, (ref_logits, rows) in places.items():
            got = torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(len(rows), -1)
            assert sc.rms_error(got, ref_logits[rows]).max() < TOL[dtype]
