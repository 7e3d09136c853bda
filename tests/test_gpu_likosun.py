"""Likosun on one GPU: every mechanism's kernel and the whole model against the plain implementation in ``ref/likosun.py``."""
import json
import os
import subprocess
import sys

import pytest
import torch

import likosun_cases as lc
from triton_distributed_b200 import ref

pytestmark = pytest.mark.gpu

TOL = {torch.float32: 1e-4, torch.bfloat16: 0.025, torch.float16: 6e-3}


def _close(got, want, dtype, factor=1.0):
    d = (got.double().cpu() - want.double().cpu()).pow(2).mean().sqrt()
    assert torch.isfinite(got).all()
    assert d <= factor * {torch.float32: 2e-6, torch.bfloat16: 6e-3, torch.float16: 8e-4}[dtype] * want.double().pow(2).mean().sqrt(), d


@pytest.fixture(autouse=True)
def _own_random_numbers():
    """The tests here draw from a fixed stream and leave the global ones as they found them."""
    with torch.random.fork_rng(devices=[0]):
        torch.manual_seed(7)
        yield


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("M,N,K", [(1, 1, 1), (5, 70, 33), (64, 64, 16), (130, 200, 257), (300, 65, 1024)])
def test_gemm_f32_is_true_fp32(M, N, K):
    from triton_distributed_b200 import ops
    a, b = torch.randn(M, K + 3, device="cuda")[:, :K], torch.randn(N, K, device="cuda")
    out = torch.full((M, N + 5), 7.0, device="cuda")
    ops.gemm_f32(a, b, out[:, :N])
    _close(out[:, :N], a.double() @ b.double().t(), torch.float32)
    assert torch.all(out[:, N:] == 7.0)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, torch.float16])
@pytest.mark.parametrize("width,center,with_bias", [(75, True, True), (1030, True, True), (2052, False, True), (1000, False, False), (2048, True, False), (5120, True, True), (9001, True, True)])
def test_embed_norm(dtype, width, center, with_bias):
    from triton_distributed_b200 import ops
    P, V = (width + 7) // 8 * 8, 50
    table = torch.zeros(V, P, device="cuda", dtype=dtype)
    table[:, :width] = torch.randn(V, width) + 0.5
    gain, bias = torch.zeros(P, device="cuda", dtype=dtype), torch.zeros(P, device="cuda", dtype=dtype)
    gain[:width] = torch.randn(width)
    bias[:width] = torch.randn(width)
    ids = torch.tensor([[3, 49, 0], [49, 7, V]], device="cuda")  # the last id is outside the table: a zero row
    state0 = torch.empty(6, P, device="cuda")
    x, h = ops.embed_norm(ids, table, 3.5, width, gain, bias if with_bias else None, 1e-3, center, state0=state0)
    rows = torch.zeros(6, width, dtype=torch.float64)
    rows[:5] = table[ids.reshape(-1)[:5], :width].double().cpu() * 3.5
    assert torch.equal(x, state0) and torch.all(x[:, width:] == 0) and torch.all(h[:, width:] == 0)
    _close(x[:, :width], rows, torch.float32)
    g, b = gain[:width].double().cpu(), bias[:width].double().cpu() * (1.0 if with_bias else 0.0)
    want = ref.layer_norm_ref(rows, g, b, 1e-3) if center else ref.rms_norm_ref(rows, g, 1e-3) + b
    _close(h[:, :width], want, dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("width,n_prev,two,gates,keep,norm", [
    (75, 1, True, True, True, True), (264, 7, False, True, True, True), (2048, 3, True, False, False, True),
    (4100, 12, True, True, True, True), (16, 0, True, True, False, True), (640, 2, True, True, True, False), (1100, 5, True, True, True, True), (6000, 1, True, True, True, True), (2500, 2, True, True, True, False)])
@pytest.mark.parametrize("T", [5, 30, 170])
def test_residual_norm(dtype, width, n_prev, two, gates, keep, norm, T):
    """Few rows take a cluster of CTAs per row (from 1024 columns on), many one CTA each."""
    from triton_distributed_b200 import ops
    P = (width + 7) // 8 * 8

    def padded(*lead, dt=dtype, scale=1.0):
        t = torch.zeros(*lead, P, device="cuda", dtype=dt)
        t[..., :width] = torch.randn(*lead, width) * scale
        return t

    x, a, b = padded(T, dt=torch.float32), padded(T), padded(T)
    wide = torch.randn(T, 3 * P + 16, device="cuda").to(dtype)       # gate logits are columns of a wider GEMM output
    ga, gb = wide[:, 8:8 + P], wide[:, 8 + 2 * P:8 + 3 * P]
    ba, bb, gain, bias = padded(), padded(), padded(), padded()
    states = torch.stack([padded(T, dt=torch.float32) for _ in range(n_prev + 1)])
    weights = torch.randn(n_prev + 1, device="cuda") if n_prev else None
    x0, st0 = x.clone(), states.clone()
    h = ops.residual_norm(x, width, 0.37, a, ga if gates else None, ba if gates else None, b if two else None,
                          gb if gates and two else None, bb if gates and two else None, states=states if n_prev else None,
                          weights=weights, keep=keep, gain=gain if norm else None, bias=bias, eps=1e-4)

    def d(t):
        return t[..., :width].double().cpu()
    inf = torch.full((T, width), torch.inf, dtype=torch.float64)     # sigmoid(inf) = 1: no gate
    subs = [(d(ga) + d(ba) if gates else inf, d(a))] + ([(d(gb) + d(bb) if gates else inf, d(b))] if two else [])
    s = ref.gated_residual_ref(d(x0), 0.37, subs)
    want = s if not n_prev else ref.depth_average_ref([d(st0[j]) for j in range(n_prev)] + [s], weights.double().cpu())
    _close(x[:, :width], want, torch.float32)
    if n_prev:
        assert torch.equal(states[:n_prev], st0[:n_prev])
        if keep:
            _close(states[n_prev][:, :width], s, torch.float32)
        else:
            assert torch.equal(states[n_prev], st0[n_prev])
    if norm:
        _close(h[:, :width], ref.layer_norm_ref(want, d(gain), d(bias), 1e-4), dtype)
        assert torch.all(h[:, width:] == 0) and torch.all(x[:, width:] == 0)
    else:
        assert h is None


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("rank,inter", [(27, 104), (512, 1032), (64, 0), (0, 2048)])
def test_latent_prep(dtype, rank, inter):
    from triton_distributed_b200 import ops
    T, pitch = 7, (rank + 7) // 8 * 8
    proj = torch.randn(T, 8 + pitch + inter + 8, device="cuda").to(dtype)
    gain = torch.zeros(max(pitch, 1), device="cuda", dtype=dtype)
    gain[:rank] = torch.randn(rank)
    cache = torch.full((4, 64, max(pitch, 1)), 9.0, device="cuda", dtype=dtype)
    slots = torch.tensor([3, 63, 64, 255, 0, -1, 100], device="cuda")
    lat, up = proj[:, 8:8 + pitch], proj[:, 8 + pitch:8 + pitch + inter]
    act = ops.latent_prep(lat if rank else None, gain if rank else None, cache if rank else None, slots if rank else None, rank, 2e-3,
                          up if inter else None)
    if rank:
        flat = cache.view(256, pitch)
        keep = slots[slots >= 0]
        want = ref.rms_norm_ref(lat[slots >= 0, :rank].double().cpu(), gain[:rank].double().cpu(), 2e-3)
        _close(flat[keep][:, :rank], want, dtype)
        assert torch.all(flat[keep][:, rank:] == 0)
        untouched = torch.ones(256, dtype=torch.bool)
        untouched[keep.cpu()] = False
        assert torch.all(flat.cpu()[untouched] == 9.0)
    if inter:
        _close(act, ref.squared_relu_ref(up.double().cpu()), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16, torch.float16])
@pytest.mark.parametrize("T,H,N,K", [(1, 1, 8, 8), (3, 5, 72, 40), (8, 16, 512, 128), (8, 2, 128, 512), (33, 3, 24, 136), (70, 2, 264, 1032), (9, 4, 16, 264)])
def test_head_linear(dtype, T, H, N, K):
    from triton_distributed_b200 import ops
    wide = torch.randn(T, H * K + 24, device="cuda").to(dtype)
    x = wide[:, 8:8 + H * K].unflatten(1, (H, K))
    w = torch.randn(H, N, K, device="cuda").to(dtype)
    _close(ops.head_linear(x, w), torch.einsum("thk,hnk->thn", x.double(), w.double()), dtype)


def _paged(seqs, pitch, page, dtype, seed=0):
    """Latents of several sequences in shuffled pages; unused slots hold NaN, which must not reach any result."""
    g = torch.Generator().manual_seed(seed)
    nb = [(s.shape[0] + page - 1) // page for s in seqs]
    perm = torch.randperm(sum(nb) + 3, generator=g)
    cache = torch.full((sum(nb) + 3, page, pitch), torch.nan)
    table = torch.zeros(len(seqs), max(nb) + 1, dtype=torch.int32)
    used = 0
    for b, s in enumerate(seqs):
        for j in range(nb[b]):
            blk = int(perm[used])
            used += 1
            table[b, j] = blk
            part = s[j * page:(j + 1) * page]
            cache[blk, : part.shape[0]] = 0.0
            cache[blk, : part.shape[0], : s.shape[1]] = part
    return cache.to(dtype).cuda(), table.cuda()


def _absorbed_ref(q, c, sink, scale, first):
    """Plain attention of [T, H, r] queries over latents as keys and values."""
    eye = torch.eye(q.shape[2], dtype=q.dtype).repeat(q.shape[1], 1)
    return ref.latent_attention_ref(q, c, eye, eye, sink, scale, first)


@pytest.mark.parametrize("dtype,variant", [(torch.bfloat16, "tc"), (torch.float16, "tc"), (torch.bfloat16, "plain"),
                                           (torch.float32, "plain")])
@pytest.mark.parametrize("H,S,rank,lens,splits,page", [
    (1, 1, 8, [1, 2, 63, 64, 65], 1, 64), (6, 1, 72, [300, 17, 128, 129], 3, 64), (16, 1, 512, [700, 64, 1], 5, 128),
    (3, 2, 40, [2, 65, 66, 130], 2, 64), (5, 7, 136, [7, 8, 70, 134], 2, 192), (33, 3, 264, [200, 3], 4, 64), (4, 31, 384, [31, 95], 1, 64),
    (64, 1, 512, [1000, 257, 129], 3, 64), (20, 2, 200, [500, 2, 256], 2, 64), (40, 1, 448, [128, 384, 770], 6, 64)])
def test_latent_attention(dtype, variant, H, S, rank, lens, splits, page):
    from triton_distributed_b200 import ops
    pitch = rank
    seqs = [torch.randn(n, rank).to(dtype) for n in lens]
    cache, table = _paged(seqs, pitch, page, dtype)
    q = (torch.randn(len(lens) * S, H, rank) * 2).to(dtype)
    sink = torch.randn(H) + 2
    scale = 1.3 / rank ** 0.5
    out = ops.latent_attention(q.cuda(), cache, torch.tensor(lens, dtype=torch.int32, device="cuda"), table, S, scale, sink.cuda(),
                               splits, variant=variant)
    want = torch.cat([_absorbed_ref(q[b * S:(b + 1) * S].double(), seqs[b].double(), sink.double(), scale, n - S)
                      for b, n in enumerate(lens)])
    _close(out, want, dtype, factor=2.0)
    no_sink = ops.latent_attention(q.cuda(), cache, torch.tensor(lens, dtype=torch.int32, device="cuda"), table, S, scale, None,
                                   splits, variant=variant)
    want0 = torch.cat([_absorbed_ref(q[b * S:(b + 1) * S].double(), seqs[b].double(), torch.full((H,), -1e30, dtype=torch.float64),
                                     scale, n - S) for b, n in enumerate(lens)])
    _close(no_sink, want0, dtype, factor=2.0)
    if variant == "tc":
        for rows in (16, 32, 64):
            other = ops.latent_attention(q.cuda(), cache, torch.tensor(lens, dtype=torch.int32, device="cuda"), table, S, scale,
                                         sink.cuda(), 1, rows_per_cta=rows, variant="tc")
            _close(other, want, dtype, factor=2.0)
    ops.check_pipeline_status()


def test_latent_attention_with_scores_that_grow():
    """Scores that rise tile after tile make the running maximum move again and again, for each row at its own pace."""
    from triton_distributed_b200 import ops
    H, rank, n = 20, 128, 1500
    c = torch.randn(n, rank) * 0.3
    c[:, 0] = torch.linspace(-40, 60, n)
    q = torch.randn(1, H, rank) * 0.3
    q[0, :, 0] = torch.linspace(-1.5, 1.5, H)
    c, q = c.bfloat16(), q.bfloat16()
    cache, table = _paged([c], rank, 64, torch.bfloat16)
    want = _absorbed_ref(q.double(), c.double(), torch.zeros(H, dtype=torch.float64), 1.0, n - 1)
    for variant in ("tc", "plain"):
        for splits in (1, 3):
            out = ops.latent_attention(q.cuda(), cache, torch.tensor([n], dtype=torch.int32, device="cuda"), table, 1, 1.0,
                                       torch.zeros(H, device="cuda"), splits, variant=variant)
            _close(out, want, torch.bfloat16, factor=2.0)
    ops.check_pipeline_status()


@pytest.mark.parametrize("variant", ["tc", "plain"])
@pytest.mark.parametrize("kv_len,S", [(1, 1), (64, 1), (65, 1), (128, 5), (190, 3), (321, 1)])
def test_latent_attention_sees_exactly_the_keys_up_to_its_own(variant, kv_len, S):
    """One key at a time gets a score that dwarfs the others: rows whose position is at or after it return its latent, rows
    before it must not notice it. Places: first key, page and tile borders, the tokens of the step themselves."""
    from triton_distributed_b200 import ops
    H, rank = 3, 64
    base = torch.randn(kv_len, rank) * 0.05
    q = torch.zeros(S, H, rank)
    q[..., 0] = 8.0
    places = sorted({0, 1, 31, 32, 62, 63, 64, 65, 127, 128, 191, 192, kv_len - S - 1, kv_len - S, kv_len - 2, kv_len - 1} & set(range(kv_len)))
    for j in places:
        c = base.clone()
        c[j] = torch.randn(rank).clamp(-1, 1)
        c[j, 0] = 8.0                                    # score 64 against about 0.4
        cache, table = _paged([c.to(torch.bfloat16)], rank, 64, torch.bfloat16, seed=j)
        out = ops.latent_attention(q.to(torch.bfloat16).cuda(), cache, torch.tensor([kv_len], dtype=torch.int32, device="cuda"), table,
                                   S, 1.0, torch.zeros(H, device="cuda"), 3, variant=variant).float().cpu()
        want = c.to(torch.bfloat16).float()[j]
        for i in range(S):
            seen = kv_len - S + i >= j
            err = (out[i] - want).abs().max()
            assert (err < 0.05) if seen else (out[i, :, 0].abs().max() < 0.5), (j, i, err)


@pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float16])
@pytest.mark.parametrize("H,dk,dv,q_lens,prefix,sink_on", [
    (2, 40, 24, [33, 1, 129], 0, True), (3, 56, 88, [128, 200], 0, True), (2, 128, 128, [257], 70, True), (1, 72, 136, [140, 60], 5, True),
    (2, 192, 64, [300], 129, True), (2, 256, 200, [130, 257], 3, True), (2, 200, 256, [64], 200, False), (4, 8, 8, [40], 0, True)])
def test_prefill_attention_vt(dtype, H, dk, dv, q_lens, prefix, sink_on):
    from triton_distributed_b200 import ops
    B = len(q_lens)
    k_lens = [n + prefix for n in q_lens]
    kv8 = (max(k_lens) + 7) // 8 * 8
    total = sum(q_lens)
    wide = torch.randn(total, H * dk + 16).to(dtype)
    q = wide.cuda()[:, 8:8 + H * dk].unflatten(1, (H, dk))
    k = torch.full((B, kv8, H, dk), 100.0)               # slots beyond a sequence hold garbage
    vt = torch.full((H, dv, B, kv8), 100.0)
    ks, vs = [], []
    for b, n in enumerate(k_lens):
        kb, vb = torch.randn(n, H, dk).to(dtype), torch.randn(n, H, dv).to(dtype)
        k[b, :n], vt[:, :, b, :n] = kb.float(), vb.permute(1, 2, 0).float()
        ks.append(kb), vs.append(vb)
    sink = (torch.randn(H) + 3) if sink_on else None
    scale = 2.0 / dk ** 0.5
    cu_q = torch.tensor([0] + list(torch.tensor(q_lens).cumsum(0)), dtype=torch.int32, device="cuda")
    cu_k = torch.arange(B + 1, dtype=torch.int32, device="cuda") * kv8
    out = ops.prefill_attention_vt(q, k.to(dtype).cuda().view(B * kv8, H, dk), vt.to(dtype).cuda().view(H, dv, B * kv8), cu_q, cu_k,
                                   torch.tensor(k_lens, dtype=torch.int32, device="cuda"), max(q_lens), scale, True,
                                   sink.cuda() if sink_on else None)
    ops.check_pipeline_status()
    at = 0
    for b, n in enumerate(q_lens):
        qb = wide[at:at + n, 8:8 + H * dk].unflatten(1, (H, dk)).double()
        want = torch.empty(n, H, dv, dtype=torch.float64)
        vis = torch.arange(k_lens[b])[None] <= (torch.arange(n) + prefix)[:, None]
        for h in range(H):
            s = torch.tensor(-1e30) if not sink_on else sink[h]
            want[:, h] = ref.sink_softmax_ref(qb[:, h] @ ks[b][:, h].double().t() * scale, s.double(), vis) @ vs[b][:, h].double()
        _close(out[at:at + n], want, dtype, factor=2.0)
        at += n


def test_prefill_attention_sees_exactly_the_keys_up_to_its_own():
    from triton_distributed_b200 import ops
    S, prefix, H, dk, dv = 150, 115, 1, 64, 64
    n = S + prefix
    kv8 = (n + 7) // 8 * 8
    q = torch.zeros(S, H, dk)
    q[..., 0] = 8.0
    for j in (0, 63, 64, 127, 128, 114, 115, 116, 191, 255, 256, n - 2, n - 1):
        k, v = torch.randn(kv8, H, dk) * 0.05, torch.zeros(kv8, H, dv)
        k[:, :, 0] = 0.0
        k[j, :, 0] = 8.0
        v[j] = 1.0
        out = ops.prefill_attention_vt(q.bfloat16().cuda(), k.bfloat16().cuda(), v.permute(1, 2, 0).contiguous().bfloat16().cuda(),
                                       torch.tensor([0, S], dtype=torch.int32, device="cuda"),
                                       torch.tensor([0, kv8], dtype=torch.int32, device="cuda"),
                                       torch.tensor([n], dtype=torch.int32, device="cuda"), S, 1.0, True, torch.zeros(H, device="cuda"))
        seen = (torch.arange(S) + prefix >= j).float()
        assert (out[:, 0, 0].float().cpu() - seen).abs().max() < 0.02, j
    ops.check_pipeline_status()


# ------------------------------------------------------------------------------------------------ the model
_refs = {}


def _case(name, n=170, seed=0):
    """(config, weights, tokens, oracle logits); computed once per module."""
    key = (name, n, seed)
    if key not in _refs:
        cfg = lc.CONFIGS[name]
        w = lc.weights_for(cfg, seed)
        toks = lc.tokens_for(cfg, n, seed)
        _refs[key] = (cfg, w, toks, ref.likosun_ref(toks, cfg, w))
    return _refs[key]


def _engine(tmp_path, name, dtype, max_length=256, seed=0):
    from triton_distributed_b200.models import Engine, ModelConfig
    cfg = lc.CONFIGS[name]
    path = lc.save(tmp_path / name, cfg, lc.weights_for(cfg, seed))
    return Engine(ModelConfig(model_name=name, checkpoint_dir=path, max_length=max_length, dtype=dtype, rank=0, world_size=1), temperature=0.0)


def _run(eng, toks, cuts, bsz=1):
    """Feed one sequence (or bsz copies' worth of different ones: toks [bsz][n]) in portions; logits of every position."""
    rows = toks if isinstance(toks[0], list) else [toks]
    ids = torch.tensor(rows, device="cuda")
    eng.start(ids.shape[0])
    out, at, i = [], 0, 0
    while at < ids.shape[1]:
        n = min(cuts[min(i, len(cuts) - 1)], ids.shape[1] - at)
        i += 1
        out.append(eng.extend(ids[:, at:at + n], want=list(range(n))).cpu().clone())
        at += n
    from triton_distributed_b200 import ops
    ops.check_pipeline_status()
    return torch.cat(out, 1)


MODES = [("odd", torch.float32), ("odd", torch.bfloat16), ("equal", torch.float32), ("equal", torch.bfloat16), ("wide", torch.float32),
         ("wide", torch.bfloat16), ("wide", torch.float16), ("large", torch.bfloat16), ("large", torch.float32)]


@pytest.mark.parametrize("name,dtype", MODES)
def test_whole_prompt_and_stream_after_every_layer(tmp_path, name, dtype):
    cfg, w, toks, (want, after) = _case(name)
    eng = _engine(tmp_path, name, dtype)
    eng.model.layer_taps = []
    got = _run(eng, toks, [len(toks)])[0]
    assert got.shape == want.shape
    assert lc.rms_error(got, want).max() < TOL[dtype]
    for i, x in enumerate(eng.model.layer_taps):
        _close(x, after[i], dtype, factor=4.0)
    assert len(eng.model.layer_taps) == len(cfg["layers"])


@pytest.mark.parametrize("name,dtype", [("odd", torch.float32), ("odd", torch.bfloat16), ("wide", torch.bfloat16), ("large", torch.bfloat16)])
@pytest.mark.parametrize("cuts", [[1], [2], [31], [3, 40, 1, 2, 64, 5, 1], [63, 1, 64, 1, 33, 8], [128, 1], [169, 1]])
def test_portions_do_not_change_the_logits(tmp_path, name, dtype, cuts):
    _, _, toks, (want, _) = _case(name)
    got = _run(_engine(tmp_path, name, dtype), toks, cuts)[0]
    assert lc.rms_error(got, want).max() < TOL[dtype]


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_slots_are_reused_without_a_trace(tmp_path, dtype):
    """A long request, then others in the same slots: as if the engine were new."""
    _, w, toks, (want, _) = _case("odd")
    eng = _engine(tmp_path, "odd", dtype)
    _run(eng, lc.tokens_for(lc.CONFIGS["odd"], 250, 9), [120, 1, 2, 90, 1])
    for cuts in ([170], [1, 2, 30, 1, 70, 1]):
        assert lc.rms_error(_run(eng, toks, cuts)[0], want).max() < TOL[dtype]
    one = _run(eng, toks[:1], [1])[0]
    assert lc.rms_error(one, want[:1]).max() < TOL[dtype]


@pytest.mark.parametrize("name,dtype", [("odd", torch.float32), ("wide", torch.bfloat16)])
def test_batches_against_each_alone(tmp_path, name, dtype):
    cfg = lc.CONFIGS[name]
    rows = [lc.tokens_for(cfg, 100, s) for s in (3, 4, 5)]
    eng = _engine(tmp_path, name, dtype)
    for cuts in ([100], [40, 2, 1, 1, 37, 3]):
        together = _run(eng, rows, cuts)
        for b, r in enumerate(rows):
            want, _ = ref.likosun_ref(r, cfg, lc.weights_for(cfg, 0))
            assert lc.rms_error(together[b], want).max() < TOL[dtype]
            alone = _run(eng, r, cuts)[0]
            assert lc.rms_error(together[b], alone).max() < TOL[dtype]


def test_long_decoding(tmp_path):
    cfg, w, toks, (want, _) = _case("odd", 420)
    for dtype in (torch.float32, torch.bfloat16):
        got = _run(_engine(tmp_path, "odd", dtype, max_length=420), toks, [20] + [1] * 400)[0]
        assert lc.rms_error(got, want).max() < TOL[dtype]


def test_extend_checks_its_input(tmp_path):
    eng = _engine(tmp_path, "odd", torch.float32, max_length=70)
    with pytest.raises(ValueError, match="start"):
        eng.extend(torch.zeros(1, 3, dtype=torch.int64, device="cuda"))
    eng.start(1)
    assert eng.extend(torch.zeros(1, 66, dtype=torch.int64, device="cuda"), want=[]) is None
    with pytest.raises(ValueError, match="max_length"):
        eng.extend(torch.zeros(1, 5, dtype=torch.int64, device="cuda"))
    assert eng.extend(torch.zeros(1, 4, dtype=torch.int64, device="cuda")).shape == (1, 1, 203)


def test_greedy_generation_through_the_engine(tmp_path):
    cfg, w = lc.CONFIGS["odd"], lc.weights_for(lc.CONFIGS["odd"], 0)
    prompts = [lc.tokens_for(cfg, 40, s) for s in (11, 20)]
    wanted = [ref.greedy_ref(p, 24, cfg, w) for p in prompts]

    def agrees(out, least_margin, at_least):
        for b, (want, margins) in enumerate(wanted):
            n = next((i for i, m in enumerate(margins) if m < least_margin), 24)   # a near tie may fall either way
            assert n >= at_least and out[b, : 40 + n].tolist() == prompts[b] + want[:n]

    ids = torch.tensor(prompts, device="cuda")
    agrees(_engine(tmp_path, "odd", torch.float32).serve(ids, gen_len=24).cpu(), 1e-3, 24)
    for no_graph in (False, True):
        e = _engine(tmp_path, "odd", torch.bfloat16)
        e.no_graph = no_graph
        agrees(e.serve(ids, gen_len=24).cpu(), 0.1, 7)
    e.temperature = 0.8                                   # top-p sampling takes the same logits
    s = e.serve(ids, gen_len=5)
    assert s.shape == (2, 45) and int(s.max()) < cfg["vocab"]


def test_named_architecture_runs():
    from triton_distributed_b200.models import Engine, ModelConfig
    eng = Engine(ModelConfig(model_name="tiny-likosun", max_length=128, rank=0, world_size=1), temperature=0.0)
    out = eng.serve(torch.randint(0, 1000, (2, 50), device="cuda"), gen_len=6)
    assert out.shape == (2, 56)
    with pytest.raises(ValueError, match="triton_dist_AR"):
        eng.model.set_fwd("torch")


def _trace(model, dtype, out, steps, max_tokens):
    exe = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "bin", "trace_run")
    return subprocess.run([sys.executable, exe, "--model", model, "--dtype", dtype, "--out", str(out), "--max-tokens", str(max_tokens)],
                          input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)


def test_trace_replay(tmp_path):
    cfg, w, toks, (want, _) = _case("odd")
    path = lc.save(tmp_path / "m", cfg, w)
    other = lc.tokens_for(cfg, 50, 8)
    want2, _ = ref.likosun_ref(other, cfg, w)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:60], "want": [59, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": toks[60:61], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[61:63], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": toks[63:], "want": [0, 1, 106]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": other, "want": [0, 49]}], "end": ["b"]}]
    places = {0: (want, [59, 3]), 1: (want, [60]), 3: (want, [63, 64, 169]), 4: (want2, [0, 49])}
    for dtype in (torch.float32, torch.bfloat16):
        out = tmp_path / str(dtype)
        r = _trace(path, str(dtype).split(".")[1], out, steps, 170)
        assert r.returncode == 0, r.stderr
        assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(5)]
        assert sorted(os.listdir(out)) == ["0.f32", "1.f32", "3.f32", "4.f32"]
        for i, (ref_logits, rows) in places.items():
            got = torch.frombuffer(bytearray((out / f"{i}.f32").read_bytes()), dtype=torch.float32).view(len(rows), -1)
            assert lc.rms_error(got, ref_logits[rows]).max() < TOL[dtype]


def test_trace_replay_of_another_model(tmp_path):
    """The same program serves the other families (bf16), and says so with exit code 3 where a family has no fp32 kernels."""
    from triton_distributed_b200.models import ARCHS, Engine, ModelConfig
    from triton_distributed_b200.models.weights import write_random_checkpoint
    write_random_checkpoint(str(tmp_path / "m"), ARCHS["tiny-qwen3"], torch.bfloat16, seed=0)
    toks = torch.randint(0, 1024, (1, 40)).tolist()
    steps = [{"step": 0, "entries": [{"id": "q", "tokens": toks[0][:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "q", "tokens": toks[0][30:31], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "q", "tokens": toks[0][31:], "want": [8]}], "end": ["q"]}]
    r = _trace(str(tmp_path / "m"), "bfloat16", tmp_path / "o", steps, 64)
    assert r.returncode == 0, r.stderr
    eng = Engine(ModelConfig(model_name="m", checkpoint_dir=str(tmp_path / "m"), max_length=64, rank=0, world_size=1), temperature=0.0)
    want = _run(eng, toks[0], [40])[0]
    for i, rows in ((0, [0, 29]), (1, [30]), (2, [39])):
        got = torch.frombuffer(bytearray((tmp_path / "o" / f"{i}.f32").read_bytes()), dtype=torch.float32).view(len(rows), -1)
        assert lc.rms_error(got, want[rows]).max() < 0.03
    assert _trace(str(tmp_path / "m"), "float32", tmp_path / "o2", steps, 64).returncode == 3
