"""Sizilorn on the CPU: configuration and registry, checkpoints, the cache, sharding of the weights, and the oracle's own
sensitivity: a mistake planted in the oracle must move the logits by far more than the GPU tests' tolerance."""
import json

import pytest
import torch

import sizilorn_cases as sc
from triton_distributed_b200 import ref
from triton_distributed_b200.models import ARCHS, AutoLLM, HybridCache, ModelConfig, Sizilorn, SizilornConfig


def test_config_round_trip_and_registry(tmp_path):
    for name, cfg in sc.CONFIGS.items():
        arch = SizilornConfig.from_dict(cfg)
        assert arch.to_dict() == cfg, name
        assert arch.num_hidden_layers == len(cfg["layers"]) and arch.vocab_size == cfg["vocab"]
    path = sc.save(tmp_path / "m", sc.CONFIGS["odd"], {"embed": torch.zeros(1)})
    assert AutoLLM.model_class(ModelConfig(model_name="x", checkpoint_dir=path)) is Sizilorn
    assert AutoLLM.model_class(ModelConfig(model_name="tiny-sizilorn")) is Sizilorn
    assert ModelConfig(model_name="tiny-sizilorn", num_layers_override=2).arch().num_hidden_layers == 2


@pytest.mark.parametrize("change", ["type", "kind", "missing"])
def test_unknown_kinds_and_missing_sizes_are_refused(tmp_path, change):
    cfg = json.loads(json.dumps(sc.CONFIGS["odd"]))
    if change == "type":
        cfg["layers"][0]["type"] = "latent_attention"      # another design's mixer
    elif change == "kind":
        cfg["layers"][0]["mlp"]["kind"] = "no_such_mlp"
    else:
        del cfg["layers"][1]["mixer"]["right"]["conv"]
    path = sc.save(tmp_path / "m", cfg, {"embed": torch.zeros(1)})
    with pytest.raises(KeyError if change == "missing" else ValueError, match="conv" if change == "missing" else "unknown"):
        ModelConfig(model_name="x", checkpoint_dir=path).arch()


def test_random_checkpoint_round_trip(tmp_path):
    from triton_distributed_b200.models.weights import (RandomSource, SafetensorsSource, read_arch_from_checkpoint, sizilorn_param_shapes,
                                                       write_random_checkpoint)
    arch = ARCHS["tiny-sizilorn"]
    write_random_checkpoint(str(tmp_path), arch, torch.bfloat16, seed=3, max_shard_bytes=1 << 20)
    assert read_arch_from_checkpoint(str(tmp_path)) == arch
    src, rnd = SafetensorsSource(str(tmp_path), device="cpu"), RandomSource(arch, torch.bfloat16, seed=3, device="cpu")
    shapes = sizilorn_param_shapes(arch)
    assert set(src.weight_map) == set(shapes) and "l0.mlp.up" not in shapes and "l0.norm2" not in shapes
    assert shapes["l1.mix.right.v.conv"] == (144, 3) and shapes["l2.mix.w1"] == (16, 264) and shapes["side.embed"] == (1000, 60)
    for name in ("l0.mix.u", "l2.mlp.down", "l1.norm2.alpha", "l1.mix.right.b", "l1.mix.right.A_log", "final.norm.b", "l0.mix.w0"):
        assert tuple(src.get(name).shape) == shapes[name] and torch.equal(src.get(name), rnd.get(name))
    assert src.get("l1.mix.right.b").abs().max() > 0        # a projection, not a bias
    model = Sizilorn(ModelConfig(model_name="x", checkpoint_dir=str(tmp_path), rank=0, world_size=1))
    assert model.layers[0].mixer.rank == 24 and model.layers[2].mixer.rank == 16   # from the tensors' shapes


def test_hybrid_cache():
    L = HybridCache.Layer
    c = HybridCache([L(states={"s": ((2, 3), torch.float32)}), L(pages={"k": (2, 8)}, states={"x": ((4,), torch.float16)})], 3, 130,
                    dtype=torch.float16, device="cpu")
    assert c.pages(1, "k").shape == (9, 64, 2, 8) and c.state(0, "s").shape == (3, 2, 3) and c.state(1, "x").dtype == torch.float16
    c.state(0, "s")[1] = 2.0
    saved, where = c.save_state(), c.state(0, "s").data_ptr()
    c.state(0, "s").add_(1.0)
    c.state(1, "x").add_(1.0)
    c.restore_state(saved)
    assert c.state(0, "s").sum() == 12.0 and c.state(1, "x").sum() == 0 and c.state(0, "s").data_ptr() == where
    c.inc_offset(5)
    c.clear()
    assert c.state(0, "s").sum() == 0 and c.kv_offset.sum() == 0 and c.state(0, "s").data_ptr() == where


def test_engine_warm_up_leaves_the_states_alone(monkeypatch):
    """The decode step runs a few times before it is captured; what it did to the states is undone."""
    from triton_distributed_b200.models import Engine
    cache = HybridCache([HybridCache.Layer(states={"s": ((2,), torch.float32)})], 1, 64, device="cpu")

    class Model:
        def make_cache(self, bsz, n):
            return cache

        def inference(self, ids, pos, kv):
            kv.state(0, "s").add_(1.0)
            return torch.zeros(1, 1, 4)

    class Stream:
        def wait_stream(self, _):
            pass

        def __enter__(self):
            pass

        def __exit__(self, *_):
            pass

    eng = Engine(ModelConfig(model_name="tiny-sizilorn", max_length=64, rank=0, world_size=1), model=Model())
    eng.start(1)
    eng._static_ids, eng._static_pos = torch.zeros(1, 1, dtype=torch.int64), torch.zeros(1, 1, dtype=torch.int64)
    monkeypatch.setattr(torch.cuda, "Stream", Stream)
    monkeypatch.setattr(torch.cuda, "current_stream", Stream)
    monkeypatch.setattr(torch.cuda, "stream", lambda s: s)
    monkeypatch.setattr(torch.cuda, "synchronize", lambda: None)
    monkeypatch.setattr(torch.cuda, "CUDAGraph", object)
    monkeypatch.setattr(torch.cuda, "graph", lambda g: Stream())
    monkeypatch.setattr(eng, "_decode_step", lambda step=eng._decode_step, left=[3]: (left.append(left.pop() - 1), step())[1] if left[0] else None)
    eng._init_cuda_graph()
    assert cache.state(0, "s").sum() == 0


def test_tensor_parallel_shards_sum_to_the_whole(tmp_path):
    """The ranks' input rows are the heads they own, and their output matrices add up."""
    cfg = sc.config(60, 40, [sc.wkv(4, 12, 44), sc.parallel((4, 2, 12, 10, 0.3, 8, 1e4, None), (4, 2, 6, 18, 4))])
    w = sc.weights_for(cfg, 5)
    path = sc.save(tmp_path / "m", cfg, w)

    def load(rank, world):
        return Sizilorn(ModelConfig(model_name="x", checkpoint_dir=path, dtype=torch.float32, rank=rank, world_size=world)).layers

    h = torch.randn(3, 40)
    o, ow = torch.randn(3, 4, 10), torch.randn(3, 4, 12)
    od = torch.randn(3, 4, 18)
    sums = [torch.zeros(3, 40) for _ in range(3)]
    for r in range(2):
        wl, pl = load(r, 2)
        mix = wl.mixer
        assert (mix.heads, mix.dim, mix.rank) == (2, 16, 8) and mix.u.shape == (32,) and mix.mu.shape == (5, 40)
        rk = (h @ mix.w_in[: mix.rows[0]].t())[:, :32].view(3, 2, 16)
        torch.testing.assert_close(rk[..., :12], (h @ w["l0.mix.r"].float().t()).view(3, 4, 12)[:, 2 * r:2 * r + 2], rtol=1e-4, atol=1e-4)
        assert torch.all(rk[..., 12:] == 0) and torch.equal(mix.u.view(2, 16)[:, :12], w["l0.mix.u"].float()[2 * r:2 * r + 2])
        parts = (h @ pl.w_in.t()).split(pl.splits, dim=1)
        q, k = parts[0].view(3, 2, 16), parts[1].view(3, 1, 16)
        torch.testing.assert_close(q[..., :12], (h @ w["l1.mix.left.q"].float().t()).view(3, 4, 12)[:, 2 * r:2 * r + 2], rtol=1e-4, atol=1e-4)
        torch.testing.assert_close(k[..., :12], (h @ w["l1.mix.left.k"].float().t()).view(3, 2, 12)[:, r:r + 1], rtol=1e-4, atol=1e-4)
        torch.testing.assert_close(parts[5][:, :2], (h @ w["l1.mix.right.b"].float().t())[:, 2 * r:2 * r + 2], rtol=1e-4, atol=1e-4)
        assert pl.right.taps.shape == (4, sum(pl.right.sizes)) and pl.right.sizes == [8, 8, 48]
        torch.testing.assert_close(pl.right.taps[:, 8:14].t(), w["l1.mix.right.k.conv"].float()[6 * r:6 * r + 6])
        for i, (x, wo, pad) in enumerate(((ow, mix.wo, 16), (o, pl.left.wo, pl.left.vdim), (od, pl.right.wo, 24))):
            xp = torch.zeros(3, 2, pad)
            xp[..., : x.shape[2]] = x[:, 2 * r:2 * r + 2]
            sums[i] += (xp.reshape(3, -1) @ wo.t())[:, :40]
    for got, x, name in zip(sums, (ow, o, od), ("l0.mix.o", "l1.mix.left.o", "l1.mix.right.o")):
        torch.testing.assert_close(got, x.reshape(3, -1) @ w[name].float().t(), rtol=1e-4, atol=1e-4)
    with pytest.raises(ValueError, match="divisible"):
        load(0, 4)


def test_rotation_tables():
    from triton_distributed_b200.layers.nvidia.gated_attn import rotation_frequencies, rotation_table
    from triton_distributed_b200.models.config import RotaryScaling, RotarySpec
    for dims, base, sc_ in ((10, 3000.0, (3.0, 1.0, 4.0, 48)), (64, 2e4, (8.0, 1.0, 4.0, 96)), (2, 10.0, None), (0, 10.0, None)):
        rot = RotarySpec(dims, base, None if sc_ is None else RotaryScaling(*sc_))
        want = ref.rotation_frequencies_ref(dims, base, None if sc_ is None else dict(zip(("factor", "low", "high", "original"), sc_)))
        torch.testing.assert_close(rotation_frequencies(rot), want, rtol=1e-12, atol=0)
        table = rotation_table(rot, 300, "cpu")
        assert table.shape == (300, dims) and table.dtype == torch.float32
        if dims:
            torch.testing.assert_close(table[299, 1::2].double(), torch.sin(299 * want), rtol=0, atol=1e-7)
    three = ref.rotation_frequencies_ref(64, 2e4, dict(factor=8.0, low=1.0, high=4.0, original=96))
    plain = ref.rotation_frequencies_ref(64, 2e4, None)
    ratio = (plain / three).tolist()
    assert ratio[0] == 1.0 and abs(ratio[-1] - 8.0) < 1e-12 and any(1.01 < r < 7.9 for r in ratio)   # all three branches


def test_oracle_mechanisms_against_other_statements():
    x = torch.randn(7, 33, dtype=torch.float64)
    torch.testing.assert_close(ref.gelu_tanh_ref(x), torch.nn.functional.gelu(x, approximate="tanh"))
    torch.testing.assert_close(ref.swish_ref(x), torch.nn.functional.silu(x))
    torch.testing.assert_close(ref.softplus_ref(20 * x), torch.nn.functional.softplus(20 * x))
    torch.testing.assert_close(ref.unit_rms_ref(x, 1e-3), torch.nn.functional.rms_norm(x, (33,), None, 1e-3))
    taps = torch.randn(33, 4, dtype=torch.float64)
    conv = torch.nn.functional.conv1d(torch.nn.functional.pad(x.t()[None], (3, 0)), taps[:, None], groups=33)[0].t()
    torch.testing.assert_close(ref.short_conv_ref(x, taps), conv)
    q, k, v = (torch.randn(9, h, 6, dtype=torch.float64) for h in (4, 2, 2))
    lib = torch.nn.functional.scaled_dot_product_attention(q.transpose(0, 1), k.transpose(0, 1).repeat_interleave(2, 0),
                                                           v.transpose(0, 1).repeat_interleave(2, 0), is_causal=True, scale=0.3)
    torch.testing.assert_close(ref.grouped_attention_ref(q, k, v, 0.3), lib.transpose(0, 1))
    r3 = torch.randn(5, 2, 8, dtype=torch.float64)
    torch.testing.assert_close(ref.rotate_pairs_ref(r3, ref.rotation_frequencies_ref(6, 100.0, None), 11), sc.rotation(r3, range(11, 16), 6, 100.0))
    # the recurrences as explicit sums over earlier tokens
    r, kk, vv = (torch.randn(6, 1, 3, dtype=torch.float64) for _ in range(3))
    w, u = torch.rand(6, 1, 3, dtype=torch.float64), torch.randn(1, 3, dtype=torch.float64)
    got, _ = ref.decayed_outer_ref(r, kk, vv, w, u)
    for t in range(6):
        want = (r[t, 0] * u[0] * kk[t, 0]).sum() * vv[t, 0]
        for j in range(t):
            want = want + (r[t, 0] * torch.prod(w[j + 1:t, 0], dim=0) * kk[j, 0]).sum() * vv[j, 0]
        torch.testing.assert_close(got[t, 0], want)
    # the delta rule with full steps, no decay and unit keys stores exactly the last value of a key
    kk = torch.eye(3, dtype=torch.float64)[[0, 1, 0, 2, 1]][:, None]
    vv = torch.randn(5, 1, 4, dtype=torch.float64)
    one = torch.ones(5, 1, dtype=torch.float64)
    o, S = ref.gated_delta_ref(kk, kk, vv, one, one)
    torch.testing.assert_close(o, vv)
    torch.testing.assert_close(S[0], torch.stack([vv[2, 0], vv[4, 0], vv[3, 0]]))


def test_planted_mistakes_show_in_the_logits(monkeypatch):
    cfg, w = sc.named("odd")
    toks = sc.tokens_for(cfg, 90)
    good, _ = ref.sizilorn_ref(toks, cfg, w)
    mod = ref.sizilorn

    def moved(cfg2=cfg, w2=w):
        return sc.rms_error(ref.sizilorn_ref(toks, cfg2, w2)[0][8:], good[8:]).median().item()

    def without(name, value=0.0):
        return {**w, name: torch.full_like(w[name], value)}

    for name, value in (("l0.norm1.b", 0.0), ("l1.norm1.alpha", 1.0), ("l2.mix.u", 0.0), ("l0.mix.mu.w", 0.0), ("l0.mix.w0", -3.0), ("l0.mix.w2", 0.0),
                        ("l2.mix.norm", 1.0), ("l1.mix.left.g", 0.0), ("l1.mix.left.k.norm", 1.0), ("l1.mix.right.a", 0.0),
                        ("l1.mix.right.dt_bias", 0.0), ("l3.mix.right.norm", 1.0), ("l3.mix.left.out", 1.0), ("l2.side.gate", 0.0),
                        ("l3.side.norm", 1.0), ("final.norm.b", 0.0)):
        assert moved(w2=without(name, value)) > 0.03, name
    shifted = dict(w)
    shifted["side.embed"] = w["side.embed"].roll(7, 1)          # another layer's part of the side embedding
    assert moved(w2=shifted) > 0.03
    flipped = {**w, "l1.mix.right.k.conv": w["l1.mix.right.k.conv"].flip(1)}
    assert moved(w2=flipped) > 0.03
    other = json.loads(json.dumps(cfg))
    other["layers"][1]["mixer"]["left"]["rot"]["scaling"] = None
    assert moved(cfg2=other) > 0.03

    def planted(name, fn):
        with monkeypatch.context() as m:
            m.setattr(mod, name, fn(getattr(mod, name)))
            return moved()

    assert planted("token_mix_ref", lambda f: lambda h, mu: h) > 0.03
    assert planted("rotate_pairs_ref", lambda f: lambda x, fr: torch.cat([f(x[..., : 2 * fr.numel()].unflatten(-1, (2, -1)).transpose(-1, -2).flatten(-2), fr)
                                                                          .unflatten(-1, (-1, 2)).transpose(-1, -2).flatten(-2), x[..., 2 * fr.numel():]], -1)) > 0.03
    assert planted("grouped_attention_ref", lambda f: lambda q, k, v, s: f(q, k[:, torch.arange(k.shape[1]) - 1], v, s)) > 0.03     # the wrong key head
    assert planted("decayed_outer_ref", lambda f: lambda r, k, v, w_, u: f(r, k, v, w_, torch.ones_like(u))) > 0.03               # bonus left out
    assert planted("gated_delta_ref", lambda f: lambda q, k, v, g, b: f(q, k, v, torch.ones_like(g), b)) > 0.03                   # no decay

    def restart(f):                                              # the state lost after 40 tokens
        def run(r, k, v, *rest):
            cut = [x[:40] if x.shape[0] == 90 else x for x in rest], [x[40:] if x.shape[0] == 90 else x for x in rest]
            a, b = f(r[:40], k[:40], v[:40], *cut[0]), f(r[40:], k[40:], v[40:], *cut[1])
            return torch.cat([a[0], b[0]]), b[1]
        return run
    for name in ("decayed_outer_ref", "gated_delta_ref"):
        with monkeypatch.context() as m:
            m.setattr(mod, name, restart(getattr(mod, name)))
            lost = ref.sizilorn_ref(toks, cfg, w)[0]
        assert sc.rms_error(lost[40:50], good[40:50]).median() > 0.03, name
        assert sc.rms_error(lost[:40], good[:40]).max() < 1e-9
