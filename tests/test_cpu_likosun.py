"""Likosun on the CPU: configuration and registry, checkpoints, sharding of the weights, and the oracle's own sensitivity: a
mistake planted in the oracle must move the logits by far more than the GPU tests' tolerance."""
import json

import pytest
import torch

import likosun_cases as lc
from triton_distributed_b200 import ref
from triton_distributed_b200.models import ARCHS, AutoLLM, Likosun, LikosunConfig, ModelConfig


def test_config_round_trip_and_registry(tmp_path):
    for name, cfg in lc.CONFIGS.items():
        arch = LikosunConfig.from_dict(cfg)
        assert arch.to_dict() == cfg, name
        assert arch.num_hidden_layers == len(cfg["layers"]) and arch.vocab_size == cfg["vocab"]
    path = lc.save(tmp_path / "m", lc.CONFIGS["odd"], {"embed": torch.zeros(1)})
    assert AutoLLM.model_class(ModelConfig(model_name="x", checkpoint_dir=path)) is Likosun
    assert AutoLLM.model_class(ModelConfig(model_name="tiny-likosun")) is Likosun
    assert AutoLLM.model_class(ModelConfig(model_name="tiny-qwen3")).__name__ == "Qwen3"
    assert AutoLLM.model_class(ModelConfig(model_name="tiny-qwen3-moe")).__name__ == "Qwen3MoE"
    assert ModelConfig(model_name="tiny-likosun", num_layers_override=2).arch().num_hidden_layers == 2


@pytest.mark.parametrize("change", ["type", "kind", "arch"])
def test_unknown_kinds_are_refused(tmp_path, change):
    cfg = json.loads(json.dumps(lc.CONFIGS["odd"]))
    if change == "type":
        cfg["layers"][0]["type"] = "no_such_mixer"
    elif change == "kind":
        cfg["layers"][0]["mlp"]["kind"] = "no_such_mlp"
    else:
        cfg["architecture"] = "NoSuchDesign"
    path = lc.save(tmp_path / "m", cfg, {"embed": torch.zeros(1)})
    with pytest.raises(ValueError, match="unknown"):
        ModelConfig(model_name="x", checkpoint_dir=path).arch()


def test_unsupported_storage_type_is_refused():
    from triton_distributed_b200.models.auto import UnsupportedDtype
    with pytest.raises(UnsupportedDtype):
        AutoLLM.from_pretrained(ModelConfig(model_name="tiny-qwen3", dtype=torch.float32, world_size=1))


def test_random_checkpoint_round_trip(tmp_path):
    from triton_distributed_b200.models.weights import (RandomSource, SafetensorsSource, likosun_param_shapes,
                                                       read_arch_from_checkpoint, write_random_checkpoint)
    arch = ARCHS["tiny-likosun"]
    write_random_checkpoint(str(tmp_path), arch, torch.bfloat16, seed=3, max_shard_bytes=1 << 20)
    assert read_arch_from_checkpoint(str(tmp_path)) == arch
    src, rnd = SafetensorsSource(str(tmp_path), device="cpu"), RandomSource(arch, torch.bfloat16, seed=3, device="cpu")
    shapes = likosun_param_shapes(arch)
    assert set(src.weight_map) == set(shapes) and "l1.mlp.up" not in shapes and "l1.rg2" not in shapes
    for name in ("l0.mix.uk", "l2.mlp.down", "l1.dwa", "l0.mix.sink", "final.norm.b"):
        assert tuple(src.get(name).shape) == shapes[name] and torch.equal(src.get(name), rnd.get(name))


def test_latent_cache_pages():
    from triton_distributed_b200.models import LatentCache
    c = LatentCache([24, 40], 3, 130, dtype=torch.float32, device="cpu")
    assert c.layer(1).shape == (9, 64, 40) and c.blocks_per_seq == 3
    pos = torch.tensor([[0, 63], [64, 65], [128, 129]])
    c.layer(1).view(-1, 40)[c.slots(pos)] = torch.arange(6.0)[:, None].expand(6, 40)
    rows = c.rows(1, 130).view(3, 130, 40)
    assert rows[0, :64, 0].tolist() == [0.0] * 63 + [1.0]
    assert rows[1, 64:66, 3].tolist() == [2.0, 3.0] and rows[2, 128:, 39].tolist() == [4.0, 5.0]
    c.blank(1, 65, 129)
    assert c.rows(1, 192).view(3, 192, 40)[:, :, 7].nonzero().tolist() == [[0, 63], [1, 64], [2, 129]]
    page = c.block_table[2, 128 // 64]
    assert c.layer(1)[page, 1, 0] == 5.0


def test_tensor_parallel_shards_sum_to_the_whole(tmp_path):
    """What a layer's sublayers contribute is the sum of the ranks' partial results (heads and inner columns are split)."""
    cfg = lc.config(60, 40, [lc.layer(4, 12, 10, 18, 0.3, 44)])
    w = lc.weights_for(cfg, 5)
    path = lc.save(tmp_path / "m", cfg, w)
    h = torch.randn(3, 40)
    q = (h @ w["l0.mix.q"].float().t()).view(3, 4, 12)
    o = torch.randn(3, 4, 10)
    up = torch.relu(h @ w["l0.mlp.up"].float().t()) ** 2
    want_a, want_f = o.reshape(3, -1) @ w["l0.mix.o"].float().t(), up @ w["l0.mlp.down"].float().t()
    got_a, got_f = torch.zeros(3, 40), torch.zeros(3, 40)
    for r in range(2):
        layer = Likosun(ModelConfig(model_name="x", checkpoint_dir=path, dtype=torch.float32, rank=r, world_size=2)).layers[0]
        a = layer.attn
        assert (a.heads, a.dim, a.vdim, a.pitch) == (2, 16, 16, 24)
        parts = (h @ layer.w_in[:, :40].t()).split(layer.splits, dim=1)
        qr = parts[0].view(3, 2, 16)
        torch.testing.assert_close(qr[..., :12], q[:, 2 * r:2 * r + 2], rtol=1e-4, atol=1e-4)
        assert torch.all(qr[..., 12:] == 0)
        op = torch.zeros(3, 2, 16)
        op[..., :10] = o[:, 2 * r:2 * r + 2]
        got_a += (op.reshape(3, -1) @ a.wo.t())[:, :40]
        got_f += (torch.relu(parts[2]) ** 2 @ layer.down.t())[:, :40]
        torch.testing.assert_close(parts[-1][:, :40], h @ w["l0.rg2"].float().t(), rtol=1e-4, atol=1e-4)
        assert torch.equal(a.sink, w["l0.mix.sink"].float()[2 * r:2 * r + 2])
    torch.testing.assert_close(got_a, want_a, rtol=1e-4, atol=1e-4)
    torch.testing.assert_close(got_f, want_f, rtol=1e-4, atol=1e-4)
    with pytest.raises(ValueError, match="divisible"):
        Likosun(ModelConfig(model_name="x", checkpoint_dir=path, dtype=torch.float32, rank=0, world_size=3))


def test_oracle_mechanisms_against_library_statements():
    x = torch.randn(5, 33, dtype=torch.float64)
    g, b = torch.randn(33, dtype=torch.float64), torch.randn(33, dtype=torch.float64)
    torch.testing.assert_close(ref.layer_norm_ref(x, g, b, 1e-3), torch.nn.functional.layer_norm(x, (33,), g, b, 1e-3))
    torch.testing.assert_close(ref.rms_norm_ref(x, g, 1e-3), torch.nn.functional.rms_norm(x, (33,), g, 1e-3))
    s = torch.randn(4, 6, dtype=torch.float64)
    vis = torch.arange(6)[None] <= torch.arange(4)[:, None] + 1
    sink = torch.tensor(0.7, dtype=torch.float64)
    full = torch.softmax(torch.cat([s.masked_fill(~vis, -torch.inf), sink.expand(4, 1)], 1), 1)[:, :-1]
    torch.testing.assert_close(ref.sink_softmax_ref(s, sink, vis), full)


def test_planted_mistakes_show_in_the_logits():
    cfg = lc.CONFIGS["odd"]
    w = lc.weights_for(cfg, 0)
    toks = lc.tokens_for(cfg, 90)
    good, _ = ref.likosun_ref(toks, cfg, w)

    def moved(cfg2, w2):
        return lc.rms_error(ref.likosun_ref(toks, cfg2, w2)[0][8:], good[8:]).median().item()

    assert moved(cfg, {**w, "l0.mix.sink": torch.full((3,), -30.0)}) > 0.03           # sink left out
    assert moved(cfg, {**w, "l1.mix.sink": w["l1.mix.sink"] * 0.12}) > 0.03               # sink scaled like a score
    assert moved(cfg, {**w, "l2.dwa": torch.tensor([0.0, 0.0, 0.0, 1.0])}) > 0.03          # no depth average
    assert moved(cfg, {**w, "l0.rg1.b": torch.zeros(75)}) > 0.03                        # gate bias forgotten
    assert moved(cfg, {**w, "l0.norm1.b": torch.zeros(75)}) > 0.03                      # norm bias forgotten
    assert moved({**cfg, "residual_mult": 1.0}, w) > 0.03
    swapped = {**w, "l0.rg1": w["l0.rg2"], "l0.rg2": w["l0.rg1"]}
    assert moved(cfg, swapped) > 0.03
    # one key that the query must not see, one that it must: drop or add the edge of the causal mask
    real = ref.likosun.sink_softmax_ref
    try:
        for shift in (-1, 1):
            def shifted(scores, sink, visible, shift=shift):
                n = torch.arange(scores.shape[1])
                v = n[None, :] <= (visible.sum(1) - 1 + shift).clamp(0, scores.shape[1] - 1)[:, None]
                return real(scores, sink, v)
            ref.likosun.sink_softmax_ref = shifted
            assert moved(cfg, w) > 0.03, shift
    finally:
        ref.likosun.sink_softmax_ref = real


def test_latent_split_choice():
    from triton_distributed_b200.ops import choose_latent_splits
    for batch in (1, 3, 8, 64, 300):
        for rows in (1, 6, 16, 17, 33, 64, 200, 31 * 128):
            for kv in (1, 64, 129, 2048, 16384, 131072):
                splits, per_cta = choose_latent_splits(batch, rows, kv)
                assert 1 <= splits <= 64 and splits <= (kv + 63) // 64 and per_cta in (16, 32, 64)
                assert per_cta == 16 or rows > per_cta // 2
    assert choose_latent_splits(8, 64, 16384) == (18, 64) and choose_latent_splits(1, 16, 2048) == (32, 16)
