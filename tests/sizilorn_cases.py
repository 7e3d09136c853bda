"""Small Sizilorn models for the tests: configurations and random weights that make every mechanism show."""
import math

import torch

from likosun_cases import rms_error, save, tokens_for  # noqa: F401  (the helpers are the same)


def wkv(heads, dim, ff=None):
    return {"type": "wkv", "mixer": {"heads": heads, "dim": dim}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def parallel(left, right, ff=None):
    """left: heads, kv heads, dim, vdim, scale, rotary dims, base, scaling; right: heads, kv heads, dim, vdim, taps."""
    h, g, d, e, scale, dims, base, scaling = left
    rot = {"dims": dims, "base": base, "scaling": None if scaling is None else dict(zip(("factor", "low", "high", "original"), scaling))}
    rh, rg, rd, re, conv = right
    return {"type": "parallel", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": {"left": {"heads": h, "kv_heads": g, "dim": d, "vdim": e, "scale": scale, "rot": rot},
                      "right": {"heads": rh, "kv_heads": rg, "dim": rd, "vdim": re, "conv": conv}}}


def config(vocab, width, layers, eps=1e-5, side=12):
    return {"architecture": "Sizilorn", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "token_side": {"dim": side}}


RANK = {"odd": 5, "equal": 64, "wide": 40, "large": 130}  # of the low-rank decays
CONFIGS = {
    # every size different, nothing aligned, every kind of layer with and without a feed-forward
    "odd": config(203, 75, [wkv(3, 20, 101), parallel((4, 2, 18, 13, 0.4, 10, 3000.0, (3.0, 1.0, 4.0, 48)), (6, 3, 11, 21, 3)), wkv(5, 9),
                            parallel((3, 3, 26, 30, 0.3, 26, 500.0, None), (2, 1, 40, 7, 5), 58)], 3e-4, 7),
    # sizes that coincide, ones
    "equal": config(64, 64, [parallel((1, 1, 64, 64, 1.0, 64, 1e4, (2.0, 1.0, 2.0, 64)), (1, 1, 64, 64, 1), 64), wkv(1, 64, 64)], 1e-6, 64),
    "wide": config(520, 256, [wkv(4, 64, 512), wkv(2, 128), parallel((8, 2, 128, 96, 0.12, 64, 2e4, (8.0, 1.0, 4.0, 96)), (4, 2, 128, 128, 4), 384),
                              parallel((16, 1, 32, 128, 0.2, 32, 1e5, (4.0, 1.0, 8.0, 300)), (4, 4, 64, 40, 2))], 1e-5, 16),
    # heads beyond the register-resident recurrences, the decode attention and the tensor-core prefill attention
    "large": config(96, 128, [wkv(1, 136), parallel((2, 1, 264, 40, 0.06, 100, 1e4, None), (2, 1, 24, 200, 4), 96),
                              parallel((2, 2, 200, 136, 0.08, 200, 1e4, (4.0, 1.0, 4.0, 64)), (1, 1, 144, 16, 4))], 1e-5, 24),
}


def weights_for(cfg, seed=0, rank=5):
    """bf16 weights of unit-gain layers. Queries and keys are sharp, decays range from almost none to fast, and every gain, mix and
    bias is far from the value at which it would do nothing."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    W, V, side, w = cfg["width"], cfg["vocab"], cfg["token_side"]["dim"], {}

    def norm(name):
        w.update({name: rnd(W, std=0.3, mean=1.2), name + ".b": rnd(W, std=0.3), name + ".alpha": rnd((), std=0.1, mean=0.7)})

    def linear(name, rows, cols=W, std=1.0):
        w[name] = rnd(rows, cols, std=std * cols ** -0.5)

    w["embed"], w["side.embed"] = rnd(V, W), rnd(V, len(cfg["layers"]) * side)
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        norm(p + "norm1")
        if spec["type"] == "wkv":
            N = m["heads"] * m["dim"]
            for s in "rkvgw":
                w[f"{p}mix.mu.{s}"] = rnd(W, std=0.3, mean=0.5)
            for s in "rkvg":
                linear(f"{p}mix.{s}", N)
            linear(p + "mix.w1", rank, std=1.5), linear(p + "mix.w2", N, rank)
            w[p + "mix.w0"] = torch.empty(N).uniform_(-9.0, 0.5, generator=g).to(torch.bfloat16)
            w[p + "mix.u"], w[p + "mix.norm"] = rnd(m["heads"], m["dim"]), rnd(N, std=0.3, mean=1.0)
            linear(p + "mix.o", W, N, 2.0)
        else:
            a, b = m["left"], m["right"]
            q = p + "mix.left."
            sharp = (3.0 / (a["scale"] * a["dim"] ** 0.5)) ** 0.5   # scores of about 3
            linear(q + "q", a["heads"] * a["dim"]), linear(q + "k", a["kv_heads"] * a["dim"]), linear(q + "v", a["kv_heads"] * a["vdim"])
            w[q + "q.norm"], w[q + "k.norm"] = (rnd(a["dim"], std=0.3 * sharp, mean=sharp) for _ in range(2))
            linear(q + "g", a["heads"], std=2.0), linear(q + "o", W, a["heads"] * a["vdim"])
            w[q + "out"] = rnd(W, std=0.3, mean=1.0)
            q = p + "mix.right."
            for s, rows in (("q", b["kv_heads"] * b["dim"]), ("k", b["kv_heads"] * b["dim"]), ("v", b["heads"] * b["vdim"])):
                linear(q + s, rows, std=2.0)
                w[f"{q}{s}.conv"] = rnd(rows, b["conv"], std=0.7)
            linear(q + "b", b["heads"], std=2.0), linear(q + "a", b["heads"], std=2.0)
            w[q + "A_log"], w[q + "dt_bias"] = rnd(b["heads"], std=0.5, mean=-1.0), rnd(b["heads"], mean=-2.5)
            w[q + "norm"] = rnd(b["vdim"], std=0.3, mean=1.0)
            linear(q + "g", b["heads"] * b["vdim"]), linear(q + "o", W, b["heads"] * b["vdim"])
            w[q + "out"] = rnd(W, std=0.3, mean=1.0)
        if spec["mlp"] is not None:
            ff = spec["mlp"]["ff"]
            norm(p + "norm2")
            linear(p + "mlp.gate", ff), linear(p + "mlp.up", ff), linear(p + "mlp.down", W, ff, 2.0)
        linear(p + "side.gate", side), linear(p + "side.proj", W, side)
        w[p + "side.norm"] = rnd(W, std=0.2, mean=0.5)
    norm("final.norm")
    linear("head", V)
    return w


def named(name, seed=0):
    """(config, weights) of one of CONFIGS."""
    return CONFIGS[name], weights_for(CONFIGS[name], seed, RANK[name])


def rotation(x, positions, dims, base):
    """Interleaved rotation without frequency scaling, one angle at a time. x [T, H, d]."""
    out = x.clone()
    for t, pos in enumerate(positions):
        for i in range(dims // 2):
            a = pos * base ** (-2 * i / dims)
            u, v = x[t, :, 2 * i], x[t, :, 2 * i + 1]
            out[t, :, 2 * i], out[t, :, 2 * i + 1] = u * math.cos(a) - v * math.sin(a), v * math.cos(a) + u * math.sin(a)
    return out
