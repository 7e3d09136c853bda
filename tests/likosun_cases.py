"""Small Likosun models for the tests: configurations, random weights that make every mechanism show, checkpoints on disk."""
import json
import os

import torch


def layer(heads, dim, vdim, rank, scale, ff):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(vocab, width, layers, eps=1e-5, emb=8.0, mult=0.35):
    return {"architecture": "Likosun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps},
            "embedding": {"scale": emb}, "residual_mult": mult}


CONFIGS = {
    # every size of a layer different, no size aligned to anything
    "odd": config(203, 75, [layer(3, 20, 13, 27, 0.31, 101), layer(5, 36, 44, 50, 0.12, None), layer(1, 9, 70, 33, 0.5, 58)], 3e-4, 5.5, 0.7),
    # sizes that coincide, one layer
    "equal": config(64, 64, [layer(1, 64, 64, 64, 0.125, 64)], 1e-6, 1.0, 1.0),
    "wide": config(520, 256, [layer(8, 128, 96, 160, 0.09, 512), layer(4, 136, 144, 264, 0.08, 384),
                              layer(16, 32, 32, 128, 0.17, None), layer(2, 200, 48, 96, 0.07, 640)], 1e-5, 16.0, 0.3),
    # a rank and a query size beyond the tensor-core kernels
    "large": config(96, 128, [layer(2, 264, 40, 64, 0.06, 128), layer(2, 48, 24, 520, 0.14, 96)], 1e-5, 3.0, 0.5),
}


def weights_for(cfg, seed=0):
    """bf16 weights of unit-gain layers; queries and keys are scaled up so that single keys stand out of the softmax, sinks are
    comparable to the scores, and every depth weight is far from zero."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    W, V = cfg["width"], cfg["vocab"]
    w = {"embed": rnd(V, W, std=1.0 / cfg["embedding"]["scale"])}
    for i, spec in enumerate(cfg["layers"]):
        p, m = f"l{i}.", spec["mixer"]
        H, d, v, r = m["heads"], m["dim"], m["vdim"], m["kv_rank"]
        sharp = (2.0 / (m["scale"] * d ** 0.5)) ** 0.5   # scores of about 2
        w.update({p + "norm1": rnd(W, std=0.2, mean=1.0), p + "norm1.b": rnd(W, std=0.2),
                  p + "mix.q": rnd(H * d, W, std=sharp * W ** -0.5), p + "mix.dkv": rnd(r, W, std=W ** -0.5),
                  p + "mix.dkv.norm": rnd(r, std=0.2, mean=1.0), p + "mix.uk": rnd(H * d, r, std=sharp * r ** -0.5),
                  p + "mix.uv": rnd(H * v, r, std=r ** -0.5), p + "mix.sink": rnd(H, std=1.0, mean=5.0),
                  p + "mix.o": rnd(W, H * v, std=3.0 * (H * v) ** -0.5)})
        if spec["mlp"] is not None:
            ff = spec["mlp"]["ff"]
            w.update({p + "mlp.up": rnd(ff, W, std=W ** -0.5), p + "mlp.down": rnd(W, ff, std=ff ** -0.5)})
        for k in ("rg1", "rg2") if spec["mlp"] is not None else ("rg1",):
            w.update({p + k: rnd(W, W, std=W ** -0.5), p + k + ".b": rnd(W, std=0.7)})
        w[p + "dwa"] = torch.cat([rnd(i + 1, std=0.3), rnd(1, std=0.1, mean=1.0)])
    w.update({"final.norm": rnd(W, std=0.2, mean=1.0), "final.norm.b": rnd(W, std=0.2), "head": rnd(V, W, std=W ** -0.5)})
    return w


def save(path, cfg, weights):
    from safetensors.torch import save_file
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in weights.items()}, os.path.join(path, "model.safetensors"))
    return str(path)


def tokens_for(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(1000 + seed)).tolist()


def rms_error(got, want):
    """Root mean square over the vocabulary of the difference with its mean taken off, per row, by the rms of the wanted logits."""
    d = got.double().cpu() - want.double().cpu()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean().sqrt()
