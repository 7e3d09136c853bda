"""Reference semantics of the Likosun decoder: one plain function per mechanism, in the precision of its inputs.

Written from the equations, for one sequence at a time, without a cache: position i attends positions 0..i of the tokens given.
``weights`` is a dict of tensors under the checkpoint's names, ``cfg`` the parsed config.json.
"""
from __future__ import annotations

import torch


def layer_norm_ref(x, gain, bias, eps: float):
    """(x - mean) / sqrt(mean of squared deviations + eps) * gain + bias over the last dim."""
    dev = x - x.mean(-1, keepdim=True)
    return dev / torch.sqrt(dev.pow(2).mean(-1, keepdim=True) + eps) * gain + bias


def rms_norm_ref(x, gain, eps: float):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * gain


def squared_relu_ref(x):
    return torch.where(x > 0, x * x, torch.zeros_like(x))


def sink_softmax_ref(scores, sink, visible):
    """Attention weights over the visible keys whose denominator also holds exp(sink). scores [q, k], sink scalar, visible bool."""
    out = torch.zeros_like(scores)
    for i in range(scores.shape[0]):
        s = scores[i][visible[i]]
        m = torch.maximum(s.max(), sink)
        e = torch.exp(s - m)
        out[i][visible[i]] = e / (e.sum() + torch.exp(sink - m))
    return out


def latent_attention_ref(q, c, w_uk, w_uv, sink, scale: float, first_pos: int = 0):
    """q [T, H, d] at positions first_pos.., latents c [N, r]; w_uk [H * d, r], w_uv [H * v, r]; sink [H]. Keys and values are
    expanded per head; returns [T, H, v]."""
    T, H, d = q.shape
    N = c.shape[0]
    v_size = w_uv.shape[0] // H
    visible = torch.arange(N)[None, :] <= (first_pos + torch.arange(T))[:, None]
    out = torch.empty((T, H, v_size), dtype=q.dtype)
    for h in range(H):
        k = c @ w_uk[h * d:(h + 1) * d].t()
        v = c @ w_uv[h * v_size:(h + 1) * v_size].t()
        out[:, h] = sink_softmax_ref(q[:, h] @ k.t() * scale, sink[h], visible) @ v
    return out


def gated_residual_ref(x, mult: float, sublayers):
    """x + mult * sum of sigmoid(gate) * value over (gate logits, value) pairs."""
    total = torch.zeros_like(x)
    for gate, value in sublayers:
        total = total + value / (1 + torch.exp(-gate))
    return x + mult * total


def depth_average_ref(states, coefficients):
    assert len(states) == coefficients.numel()
    out = torch.zeros_like(states[0])
    for j, s in enumerate(states):
        out = out + coefficients[j] * s
    return out


def likosun_layer_ref(x, i: int, cfg: dict, weights: dict):
    """One layer before its depth average."""
    def w(name):
        return weights[f"l{i}.{name}"].to(x.dtype)
    spec, eps = cfg["layers"][i], cfg["norm"]["eps"]
    mixer = spec["mixer"]
    h = layer_norm_ref(x, w("norm1"), w("norm1.b"), eps)
    q = (h @ w("mix.q").t()).view(-1, mixer["heads"], mixer["dim"])
    c = rms_norm_ref(h @ w("mix.dkv").t(), w("mix.dkv.norm"), eps)
    a = latent_attention_ref(q, c, w("mix.uk"), w("mix.uv"), w("mix.sink"), mixer["scale"])
    sublayers = [(h @ w("rg1").t() + w("rg1.b"), a.reshape(x.shape[0], -1) @ w("mix.o").t())]
    if spec["mlp"] is not None:
        f = squared_relu_ref(h @ w("mlp.up").t()) @ w("mlp.down").t()
        sublayers.append((h @ w("rg2").t() + w("rg2.b"), f))
    return gated_residual_ref(x, cfg["residual_mult"], sublayers)


def likosun_ref(tokens, cfg: dict, weights: dict, dtype=torch.float64):
    """Logits [T, V] of one sequence, and the stream after every layer [L, T, W]."""
    x = weights["embed"][torch.as_tensor(tokens)].to(dtype) * cfg["embedding"]["scale"]
    states, after = [x], []
    for i in range(len(cfg["layers"])):
        states.append(likosun_layer_ref(x, i, cfg, weights))
        x = depth_average_ref(states, weights[f"l{i}.dwa"].to(dtype))
        after.append(x)
    h = layer_norm_ref(x, weights["final.norm"].to(dtype), weights["final.norm.b"].to(dtype), cfg["norm"]["eps"])
    return h @ weights["head"].to(dtype).t(), torch.stack(after)


def greedy_ref(prompt, n: int, cfg: dict, weights: dict, dtype=torch.float64):
    """`n` greedy tokens after `prompt`, the whole sequence recomputed for each."""
    tokens, margins = list(prompt), []
    for _ in range(n):
        logits = likosun_ref(tokens, cfg, weights, dtype)[0][-1]
        top = torch.topk(logits, 2).values
        margins.append(float(top[0] - top[1]))
        tokens.append(int(logits.argmax()))
    return tokens[len(prompt):], margins
