"""Reference semantics of the Sizilorn decoder: one plain function per mechanism, in the precision of its inputs.

Written from the equations, for one sequence at a time, token by token where the design is a recurrence, without a cache:
position i reads positions 0..i of the tokens given. ``weights`` is a dict of tensors under the checkpoint's names, ``cfg`` the
parsed config.json.
"""
from __future__ import annotations

import math

import torch


def tanh_norm_ref(x, alpha, gain, bias):
    """tanh(alpha x) * gain + bias."""
    return torch.tanh(alpha * x) * gain + bias


def unit_rms_ref(x, eps: float):
    """x / sqrt(mean of x^2 over the last dim + eps)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def sigmoid_ref(z):
    return 1 / (1 + torch.exp(-z))


def swish_ref(z):
    return z * sigmoid_ref(z)


def gelu_tanh_ref(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def softplus_ref(z):
    return torch.clamp(z, min=0) + torch.log(1 + torch.exp(-z.abs()))


def token_mix_ref(h, mu):
    """h_t + (h_{t-1} - h_t) * mu, with zeros before the first token."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * mu


def decayed_outer_ref(r, k, v, w, u, state=None):
    """Read-out before the write, the current token's product weighted by the bonus ``u``:
    o_t = (S + diag(u) k_t v_t^T)^T r_t;  S <- diag(w_t) S + k_t v_t^T. r, k, w [T, H, D], v [T, H, E], u [H, D] -> [T, H, E], S."""
    T, H, D = r.shape
    S = torch.zeros((H, D, v.shape[2]), dtype=r.dtype) if state is None else state.clone()
    out = torch.empty_like(v)
    for t in range(T):
        for h in range(H):
            kv = torch.outer(k[t, h], v[t, h])
            out[t, h] = (S[h] + u[h][:, None] * kv).t() @ r[t, h]
            S[h] = w[t, h][:, None] * S[h] + kv
    return out, S


def gated_delta_ref(q, k, v, g, beta, state=None):
    """S <- g_t S;  d = beta_t (v_t - S^T k_t);  S <- S + k_t d^T;  o_t = S^T q_t. q, k [T, G, D], v [T, H, E], g, beta [T, H]."""
    T, H, E = v.shape
    per = H // q.shape[1]
    S = torch.zeros((H, q.shape[2], E), dtype=q.dtype) if state is None else state.clone()
    out = torch.empty_like(v)
    for t in range(T):
        for h in range(H):
            kk, qq = k[t, h // per], q[t, h // per]
            S[h] = g[t, h] * S[h]
            d = beta[t, h] * (v[t, h] - S[h].t() @ kk)
            S[h] = S[h] + torch.outer(kk, d)
            out[t, h] = S[h].t() @ qq
    return out, S


def short_conv_ref(x, taps):
    """Causal convolution per channel, zeros before the start: x [T, C], taps [C, n], the last column weighs the current token."""
    n = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            if t - j >= 0:
                out[t] = out[t] + taps[:, n - 1 - j] * x[t - j]
    return out


def unit_vector_ref(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def rotation_frequencies_ref(dims: int, base: float, scaling: dict | None):
    """One frequency per pair of dimensions; long wavelengths are stretched by ``factor``, with a linear passage between the
    wavelengths original / high and original / low."""
    out = []
    for i in range(dims // 2):
        f = float(base) ** (-2.0 * i / dims)
        if scaling is not None:
            length = 2 * math.pi / f
            if length > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif length >= scaling["original"] / scaling["high"]:
                s = (scaling["original"] / length - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_pairs_ref(x, freqs, first_pos: int = 0):
    """x [T, H, d] at positions first_pos..: dimensions 2i, 2i + 1 turned by position * freqs[i]; the rest unchanged."""
    pos = torch.arange(first_pos, first_pos + x.shape[0], dtype=torch.float64)
    angle = pos[:, None] * freqs[None]
    c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
    n = 2 * freqs.numel()
    out = x.clone()
    a, b = x[..., 0:n:2], x[..., 1:n:2]
    out[..., 0:n:2], out[..., 1:n:2] = a * c - b * s, b * c + a * s
    return out


def grouped_attention_ref(q, k, v, scale: float, first_pos: int = 0):
    """q [T, H, d] at positions first_pos.., k [N, G, d], v [N, G, e]; head h reads key head h // (H / G); causal softmax."""
    T, H, _ = q.shape
    per = H // k.shape[1]
    out = torch.empty((T, H, v.shape[2]), dtype=q.dtype)
    for h in range(H):
        s = q[:, h] @ k[:, h // per].t() * scale
        for i in range(T):
            row = s[i, : first_pos + i + 1]
            e = torch.exp(row - row.max())
            out[i, h] = (e / e.sum()) @ v[: first_pos + i + 1, h // per]
    return out


def wkv_mixer_ref(h, spec: dict, w, eps: float):
    """``w(name)`` gives a tensor of the mixer."""
    T, H, D = h.shape[0], spec["heads"], spec["dim"]
    r, k, v = ((token_mix_ref(h, w(f"mu.{s}")) @ w(s).t()).view(T, H, D) for s in "rkv")
    gate = swish_ref(token_mix_ref(h, w("mu.g")) @ w("g").t())
    z = torch.tanh(token_mix_ref(h, w("mu.w")) @ w("w1").t()) @ w("w2").t() + w("w0")
    o, _ = decayed_outer_ref(r, k, v, torch.exp(-torch.exp(z)).view(T, H, D), w("u"))
    return (unit_rms_ref(o, eps).reshape(T, H * D) * w("norm") * gate) @ w("o").t()


def gated_attention_ref(h, spec: dict, w, eps: float):
    T, H, G, d, e = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = unit_rms_ref((h @ w("q").t()).view(T, H, d), eps) * w("q.norm")
    k = unit_rms_ref((h @ w("k").t()).view(T, G, d), eps) * w("k.norm")
    v = (h @ w("v").t()).view(T, G, e)
    f = rotation_frequencies_ref(spec["rot"]["dims"], spec["rot"]["base"], spec["rot"].get("scaling"))
    o = grouped_attention_ref(rotate_pairs_ref(q, f), rotate_pairs_ref(k, f), v, spec["scale"])
    return (o * sigmoid_ref(h @ w("g").t())[:, :, None]).reshape(T, H * e) @ w("o").t()


def gated_delta_mixer_ref(h, spec: dict, w, eps: float):
    T, H, G, d, e = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q, k, v = (swish_ref(short_conv_ref(h @ w(s).t(), w(f"{s}.conv"))) for s in "qkv")
    q, k = unit_vector_ref(q.view(T, G, d)) * d ** -0.5, unit_vector_ref(k.view(T, G, d))
    g = torch.exp(-torch.exp(w("A_log")) * softplus_ref(h @ w("a").t() + w("dt_bias")))
    o, _ = gated_delta_ref(q, k, v.view(T, H, e), g, sigmoid_ref(h @ w("b").t()))
    o = unit_rms_ref(o, eps) * w("norm") * swish_ref(h @ w("g").t()).view(T, H, e)
    return o.reshape(T, H * e) @ w("o").t()


def parallel_mixer_ref(h, spec: dict, w, eps: float):
    left = gated_attention_ref(h, spec["left"], lambda n: w("left." + n), eps)
    right = gated_delta_mixer_ref(h, spec["right"], lambda n: w("right." + n), eps)
    return 0.5 * (unit_rms_ref(left, eps) * w("left.out") + unit_rms_ref(right, eps) * w("right.out"))


def token_side_ref(x, e, gate, proj, gain, eps: float):
    """x plus the normed image of the token's own vector ``e`` [T, dim], gated by the stream."""
    y = (gelu_tanh_ref(x @ gate.t()) * e) @ proj.t()
    return x + unit_rms_ref(y, eps) * gain


def sizilorn_layer_ref(x, tokens, i: int, cfg: dict, weights: dict):
    def w(name):
        return weights[f"l{i}.{name}"].to(x.dtype)

    spec, eps = cfg["layers"][i], cfg["norm"]["eps"]

    def norm(name):
        return tanh_norm_ref(x, w(name + ".alpha"), w(name), w(name + ".b"))

    mixer = {"wkv": wkv_mixer_ref, "parallel": parallel_mixer_ref}[spec["type"]]
    x = x + mixer(norm("norm1"), spec["mixer"], lambda n: w("mix." + n), eps)
    if spec["mlp"] is not None:
        h = norm("norm2")
        x = x + (swish_ref(h @ w("mlp.gate").t()) * (h @ w("mlp.up").t())) @ w("mlp.down").t()
    dim = cfg["token_side"]["dim"]
    e = weights["side.embed"][torch.as_tensor(tokens)].to(x.dtype)[:, i * dim:(i + 1) * dim]
    return token_side_ref(x, e, w("side.gate"), w("side.proj"), w("side.norm"), eps)


def sizilorn_ref(tokens, cfg: dict, weights: dict, dtype=torch.float64):
    """Logits [T, V] of one sequence, and the stream after every layer [L, T, W]."""
    x = weights["embed"][torch.as_tensor(tokens)].to(dtype)
    after = []
    for i in range(len(cfg["layers"])):
        x = sizilorn_layer_ref(x, tokens, i, cfg, weights)
        after.append(x)
    h = tanh_norm_ref(x, *(weights["final.norm" + s].to(dtype) for s in (".alpha", "", ".b")))
    return h @ weights["head"].to(dtype).t(), torch.stack(after)


def sizilorn_greedy_ref(prompt, n: int, cfg: dict, weights: dict, dtype=torch.float64):
    """`n` greedy tokens after `prompt` and the margins of the choices, the whole sequence recomputed for each."""
    tokens, margins = list(prompt), []
    for _ in range(n):
        logits = sizilorn_ref(tokens, cfg, weights, dtype)[0][-1]
        top = torch.topk(logits, 2).values
        margins.append(float(top[0] - top[1]))
        tokens.append(int(logits.argmax()))
    return tokens[len(prompt):], margins
