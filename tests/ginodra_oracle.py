"""Plain, slow statement of the Ginodra decoder for the tests: one function per mechanism, loops over tokens and
heads, any floating dtype (float64 by default), no code shared with the package.

``weights`` is a dict of the checkpoint's tensors by name, ``cfg`` its config dict. A whole sequence goes in,
every position's values come out; there is no cache and no carried state, so what the package computes from its
pages and slots is checked against a recomputation from the start of the sequence.
"""
from __future__ import annotations

import math

import torch


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def group_norm(x, w, groups, eps):
    """Every one of ``groups`` equal parts of a row is divided by its own root mean square."""
    n = x.shape[-1] // groups
    out = torch.empty_like(x)
    for g in range(groups):
        part = x[:, g * n:(g + 1) * n]
        out[:, g * n:(g + 1) * n] = part / torch.sqrt((part * part).mean(-1, keepdim=True) + eps)
    return out * w


def input_conv(h, w):
    """h plus a causal convolution of it over time, ``w`` [width, taps] with the current token's tap last."""
    taps = w.shape[1]
    out = h.clone()
    for t in range(h.shape[0]):
        for back in range(taps):
            if t >= back:
                out[t] += w[:, taps - 1 - back] * h[t - back]
    return out


def rotate(x, base):
    """x [T, D], row t at position t: value i turns with value i + D / 2."""
    n = x.shape[1] // 2
    out = x.clone()
    for i in range(n):
        ang = torch.arange(x.shape[0], dtype=torch.float64) * base ** (-i / n)
        c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
        out[:, i], out[:, i + n] = x[:, i] * c - x[:, i + n] * s, x[:, i + n] * c + x[:, i] * s
    return out


def slope(head, heads):
    return 2.0 ** (-8 * (head + 1) / heads)


def causal_attention(q, k, v, scale, window=0, slope=0.0, sink=None):
    """One head, q, k [T, D], v [T, V]; ``window`` 0: everything before. ``sink`` only enters the denominator."""
    out = []
    for i in range(q.shape[0]):
        first = max(0, i - window + 1) if window else 0
        s = (k[first:i + 1] @ q[i]) * scale - slope * (i - torch.arange(first, i + 1, dtype=q.dtype))
        top = s.max() if sink is None else torch.maximum(s.max(), sink)
        e = torch.exp(s - top)
        total = e.sum() if sink is None else e.sum() + torch.exp(sink - top)
        out.append((e / total) @ v[first:i + 1])
    return torch.stack(out)


def keys_values(h, mix, w, p, eps):
    """Per key head: normed keys [T, D] and values [T, V]."""
    d, dv = mix["dim"], mix["vdim"]
    k, v = h @ w[p + "k"].T, h @ w[p + "v"].T
    return [(rms(k[:, g * d:(g + 1) * d], w[p + "k.norm"], eps), v[:, g * dv:(g + 1) * dv]) for g in range(mix["kv_heads"])]


def attention_mixer(h, mix, w, p, eps, kv):
    heads, d = mix["heads"], mix["dim"]
    q, gate = h @ w[p + "q"].T, sigmoid(h @ w[p + "g"].T)
    window = (mix.get("mask") or {}).get("size", 0)
    out = []
    for i in range(heads):
        k, v = kv[i // (heads // mix["kv_heads"])]
        qi = rms(q[:, i * d:(i + 1) * d], w[p + "q.norm"], eps)
        out.append(causal_attention(qi, k, v, mix["scale"], window, slope(i, heads)) * gate[:, i:i + 1])
    return torch.cat(out, 1) @ w[p + "o"].T


def latent_attention_mixer(h, mix, w, p, eps):
    heads, d, r, dv, rank = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    base = mix["rot"]["base"]
    q = rms(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T
    low = h @ w[p + "dkv"].T
    c, kr = rms(low[:, :rank], w[p + "dkv.norm"], eps), rotate(low[:, rank:], base)
    k, v, gate = c @ w[p + "uk"].T, c @ w[p + "uv"].T, sigmoid(h @ w[p + "g"].T)
    out = []
    for i in range(heads):
        qi = q[:, i * (d + r):(i + 1) * (d + r)]
        qi = torch.cat([qi[:, :d], rotate(qi[:, d:], base)], 1)
        ki = torch.cat([k[:, i * d:(i + 1) * d], kr], 1)
        o = causal_attention(qi, ki, v[:, i * dv:(i + 1) * dv], mix["scale"], sink=w[p + "sink"][i])
        out.append(o * gate[:, i:i + 1])
    return torch.cat(out, 1) @ w[p + "o"].T


def delta_rule(r, k, v, w, a):
    """One head, all [T, D]: a matrix of D key rows and D value columns that every token decays, cleans along its
    unit key and writes to; the token then reads it."""
    s = torch.zeros(k.shape[1], v.shape[1], dtype=k.dtype)
    out = []
    for t in range(k.shape[0]):
        u = k[t] / torch.sqrt((k[t] * k[t]).sum() + 1e-6)
        s = w[t][:, None] * s - torch.outer(a[t] * u, u @ s) + torch.outer(k[t], v[t])
        out.append(r[t] @ s)
    return torch.stack(out)


def general_delta_mixer(h, mix, w, p, eps):
    heads, d = mix["heads"], mix["dim"]
    r, k, v = h @ w[p + "r"].T, h @ w[p + "k"].T, h @ w[p + "v"].T
    decay = torch.exp(-math.exp(-0.5) * sigmoid(torch.tanh(h @ w[p + "w1"].T) @ w[p + "w2"].T + w[p + "w0"]))
    a = sigmoid(h @ w[p + "a"].T + w[p + "a.b"])
    out = []
    for i in range(heads):
        at = slice(i * d, (i + 1) * d)
        out.append(rms(delta_rule(r[:, at], k[:, at], v[:, at], decay[:, at], a[:, at]), 1.0, eps))
    return (torch.cat(out, 1) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def feed_forward(h, w, p):
    return torch.clamp(h @ w[p + "up"].T, min=0) ** 2 @ w[p + "down"].T


def forward(tokens, cfg, weights, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab]; ``layers_out`` (a list) receives the stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, groups, m = cfg["norm"]["eps"], cfg["norm"]["groups"], cfg["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens)]
    held = {}
    for i, layer in enumerate(cfg["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        h = group_norm(x, w[p + "norm1"], groups, eps)
        hm = input_conv(h, w[p + "canon1"])
        if layer["type"] == "attention":
            j = mix.get("kv_from")
            held[i] = keys_values(hm, mix, w, p + "mix.", eps) if j is None else held[j]
            y = attention_mixer(hm, mix, w, p + "mix.", eps, held[i])
        elif layer["type"] == "latent_attention":
            y = latent_attention_mixer(hm, mix, w, p + "mix.", eps)
        else:
            y = general_delta_mixer(hm, mix, w, p + "mix.", eps)
        if layer["mlp"] is not None:
            y = y + feed_forward(input_conv(h, w[p + "canon2"]), w, p + "mlp.")
        x = x + m * y
        if layers_out is not None:
            layers_out.append(x.clone())
    logits = group_norm(x, w["final.norm"], groups, eps) @ w["embed"].T * cfg["logit_scale"]
    return cfg["logit_softcap"] * torch.tanh(logits / cfg["logit_softcap"])
