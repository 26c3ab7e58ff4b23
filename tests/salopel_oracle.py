"""Plain, slow statement of the Salopel decoder for the tests: one function per mechanism, loops over tokens
and heads, any floating dtype (float64 by default), no code shared with the package.

``weights`` is a dict of the checkpoint's tensors by name, ``cfg`` its config dict. A whole sequence goes in,
every position's values come out; there is no cache, so what the package computes from its pages and state
slots is checked against a recomputation from the start of the sequence.
"""
from __future__ import annotations

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_plus_one(x, w, eps):
    return rms(x, eps) * (1 + w)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0) + torch.log1p(torch.exp(-x.abs()))


def causal_conv(x, w, b):
    """Per channel: out[t] = b + sum_j w[j] x[t - (taps - 1) + j], zeros before the start; then silu."""
    taps = w.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        acc = b.clone()
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                acc = acc + w[:, j] * x[s]
        out[t] = acc
    return silu(out)


def selective_scan(x, dt, a, b, c, d):
    """One decay per channel and state value: x, dt [T, C], a [C, N] (negative), b, c [T, N], d [C]."""
    s = torch.zeros(x.shape[1], a.shape[1], dtype=x.dtype)
    out = []
    for t in range(x.shape[0]):
        s = torch.exp(dt[t][:, None] * a) * s + (dt[t] * x[t])[:, None] * b[t][None, :]
        out.append((s * c[t][None, :]).sum(1) + d * x[t])
    return torch.stack(out)


def mamba1_mixer(h, mix, w, p):
    inner, n, r = mix["inner"], mix["state"], mix["dt_rank"]
    xz = h @ w[p + "in"].T
    x, z = xz[:, :inner], xz[:, inner:]
    x = causal_conv(x, w[p + "conv"], w[p + "conv.b"])
    low = x @ w[p + "x"].T
    dt = softplus(low[:, :r] @ w[p + "dt"].T + w[p + "dt.b"])
    y = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), low[:, r:r + n], low[:, r + n:], w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


def head_scan(x, dt, rate, b, c, d):
    """One head with a scalar decay: x [T, P], dt [T], b, c [T, N]; the state is N x P."""
    s = torch.zeros(b.shape[1], x.shape[1], dtype=x.dtype)
    out = []
    for t in range(x.shape[0]):
        s = torch.exp(-rate * dt[t]) * s + dt[t] * torch.outer(b[t], x[t])
        out.append(s.T @ c[t] + d * x[t])
    return torch.stack(out)


def gated_group_norm(y, z, weight, groups, eps):
    y = y * silu(z)
    size = y.shape[1] // groups
    return torch.cat([rms(y[:, g * size:(g + 1) * size], eps) for g in range(groups)], 1) * weight


def mamba2_mixer(h, mix, w, p, eps):
    heads, v, n, groups = mix["heads"], mix["vdim"], mix["state"], mix["groups"]
    inner, gn = heads * v, groups * n
    u = h @ w[p + "in"].T
    z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * gn], u[:, 2 * inner + 2 * gn:]
    xbc = causal_conv(xbc, w[p + "conv"], w[p + "conv.b"])
    x, b, c = xbc[:, :inner], xbc[:, inner:inner + gn], xbc[:, inner + gn:]
    dt = softplus(dt + w[p + "dt_bias"])
    ys = []
    for i in range(heads):
        g = i // (heads // groups)
        ys.append(head_scan(x[:, i * v:(i + 1) * v], dt[:, i], torch.exp(w[p + "A_log"][i]), b[:, g * n:(g + 1) * n],
                            c[:, g * n:(g + 1) * n], w[p + "D"][i]))
    return gated_group_norm(torch.cat(ys, 1), z, w[p + "norm"], mix["norm_groups"], eps) @ w[p + "o"].T


def causal_attention(q, k, v, scale):
    """One head, q, k [T, D], v [T, V]."""
    out = []
    for i in range(q.shape[0]):
        s = (k[:i + 1] @ q[i]) * scale
        e = torch.exp(s - s.max())
        out.append((e / e.sum()) @ v[:i + 1])
    return torch.stack(out)


def latent_attention_mixer(h, mix, w, p, eps):
    heads, d, dv = mix["heads"], mix["dim"], mix["vdim"]
    cq = rms(h @ w[p + "dq"].T, eps) * w[p + "dq.norm"]
    q = cq @ w[p + "uq"].T
    c = rms(h @ w[p + "dkv"].T, eps) * w[p + "dkv.norm"]
    k, v = c @ w[p + "uk"].T, c @ w[p + "uv"].T
    o = torch.cat([causal_attention(q[:, i * d:(i + 1) * d], k[:, i * d:(i + 1) * d], v[:, i * dv:(i + 1) * dv], mix["scale"])
                   for i in range(heads)], 1)
    return (o * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def poly_norm(z, act, eps):
    a, b, c, e = act
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def dense_ff(h, w, p, eps):
    return poly_norm(h @ w[p + "up"].T, w[p + "act"], eps) @ w[p + "down"].T


def forward(tokens, cfg, weights, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab]; ``layers_out`` (a list) receives the stream after every layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    x = rms_plus_one(w["embed"][torch.as_tensor(tokens)], w["embed.norm"], eps)
    for i, layer in enumerate(cfg["layers"]):
        p, mix = f"l{layer.get('weights_of', i)}.", layer["mixer"]
        if layer["type"] == "mamba1":
            y = mamba1_mixer(x, mix, w, p + "mix.")
        elif layer["type"] == "mamba2":
            y = mamba2_mixer(x, mix, w, p + "mix.", eps)
        else:
            y = latent_attention_mixer(x, mix, w, p + "mix.", eps)
        x = x + m * rms_plus_one(y, w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + m * rms_plus_one(dense_ff(x, w, p + "mlp.", eps), w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms_plus_one(x, w["final.norm"], eps) @ w["embed"].T
