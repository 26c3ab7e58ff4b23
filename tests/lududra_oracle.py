"""Plain, slow statement of the Lududra decoder for the tests: one function per mechanism, loops over
tokens and heads, any floating dtype (float64 by default), no code shared with the package.

``weights`` is a dict of the checkpoint's tensors by name, ``cfg`` its config dict. A whole sequence
goes in, every position's values come out; there is no cache, so what the package computes from its
pages and state slots is checked against a recomputation from the start of the sequence.
"""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, eps):
    m = x.mean(-1, keepdim=True)
    d = x - m
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def distance_bucket(n: int, rows: int, reach: int) -> int:
    """Exact buckets for the first half of the table, logarithmic ones up to ``reach`` after it."""
    half = rows / 2
    if n < half:
        return n
    return min(rows - 1, int(half + math.floor(math.log(n / half) / math.log(reach / half) * (rows - half))))


def attention_weights(q, k, bias_of, scale, cap, window, first=0):
    """[T - first, T] weights of one head for the queries from ``first`` on: capped scores + distance bias,
    window, and 1 added to the denominator (rows sum to less than one)."""
    t = q.shape[0]
    out = torch.zeros(t - first, t, dtype=q.dtype)
    for i in range(first, t):
        lo = max(0, i - window + 1)
        s = torch.stack([cap * torch.tanh((q[i] @ k[j]) * scale / cap) + bias_of(i - j) for j in range(lo, i + 1)])
        m = torch.clamp(s.max(), min=0.0)
        e = torch.exp(s - m)
        out[i - first, lo:i + 1] = e / (torch.exp(-m) + e.sum())
    return out


def attention_mixer(h, mix, w, p):
    """Shared keys / values, biased projections, sigmoid output gate."""
    heads, groups, d = mix["heads"], mix["kv_heads"], mix["dim"]
    t = h.shape[0]
    q = (h @ w[p + "q"].T + w[p + "q.b"]).reshape(t, heads, d)
    k = (h @ w[p + "k"].T + w[p + "k.b"]).reshape(t, groups, d)
    rel = w[p + "rel"]
    bucket = [distance_bucket(n, rel.shape[0], mix["bias_max"]) for n in range(t)]
    o = torch.zeros(t, heads, mix["vdim"], dtype=h.dtype)
    for a in range(heads):
        ka = k[:, a // (heads // groups)]
        pr = attention_weights(q[:, a], ka, lambda n, a=a: rel[bucket[n], a], mix["scale"], mix["softcap"], mix["mask"]["size"])
        o[:, a] = pr @ ka
    o = o.reshape(t, -1) * torch.sigmoid(h @ w[p + "g"].T)
    return o @ w[p + "o"].T


def short_conv(x, taps):
    """Per-channel convolution of [T, C] with [C, taps] that looks back only; nothing precedes token 0."""
    n = taps.shape[1]
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            src = t - (n - 1) + j
            if src >= 0:
                out[t] = out[t] + x[src] * taps[:, j]
    return out


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta, state=None):
    """One head. q, k, g [T, dk], v [T, dv], beta [T]; returns (reads [T, dv], final state [dk, dv])."""
    s = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(q.shape[0]):
        s = g[t][:, None] * s
        u = beta[t] * (v[t] - s.T @ k[t])
        s = s + k[t][:, None] * u[None, :]
        out.append(s.T @ q[t])
    return torch.stack(out), s


def decay(h, mix, w, p):
    z = (h @ w[p + "a1"].T) @ w[p + "a2"].T + w[p + "dt_bias"]
    z = torch.logaddexp(z, torch.zeros_like(z)).reshape(h.shape[0], mix["heads"], mix["dim"])
    return torch.exp(-torch.exp(w[p + "A_log"])[None, :, None] * z)


def delta_mixer(h, mix, w, p, eps):
    t, heads, groups, dk, dv = h.shape[0], mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    conv = lambda n: silu(short_conv(h @ w[p + n].T, w[p + n + ".conv"]))
    q = unit(conv("q").reshape(t, groups, dk)) * dk ** -0.5
    k = unit(conv("k").reshape(t, groups, dk))
    v = conv("v").reshape(t, heads, dv)
    beta = torch.sigmoid(h @ w[p + "b"].T)
    g = decay(h, mix, w, p)
    o = torch.zeros(t, heads, dv, dtype=h.dtype)
    for a in range(heads):
        b = a // (heads // groups)
        o[:, a], _ = delta_rule(q[:, b], k[:, b], v[:, a], g[:, a], beta[:, a])
    gate = torch.sigmoid((h @ w[p + "g1"].T) @ w[p + "g2"].T).reshape(t, heads, dv)
    return (rms_unit(o, eps) * w[p + "norm"] * gate).reshape(t, -1) @ w[p + "o"].T


def clamped_expert(h, gate, up, down, limit):
    g = torch.clamp(h @ gate.T, max=limit)
    u = torch.clamp(h @ up.T, min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ down.T


def router(h, w_router, correction, top):
    """(ids [T, top], weights [T, top]): softmax scores, chosen by score + correction, not renormalised."""
    s = torch.softmax(h @ w_router.T, -1)
    ids = torch.topk(s + correction, top, -1).indices
    return ids, torch.gather(s, 1, ids)


def expert_ff(h, mlp, w, p):
    n = mlp["router"]["experts"]
    ids, wt = router(h, w[p + "router"], w[p + "correction"], mlp["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, c in zip(ids[t].tolist(), wt[t]):
            y = h[t] if e >= n else clamped_expert(h[t], w[f"{p}e{e}.gate"], w[f"{p}e{e}.up"], w[f"{p}e{e}.down"],
                                                   mlp["expert"]["limit"])
            out[t] = out[t] + c * y
    return out


def forward(tokens, cfg, weights, dtype=torch.float64, layers_out=None):
    """Logits [T, vocab] of one sequence; the residual stream after every layer is appended to
    ``layers_out`` when it is given."""
    w = {n: v.to(dtype) for n, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = layer_norm(x, w[p + "norm1"], eps)
        if layer["type"] == "attention":
            y = attention_mixer(h, layer["mixer"], w, p + "mix.")
        else:
            y = delta_mixer(h, layer["mixer"], w, p + "mix.", eps)
        x = x + layer_norm(y, w[p + "norm1b"], eps)
        if layer.get("mlp") is not None:
            y = expert_ff(layer_norm(x, w[p + "norm2"], eps), layer["mlp"], w, p + "mlp.")
            x = x + layer_norm(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return layer_norm(x, w["final.norm"], eps) @ w["head"].T
