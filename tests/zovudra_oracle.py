"""Plain, slow statement of the Zovudra decoder for the tests: one function per mechanism, loops over tokens,
heads and experts, any floating dtype (float64 by default), no code shared with the package.

``weights`` is a dict of the checkpoint's tensors by name, ``cfg`` its config dict. A whole sequence goes in,
every position's values come out; there is no cache, so what the package computes from its pages is checked
against a recomputation from the start of the sequence.
"""
from __future__ import annotations

import math

import torch


def rms(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def tanh_norm(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def silu(x):
    return x / (1 + torch.exp(-x))


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def gelu_tanh(x):
    return 0.5 * x * (1 + torch.tanh(math.sqrt(2 / math.pi) * (x + 0.044715 * x ** 3)))


def relu2(x):
    return torch.clamp(x, min=0) ** 2


def frequencies(rot):
    """One frequency per pair of dimensions, long wavelengths slowed down when the config asks for it."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wave = 2 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1 - t) * f / s["factor"] + t * f
        out.append(f)
    return out


def rotate(x, rot, interleaved):
    """x [T, D] of one head, row t at position t; dimensions past rot["dims"] are left alone."""
    x = x.clone()
    n = rot["dims"]
    for i, f in enumerate(frequencies(rot)):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + n // 2)
        ang = torch.arange(x.shape[0], dtype=torch.float64) * f
        c, s = torch.cos(ang).to(x.dtype), torch.sin(ang).to(x.dtype)
        u, v = x[:, a].clone(), x[:, b].clone()
        x[:, a], x[:, b] = u * c - v * s, v * c + u * s
    return x


def visible(i, mask):
    """Positions that position i attends to."""
    size, first = (mask or {}).get("size", 0), (mask or {}).get("keep_first", 0)
    return [j for j in range(i + 1) if size <= 0 or i - j < size or j < first]


def masked_attention(q, k, v, scale, mask, first=0):
    """One head, q, k [T, D], v [T, V]; outputs from position ``first`` on."""
    out = []
    for i in range(first, q.shape[0]):
        at = visible(i, mask)
        s = (k[at] @ q[i]) * scale
        e = torch.exp(s - s.max())
        out.append((e / e.sum()) @ v[at])
    return torch.stack(out)


def attention_mixer(h, mix, w, p, eps):
    heads, groups, d, dv = mix["heads"], mix["kv_heads"], mix["dim"], mix["vdim"]
    q = rms(h @ w[p + "q"].T, w[p + "q.norm"], eps)
    k = rms(h @ w[p + "k"].T, w[p + "k.norm"], eps)
    v = h @ w[p + "v"].T
    out = []
    for i in range(heads):
        g = i // (heads // groups)
        out.append(masked_attention(rotate(q[:, i * d:(i + 1) * d], mix["rot"], False), rotate(k[:, g * d:(g + 1) * d], mix["rot"], False),
                                    v[:, g * dv:(g + 1) * dv], mix["scale"], mix.get("mask")))
    return torch.cat(out, 1) @ w[p + "o"].T


def latent_attention_mixer(h, mix, w, p, eps):
    heads, d, r, dv, rank = mix["heads"], mix["dim"], mix["rot_dim"], mix["vdim"], mix["kv_rank"]
    rot = dict(mix["rot"], dims=r)
    q = rms(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T
    low = h @ w[p + "dkv"].T
    c = rms(low[:, :rank], w[p + "dkv.norm"], eps)
    kr = rotate(low[:, rank:], rot, True)
    k, v = c @ w[p + "uk"].T, c @ w[p + "uv"].T
    out = []
    for i in range(heads):
        qi = q[:, i * (d + r):(i + 1) * (d + r)]
        qi = torch.cat([qi[:, :d], rotate(qi[:, d:], rot, True)], 1)
        ki = torch.cat([k[:, i * d:(i + 1) * d], kr], 1)
        out.append(masked_attention(qi, ki, v[:, i * dv:(i + 1) * dv], mix["scale"], mix.get("mask")))
    return torch.cat(out, 1) @ w[p + "o"].T


def dense_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def small_ff(h, w, p):
    return relu2(h @ w[p + "up"].T) @ w[p + "down"].T


def choose(scores, router):
    """Expert indices of one token: the best ``top`` among the experts of the best groups."""
    n = len(scores)
    grp = router.get("groups")
    allowed = list(range(n))
    if grp:
        size = n // grp["count"]
        value = [sum(sorted(scores[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(grp["count"])]
        best = sorted(range(grp["count"]), key=lambda g: (-value[g], g))[:grp["keep"]]
        allowed = [e for e in allowed if e // size in best]
    return sorted(allowed, key=lambda e: (-scores[e], e))[:router["top"]]


def clearance(scores, router):
    """How far one token's choice is from another one: the smallest gap between what was taken and what was left."""
    n, out = len(scores), []
    grp = router.get("groups")
    allowed = list(range(n))
    if grp:
        size = n // grp["count"]
        value = [sum(sorted(scores[g * size:(g + 1) * size], reverse=True)[:2]) for g in range(grp["count"])]
        best = sorted(range(grp["count"]), key=lambda g: -value[g])
        out += [value[a] - value[b] for a, b in zip(best[grp["keep"] - 1:], best[grp["keep"]:][:1])]
        allowed = [e for e in allowed if e // size in best[:grp["keep"]]]
    rest = sorted((scores[e] for e in allowed), reverse=True)
    out += [a - b for a, b in zip(rest[router["top"] - 1:], rest[router["top"]:][:1])]
    return min(out, default=1.0)


def moe_ff(h, mlp, w, p, clear=None):
    r = mlp["router"]
    scores = sigmoid(h @ w[p + "router"].T)
    if clear is not None:
        clear.append([clearance(row, r) for row in scores.tolist()])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        ids = choose(scores[t].tolist(), r)
        total = sum(scores[t, e] for e in ids) + 1e-20
        for e in ids:
            out[t] += scores[t, e] / total * r.get("scale", 1.0) * small_ff(h[t:t + 1], w, f"{p}e{e}.")[0]
    if mlp.get("shared"):
        out = out + sigmoid(h @ w[p + "shared.sg"].T) * small_ff(h, w, p + "shared.")
    return out


def side_input(x, e, w, p, eps):
    """What a layer adds from its part ``e`` [T, dim] of the tokens' second embedding."""
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return rms(y, w[p + "norm"], eps)


def forward(tokens, cfg, weights, dtype=torch.float64, layers_out=None, clear=None):
    """Logits [T, vocab]; ``layers_out`` (a list) receives the stream after every layer, ``clear`` the tokens'
    :func:`clearance` in every routed layer."""
    w = {n: t.to(dtype) for n, t in weights.items()}
    eps, ids = cfg["norm"]["eps"], torch.as_tensor(tokens)
    norm = lambda v, name: tanh_norm(v, w[name + ".alpha"], w[name], w[name + ".b"])
    x = w["embed"][ids] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p, mix, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        mixer = attention_mixer if layer["type"] == "attention" else latent_attention_mixer
        x = x + mixer(norm(x, p + "norm1"), mix, w, p + "mix.", eps)
        if mlp is not None:
            h = norm(x, p + "norm2")
            x = x + (dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else moe_ff(h, mlp, w, p + "mlp.", clear))
        if cfg.get("token_side"):
            n = cfg["token_side"]["dim"]
            x = x + side_input(x, w["side.embed"][ids, i * n:(i + 1) * n], w, p + "side.", eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ w["head"].T
