"""Ginodra: latent attention with sinks, windowed attention with linear distance biases and shared keys, and a generalized
delta rule, each beside a feed-forward that reads the same norm, around a 32-bit residual stream.

This file maps the design's ``config.json`` and tensor names onto the generic pieces: per-layer
:class:`~.config.LayerSpec` records and the mixers of :mod:`.mixers`. What the design fixes is stated here: RMS norms in equal
parts, a short convolution on what every sublayer reads, one gate number per attention head, split halves turned in latent
attention, head norms and no rotation in attention, relu squared feed-forwards, the embedding as output head.

    per layer, x the stream, m a constant, N the layer's norm, C1 C2 its convolutions over time:
        h = N x,   x += m (M(h + C1 h) + F(h + C2 h))
    with M the layer's mixer and F its feed-forward (a layer can lack F); logits = c tanh(s E N_final x / c)
"""
from __future__ import annotations

from typing import Callable, Optional

import torch

from .config import DenseSpec, LayerSpec, MixerSpec, RotarySpec, TransformerConfig
from .mixers import BiasedAttention, DenseFeedForward, GeneralDeltaMixer, LatentAttention, ParallelBlock, pad_cols, pad_rows, pad_to


def _mixer(kind: str, m: dict, layers: list) -> MixerSpec:
    heads, dim = int(m["heads"]), int(m["dim"])
    if kind == "general_delta":
        return MixerSpec(kind=kind, heads=heads, kv_heads=heads, dim=dim, vdim=dim)
    mask = m.get("mask") or {}
    common = dict(kind=kind, heads=heads, dim=dim, vdim=int(m["vdim"]), scale=float(m["scale"]), window=int(mask.get("size") or 0), head_gate=True)
    if kind == "attention":
        kv, source = int(m["kv_heads"]), m.get("kv_from")
        if heads % kv:
            raise ValueError(f"attention: {heads} heads do not divide over {kv} key heads")
        if source is not None:
            s = layers[int(source)]
            same = all(int(s["mixer"].get(n) or 0) == int(m[n]) for n in ("kv_heads", "dim", "vdim"))
            if s["type"] != "attention" or s["mixer"].get("kv_from") is not None or not same:
                raise ValueError(f"attention: layer {source} has no keys and values of {kv} x {dim} / {m['vdim']} to share")
        return MixerSpec(**common, kv_heads=kv, head_norm=True, slope_bias=True, kv_from=None if source is None else int(source))
    if kind == "latent_attention":
        rot = int(m["rot_dim"])
        return MixerSpec(**common, kv_heads=1, q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), rot_dim=rot,
                         rot=RotarySpec(dims=rot, base=float(m["rot"]["base"])) if rot else None)
    raise ValueError(f"unknown mixer type '{kind}'")


def _dense(m: Optional[dict]) -> Optional[DenseSpec]:
    if m is None:
        return None
    if m.get("kind", "dense") != "dense":
        raise ValueError(f"unknown feed-forward kind '{m['kind']}'")
    return DenseSpec(ffn=int(m["ff"]), act="relu2")


def config_from(d: dict) -> TransformerConfig:
    layers = d["layers"]
    specs = []
    for i, layer in enumerate(layers):
        spec = LayerSpec(_mixer(layer["type"], layer["mixer"], layers), dense=_dense(layer.get("mlp")))
        if spec.mixer.kv_from is not None and not 0 <= spec.mixer.kv_from < i:
            raise ValueError(f"layer {i}: it reads the keys of layer {spec.mixer.kv_from}, which does not come before it")
        specs.append(spec)
    width, groups = int(d["width"]), int(d["norm"].get("groups") or 1)
    if width % groups:
        raise ValueError(f"a norm of {width} values does not divide into {groups} parts")
    eos = d.get("eos_token_id")
    eos = () if eos is None else tuple(eos) if isinstance(eos, (list, tuple)) else (int(eos),)
    att = next((ls.mixer for ls in specs if ls.mixer.kind == "attention"), specs[0].mixer if specs else MixerSpec())
    return TransformerConfig(arch="ginodra", vocab_size=int(d["vocab"]), hidden_size=width, num_layers=len(specs), num_heads=att.heads,
                             num_kv_heads=att.kv_heads, head_dim=att.dim,
                             ffn_size=max((ls.dense.ffn for ls in specs if ls.dense is not None), default=0),
                             rms_eps=float(d["norm"]["eps"]), norm_groups=groups, parallel_residual=True, shared_parallel_norm=True,
                             residual_multiplier=float(d.get("residual_mult", 1.0)), logits_scale=float(d.get("logit_scale", 1.0)),
                             logit_softcap=float(d.get("logit_softcap") or 0.0), tie_embeddings=True, max_position=1 << 20,
                             input_conv=int((d.get("canon") or {}).get("taps") or 0), layer_specs=tuple(specs),
                             bos_token_id=int(d.get("bos_token_id") or 0), eos_token_ids=eos)


def load_layers(model, need: Callable[[str], torch.Tensor]) -> None:
    """Checkpoint tensors (``embed``, ``l<i>.norm1``, ``l<i>.canon1`` / ``2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``) ->
    the decoder's layers. ``need(name)`` returns a tensor on any device."""
    from .transformer import LayerWeights
    cfg, w, dev, eps = model.cfg, model.cfg.hidden_size, model.device, model.cfg.rms_eps
    wp = pad_to(w, 8)
    vec = lambda name: need(name).to(torch.bfloat16).to(dev).contiguous()
    # one table for both ends: rows padded for the output product, ids are below the vocabulary
    emb = need("embed")
    model.lm_head = model._lw(pad_rows(pad_cols(emb, wp), pad_to(emb.shape[0], 128)).to(torch.bfloat16))
    model.embed = model.lm_head.weight
    model.final_norm = vec("final.norm")
    model.layers = []
    for i, spec in enumerate(cfg.layer_specs):
        p, m = f"l{i}.", spec.mixer
        mix, mlp = (lambda name: need(p + "mix." + name)), (lambda name: need(p + "mlp." + name))
        lw = LayerWeights(in_norm=vec(p + "norm1"), qkv=None, o=None, post_norm=None)
        if m.kind == "attention":
            kv = {} if m.kv_from is not None else dict(k=mix("k"), v=mix("v"), k_norm=mix("k.norm"))
            mixer = BiasedAttention(m, w, dev, q=mix("q"), gate=mix("g"), q_norm=mix("q.norm"), eps=eps, o=None, **kv)
        elif m.kind == "latent_attention":
            mixer = LatentAttention(m, w, eps, dev, dq=mix("dq"), dq_norm=mix("dq.norm"), uq=mix("uq"), dkv=mix("dkv"), dkv_norm=mix("dkv.norm"),
                                    uk=mix("uk"), uv=mix("uv"), g=mix("g"), sinks=mix("sink"), o=None)
        else:
            mixer = GeneralDeltaMixer(m, w, eps, dev, r=mix("r"), k=mix("k"), v=mix("v"), a=mix("a"), a_bias=mix("a.b"), g=mix("g"), w1=mix("w1"),
                                      w2=mix("w2"), w0=mix("w0"), norm=mix("norm"), o=None)
        ffn = None if spec.dense is None else DenseFeedForward(spec.dense, w, eps, dev, up=mlp("up"), down=None)
        lw.attn_module = ParallelBlock(mixer, ffn, w, dev, o=mix("o"), down=None if ffn is None else mlp("down"))
        if cfg.input_conv:
            taps = [need(p + "canon1")] + ([] if ffn is None else [need(p + "canon2")])
            lw.input_conv = torch.stack([pad_rows(t, wp).t() for t in taps]).float().to(dev).contiguous()
        model.layers.append(lw)


def tensor_shapes(cfg: TransformerConfig) -> dict[str, tuple]:
    """Names and shapes of a checkpoint of this configuration (synthetic weights, tests)."""
    w, taps = cfg.hidden_size, cfg.input_conv
    out: dict[str, tuple] = {"embed": (cfg.vocab_size, w)}
    for i, spec in enumerate(cfg.layer_specs):
        m, x, y = spec.mixer, f"l{i}.mix.", f"l{i}.mlp."
        h, d, v = m.heads, m.dim, m.vdim
        out[f"l{i}.norm1"] = (w,)
        if m.kind == "attention":
            out.update({x + "q": (h * d, w), x + "q.norm": (d,), x + "g": (h, w), x + "o": (w, h * v)})
            if m.kv_from is None:
                out.update({x + "k": (m.kv_heads * d, w), x + "v": (m.kv_heads * v, w), x + "k.norm": (d,)})
        elif m.kind == "latent_attention":
            q, r, t = m.q_rank, m.kv_rank, m.rot_dim
            out.update({x + "dq": (q, w), x + "dq.norm": (q,), x + "uq": (h * (d + t), q), x + "dkv": (r + t, w), x + "dkv.norm": (r,),
                        x + "uk": (h * d, r), x + "uv": (h * v, r), x + "sink": (h,), x + "g": (h, w), x + "o": (w, h * v)})
        else:
            c, r = h * d, m.rank or d
            out.update({x + n: (c, w) for n in ("r", "k", "v", "g", "a")})
            out.update({x + "a.b": (c,), x + "w1": (r, w), x + "w2": (c, r), x + "w0": (c,), x + "norm": (c,), x + "o": (w, c)})
        if taps:
            out[f"l{i}.canon1"] = (w, taps)
        if spec.dense is not None:
            out.update({y + "up": (spec.dense.ffn, w), y + "down": (w, spec.dense.ffn)})
            if taps:
                out[f"l{i}.canon2"] = (w, taps)
    out["final.norm"] = (w,)
    return out


def random_tensor(name: str, shape: tuple, device, seed: int, std: float) -> torch.Tensor:
    """Synthetic value of one checkpoint tensor, generated on ``device``."""
    from ... import ops
    leaf = name.rsplit(".", 1)[-1]
    full = lambda v: torch.full(shape, v, dtype=torch.bfloat16, device=device)
    if "norm" in leaf:
        return full(1.0)
    if leaf == "w0":
        return full(-4.0)
    if leaf in ("sink", "b"):
        return full(0.0)
    n = 1
    for s in shape:
        n *= s
    t = torch.empty(1, n, dtype=torch.bfloat16, device=device)
    ops.fill_random_(t, seed, 1.0 if name == "embed" else 0.3 if leaf.startswith("canon") else std)
    return t.reshape(shape)
