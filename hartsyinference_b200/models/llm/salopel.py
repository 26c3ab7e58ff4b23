"""Salopel: state-space layers of two kinds and latent attention over a 32-bit residual stream, with norms on the
sublayers' outputs only and layers that share weights.

This file maps the design's ``config.json`` and tensor names onto the generic pieces: per-layer
:class:`~.config.LayerSpec` records and the mixers of :mod:`.mixers`. What the design fixes is stated here: RMS
norms stored around zero, a normed embedding that is also the output head, an output gate and no positions in
attention, the activation of normed powers.

    per layer, x the stream, N.. its RMS norms, m a constant:   x += m N1 M(x),   then   x += m N2 F(x)
    with M the layer's mixer and F its feed-forward (a layer can lack F); logits = E N_final x, x_0 = N_embed E[token]
"""
from __future__ import annotations

from typing import Callable, Optional

import torch

from .config import DenseSpec, LayerSpec, MixerSpec, TransformerConfig
from .mixers import ChannelScanMixer, DenseFeedForward, HeadScanMixer, LatentAttention, pad_cols, pad_rows, pad_to


def _mixer(kind: str, m: dict) -> MixerSpec:
    if kind == "mamba1":
        return MixerSpec(kind="channel_scan", inner=int(m["inner"]), state=int(m["state"]), rank=int(m["dt_rank"]), conv=int(m["conv"]))
    if kind == "mamba2":
        return MixerSpec(kind="head_scan", heads=int(m["heads"]), kv_heads=int(m["groups"]), vdim=int(m["vdim"]), state=int(m["state"]),
                         groups=int(m["groups"]), norm_groups=int(m["norm_groups"]), conv=int(m["conv"]))
    if kind == "latent_attention":
        return MixerSpec(kind=kind, heads=int(m["heads"]), kv_heads=1, dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                         q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), out_gate=True)
    raise ValueError(f"unknown mixer type '{kind}'")


def _dense(m: Optional[dict]) -> Optional[DenseSpec]:
    if m is None:
        return None
    if m.get("kind", "dense") != "dense":
        raise ValueError(f"unknown feed-forward kind '{m['kind']}'")
    return DenseSpec(ffn=int(m["ff"]), act="poly_norm")


def config_from(d: dict) -> TransformerConfig:
    layers = d["layers"]

    def owner(i: int) -> Optional[int]:
        seen = {i}
        j = layers[i].get("weights_of")
        while j is not None and layers[j].get("weights_of") is not None and j not in seen:
            seen.add(j)
            j = layers[j]["weights_of"]
        if j in seen:
            raise ValueError(f"layer {i}: its weights lead back to itself")
        return j

    specs = tuple(LayerSpec(_mixer(layer["type"], layer["mixer"]), dense=_dense(layer.get("mlp")), weights_of=owner(i))
                  for i, layer in enumerate(layers))
    eos = d.get("eos_token_id")
    eos = () if eos is None else tuple(eos) if isinstance(eos, (list, tuple)) else (int(eos),)
    att = next((ls.mixer for ls in specs if ls.mixer.kind == "latent_attention"), MixerSpec())
    return TransformerConfig(arch="salopel", vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), num_layers=len(specs),
                             num_heads=att.heads, num_kv_heads=1, head_dim=att.dim,
                             ffn_size=max((ls.dense.ffn for ls in specs if ls.dense is not None), default=0),
                             rms_eps=float(d["norm"]["eps"]), norm_plus_one=True, pre_norm=False, post_norms=True, embed_norm=True,
                             residual_multiplier=float(d["residual_mult"]), tie_embeddings=True, use_rope=False, max_position=1 << 20,
                             layer_specs=specs, bos_token_id=int(d.get("bos_token_id") or 0), eos_token_ids=eos)


def load_layers(model, need: Callable[[str], torch.Tensor]) -> None:
    """Checkpoint tensors (``embed``, ``embed.norm``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``) -> the
    decoder's layers. ``need(name)`` returns a tensor on any device."""
    from .transformer import LayerWeights
    cfg, w, dev, eps = model.cfg, model.cfg.hidden_size, model.device, model.cfg.rms_eps
    vec = lambda name: need(name).to(torch.bfloat16).to(dev).contiguous()
    # one table for both ends: rows padded for the output product, ids are below the vocabulary
    emb = need("embed")
    model.lm_head = model._lw(pad_rows(pad_cols(emb, pad_to(w, 8)), pad_to(emb.shape[0], 128)).to(torch.bfloat16))
    model.embed = model.lm_head.weight
    model.embed_norm_w, model.final_norm = vec("embed.norm"), vec("final.norm")
    built: dict[int, LayerWeights] = {}

    def build(i: int) -> LayerWeights:
        spec, p = cfg.layer_specs[i], f"l{i}."
        m, mix, mlp = spec.mixer, (lambda n: need(p + "mix." + n)), (lambda n: need(p + "mlp." + n))
        lw = LayerWeights(in_norm=None, qkv=None, o=None, post_norm=None, post_attn_norm=vec(p + "norm1"))
        if m.kind == "channel_scan":
            lw.attn_module = ChannelScanMixer(m, w, dev, w_in=mix("in"), conv=mix("conv"), conv_bias=mix("conv.b"), x=mix("x"), dt=mix("dt"),
                                              dt_bias=mix("dt.b"), a_log=mix("A_log"), d=mix("D"), o=mix("o"))
        elif m.kind == "head_scan":
            lw.attn_module = HeadScanMixer(m, w, eps, dev, w_in=mix("in"), conv=mix("conv"), conv_bias=mix("conv.b"), dt_bias=mix("dt_bias"),
                                           a_log=mix("A_log"), d=mix("D"), norm=mix("norm"), o=mix("o"))
        else:
            lw.attn_module = LatentAttention(m, w, eps, dev, dq=mix("dq"), dq_norm=mix("dq.norm"), uq=mix("uq"), dkv=mix("dkv"),
                                             dkv_norm=mix("dkv.norm"), uk=mix("uk"), uv=mix("uv"), g=mix("g"), o=mix("o"))
        if spec.dense is not None:
            lw.post_ffn_norm = vec(p + "norm2")
            lw.ffn_module = DenseFeedForward(spec.dense, w, eps, dev, up=mlp("up"), down=mlp("down"), coef=mlp("act"))
        return lw

    model.layers = []
    for i, spec in enumerate(cfg.layer_specs):
        j = i if spec.weights_of is None else spec.weights_of
        if j not in built:
            built[j] = build(j)
        model.layers.append(built[j])


def tensor_shapes(cfg: TransformerConfig) -> dict[str, tuple]:
    """Names and shapes of a checkpoint of this configuration (synthetic weights, tests)."""
    w = cfg.hidden_size
    out: dict[str, tuple] = {"embed": (cfg.vocab_size, w), "embed.norm": (w,)}
    for i, spec in enumerate(cfg.layer_specs):
        if spec.weights_of is not None:
            continue
        m, x, y = spec.mixer, f"l{i}.mix.", f"l{i}.mlp."
        out[f"l{i}.norm1"] = (w,)
        if m.kind == "channel_scan":
            c, n, r = m.inner, m.state, m.rank
            out.update({x + "in": (2 * c, w), x + "conv": (c, m.conv), x + "conv.b": (c,), x + "x": (r + 2 * n, c), x + "dt": (c, r),
                        x + "dt.b": (c,), x + "A_log": (c, n), x + "D": (c,), x + "o": (w, c)})
        elif m.kind == "head_scan":
            c, gn = m.heads * m.vdim, m.groups * m.state
            out.update({x + "in": (2 * c + 2 * gn + m.heads, w), x + "conv": (c + 2 * gn, m.conv), x + "conv.b": (c + 2 * gn,),
                        x + "dt_bias": (m.heads,), x + "A_log": (m.heads,), x + "D": (m.heads,), x + "norm": (c,), x + "o": (w, c)})
        else:
            h, r, q = m.heads, m.kv_rank, m.q_rank
            out.update({x + "dq": (q, w), x + "dq.norm": (q,), x + "uq": (h * m.dim, q), x + "dkv": (r, w), x + "dkv.norm": (r,),
                        x + "uk": (h * m.dim, r), x + "uv": (h * m.vdim, r), x + "g": (h * m.vdim, w), x + "o": (w, h * m.vdim)})
        if spec.dense is not None:
            out.update({f"l{i}.norm2": (w,), y + "up": (spec.dense.ffn, w), y + "down": (w, spec.dense.ffn), y + "act": (4,)})
    out["final.norm"] = (w,)
    return out


def random_tensor(name: str, shape: tuple, device, seed: int, std: float) -> torch.Tensor:
    """Synthetic value of one checkpoint tensor, generated on ``device``."""
    from ... import ops
    leaf = name.rsplit(".", 1)[-1]
    full = lambda v: torch.full(shape, v, dtype=torch.bfloat16, device=device)
    if leaf == "norm" and ".mix." in name or leaf == "D":
        return full(1.0)
    if "norm" in leaf or leaf == "A_log":
        return full(0.0)
    if leaf == "dt_bias" or name.endswith(".dt.b"):
        return full(-4.0)
    if leaf == "act":
        return full(0.25)
    n = 1
    for s in shape:
        n *= s
    t = torch.empty(1, n, dtype=torch.bfloat16, device=device)
    ops.fill_random_(t, seed, 0.3 if leaf == "conv" else std)
    return t.reshape(shape)
