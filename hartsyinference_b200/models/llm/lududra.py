"""Lududra: windowed attention and channel-wise gated delta-rule layers over a 32-bit residual stream
with sandwich LayerNorms, and routed experts with pass-through outputs.

This file maps the design's ``config.json`` and tensor names onto the generic pieces: per-layer
:class:`~.config.LayerSpec` records and the mixers of :mod:`.mixers`. What the design fixes is stated
here: the attention sink has score 0, keys serve as values, q and k carry biases, the output gate is on,
router scores are a softmax that is not renormalised after the choice, and the expert gate uses 1.702.

    per layer, x the stream and N.. its LayerNorms:   x += N1b M(N1 x),   then   x += N2b E(N2 x)
    with M the layer's mixer and E its experts (a layer can lack E); logits = W_head N_final x
"""
from __future__ import annotations

from typing import Callable, Optional

import torch

from .config import LayerSpec, MixerSpec, MoeConfig, TransformerConfig
from .mixers import BiasedAttention, DeltaMixer, build_experts, pad_cols, pad_to
from .moe import MoeFeedForward


def _mixer(kind: str, m: dict) -> MixerSpec:
    common = dict(kind=kind, heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
    if common["heads"] % common["kv_heads"]:
        raise ValueError(f"{kind}: {common['heads']} heads do not divide over {common['kv_heads']} key heads")
    if kind == "attention":
        if common["dim"] != common["vdim"]:
            raise ValueError("attention: the values are the keys, dim and vdim must be equal")
        return MixerSpec(**common, scale=float(m["scale"]), softcap=float(m.get("softcap") or 0.0),
                         window=int((m.get("mask") or {}).get("size") or 0), bias_reach=int(m.get("bias_max") or 0),
                         shared_kv=True, qk_bias=True, out_gate=True, sink=0.0)
    if kind == "channel_delta":
        return MixerSpec(**common, conv=int(m["conv"]))
    raise ValueError(f"unknown mixer type '{kind}'")


def _experts(m: Optional[dict]) -> Optional[MoeConfig]:
    if m is None:
        return None
    if m.get("kind", "moe") != "moe":
        raise ValueError(f"unknown feed-forward kind '{m['kind']}'")
    r, e = m["router"], m["expert"]
    return MoeConfig(num_experts=int(r["experts"]), top_k=int(r["top"]), identity_experts=int(r.get("identity") or 0),
                     expert_ffn=int(e["ff"]), glu_limit=float(e["limit"]), scoring="softmax", norm_topk_prob=False,
                     use_correction_bias=True, exact_router=True)


def lududra_config(d: dict) -> TransformerConfig:
    specs = tuple(LayerSpec(_mixer(layer["type"], layer["mixer"]), _experts(layer.get("mlp"))) for layer in d["layers"])
    eos = d.get("eos_token_id")
    eos = () if eos is None else tuple(eos) if isinstance(eos, (list, tuple)) else (int(eos),)
    first = specs[0].mixer
    return TransformerConfig(arch="lududra", vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), num_layers=len(specs),
                             num_heads=first.heads, num_kv_heads=first.kv_heads, head_dim=first.dim,
                             ffn_size=max((ls.moe.expert_ffn for ls in specs if ls.moe is not None), default=0),
                             rms_eps=float(d["norm"]["eps"]), norm_type="layernorm", post_norms=True, use_rope=False,
                             embed_scale=float(d["embedding"]["scale"]), max_position=1 << 20, layer_specs=specs,
                             bos_token_id=int(d.get("bos_token_id") or 0), eos_token_ids=eos)


config_from = lududra_config


def load_layers(model, need: Callable[[str], torch.Tensor]) -> None:
    """Checkpoint tensors (``embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``)
    -> the decoder's layers. ``need(name)`` returns a tensor on any device."""
    from .transformer import LayerWeights
    cfg, w = model.cfg, model.cfg.hidden_size
    wp = pad_to(w, 8)
    dev = lambda t: t.to(torch.bfloat16).to(model.device).contiguous()
    vec = lambda name: dev(need(name))
    model.embed = dev(pad_cols(need("embed"), wp))
    model.lm_head = model._lw(pad_cols(need("head"), wp), pad_rows=128)
    model.final_norm = vec("final.norm")
    model.layers = []
    for i, spec in enumerate(cfg.layer_specs):
        p = f"l{i}."
        lw = LayerWeights(in_norm=vec(p + "norm1"), qkv=None, o=None, post_norm=None, post_attn_norm=vec(p + "norm1b"))
        m, mix = spec.mixer, lambda n, p=p: need(p + "mix." + n)
        if m.kind == "attention":
            lw.attn_module = BiasedAttention(m, w, model.device, q=mix("q"), k=mix("k"), v=None, o=mix("o"), q_bias=mix("q.b"),
                                             k_bias=mix("k.b"), gate=mix("g"), rel=mix("rel"))
        else:
            lw.attn_module = DeltaMixer(m, w, cfg.rms_eps, model.device, q=mix("q"), k=mix("k"), v=mix("v"), b=mix("b"),
                                        o=mix("o"), conv=(mix("q.conv"), mix("k.conv"), mix("v.conv")), a_log=mix("A_log"),
                                        dt_bias=mix("dt_bias"), norm=mix("norm"), a1=mix("a1"), a2=mix("a2"), g1=mix("g1"),
                                        g2=mix("g2"))
        if spec.moe is not None:
            lw.post_norm, lw.post_ffn_norm = vec(p + "norm2"), vec(p + "norm2b")
            f = lambda n, p=p: need(p + "mlp." + n)
            experts = ((f(f"e{e}.gate"), f(f"e{e}.up"), f(f"e{e}.down")) for e in range(spec.moe.num_experts))
            weights = build_experts(spec.moe, w, model.device, f("router"), f("correction"), experts)
            lw.ffn_module = MoeFeedForward(cfg, weights, moe=spec.moe, hidden=wp)
        model.layers.append(lw)


def tensor_shapes(cfg: TransformerConfig) -> dict[str, tuple]:
    """Names and shapes of a checkpoint of this configuration (synthetic weights, tests)."""
    w = cfg.hidden_size
    out: dict[str, tuple] = {"embed": (cfg.vocab_size, w)}
    for i, spec in enumerate(cfg.layer_specs):
        p, m = f"l{i}.", spec.mixer
        out.update({p + n: (w,) for n in (("norm1", "norm1b") + (("norm2", "norm2b") if spec.moe is not None else ()))})
        x = p + "mix."
        if m.kind == "attention":
            hq, hk = m.heads * m.dim, m.kv_heads * m.dim
            out.update({x + "q": (hq, w), x + "q.b": (hq,), x + "k": (hk, w), x + "k.b": (hk,), x + "rel": (m.bias_rows, m.heads),
                        x + "g": (hq, w), x + "o": (w, hq)})
        else:
            qk, hv, r = m.kv_heads * m.dim, m.heads * m.vdim, m.rank or m.dim
            for n, c in (("q", qk), ("k", qk), ("v", hv)):
                out.update({x + n: (c, w), x + n + ".conv": (c, m.conv)})
            out.update({x + "b": (m.heads, w), x + "A_log": (m.heads,), x + "norm": (m.vdim,), x + "a1": (r, w),
                        x + "a2": (m.heads * m.dim, r), x + "dt_bias": (m.heads * m.dim,), x + "g1": (r, w), x + "g2": (hv, r),
                        x + "o": (w, hv)})
        if spec.moe is not None:
            y, e = p + "mlp.", spec.moe
            for j in range(e.num_experts):
                out.update({f"{y}e{j}.gate": (e.expert_ffn, w), f"{y}e{j}.up": (e.expert_ffn, w), f"{y}e{j}.down": (w, e.expert_ffn)})
            out.update({y + "router": (e.choices, w), y + "correction": (e.choices,)})
    out.update({"final.norm": (w,), "head": (cfg.vocab_size, w)})
    return out


def random_tensor(name: str, shape: tuple, device, seed: int, std: float) -> torch.Tensor:
    """Synthetic value of one checkpoint tensor, generated on ``device``."""
    from ... import ops
    leaf = name.rsplit(".", 1)[-1]
    if "norm" in leaf:
        return torch.ones(shape, dtype=torch.bfloat16, device=device)
    if leaf in ("A_log", "correction"):
        return torch.zeros(shape, dtype=torch.bfloat16, device=device)
    n = 1
    for s in shape:
        n *= s
    t = torch.empty(1, n, dtype=torch.bfloat16, device=device)
    ops.fill_random_(t, seed, 0.3 if leaf == "conv" else std)
    return t.reshape(shape)
