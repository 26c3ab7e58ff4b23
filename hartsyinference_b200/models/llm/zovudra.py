"""Zovudra: windowed attention with kept first tokens and windowed latent attention over a 32-bit residual stream, norms
without statistics, small ungated experts, and a second token embedding that enters every layer.

This file maps the design's ``config.json`` and tensor names onto the generic pieces: per-layer
:class:`~.config.LayerSpec` records and the mixers of :mod:`.mixers`. What the design fixes is stated here: the norm is
tanh(alpha x) w + b; attention norms q and k over all their heads and turns split halves, latent attention turns pairs of
neighbours; dense feed-forwards are gated by silu, experts square a relu; experts are chosen by sigmoid scores inside the best
groups, their weights sum to the router's scale, and a shared expert has a sigmoid gate of its own.

    per layer, x the stream, N1 N2 its norms, s the layer's part of the token's second embedding:
        x += M(N1 x),   x += F(N2 x),   x += R(P (gelu(G x) * s))
    with M the layer's mixer, F its feed-forward (a layer can lack F), R an RMS norm; logits = W_head N_final x
"""
from __future__ import annotations

from typing import Callable

import torch

from .config import DenseSpec, LayerSpec, MixerSpec, MoeConfig, RopeScaling, RotarySpec, TransformerConfig
from .mixers import BiasedAttention, DenseFeedForward, LatentAttention, TokenInput, build_experts, pad_cols, pad_head_rows, pad_to
from .moe import MoeFeedForward


def _rotary(r: dict, dims: int, interleaved: bool) -> RotarySpec:
    s = r.get("scaling")
    scaling = RopeScaling() if not s else RopeScaling(kind="llama3", factor=float(s["factor"]), low_freq_factor=float(s["low"]),
                                                      high_freq_factor=float(s["high"]), original_max_position=float(s["original"]))
    return RotarySpec(dims=dims, base=float(r["base"]), interleaved=interleaved, scaling=scaling)


def _mixer(kind: str, m: dict) -> MixerSpec:
    mask = m.get("mask") or {}
    common = dict(kind=kind, heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]), window=int(mask.get("size") or 0))
    if kind == "attention":
        kv, rot = int(m["kv_heads"]), int(m["rot"]["dims"])
        if common["heads"] % kv:
            raise ValueError(f"attention: {common['heads']} heads do not divide over {kv} key heads")
        if rot % 2 or rot > common["dim"]:
            raise ValueError(f"attention: {rot} of {common['dim']} dimensions cannot be turned")
        return MixerSpec(**common, kv_heads=kv, keep_first=int(mask.get("keep_first") or 0), rot=_rotary(m["rot"], rot, False), qk_norm=True)
    if kind == "latent_attention":
        rot = int(m["rot_dim"])
        return MixerSpec(**common, kv_heads=1, q_rank=int(m["q_rank"]), kv_rank=int(m["kv_rank"]), rot_dim=rot, rot=_rotary(m["rot"], rot, True))
    raise ValueError(f"unknown mixer type '{kind}'")


def _experts(m: dict) -> MoeConfig:
    r, shared = m["router"], m.get("shared")
    groups = r.get("groups") or {}
    moe = MoeConfig(num_experts=int(r["experts"]), top_k=int(r["top"]), expert_ffn=int(m["expert"]["ff"]), expert_act="relu2", scoring="sigmoid",
                    norm_topk_prob=True, routed_scaling_factor=float(r.get("scale", 1.0)), n_group=int(groups.get("count", 1)),
                    topk_group=int(groups.get("keep", 1)), exact_router=True, num_shared_experts=0 if shared is None else 1,
                    shared_ffn=0 if shared is None else int(shared["ff"]), shared_gate=shared is not None)
    n, k = moe.n_group, moe.topk_group
    if moe.num_experts % n or n > 32 or k > n or moe.top_k > 32 or moe.top_k > moe.num_experts // n * k:
        raise ValueError(f"router: {moe.top_k} of {moe.num_experts} experts in {k} of {n} groups is not supported")
    return moe


def _layer(layer: dict) -> LayerSpec:
    mixer, mlp = _mixer(layer["type"], layer["mixer"]), layer.get("mlp")
    if mlp is None:
        return LayerSpec(mixer)
    if mlp["kind"] == "dense":
        return LayerSpec(mixer, dense=DenseSpec(ffn=int(mlp["ff"]), act="silu"))
    if mlp["kind"] == "moe":
        return LayerSpec(mixer, _experts(mlp))
    raise ValueError(f"unknown feed-forward kind '{mlp['kind']}'")


def config_from(d: dict) -> TransformerConfig:
    specs = tuple(_layer(layer) for layer in d["layers"])
    eos = d.get("eos_token_id")
    eos = () if eos is None else tuple(eos) if isinstance(eos, (list, tuple)) else (int(eos),)
    att = next((ls.mixer for ls in specs if ls.mixer.kind == "attention"), specs[0].mixer if specs else MixerSpec())
    ffn = max((ls.dense.ffn if ls.dense is not None else ls.moe.expert_ffn for ls in specs if ls.dense is not None or ls.moe is not None), default=0)
    return TransformerConfig(arch="zovudra", vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), num_layers=len(specs), num_heads=att.heads,
                             num_kv_heads=att.kv_heads, head_dim=att.dim, ffn_size=ffn, rms_eps=float(d["norm"]["eps"]), norm_type="tanh",
                             embed_scale=float(d["embedding"]["scale"]), max_position=1 << 20, layer_specs=specs,
                             token_side=int((d.get("token_side") or {}).get("dim") or 0), bos_token_id=int(d.get("bos_token_id") or 0),
                             eos_token_ids=eos)


def load_layers(model, need: Callable[[str], torch.Tensor]) -> None:
    """Checkpoint tensors (``embed``, ``side.embed``, ``l<i>.norm1``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``l<i>.side.*``,
    ``final.norm``, ``head``) -> the decoder's layers. ``need(name)`` returns a tensor on any device."""
    from ...ops import TanhNorm
    from .transformer import LayerWeights
    cfg, w, dev, eps, n = model.cfg, model.cfg.hidden_size, model.device, model.cfg.rms_eps, model.cfg.token_side
    wp = pad_to(w, 8)
    vec = lambda name: need(name).to(torch.bfloat16).to(dev).contiguous()
    norm = lambda name: TanhNorm(float(need(name + ".alpha").float().reshape(-1)[0]), vec(name), vec(name + ".b"))
    model.embed = pad_cols(need("embed"), wp).to(torch.bfloat16).to(dev).contiguous()
    model.lm_head = model._lw(pad_cols(need("head"), wp), pad_rows=128)
    model.final_norm = norm("final.norm")
    side = None
    if n:                                     # [vocab, layers * n], every layer's columns padded to 8
        np_ = pad_to(n, 8)
        side = pad_head_rows(need("side.embed").t().contiguous(), cfg.num_layers, n, np_).t().to(torch.bfloat16).to(dev).contiguous()
    model.layers = []
    for i, spec in enumerate(cfg.layer_specs):
        p, m = f"l{i}.", spec.mixer
        mix, mlp = (lambda name: need(p + "mix." + name)), (lambda name: need(p + "mlp." + name))
        lw = LayerWeights(in_norm=norm(p + "norm1"), qkv=None, o=None, post_norm=None)
        if m.kind == "attention":
            lw.attn_module = BiasedAttention(m, w, dev, q=mix("q"), k=mix("k"), v=mix("v"), o=mix("o"), q_norm=mix("q.norm"), k_norm=mix("k.norm"),
                                             eps=eps)
        else:
            lw.attn_module = LatentAttention(m, w, eps, dev, dq=mix("dq"), dq_norm=mix("dq.norm"), uq=mix("uq"), dkv=mix("dkv"),
                                             dkv_norm=mix("dkv.norm"), uk=mix("uk"), uv=mix("uv"), o=mix("o"))
        if spec.dense is not None or spec.moe is not None:
            lw.post_norm = norm(p + "norm2")
        if spec.dense is not None:
            lw.ffn_module = DenseFeedForward(spec.dense, w, eps, dev, gate=mlp("gate"), up=mlp("up"), down=mlp("down"))
        elif spec.moe is not None:
            experts = ((None, mlp(f"e{e}.up"), mlp(f"e{e}.down")) for e in range(spec.moe.num_experts))
            shared = (mlp("shared.up"), mlp("shared.down"), mlp("shared.sg")) if spec.moe.shared_gate else None
            lw.ffn_module = MoeFeedForward(cfg, build_experts(spec.moe, w, dev, mlp("router"), None, experts, shared), moe=spec.moe, hidden=wp)
        if n:
            lw.side_module = TokenInput(n, w, dev, table=side[:, i * np_:(i + 1) * np_], gate=need(p + "side.gate"), proj=need(p + "side.proj"))
            lw.side_norm = vec(p + "side.norm")
        model.layers.append(lw)


def tensor_shapes(cfg: TransformerConfig) -> dict[str, tuple]:
    """Names and shapes of a checkpoint of this configuration (synthetic weights, tests)."""
    w, n = cfg.hidden_size, cfg.token_side
    out: dict[str, tuple] = {"embed": (cfg.vocab_size, w)}
    norm = lambda name: {name: (w,), name + ".b": (w,), name + ".alpha": ()}
    if n:
        out["side.embed"] = (cfg.vocab_size, cfg.num_layers * n)
    for i, spec in enumerate(cfg.layer_specs):
        m, x, y, z = spec.mixer, f"l{i}.mix.", f"l{i}.mlp.", f"l{i}.side."
        h, d, v = m.heads, m.dim, m.vdim
        out.update(norm(f"l{i}.norm1"))
        if m.kind == "attention":
            out.update({x + "q": (h * d, w), x + "k": (m.kv_heads * d, w), x + "v": (m.kv_heads * v, w), x + "q.norm": (h * d,),
                        x + "k.norm": (m.kv_heads * d,), x + "o": (w, h * v)})
        else:
            q, r, t = m.q_rank, m.kv_rank, m.rot_dim
            out.update({x + "dq": (q, w), x + "dq.norm": (q,), x + "uq": (h * (d + t), q), x + "dkv": (r + t, w), x + "dkv.norm": (r,),
                        x + "uk": (h * d, r), x + "uv": (h * v, r), x + "o": (w, h * v)})
        if spec.dense is not None or spec.moe is not None:
            out.update(norm(f"l{i}.norm2"))
        if spec.dense is not None:
            f = spec.dense.ffn
            out.update({y + "gate": (f, w), y + "up": (f, w), y + "down": (w, f)})
        elif spec.moe is not None:
            e = spec.moe
            for j in range(e.num_experts):
                out.update({f"{y}e{j}.up": (e.expert_ffn, w), f"{y}e{j}.down": (w, e.expert_ffn)})
            out[y + "router"] = (e.num_experts, w)
            if e.shared_gate:
                out.update({y + "shared.up": (e.shared_ffn, w), y + "shared.down": (w, e.shared_ffn), y + "shared.sg": (1, w)})
        if n:
            out.update({z + "gate": (n, w), z + "proj": (w, n), z + "norm": (w,)})
    out.update({**norm("final.norm"), "head": (cfg.vocab_size, w)})
    return out


def random_tensor(name: str, shape: tuple, device, seed: int, std: float) -> torch.Tensor:
    """Synthetic value of one checkpoint tensor, generated on ``device``."""
    from ... import ops
    leaf = name.rsplit(".", 1)[-1]
    full = lambda v: torch.full(shape, v, dtype=torch.bfloat16, device=device)
    if leaf == "alpha":
        return full(0.5)
    if leaf == "b":
        return full(0.0)
    if "norm" in leaf:
        return full(1.0)
    n = 1
    for s in shape:
        n *= s
    t = torch.empty(1, n, dtype=torch.bfloat16, device=device)
    ops.fill_random_(t, seed, 1.0 if name in ("embed", "side.embed") else std)
    return t.reshape(shape)
