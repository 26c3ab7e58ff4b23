"""``bench.py --preset ginodra``: prefill and decode throughput of the Ginodra design at sizes that resemble a real
model's layers (random weights, a few layers), beside the closest models the framework already serves at equal
size, all through the same engine in bf16:

* a DeepSeek-type decoder of the same width, heads, latents, layer count and feed-forward parameters (latent attention with
  a rotated part and a gated feed-forward in every layer), and
* a Qwen3-type decoder (grouped-query attention with normed and rotated heads, a gated feed-forward in every layer).

Throughput comes from CUDA events around ``LLMEngine.step``; e2e from host time around the same steps. Then every
kernel the design adds or extends is timed alone beside the like kernel of the existing models, with its share of the
measured copy bandwidth or GEMM peak (inputs flushed from L2 before every launch).
"""
from __future__ import annotations

import torch

from bench_mixers import VOCAB, Timer, serve
from hartsyinference_b200 import ops
from hartsyinference_b200.models.llm import config as C
from hartsyinference_b200.models.llm.ginodra import config_from
from hartsyinference_b200.models.llm.rope import Rotary
from hartsyinference_b200.models.llm.transformer import DecoderModel
from hartsyinference_b200.ops import _native as N

# width, layers in fours (latent attention, attention, attention on the keys before it, delta rule), heads of 128, key
# heads, feed-forward
SIZES = {
    "2k": dict(width=2048, layers=8, heads=16, kv=4, ff=8192),
    "4k": dict(width=4096, layers=4, heads=32, kv=8, ff=16384),
}
D, ROT, RANK, QRANK, GROUPS, WINDOW, TAPS = 128, 64, 512, 1024, 8, 1024, 4


def ginodra_cfg(s: dict) -> C.TransformerConfig:
    mlp = {"kind": "dense", "ff": s["ff"]}
    lat = {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": s["heads"], "dim": D, "rot_dim": ROT, "vdim": D, "kv_rank": RANK, "q_rank": QRANK,
                                                             "scale": (D + ROT) ** -0.5, "rot": {"base": 1e6, "dims": ROT}}}
    att = lambda source: {"type": "attention", "mlp": mlp, "mixer": {"heads": s["heads"], "kv_heads": s["kv"], "dim": D, "vdim": D, "scale": D ** -0.5,
                                                                     "mask": {"size": WINDOW}, **({} if source is None else {"kv_from": source})}}
    delta = {"type": "general_delta", "mlp": mlp, "mixer": {"heads": s["heads"], "dim": D}}
    layers = [(lat, att(None), att(i - 1), delta)[i % 4] for i in range(s["layers"])]
    return config_from({"architecture": "Ginodra", "norm": {"eps": 1e-6, "groups": GROUPS}, "canon": {"taps": TAPS}, "residual_mult": 0.5, "logit_scale": 0.5,
                        "logit_softcap": 30.0, "vocab": VOCAB, "width": s["width"], "layers": layers})


def gated(ff: int) -> int:
    """Gated feed-forward (three matrices) with the parameters of an ungated one."""
    return (2 * ff // 3 + 127) // 128 * 128


def latent_cfg(s: dict) -> C.TransformerConfig:
    return C.TransformerConfig(arch="deepseek_v3", vocab_size=VOCAB, hidden_size=s["width"], num_layers=s["layers"], num_heads=s["heads"],
                               num_kv_heads=s["heads"], head_dim=D + ROT, ffn_size=gated(s["ff"]), rope_dim=ROT, tie_embeddings=True,
                               mla=C.MlaConfig(q_lora_rank=QRANK, kv_lora_rank=RANK, qk_nope_head_dim=D, qk_rope_head_dim=ROT, v_head_dim=D))


def attention_cfg(s: dict) -> C.TransformerConfig:
    return C.TransformerConfig(arch="qwen3", vocab_size=VOCAB, hidden_size=s["width"], num_layers=s["layers"], num_heads=s["heads"],
                               num_kv_heads=s["kv"], head_dim=D, ffn_size=gated(s["ff"]), qk_norm=True, tie_embeddings=True)


class _Positions:
    def __init__(self, positions):
        self.positions, self.plan = positions, None


# ------------------------------------------------------------------------------------------ kernels
def kernels(s: dict, dev) -> dict:
    """{kernel: {"decode" (64 rows): [new, like], "prefill" (8192 rows): [new, like]}}"""
    tm = Timer(dev)
    w, h, kv, ff = (s[n] for n in ("width", "heads", "kv", "ff"))
    bf = lambda *sh: torch.randn(*sh, device=dev).to(torch.bfloat16)
    i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=dev)
    ones = torch.ones(max(w, h * D, QRANK), dtype=torch.bfloat16, device=dev)
    taps = torch.randn(2, TAPS, w, device=dev)
    out: dict = {}

    def put(name, phase, new, like):
        out.setdefault(name, {})[phase] = {"new": new, "like": like}

    for phase, t in (("decode", 64), ("prefill", 8192)):
        seqs, ctx = (64, 2048) if phase == "decode" else (4, 2048)
        decode = phase == "decode"
        pos = torch.full((t,), ctx - 1, dtype=torch.int32, device=dev) if decode else torch.arange(t, dtype=torch.int32, device=dev) % ctx
        cu = None if decode else torch.arange(0, t + 1, ctx, dtype=torch.int32, device=dev)
        sl = torch.arange(seqs, dtype=torch.int32, device=dev)
        # ---- norm in groups, convolutions of the sublayers' inputs
        x, y = torch.randn(t, w, device=dev), bf(t, w)
        kw = dict(dim=w, eps=1e-6, layernorm=False, dtype=torch.bfloat16, mult=0.5, groups=GROUPS)
        state = torch.zeros(seqs, TAPS - 1, w, dtype=torch.bfloat16, device=dev)
        norm = tm.row(lambda: ops.norm(y, ones[:w], residual=y), t * w * 8)
        put("residual_norm (groups) / norm", phase, tm.row(lambda: ops.residual_norm(x, y, None, ones[:w], **kw), t * w * 12), norm)
        conv = lambda: ops.short_conv(y, taps[0], None, state, pos, cu, sl)
        held = seqs * (TAPS - 1) * w * 4
        if decode:
            def norm_conv():
                ops.norm(y, ones[:w], residual=y)
                conv()
            put("residual_norm with both convolutions / norm + short_conv", phase,
                tm.row(lambda: ops.residual_norm(x, y, None, ones[:w], conv=(taps, state, pos, sl), **kw), t * w * 14 + held + 2 * TAPS * w * 4),
                tm.row(norm_conv, t * w * 12 + held + TAPS * w * 4))
        else:
            put("input_conv / short_conv", phase, tm.row(lambda: ops.input_conv(y, taps, state, pos, cu, sl), t * w * 6), tm.row(conv, t * w * 4))
        # ---- feed-forward and output products (vendor-free GEMM in both): activation in the epilogue, one product for both outputs
        up, gate_up = ops.LinearWeight(bf(ff, w)), ops.LinearWeight(bf(2 * gated(ff), w))
        o, down, both = ops.LinearWeight(bf(w, h * D)), ops.LinearWeight(bf(w, ff)), ops.LinearWeight(bf(w, h * D + ff))
        buf, act = bf(t, h * D + ff), bf(t, ff)
        a = bf(t, h * D)
        put("up product with relu squared / gate|up product + glu", phase,
            tm.row(lambda: ops.linear_act(y, up, "relu2", out=buf[:, h * D:]), ff * w * 2 + t * (w + ff) * 2, 2.0 * t * w * ff),
            tm.row(lambda: ops.glu(ops.linear(y, gate_up, defer=decode)), 2 * gated(ff) * w * 2 + t * (w + 5 * gated(ff)) * 2, 4.0 * t * w * gated(ff)))
        put("joint output product / output + down product", phase,
            tm.row(lambda: ops.linear(buf, both), (h * D + ff) * w * 2 + t * (h * D + ff + w) * 2, 2.0 * t * w * (h * D + ff)),
            tm.row(lambda: (ops.linear(a, o), ops.linear(act, down)), (h * D + ff) * w * 2 + t * (h * D + ff + 2 * w) * 2, 2.0 * t * w * (h * D + ff)))
        # ---- grouped-query attention: 64 contexts of 2048 tokens, or four whole prompts
        per = ctx // 16
        kc, vc = bf(seqs * per, kv, 16, D), bf(seqs * per, kv, 16, D)
        table = torch.randperm(seqs * per, device=dev).to(torch.int32).reshape(seqs, per)
        lens = torch.full((seqs,), ctx, dtype=torch.int32, device=dev)
        wslots = torch.randperm(seqs * ctx, device=dev)[:t].contiguous()
        p = bf(t, (h + 2 * kv) * D)
        inv = Rotary(C.RotarySpec(D, 1e6), dev).hi
        nb = t * (h + 2 * kv) * D * 4
        put("head_norm_store / rope_kv", phase,
            tm.row(lambda: ops.qk_rope_store(p, h, kc, vc, wslots, q_norm=ones[:D], k_norm=ones[:D], eps=1e-6, per_head=True), nb),
            tm.row(lambda: ops.rope_kv(p, pos, h, kv, D, k_cache=kc, v_cache=vc, slot_mapping=wslots, inv_freq=inv, q_norm_w=ones[:D], k_norm_w=ones[:D]), nb))
        q, g = bf(t, h * D), bf(t, h)
        q3 = q.view(t, h, D)
        slopes, sinks = torch.rand(h, device=dev), torch.zeros(h, device=dev)
        ext = dict(heads=h, max_kv_len=ctx, scale=0.1, window=WINDOW, slopes=slopes, gate=g, head_gate=True)
        if decode:
            nb = (seqs * WINDOW * kv * 2 + 2 * t * h) * D * 2
            put("attn_biased (window, slopes, gate) / attn_decode (window)", phase, tm.row(lambda: ops.attn_biased(q, kc, vc, table, lens, None, **ext), nb),
                tm.row(lambda: ops.attn_decode(q3, kc, vc, table, lens, 0.1, window=WINDOW, max_kv_len=ctx), nb))
        else:
            fl = 4.0 * seqs * (WINDOW * (WINDOW + 1) / 2 + (ctx - WINDOW) * WINDOW) * h * D
            put("attn_biased (window, slopes, gate) / attn_prefill (window)", phase,
                tm.row(lambda: ops.attn_biased(q, kc, vc, table, lens, cu, max_q_len=ctx, **ext), 4 * t * h * D * 2, fl),
                tm.row(lambda: ops.attn_prefill_paged(q3, kc, vc, table, lens, cu, ctx, causal=True, scale=0.1, window=WINDOW), 4 * t * h * D * 2, fl))
        # ---- latent attention
        row = RANK + ROT
        cache, cache2 = bf(seqs * per, 1, 16, row), bf(seqs * per, 16, row)
        rot = Rotary(C.RotarySpec(ROT, 1e6, True), dev)
        ct = rot.table(_Positions(pos))
        if decode:
            ql = bf(t, h * row)
            fl = 2.0 * t * ctx * h * (2 * RANK + ROT)
            nb = seqs * ctx * row * 2 + t * h * (2 * RANK + ROT) * 2
            put("latent_attn (sinks) / mla_attn", phase,
                tm.row(lambda: ops.latent_attn(ql, cache, table, lens, h, 0.05, max_kv_len=ctx, v_dim=RANK, sinks=sinks), nb, fl),
                tm.row(lambda: ops.mla_attn(ql.view(t, h, row), cache2, table, lens, 0.05, max_kv_len=ctx), nb, fl))
            uv, vo, lat = ops.LinearWeight(bf(h * D, RANK)), torch.empty(t, h * D, dtype=torch.bfloat16, device=dev), bf(t, h * RANK)
            nb = h * RANK * D * 2 + t * h * (RANK + D) * 2
            put("head_linear (W_uv, gate) / colbatched_linear", phase, tm.row(lambda: ops.head_linear(lat, uv, h, gate=g, head_gate=True, out=vo), nb),
                tm.row(lambda: ops.colbatched_linear(lat, uv.weight, h, RANK, vo, D), nb))
        else:
            qn, kvx, o2, c = bf(t, h * (D + ROT)), bf(t, 2 * h * D), torch.empty(t, h * D, dtype=torch.bfloat16, device=dev), bf(t, row)
            fl = 2.0 * seqs * ctx * (ctx + 1) / 2 * h * (2 * D + ROT)
            kch, vch = bf(seqs * per, h, 16, D), bf(seqs * per, h, 16, D)
            put("attn_runs (keys of 192, sinks, gate) / attn_prefill (128)", phase,
                tm.row(lambda: ops.attn_runs(qn, kvx[:, :h * D], kvx[:, h * D:], o2, cu[:-1].contiguous(), lens, cu, lens, heads=h, max_q_len=ctx, scale=0.07,
                                             k_shared=c[:, RANK:], table=ct, sinks=sinks, gate=g, head_gate=True), t * h * (4 * D + ROT) * 2, fl),
                tm.row(lambda: ops.attn_prefill_paged(q3, kch, vch, table, lens, cu, ctx, causal=True, scale=0.1), 4 * t * h * D * 2,
                       4.0 * seqs * ctx * (ctx + 1) / 2 * h * D))
        # ---- delta rule beside the one with a step size per head (its convolution included)
        n = h * D
        gw = ops.GeneralDeltaWeights(decay_bias=torch.full((n,), -4.0, device=dev), rate_bias=torch.zeros(n, device=dev), norm=ones[:n], heads=h, dk=D, dv=D,
                                     d_true=D, eps=1e-6)
        dw = ops.DeltaWeights(conv=torch.randn(4, 3 * n, device=dev), decay_rate=torch.ones(h, device=dev), dt_bias=torch.zeros(n, device=dev),
                              norm=ones[:D], heads=h, kv_heads=h, dk=D, dv=D, dk_true=D, dv_true=D, eps=1e-6)
        st, cs = torch.zeros(seqs, h, D, D, device=dev), torch.zeros(seqs, 3, 3 * n, dtype=torch.bfloat16, device=dev)
        five = torch.full((t,), 5, dtype=torch.int32, device=dev)
        gp, gz, dp, dz = bf(t, 5 * n + D), bf(t, n), bf(t, 3 * n + h), bf(t, 2 * n)
        put("general_delta / delta_mix", phase, tm.row(lambda: ops.general_delta(gp, gz, gw, st, five, cu, sl), t * 7 * n * 2 + seqs * n * D * 8),
            tm.row(lambda: ops.delta_mix(dp, dz, dw, cs, st, five, cu, sl, 3 * n), t * (3 * n + h + 3 * n) * 2 + seqs * n * D * 8))
        # ---- logits of the rows that are sampled
        if decode:
            lg, gu = bf(t, VOCAB), bf(t, 2 * VOCAB)
            put("cap_logits / glu", phase, tm.row(lambda: ops.cap_logits(lg, 0.5, 30.0), t * VOCAB * 6), tm.row(lambda: ops.glu(gu), t * VOCAB * 6))
    return out


def run(args, device, sampler) -> dict:
    torch.manual_seed(0)
    res: dict = {}
    steps, warm = args.steps, max(args.warmup, 3)
    sampler.start()
    headline = None
    for name, s in SIZES.items():
        r = res[name] = {"size": {**s, "head_dim": D, "rot_dim": ROT, "kv_rank": RANK, "q_rank": QRANK, "norm_groups": GROUPS, "window": WINDOW,
                                  "taps": TAPS}}
        for kind, cfg in (("ginodra", ginodra_cfg(s)), ("latent", latent_cfg(s)), ("attention", attention_cfg(s))):
            model = DecoderModel(cfg, device)
            model.random_init(seed=0)
            r[f"{kind} params"] = cfg.param_count()
            for b in (64, 8, 1):
                r[f"{kind} b{b}"] = serve(model, b, 2048, steps, warm)
            if kind == "ginodra" and headline is None:
                headline = r["ginodra b64"]["decode"]
            del model
            torch.cuda.empty_cache()
        r["kernels"] = kernels(s, device)
        torch.cuda.empty_cache()
    N.check_status(device)
    return {"metric": "decode tok/s (Ginodra layers, bf16, 64 x 2048-token contexts)", "value": headline["tok_s"], "unit": "tokens/s", "n_gpus": 1,
            "steps": steps, "warmup": warm, "ms_per_step": headline["ms_per_step"], "higher_is_better": True, "scaling": "strong",
            "vs_baseline": None, "dtype": "bf16", "data": "synthetic: random-init weights, uniform-random prompt token ids",
            "config": {"model": "ginodra 2k", "global_batch": 64, "seq_len": 2048, "parallelism": "tp1", "kv_page": 16,
                       "l2": "model steps: weights >> 126 MB; kernels: L2 flushed before every launch"},
            "e2e": {"value": headline["e2e_tok_s"], "unit": "tokens/s", "ms_per_step": headline["e2e_ms_per_step"],
                    "h2d_bytes_per_step": headline["h2d"], "d2h_bytes_per_step": headline["d2h"]},
            "gpu_launches": headline["launches"] * steps, "clocks": sampler.stop(), "sizes": res}
