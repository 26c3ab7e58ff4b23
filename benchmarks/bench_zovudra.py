"""``bench.py --preset zovudra``: prefill and decode throughput of the Zovudra design at sizes that resemble a real
model's layers (random weights, a few layers), beside the closest models the framework already serves at equal
size, all through the same engine in bf16:

* a DeepSeek-type decoder of the same width, heads, latents, experts and layer count (latent attention with a rotated
  part, gated experts chosen in groups and a shared expert in every layer), and
* a Qwen3-MoE-type decoder (grouped-query attention with normed and rotated heads, gated experts in every layer).

Throughput comes from CUDA events around ``LLMEngine.step``; e2e from host time around the same steps. Then every
kernel the design adds or extends is timed alone beside the like kernel of the existing models, with its share of the
measured copy bandwidth or GEMM peak (inputs flushed from L2 before every launch).
"""
from __future__ import annotations

import torch

from bench_mixers import VOCAB, Timer, serve
from hartsyinference_b200 import ops
from hartsyinference_b200.models.llm import config as C
from hartsyinference_b200.models.llm.rope import Rotary
from hartsyinference_b200.models.llm.transformer import DecoderModel
from hartsyinference_b200.models.llm.zovudra import config_from
from hartsyinference_b200.ops import _native as N

# width, layers (attention and latent attention in turn), heads of 128, key heads, experts, chosen, expert size, token input
SIZES = {
    "2k": dict(width=2048, layers=8, heads=16, kv=4, experts=64, top=6, ff=1024, side=256),
    "4k": dict(width=4096, layers=4, heads=32, kv=8, experts=32, top=4, ff=2048, side=256),
}
D, ROT, RANK, QRANK, GROUPS, KEEP, WINDOW, FIRST = 128, 64, 512, 1024, 8, 4, 1024, 4


def zovudra_cfg(s: dict) -> C.TransformerConfig:
    mlp = {"kind": "moe", "expert": {"ff": s["ff"]}, "shared": {"ff": s["ff"]},
           "router": {"experts": s["experts"], "top": s["top"], "groups": {"count": GROUPS, "keep": KEEP}, "scale": 1.0}}
    att = {"type": "attention", "mlp": mlp, "mixer": {"heads": s["heads"], "kv_heads": s["kv"], "dim": D, "vdim": D, "scale": D ** -0.5,
                                                      "mask": {"size": WINDOW, "keep_first": FIRST}, "rot": {"base": 1e6, "dims": D}}}
    lat = {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": s["heads"], "dim": D, "rot_dim": ROT, "vdim": D, "kv_rank": RANK, "q_rank": QRANK,
                                                             "scale": (D + ROT) ** -0.5, "mask": {"size": WINDOW}, "rot": {"base": 1e6, "dims": ROT}}}
    return config_from({"architecture": "Zovudra", "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "token_side": {"dim": s["side"]},
                        "vocab": VOCAB, "width": s["width"], "layers": [(att, lat)[i % 2] for i in range(s["layers"])]})


def latent_moe_cfg(s: dict) -> C.TransformerConfig:
    return C.TransformerConfig(arch="deepseek_v3", vocab_size=VOCAB, hidden_size=s["width"], num_layers=s["layers"], num_heads=s["heads"],
                               num_kv_heads=s["heads"], head_dim=D + ROT, ffn_size=s["ff"], rope_dim=ROT,
                               mla=C.MlaConfig(q_lora_rank=QRANK, kv_lora_rank=RANK, qk_nope_head_dim=D, qk_rope_head_dim=ROT, v_head_dim=D),
                               moe=C.MoeConfig(num_experts=s["experts"], top_k=s["top"], expert_ffn=s["ff"], num_shared_experts=1, shared_ffn=s["ff"],
                                               scoring="sigmoid", norm_topk_prob=True, n_group=GROUPS, topk_group=KEEP))


def attention_moe_cfg(s: dict) -> C.TransformerConfig:
    return C.TransformerConfig(arch="qwen3_moe", vocab_size=VOCAB, hidden_size=s["width"], num_layers=s["layers"], num_heads=s["heads"],
                               num_kv_heads=s["kv"], head_dim=D, ffn_size=s["ff"], qk_norm=True,
                               moe=C.MoeConfig(num_experts=s["experts"], top_k=s["top"], expert_ffn=s["ff"], norm_topk_prob=True))


class _Positions:
    def __init__(self, positions):
        self.positions, self.plan = positions, None


# ------------------------------------------------------------------------------------------ kernels
def kernels(s: dict, dev) -> dict:
    """{kernel: {"decode" (64 rows): [new, like], "prefill" (8192 rows): [new, like]}}"""
    tm = Timer(dev)
    w, h, kv, ff, e, top, side = (s[n] for n in ("width", "heads", "kv", "ff", "experts", "top", "side"))
    bf = lambda *sh: torch.randn(*sh, device=dev).to(torch.bfloat16)
    i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=dev)
    ones = torch.ones(max(w, h * D, QRANK), dtype=torch.bfloat16, device=dev)
    out: dict = {}

    def put(name, phase, new, like):
        out.setdefault(name, {})[phase] = {"new": new, "like": like}

    for phase, t in (("decode", 64), ("prefill", 8192)):
        seqs, ctx = (64, 2048) if phase == "decode" else (4, 2048)
        decode = phase == "decode"
        pos = torch.full((t,), ctx - 1, dtype=torch.int32, device=dev) if decode else torch.arange(t, dtype=torch.int32, device=dev) % ctx
        # ---- norms, token input
        x, y = torch.randn(t, w, device=dev), bf(t, w)
        tanh = ops.TanhNorm(0.5, ones[:w], torch.zeros(w, dtype=torch.bfloat16, device=dev))
        kw = dict(dim=w, eps=1e-6, layernorm=False, dtype=torch.bfloat16)
        norm = tm.row(lambda: ops.norm(y, ones[:w], residual=y), t * w * 8)
        put("residual_norm (tanh) / norm", phase, tm.row(lambda: ops.residual_norm(x, y, None, tanh, **kw), t * w * 12), norm)
        put("residual_norm (RMS in, tanh out) / norm", phase, tm.row(lambda: ops.residual_norm(x, y, ones[:w], tanh, **kw), t * w * 12), norm)
        pairs = t * top
        rows, slot = bf(pairs, w), torch.randperm(pairs, device=dev).to(torch.int32).reshape(t, top)
        wts, ids0, ew, comb = torch.rand(t, top, device=dev), torch.zeros(t, top, dtype=torch.int32, device=dev), torch.rand(t, device=dev), bf(t, w)
        rr = ops.RoutedRows(rows, slot, ids0, wts, None, e, y, ew)

        def combine_norm():
            ops.moe_combine(rows, slot, wts, comb, accumulate=True)
            ops.norm(comb, ones[:w], residual=y)
        put("residual_norm (expert rows, shared rows) / moe_combine + norm", phase,
            tm.row(lambda: ops.residual_norm(x, rr, None, None, plain=True, **kw), (pairs + t) * w * 2 + t * w * 10),
            tm.row(combine_norm, (pairs + 2 * t) * w * 2 + t * w * 8))
        tab, ids = bf(VOCAB, s["layers"] * side), torch.randint(0, VOCAB, (t,), dtype=torch.int32, device=dev)
        u, gu = bf(t, side), bf(t, 2 * side)
        put("side_gate / glu", phase, tm.row(lambda: ops.side_gate(u, ids, tab[:, side:2 * side]), t * side * 6), tm.row(lambda: ops.glu(gu), t * side * 6))
        # ---- experts
        rw, rg = ops.LinearWeight(bf(e, w)), ops.LinearWeight(bf(e + 1, w))
        route = lambda: ops.moe_route(ops.linear(y, rw), None, top, n_group=GROUPS, topk_group=KEEP, sigmoid=True, norm_topk=True)
        put("router (groups, gate) / linear + moe_route", phase,
            tm.row(lambda: ops.router(y, rg, None, top, sigmoid=True, norm_topk=True, n_group=GROUPS, topk_group=KEEP, gate=True),
                   t * w * 2 + e * w * 2, 2.0 * t * w * e), tm.row(route, t * w * 2 + e * w * 2, 2.0 * t * w * e))
        ids_e = route()[0]
        cap = ops.moe_block_capacity(t, top, e)
        xs = torch.zeros((pairs + cap - 1) // cap * cap + e * cap, w, dtype=torch.bfloat16, device=dev)
        plan = ops.moe_dispatch_dynamic(y, ids_e, 0, e, cap, xs)
        used = len(ids_e.unique())
        up, gup = ops.LinearWeight(bf(e * ff, w)), ops.LinearWeight(bf(e * 2 * ff, w))
        put("grouped product with relu squared / grouped product + glu", phase,
            tm.row(lambda: ops.grouped_linear_dynamic(xs, up, e, plan, act="relu2"), used * ff * w * 2 + pairs * (w + ff) * 2, 2.0 * pairs * w * ff),
            tm.row(lambda: ops.glu(ops.grouped_linear_dynamic(xs, gup, e, plan)), used * 2 * ff * w * 2 + pairs * (w + 5 * ff) * 2, 4.0 * pairs * w * ff))
        del up, gup, xs
        # ---- grouped-query attention: 64 contexts of 2048 tokens, or four whole prompts
        per = ctx // 16
        kc, vc = bf(seqs * per, kv, 16, D), bf(seqs * per, kv, 16, D)
        table = torch.randperm(seqs * per, device=dev).to(torch.int32).reshape(seqs, per)
        lens = torch.full((seqs,), ctx, dtype=torch.int32, device=dev)
        cu = None if decode else torch.arange(0, t + 1, ctx, dtype=torch.int32, device=dev)
        wslots = torch.randperm(seqs * ctx, device=dev)[:t].contiguous()
        p = bf(t, (h + 2 * kv) * D)
        rotary = Rotary(C.RotarySpec(D, 1e6), dev)
        narrow, wide = tab[:, :D].contiguous(), tab[:, :RANK + ROT].contiguous()
        cs, inv = rotary.table(_Positions(pos)), rotary.hi
        put("rope_table / embedding (as many bytes)", phase, tm.row(lambda: ops.rope_table(pos, rotary.hi, rotary.lo), t * D * 4),
            tm.row(lambda: ops.embedding(ids, narrow), t * D * 4))
        nb = t * (h + 2 * kv) * D * 4
        put("qk_rope_store / rope_kv", phase,
            tm.row(lambda: ops.qk_rope_store(p, h, kc, vc, wslots, table=cs, q_norm=ones[:h * D], k_norm=ones[:kv * D], eps=1e-6), nb + t * D * 4),
            tm.row(lambda: ops.rope_kv(p, pos, h, kv, D, k_cache=kc, v_cache=vc, slot_mapping=wslots, inv_freq=inv, q_norm_w=ones[:D], k_norm_w=ones[:D]), nb))
        q = bf(t, h * D)
        q3 = q.view(t, h, D)
        seen = WINDOW + FIRST
        nb = (seqs * WINDOW * kv * 2 + 2 * t * h) * D * 2
        if decode:
            put("attn_biased (window, kept tokens) / attn_decode (window)", phase,
                tm.row(lambda: ops.attn_biased(q, kc, vc, table, lens, None, heads=h, max_kv_len=ctx, scale=0.1, window=WINDOW, keep_first=FIRST), nb),
                tm.row(lambda: ops.attn_decode(q3, kc, vc, table, lens, 0.1, window=WINDOW, max_kv_len=ctx), nb))
        else:
            fl = 4.0 * seqs * (WINDOW * (WINDOW + 1) / 2 + (ctx - WINDOW) * seen) * h * D
            put("attn_biased (window, kept tokens) / attn_prefill (window)", phase,
                tm.row(lambda: ops.attn_biased(q, kc, vc, table, lens, cu, heads=h, max_q_len=ctx, max_kv_len=ctx, scale=0.1, window=WINDOW, keep_first=FIRST),
                       4 * t * h * D * 2, fl),
                tm.row(lambda: ops.attn_prefill_paged(q3, kc, vc, table, lens, cu, ctx, causal=True, scale=0.1, window=WINDOW), 4 * t * h * D * 2, fl))
        # ---- latent attention
        row = RANK + ROT
        cache, cache2 = bf(seqs * per, 1, 16, row), bf(seqs * per, 16, row)
        rot = Rotary(C.RotarySpec(ROT, 1e6, True), dev)
        ct = rot.table(_Positions(pos))
        pt, kv576, qn = bf(t, QRANK + row), bf(t, row), bf(t, h * (D + ROT))
        qa = torch.empty(t, h, row, dtype=torch.bfloat16, device=dev)
        put("latent_prep / mla_prep", phase,
            tm.row(lambda: ops.latent_prep(pt, 0, QRANK, ones[:QRANK], QRANK, RANK, ones[:RANK], cache, wslots, 1e-6, ct), t * (QRANK + row) * 4),
            tm.row(lambda: ops.mla_prep(kv576, ones[:RANK], qn, qa, cache2, pos, wslots, rot.hi, h, D + ROT, D), t * (row * 4 + h * ROT * 4)))
        if decode:
            short = torch.full((seqs,), WINDOW, dtype=torch.int32, device=dev)
            ql = bf(t, h * row)
            fl = 2.0 * t * WINDOW * h * (2 * RANK + ROT)
            nb = seqs * WINDOW * row * 2 + t * h * (2 * RANK + ROT) * 2
            put("latent_attn (window) / mla_attn (contexts of that length)", phase,
                tm.row(lambda: ops.latent_attn(ql, cache, table, lens, h, 0.05, max_kv_len=ctx, v_dim=RANK, window=WINDOW), nb, fl),
                tm.row(lambda: ops.mla_attn(ql.view(t, h, row), cache2, table, short, 0.05, max_kv_len=WINDOW), nb, fl))
            uk, uv = ops.LinearWeight(bf(h * RANK, D)), ops.LinearWeight(bf(h * D, RANK))
            vo, lat = torch.empty(t, h * D, dtype=torch.bfloat16, device=dev), bf(t, h * RANK)
            nb = h * RANK * D * 2 + t * h * (row + D + ROT) * 2
            put("head_linear (W_uk, turned tail) / colbatched_linear", phase, tm.row(lambda: ops.head_linear(qn, uk, h, tail=ROT, table=ct), nb),
                tm.row(lambda: ops.colbatched_linear(qn, uk.weight, h, D + ROT, qa.view(t, -1), row), nb - t * h * ROT * 4))
            nb = h * RANK * D * 2 + t * h * (RANK + D) * 2
            put("head_linear (W_uv) / colbatched_linear", phase, tm.row(lambda: ops.head_linear(lat, uv, h), nb),
                tm.row(lambda: ops.colbatched_linear(lat, uv.weight, h, RANK, vo, D), nb))
        else:
            kvx, o = bf(t, 2 * h * D), torch.empty(t, h * D, dtype=torch.bfloat16, device=dev)
            gathered, starts, zero, ids4 = bf(t, row), cu[:-1].contiguous(), i32(0, 0, 0, 0), i32(0, 1, 2, 3)
            keys = seqs * (WINDOW * (WINDOW + 1) / 2 + (ctx - WINDOW) * WINDOW)
            fl = 2.0 * keys * h * (2 * D + ROT)
            nb = t * h * (4 * D + ROT) * 2
            kch, vch = bf(seqs * per, h, 16, D), bf(seqs * per, h, 16, D)
            runs = lambda k, v, c: ops.attn_runs(qn, k, v, o, starts, lens, cu, lens, heads=h, max_q_len=ctx, scale=0.07, window=WINDOW,
                                                 k_shared=c[:, RANK:], table=ct)
            put("attn_runs (keys of 192, window) / attn_prefill (128, window)", phase, tm.row(lambda: runs(kvx[:, :h * D], kvx[:, h * D:], gathered), nb, fl),
                tm.row(lambda: ops.attn_prefill_paged(q3, kch, vch, table, lens, cu, ctx, causal=True, scale=0.1, window=WINDOW), 4 * t * h * D * 2, 4.0 * keys * h * D))
            upw = ops.LinearWeight(bf(2 * h * D, RANK))

            def latent():                       # gather, expansion and attention of the prompts
                c = ops.latent_gather(cache, table, ids4, cu, t, ctx, zero)
                kvs = ops.linear(c[:, :RANK], upw)
                runs(kvs[:, :h * D], kvs[:, h * D:], c)
            r = torch.arange(t, device=dev)
            rseq, rlen = (r // ctx).to(torch.int32), (r % ctx + 1).to(torch.int32)
            q576 = bf(t, h, row)
            put("gather + expansion + attn_runs / mla_attn (no window)", phase, tm.row(latent, nb, fl + 4.0 * t * RANK * h * D),
                tm.row(lambda: ops.mla_attn(q576, cache2, table, rlen, 0.05, row_seq=rseq, max_kv_len=ctx), t * h * (2 * RANK + ROT) * 2,
                       2.0 * seqs * ctx * (ctx + 1) / 2 * h * (2 * RANK + ROT)))
            put("latent_gather / embedding", phase, tm.row(lambda: ops.latent_gather(cache, table, ids4, cu, t, ctx, zero), t * row * 4),
                tm.row(lambda: ops.embedding(ids, wide), t * row * 4))
    return out


def run(args, device, sampler) -> dict:
    torch.manual_seed(0)
    res: dict = {}
    steps, warm = args.steps, max(args.warmup, 3)
    sampler.start()
    headline = None
    for name, s in SIZES.items():
        r = res[name] = {"size": {**s, "head_dim": D, "rot_dim": ROT, "kv_rank": RANK, "q_rank": QRANK, "groups": [GROUPS, KEEP], "window": WINDOW,
                                  "keep_first": FIRST}}
        for kind, cfg in (("zovudra", zovudra_cfg(s)), ("latent_moe", latent_moe_cfg(s)), ("attention_moe", attention_moe_cfg(s))):
            model = DecoderModel(cfg, device)
            model.random_init(seed=0)
            for b in (64, 8, 1):
                r[f"{kind} b{b}"] = serve(model, b, 2048, steps, warm)
            if kind == "zovudra" and headline is None:
                headline = r["zovudra b64"]["decode"]
            del model
            torch.cuda.empty_cache()
        r["kernels"] = kernels(s, device)
        torch.cuda.empty_cache()
    N.check_status(device)
    return {"metric": "decode tok/s (Zovudra layers, bf16, 64 x 2048-token contexts)", "value": headline["tok_s"], "unit": "tokens/s", "n_gpus": 1,
            "steps": steps, "warmup": warm, "ms_per_step": headline["ms_per_step"], "higher_is_better": True, "scaling": "strong",
            "vs_baseline": None, "dtype": "bf16", "data": "synthetic: random-init weights, uniform-random prompt token ids",
            "config": {"model": "zovudra 2k", "global_batch": 64, "seq_len": 2048, "parallelism": "tp1", "kv_page": 16,
                       "l2": "model steps: weights >> 126 MB; kernels: L2 flushed before every launch"},
            "e2e": {"value": headline["e2e_tok_s"], "unit": "tokens/s", "ms_per_step": headline["e2e_ms_per_step"],
                    "h2d_bytes_per_step": headline["h2d"], "d2h_bytes_per_step": headline["d2h"]},
            "gpu_launches": headline["launches"] * steps, "clocks": sampler.stop(), "sizes": res}
