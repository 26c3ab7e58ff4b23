"""``bench.py --preset salopel``: prefill and decode throughput of the Salopel design at sizes that resemble a real
model's layers (random weights, a few layers), beside the closest models the framework already serves at equal
size:

* a DeepSeek-type decoder of the same width, heads, latents and layer count (latent attention with a rotated part
  and a dense gated feed-forward in every layer, through the same engine, bf16), and
* the Mamba-2 language model of the same width and layer count, which serves one request at a time (its scan
  kernel takes 32 state rows per head).

Throughput comes from CUDA events around ``LLMEngine.step``; e2e from host time around the same steps. Then every
kernel the design adds is timed alone beside the like kernel of the existing models, with its share of the measured
copy bandwidth or GEMM peak (inputs flushed from L2 before every launch).
"""
from __future__ import annotations

import torch

from bench_mixers import VOCAB, Timer, serve
from hartsyinference_b200 import ops
from hartsyinference_b200.models.llm import config as C
from hartsyinference_b200.models.llm.salopel import config_from
from hartsyinference_b200.models.llm.transformer import DecoderModel
from hartsyinference_b200.ops import _native as N

# width, layers in fours (per-head scan, selective scan, per-head scan, attention + feed-forward), scan channels,
# attention heads of 128, feed-forward
SIZES = {
    "2k": dict(width=2048, layers=8, inner=4096, heads=16, ff=8192),
    "4k": dict(width=4096, layers=4, inner=8192, heads=32, ff=16384),
}
D, RANK, QRANK, STATE1, STATE2, P = 128, 512, 1024, 16, 128, 64


def salopel_cfg(s: dict) -> C.TransformerConfig:
    head = {"type": "mamba2", "mlp": None, "mixer": {"heads": s["inner"] // P, "vdim": P, "state": STATE2, "groups": 1, "norm_groups": 1, "conv": 4}}
    chan = {"type": "mamba1", "mlp": None, "mixer": {"inner": s["inner"], "state": STATE1, "dt_rank": s["width"] // 16, "conv": 4}}
    att = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": s["ff"]},
           "mixer": {"heads": s["heads"], "dim": D, "vdim": D, "kv_rank": RANK, "q_rank": QRANK, "scale": D ** -0.5}}
    return config_from({"architecture": "Salopel", "norm": {"eps": 1e-6}, "residual_mult": 0.5, "vocab": VOCAB, "width": s["width"],
                        "layers": [(head, chan, head, att)[i % 4] for i in range(s["layers"])]})


def latent_cfg(s: dict) -> C.TransformerConfig:
    return C.TransformerConfig(arch="deepseek_v3", vocab_size=VOCAB, hidden_size=s["width"], num_layers=s["layers"], num_heads=s["heads"],
                               num_kv_heads=s["heads"], head_dim=D + 64, ffn_size=s["ff"], rope_dim=64,
                               mla=C.MlaConfig(q_lora_rank=QRANK, kv_lora_rank=RANK, qk_nope_head_dim=D, qk_rope_head_dim=64, v_head_dim=D))


def mamba2(s: dict, dev):
    from hartsyinference_b200.models.ssm import Mamba2Config, Mamba2Model
    return Mamba2Model(Mamba2Config(vocab_size=VOCAB, d_model=s["width"], n_layer=s["layers"], d_state=32, head_dim=P, expand=s["inner"] // s["width"]), dev)


def serve_one(model, prompt_len: int, steps: int) -> dict:
    ev = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
    toks = torch.randint(0, VOCAB, (prompt_len,), dtype=torch.int32)
    model.forward(toks, model.new_state())
    st = model.new_state()
    ev[0].record()
    h = model.forward(toks, st)
    ev[1].record()
    for _ in range(steps):
        h = model.forward(model.logits(h[-1:]).argmax(-1).to(torch.int32), st)
    ev[2].record()
    torch.cuda.synchronize()
    a, b = ev[0].elapsed_time(ev[1]), ev[1].elapsed_time(ev[2])
    return {"prefill": {"tokens": prompt_len, "device_ms": a, "tok_s": prompt_len / a * 1e3},
            "decode": {"batch": 1, "context": prompt_len, "ms_per_step": b / steps, "tok_s": steps / b * 1e3}}


# ------------------------------------------------------------------------------------------ kernels
def kernels(s: dict, dev) -> dict:
    """{kernel: {"decode" (64 rows): [new, like], "prefill" (8192 rows): [new, like]}}"""
    tm = Timer(dev)
    w, h, ff, inner = s["width"], s["heads"], s["ff"], s["inner"]
    heads2 = inner // P
    bf = lambda *sh: torch.randn(*sh, device=dev).to(torch.bfloat16)
    f32 = lambda *sh: torch.rand(*sh, device=dev)
    ones = torch.ones(max(w, inner), dtype=torch.bfloat16, device=dev)
    out: dict = {}

    def put(name, phase, new, like):
        out.setdefault(name, {})[phase] = {"new": new, "like": like}

    for phase, t in (("decode", 64), ("prefill", 8192)):
        nseq = 64 if phase == "decode" else 4
        cu = None if phase == "decode" else torch.arange(0, t + 1, t // 4, dtype=torch.int32, device=dev)
        slots = torch.arange(nseq, dtype=torch.int32, device=dev)
        pos = torch.full((t,), 5, dtype=torch.int32, device=dev)
        runs = None if phase == "decode" else [(t // 4, t // 4)] * 4
        # ---- norms and activation
        x, y = torch.randn(t, w, device=dev), bf(t, w)
        kw = dict(dim=w, eps=1e-6, layernorm=False, dtype=torch.bfloat16, plus_one=True, mult=0.5, plain=True)
        like = tm.row(lambda: ops.norm(y, ones[:w], residual=y), t * w * 8)
        put("residual_norm / norm", phase, tm.row(lambda: ops.residual_norm(x, y, ones[:w], None, **kw), t * w * (4 + 4 + 2 + 2)), like)
        table, ids = bf(VOCAB, w), torch.randint(0, VOCAB, (t,), dtype=torch.int32, device=dev)
        put("embedding_norm / embedding", phase, tm.row(lambda: ops.embedding_norm(ids, table, ones[:w], dim=w, eps=1e-6, plus_one=True), t * w * 8),
            tm.row(lambda: ops.embedding(ids, table), t * w * 4))
        z, coef = bf(t, ff), f32(4)
        gu = bf(t, 2 * ff)
        put("poly_norm / glu", phase, tm.row(lambda: ops.poly_norm(z, coef, ff, 1e-6), t * ff * 4), tm.row(lambda: ops.glu(gu), t * ff * 6))
        yi, zi = bf(t, inner), bf(t, inner)
        put("gated_norm / norm", phase, tm.row(lambda: ops.gated_norm(yi, zi, ones[:inner], 1, 1e-6, heads2, P), t * inner * 6),
            tm.row(lambda: ops.norm(yi, ones[:inner], residual=yi), t * inner * 8))
        # ---- recurrent mixers
        ch = inner + 2 * STATE2
        proj, cw, cb = bf(t, ch + inner + heads2), f32(4, ch), f32(ch)
        cs = torch.zeros(nseq, 3, ch, dtype=torch.bfloat16, device=dev)
        conv = lambda: ops.short_conv(proj[:, inner:inner + ch], cw, cb, cs, pos, cu, slots)
        seq = torch.cat([cs[0], proj[:t // nseq, inner:inner + ch]], 0)

        def torch_conv():                       # the convolution of the Mamba models, one sequence
            f = seq.float()
            return torch.nn.functional.silu((f.unfold(0, 4, 1) * cw.t()[None]).sum(-1) + cb).to(torch.bfloat16)
        put("short_conv / tensor-op convolution (one sequence)", phase, tm.row(conv, t * ch * 4 + nseq * ch * 12),
            tm.row(torch_conv, t // nseq * ch * 4))
        cwt = ops.ChannelScanWeights(a=-f32(inner, STATE1), dt_bias=f32(inner) - 4, d=f32(inner))
        st1 = torch.zeros(nseq, inner, STATE1, device=dev)
        xc, dtl, bc, zc = bf(t, inner), bf(t, inner), bf(t, 2 * STATE1), bf(t, inner)
        one = t // nseq
        dts, bs, c1 = f32(one, inner), bf(one, STATE1), bf(one, STATE1)
        put("channel_scan / selective_scan (one sequence)", phase,
            tm.row(lambda: ops.channel_scan(xc, dtl, bc, 0, STATE1, zc, cwt, st1, pos, cu, slots), t * inner * 8 + nseq * inner * STATE1 * 8),
            tm.row(lambda: ops.selective_scan(xc[:one], dts, cwt.a, bs, c1, cwt.d, st1[0]), one * inner * 8 + inner * STATE1 * 8))
        hw = ops.HeadScanWeights(rate=f32(heads2), dt_bias=f32(heads2) - 4, d=f32(heads2), heads=heads2, groups=1, n=STATE2, p=P)
        st2 = torch.zeros(nseq, heads2, STATE2, P, device=dev)
        xbc, dth = bf(t, ch), bf(t, heads2)
        new = tm.row(lambda: ops.head_scan(xbc, dth, hw, st2, pos, cu, slots, runs), t * (ch + inner) * 2 + nseq * heads2 * STATE2 * P * 8)
        # the same count of state values through the Mamba-2 model's kernel (32 rows per channel, one sequence)
        c32 = inner * STATE2 // 32
        xs, ds, b32, a32, d32 = bf(one, c32), f32(one, c32), bf(one, 32), -f32(c32, 32), f32(c32)
        h32 = torch.zeros(c32, 32, device=dev)
        put("head_scan / selective_scan (as many state values, one sequence)", phase, new,
            tm.row(lambda: ops.selective_scan(xs, ds, a32, b32, b32, d32, h32), one * c32 * 8 + c32 * 32 * 8))
        dh = heads2 // 2                        # delta rule with as many state values: heads of 128 x 128
        dch = 3 * dh * 128
        dw = ops.DeltaWeights(conv=f32(4, dch), decay_rate=f32(dh), dt_bias=f32(dh * 128), norm=ones[:128], heads=dh, kv_heads=dh, dk=128, dv=128,
                              dk_true=128, dv_true=128, eps=1e-6)
        dcs, dst = torch.zeros(nseq, 3, dch, dtype=torch.bfloat16, device=dev), torch.zeros(nseq, dh, 128, 128, device=dev)
        dp, dz = bf(t, dch + dh), bf(t, 2 * dh * 128)

        def head_mixer():
            return ops.gated_norm(ops.head_scan(conv(), dth, hw, st2, pos, cu, slots, runs), zi, ones[:inner], 1, 1e-6, heads2, P)
        put("conv + head_scan + gated_norm / delta_mix", phase,
            tm.row(head_mixer, t * (ch + 2 * inner) * 2 + nseq * heads2 * STATE2 * P * 8),
            tm.row(lambda: ops.delta_mix(dp, dz, dw, dcs, dst, pos, cu, slots, dch), t * (dch + 3 * dh * 128) * 2 + nseq * dh * 128 * 128 * 8))
        # ---- latent attention: 64 sequences of 2048 tokens at decode, four whole prompts of 2048 at prefill
        seqs, ctx = nseq, 2048
        per = ctx // 16
        cache, cache2 = bf(seqs * per, 1, 16, RANK), bf(seqs * per, 16, RANK + 64)
        btab = torch.randperm(seqs * per, device=dev).to(torch.int32).reshape(seqs, per)
        lens = torch.full((seqs,), ctx, dtype=torch.int32, device=dev)
        gate = bf(t, h * D)
        ptok = bf(t, QRANK + RANK)
        wslots = torch.randperm(seqs * ctx, device=dev)[:t].contiguous()
        inv = torch.rand(32, device=dev)
        kv576, qn, qa = bf(t, RANK + 64), bf(t, h * (D + 64)), torch.empty(t, h, RANK + 64, dtype=torch.bfloat16, device=dev)
        put("latent_prep / mla_prep", phase,
            tm.row(lambda: ops.latent_prep(ptok, 0, QRANK, ones[:QRANK], QRANK, RANK, ones[:RANK], cache, wslots, 1e-6), t * (QRANK + RANK) * 4),
            tm.row(lambda: ops.mla_prep(kv576, ones[:RANK], qn, qa, cache2, pos, wslots, inv, h, D + 64, D), t * ((RANK + 64) * 4 + h * 64 * 4)))
        if phase == "decode":
            ql, q576 = bf(t, h * RANK), bf(t, h, RANK + 64)
            put("latent_attn / mla_attn", phase,
                tm.row(lambda: ops.latent_attn(ql, cache, btab, lens, h, 0.05, max_kv_len=ctx), seqs * ctx * RANK * 2 + 2 * t * h * RANK * 2,
                       4.0 * t * ctx * h * RANK),
                tm.row(lambda: ops.mla_attn(q576, cache2, btab, lens, 0.05, max_kv_len=ctx), seqs * ctx * (RANK + 64) * 2 + t * h * (2 * RANK + 64) * 2,
                       2.0 * t * ctx * h * (2 * RANK + 64)))
            qd, uk, uv = bf(t, h * D), ops.LinearWeight(bf(h * RANK, D)), ops.LinearWeight(bf(h * D, RANK))
            qab, vo, lat = torch.empty(t, h * RANK, dtype=torch.bfloat16, device=dev), torch.empty(t, h * D, dtype=torch.bfloat16, device=dev), bf(t, h * RANK)
            nb = h * RANK * D * 2 + t * h * (RANK + D) * 2
            put("head_linear (W_uk) / colbatched_linear", phase, tm.row(lambda: ops.head_linear(qd, uk, h), nb),
                tm.row(lambda: ops.colbatched_linear(qd, uk.weight, h, D, qab, RANK), nb))
            put("head_linear (W_uv, gate) / colbatched_linear", phase, tm.row(lambda: ops.head_linear(lat, uv, h, gate=gate), nb + t * h * D * 2),
                tm.row(lambda: ops.colbatched_linear(lat, uv.weight, h, RANK, vo, D), nb))
        else:
            q, kvx, o = bf(t, h * D), bf(t, 2 * h * D), torch.empty(t, h * D, dtype=torch.bfloat16, device=dev)
            starts, qlens = cu[:-1].contiguous(), lens
            flops = 4.0 * seqs * ctx * (ctx + 1) / 2 * h * D
            kc, vc = bf(seqs * per, h, 16, D), bf(seqs * per, h, 16, D)
            q3 = q.view(t, h, D)
            put("attn_runs / attn_prefill", phase,
                tm.row(lambda: ops.attn_runs(q, kvx[:, :h * D], kvx[:, h * D:], o, starts, qlens, cu, lens, heads=h, max_q_len=ctx, scale=0.1, gate=gate),
                       5 * t * h * D * 2, flops),
                tm.row(lambda: ops.attn_prefill_paged(q3, kc, vc, btab, lens, cu, ctx), 4 * t * h * D * 2, flops))
            up = ops.LinearWeight(bf(2 * h * D, RANK))
            ids4 = torch.arange(4, dtype=torch.int32, device=dev)

            def latent():                       # gather, expansion and attention of the prompts
                c = ops.latent_gather(cache, btab, ids4, cu, t, ctx)
                kv = ops.linear(c, up)
                ops.attn_runs(q, kv[:, :h * D], kv[:, h * D:], o, starts, qlens, cu, lens, heads=h, max_q_len=ctx, scale=0.1, gate=gate)
            rows = torch.arange(t, device=dev)
            rseq, rlen = (rows // ctx).to(torch.int32), (rows % ctx + 1).to(torch.int32)
            q576 = bf(t, h, RANK + 64)
            put("gather + expansion + attn_runs / mla_attn", phase, tm.row(latent, 5 * t * h * D * 2, flops + 4.0 * t * RANK * h * D),
                tm.row(lambda: ops.mla_attn(q576, cache2, btab, rlen, 0.05, row_seq=rseq, max_kv_len=ctx), t * h * (2 * RANK + 64) * 2,
                       2.0 * seqs * ctx * (ctx + 1) / 2 * h * (2 * RANK + 64)))
            put("latent_gather / embedding", phase, tm.row(lambda: ops.latent_gather(cache, btab, ids4, cu, t, ctx), t * RANK * 4),
                tm.row(lambda: ops.embedding(ids, table[:, :RANK].contiguous()), t * RANK * 4))
    return out


def run(args, device, sampler) -> dict:
    torch.manual_seed(0)
    res: dict = {}
    steps, warm = args.steps, max(args.warmup, 3)
    sampler.start()
    headline = None
    for name, s in SIZES.items():
        r = res[name] = {"size": {**s, "head_dim": D, "kv_rank": RANK, "q_rank": QRANK, "states": [STATE1, STATE2], "scan_head": P}}
        for kind, cfg in (("salopel", salopel_cfg(s)), ("latent_dense", latent_cfg(s))):
            model = DecoderModel(cfg, device)
            model.random_init(seed=0)
            for b in (64, 8, 1):
                r[f"{kind} b{b}"] = serve(model, b, 2048, steps, warm)
            if kind == "salopel" and headline is None:
                headline = r["salopel b64"]["decode"]
            del model
            torch.cuda.empty_cache()
        m = mamba2(s, device)
        r["mamba2 b1"] = serve_one(m, 2048, 8)
        del m
        torch.cuda.empty_cache()
        r["kernels"] = kernels(s, device)
        torch.cuda.empty_cache()
    N.check_status(device)
    return {"metric": "decode tok/s (Salopel layers, bf16, 64 x 2048-token contexts)", "value": headline["tok_s"], "unit": "tokens/s", "n_gpus": 1,
            "steps": steps, "warmup": warm, "ms_per_step": headline["ms_per_step"], "higher_is_better": True, "scaling": "strong",
            "vs_baseline": None, "dtype": "bf16", "data": "synthetic: random-init weights, uniform-random prompt token ids",
            "config": {"model": "salopel 2k", "global_batch": 64, "seq_len": 2048, "parallelism": "tp1", "kv_page": 16,
                       "l2": "model steps: weights + state >> 126 MB; kernels: L2 flushed before every launch"},
            "e2e": {"value": headline["e2e_tok_s"], "unit": "tokens/s", "ms_per_step": headline["e2e_ms_per_step"],
                    "h2d_bytes_per_step": headline["h2d"], "d2h_bytes_per_step": headline["d2h"]},
            "gpu_launches": headline["launches"] * steps, "clocks": sampler.stop(), "sizes": res}
