"""``bench.py --preset lududra``: prefill and decode throughput of the Lududra design at sizes that resemble a
real model's layers (random weights, a few layers), beside the closest models the framework already serves
at equal size:

* a Qwen3-MoE-type decoder of the same width, heads, experts and layer count (grouped-query attention and
  routed experts through the same engine and grouped GEMMs, bf16), and
* the Qwen3.5 hybrid (gated DeltaNet + attention), the only other delta-rule model, which steps token by
  token in tensor ops and serves one request at a time.

Throughput comes from CUDA events around ``LLMEngine.step``; e2e from host time around the same steps. Then
every kernel the design adds is timed alone beside the like kernel of the existing models, with its share
of the measured copy bandwidth or GEMM peak (inputs flushed from L2 before every launch).
"""
from __future__ import annotations

import json
import os
import time

import torch

from hartsyinference_b200 import ops
from hartsyinference_b200.engine import LLMEngine, SamplingParams
from hartsyinference_b200.models.llm import config as C
from hartsyinference_b200.models.llm.lududra import lududra_config
from hartsyinference_b200.models.llm.transformer import DecoderModel
from hartsyinference_b200.ops import _native as N

# width, layers (every fourth is attention), heads of 128, key heads of attention, experts + pass-through, chosen, expert size
SIZES = {
    "2k": dict(width=2048, layers=8, heads=16, kv=2, experts=64, identity=8, top=6, ff=1024),
    "4k": dict(width=4096, layers=4, heads=32, kv=4, experts=32, identity=8, top=4, ff=2048),
}
WINDOW, VOCAB, D = 1024, 32768, 128


def lududra_cfg(s: dict) -> C.TransformerConfig:
    mlp = {"kind": "moe", "expert": {"ff": s["ff"], "limit": 7.0},
           "router": {"experts": s["experts"], "identity": s["identity"], "top": s["top"]}}
    delta = {"type": "channel_delta", "mlp": mlp, "mixer": {"heads": s["heads"], "kv_heads": s["heads"], "dim": D, "vdim": D, "conv": 4}}
    att = {"type": "attention", "mlp": mlp, "mixer": {"heads": s["heads"], "kv_heads": s["kv"], "dim": D, "vdim": D, "bias_max": 512,
                                                      "mask": {"size": WINDOW}, "scale": D ** -0.5, "softcap": 30.0}}
    return lududra_config({"architecture": "Lududra", "embedding": {"scale": 1.0}, "norm": {"eps": 1e-6}, "vocab": VOCAB,
                           "width": s["width"], "layers": [att if i % 4 == 3 else delta for i in range(s["layers"])]})


def attention_moe_cfg(s: dict) -> C.TransformerConfig:
    return C.TransformerConfig(arch="qwen3_moe", vocab_size=VOCAB, hidden_size=s["width"], num_layers=s["layers"], num_heads=s["heads"],
                               num_kv_heads=s["kv"], head_dim=D, ffn_size=s["ff"], qk_norm=True,
                               moe=C.MoeConfig(num_experts=s["experts"], top_k=s["top"], expert_ffn=s["ff"], norm_topk_prob=True))


def qwen35_model(s: dict, dev):
    from hartsyinference_b200.models.ssm.qwen35 import Qwen35Config, Qwen35Model
    types = tuple("full_attention" if i % 4 == 3 else "linear_attention" for i in range(s["layers"]))
    cfg = Qwen35Config(vocab_size=VOCAB, hidden=s["width"], layers=s["layers"], heads=s["heads"], kv_heads=s["kv"], head_dim=D,
                       lin_k_heads=s["heads"], lin_v_heads=s["heads"], lin_k_dim=D, lin_v_dim=D, layer_types=types, experts=s["experts"],
                       top_k=s["top"], expert_ffn=s["ff"], shared_ffn=128)
    w, h, hd = s["width"], s["heads"], s["heads"] * D
    shape = {"embed_tokens.weight": (VOCAB, w), "mlp.gate.weight": (s["experts"], w), "experts.gate_up_proj": (s["experts"], 2 * s["ff"], w),
             "experts.down_proj": (s["experts"], w, s["ff"]), "gate_proj.weight": (128, w), "up_proj.weight": (128, w), "down_proj.weight": (w, 128),
             "shared_expert_gate.weight": (1, w), "in_proj_qkv.weight": (3 * hd, w), "in_proj_z.weight": (hd, w), "in_proj_b.weight": (h, w),
             "in_proj_a.weight": (h, w), "conv1d.weight": (3 * hd, 1, 4), "dt_bias": (h,), "A_log": (h,), "out_proj.weight": (w, hd),
             "q_proj.weight": (2 * hd, w), "k_proj.weight": (s["kv"] * D, w), "v_proj.weight": (s["kv"] * D, w), "o_proj.weight": (w, hd)}

    def get(name):
        if name == "lm_head.weight":
            return torch.randn(VOCAB, w, device=dev, dtype=torch.bfloat16) * 0.02
        for k, v in shape.items():
            if name.endswith(k):
                return torch.randn(v, device=dev, dtype=torch.bfloat16) * 0.02
        return torch.zeros(D if name.endswith(("linear_attn.norm.weight", "q_norm.weight", "k_norm.weight")) else w, device=dev, dtype=torch.bfloat16)
    return Qwen35Model(cfg, dev, get)


# ------------------------------------------------------------------------------------------ models
def serve(model, batch: int, prompt_len: int, steps: int, warmup: int) -> dict:
    """Prefill of ``batch`` prompts, then decode steps of the whole batch."""
    spare = batch * prompt_len // 8192 + 8           # early prompts decode beside the later ones' chunks
    total = prompt_len + steps + warmup + spare
    pages = (total + 15) // 16 + 1
    eng = LLMEngine(model, num_pages=batch * pages + 8, page_size=16, max_batch=batch, prefill_chunk=8192, max_model_len=pages * 16)
    g = torch.Generator().manual_seed(1)
    prompts = torch.randint(0, VOCAB, (batch, prompt_len), generator=g).tolist()
    params = SamplingParams(greedy=True, ignore_eos=True, max_tokens=steps + warmup + spare)
    eng.time_steps = True
    out = {}
    for timed in (False, True):                    # the first prefill warms up
        ids = [eng.add_request(p, params) for p in prompts]
        ms, launches = 0.0, 0
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        while any(not eng.requests[i].output for i in ids):
            eng.step()
            ms += eng.device_ms_last
            launches += eng.kernel_launches_last
        wall = time.perf_counter() - t0
        if not timed:
            for i in ids:
                eng.cancel(i)
    out["prefill"] = {"tokens": batch * prompt_len, "device_ms": ms, "tok_s": batch * prompt_len / ms * 1e3,
                      "e2e_tok_s": batch * prompt_len / wall, "launches": launches}
    for _ in range(warmup):
        eng.step()
    ms, launches, h2d, d2h = 0.0, 0, 0, 0
    torch.cuda.synchronize()
    t0 = time.perf_counter()
    for _ in range(steps):
        assert len(eng.step()) == batch
        ms += eng.device_ms_last
        launches += eng.kernel_launches_last
        h2d += eng.h2d_bytes_last
        d2h += eng.d2h_bytes_last
    wall = time.perf_counter() - t0
    out["decode"] = {"batch": batch, "context": prompt_len, "ms_per_step": ms / steps, "tok_s": batch * steps / ms * 1e3,
                     "e2e_tok_s": batch * steps / wall, "e2e_ms_per_step": wall / steps * 1e3, "launches": launches // steps, "h2d": h2d // steps,
                     "d2h": d2h // steps}
    return out


def serve_qwen35(model, prompt_len: int, steps: int) -> dict:
    ev = [torch.cuda.Event(enable_timing=True) for _ in range(3)]
    toks = torch.randint(0, VOCAB, (prompt_len,))
    model.forward(toks[:4], model.new_state())
    st = model.new_state()
    ev[0].record()
    h = model.forward(toks, st)
    ev[1].record()
    for _ in range(steps):
        h = model.forward(model.logits(h[-1:]).argmax(-1).cpu(), st)
    ev[2].record()
    torch.cuda.synchronize()
    a, b = ev[0].elapsed_time(ev[1]), ev[1].elapsed_time(ev[2])
    return {"prefill": {"tokens": prompt_len, "device_ms": a, "tok_s": prompt_len / a * 1e3},
            "decode": {"batch": 1, "context": prompt_len, "ms_per_step": b / steps, "tok_s": steps / b * 1e3}}


# ------------------------------------------------------------------------------------------ kernels
class Timer:
    def __init__(self, dev):
        self.flush = torch.empty(256 << 20, dtype=torch.uint8, device=dev)
        p = os.path.join(os.path.dirname(os.path.dirname(os.path.abspath(__file__))), "MEASURED_PEAKS.json")
        peaks = json.load(open(p)) if os.path.exists(p) else {"hbm_gbs": 6650.0, "bf16_tflops": 1590.0}
        self.hbm, self.tc = peaks["hbm_gbs"] * 1e9, peaks["bf16_tflops"] * 1e12

    def us(self, fn, n: int = 12) -> float:
        for _ in range(3):
            fn()
        ts = []
        for _ in range(n):
            self.flush.zero_()
            torch.cuda._sleep(600_000)             # the host gets ahead of the device: launch cost stays out
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            torch.cuda.synchronize()
            ts.append(a.elapsed_time(b) * 1e3)
        return sorted(ts)[len(ts) // 2]

    def row(self, fn, nbytes: float = 0.0, flops: float = 0.0) -> dict:
        """The roof is the slower of moving the bytes and doing the tensor-core operations."""
        t = self.us(fn)
        roof = max(nbytes / self.hbm, flops / self.tc) * 1e6
        return {"us": round(t, 1), "roof_us": round(roof, 2), "of_measured": round(roof / t, 3)}


def kernels(s: dict, dev) -> dict:
    """{kernel: {"decode" (64 rows): [new, like], "prefill" (8192 rows): [new, like]}}"""
    tm = Timer(dev)
    w, h, kv, ff = s["width"], s["heads"], s["kv"], s["ff"]
    choices = s["experts"] + s["identity"]
    bf = lambda *sh: torch.randn(*sh, device=dev).to(torch.bfloat16)
    ones = torch.ones(w, dtype=torch.bfloat16, device=dev)
    out: dict = {}

    def put(name, phase, new, like):
        out.setdefault(name, {})[phase] = {"new": new, "like": like}

    for phase, t in (("decode", 64), ("prefill", 8192)):
        x, y = torch.randn(t, w, device=dev), bf(t, w)
        kw = dict(dim=w, eps=1e-6, layernorm=True, dtype=torch.bfloat16)
        put("residual_norm / norm", phase, tm.row(lambda: ops.residual_norm(x, y, ones, ones, **kw), t * w * (4 + 4 + 2 + 2)),
            tm.row(lambda: ops.norm(y, ones, residual=y), t * w * 8))
        rw, bias = ops.LinearWeight(bf(choices, w)), torch.zeros(choices, device=dev)
        put("router / linear + moe_route", phase, tm.row(lambda: ops.router(y, rw, bias, s["top"]), t * w * 2 + choices * w * 2, 2.0 * t * w * choices),
            tm.row(lambda: ops.moe_route(ops.linear(y, rw), bias, s["top"]), t * w * 2 + choices * w * 2, 2.0 * t * w * choices))
        rows = t * s["top"]
        gu = bf(rows, 2 * ff)
        put("glu_clamped / glu", phase, tm.row(lambda: ops.glu_clamped(gu, 7.0, 1.702), rows * ff * 6), tm.row(lambda: ops.glu(gu), rows * ff * 6))
        # attention: 64 sequences of 2048 tokens at decode, four whole prompts of 2048 at prefill
        seqs, ctx = (64, 2048) if phase == "decode" else (4, 2048)
        per = ctx // 16
        kc, vc = bf(seqs * per, kv, 16, D), bf(seqs * per, kv, 16, D)
        table = torch.randperm(seqs * per, device=dev).to(torch.int32).reshape(seqs, per)
        lens = torch.full((seqs,), ctx, dtype=torch.int32, device=dev)
        q, gate = bf(t, h * D), bf(t, h * D)
        dist, sinks = torch.randn(h, 513, device=dev), torch.zeros(h, device=dev)
        cu = None if phase == "decode" else torch.arange(0, t + 1, ctx, dtype=torch.int32, device=dev)
        ql = 1 if phase == "decode" else ctx
        seen = sum(min(i + 1, WINDOW) for i in range(ctx - ql, ctx)) * seqs            # (query, key) pairs per head
        kvb = seqs * (min(ctx, WINDOW) if phase == "decode" else ctx) * kv * D * 2
        io = t * h * D * 2
        put("attn_biased / attn", phase,
            tm.row(lambda: ops.attn_biased(q, kc, None, table, lens, cu, heads=h, max_q_len=ql, max_kv_len=ctx, scale=0.1, softcap=30.0,
                                           window=WINDOW, dist_bias=dist, sinks=sinks, gate=gate), kvb + 3 * io, 4.0 * seen * h * D),
            tm.row((lambda: ops.attn_decode(q.view(t, h, D), kc, vc, table, lens, window=WINDOW, max_kv_len=ctx)) if phase == "decode" else
                   (lambda: ops.attn_prefill_paged(q.view(t, h, D), kc, vc, table, lens, cu, ql, window=WINDOW)), 2 * kvb + 2 * io, 4.0 * seen * h * D))
        slots = torch.randperm(seqs * ctx, device=dev)[:t].contiguous()
        qkv, pos = bf(t, (h + 2 * kv) * D), torch.arange(t, dtype=torch.int32, device=dev)
        put("kv_store / rope_kv", phase, tm.row(lambda: ops.kv_store(qkv[:, h * D:(h + kv) * D], kc, slots), t * kv * D * 4),
            tm.row(lambda: ops.rope_kv(qkv, pos, h, kv, D, k_cache=kc, v_cache=vc, slot_mapping=slots), t * (h + 2 * kv) * D * 4))
        # delta rule against the state-space scan with as many state values per token (d_state 16: 8 x the channels)
        ch = 3 * h * D
        dw = ops.DeltaWeights(conv=torch.randn(4, ch, device=dev), decay_rate=torch.ones(h, device=dev), dt_bias=torch.zeros(h * D, device=dev),
                              norm=torch.ones(D, dtype=torch.bfloat16, device=dev), heads=h, kv_heads=h, dk=D, dv=D, dk_true=D, dv_true=D, eps=1e-6)
        nseq = 64 if phase == "decode" else 4
        cs, st = torch.zeros(nseq, 3, ch, dtype=torch.bfloat16, device=dev), torch.zeros(nseq, h, D, D, device=dev)
        proj, z = bf(t, ch + h), bf(t, 2 * h * D)
        p0 = torch.full((t,), 5, dtype=torch.int32, device=dev)
        sl = torch.arange(nseq, dtype=torch.int32, device=dev)
        traffic = t * (ch + 3 * h * D) * 2 + nseq * h * D * D * 8
        new = tm.row(lambda: ops.delta_mix(proj, z, dw, cs, st, p0, cu, sl, ch), traffic)
        c, ns, steps = h * D * D // 16, 16, (1 if phase == "decode" else t)
        xs, dts = bf(steps, c), torch.rand(steps, c, device=dev)
        a, b, cc, dd = -torch.rand(c, ns, device=dev), torch.randn(steps, ns, device=dev), torch.randn(steps, ns, device=dev), torch.ones(c, device=dev)
        h0 = torch.zeros(c, ns, device=dev)
        try:
            like = tm.row(lambda: ops.selective_scan(xs, dts, a, b, cc, dd, h0), steps * c * 8 + c * ns * 12)
        except Exception as e:            # keep the table when the comparison does not take these sizes
            like = {"unavailable": f"{type(e).__name__}: {e}"}
        put("delta_mix / selective_scan", phase, new, like)
    return out


def run(args, device, sampler) -> dict:
    torch.manual_seed(0)
    res: dict = {}
    steps, warm = args.steps, max(args.warmup, 3)
    sampler.start()
    headline = None
    for name, s in SIZES.items():
        r = res[name] = {"size": {**s, "head_dim": D, "window": WINDOW}}
        for kind, cfg in (("lududra", lududra_cfg(s)), ("attention_moe", attention_moe_cfg(s))):
            model = DecoderModel(cfg, device)
            model.random_init(seed=0)
            for b in (64, 8, 1):
                r[f"{kind} b{b}"] = serve(model, b, 2048, steps, warm)
            if kind == "lududra" and headline is None:
                headline = r["lududra b64"]["decode"]
            del model
            torch.cuda.empty_cache()
        m = qwen35_model(s, device)
        r["qwen3_5 b1"] = serve_qwen35(m, 128, 8)
        del m
        torch.cuda.empty_cache()
        r["kernels"] = kernels(s, device)
        torch.cuda.empty_cache()
    N.check_status(device)
    return {"metric": "decode tok/s (Lududra layers, bf16, 64 x 2048-token contexts)", "value": headline["tok_s"], "unit": "tokens/s", "n_gpus": 1,
            "steps": steps, "warmup": warm, "ms_per_step": headline["ms_per_step"], "higher_is_better": True, "scaling": "strong",
            "vs_baseline": None, "dtype": "bf16", "data": "synthetic: random-init weights, uniform-random prompt token ids",
            "config": {"model": "lududra 2k", "global_batch": 64, "seq_len": 2048, "parallelism": "tp1", "kv_page": 16,
                       "l2": "model steps: weights + state >> 126 MB; kernels: L2 flushed before every launch"},
            "e2e": {"value": headline["e2e_tok_s"], "unit": "tokens/s", "ms_per_step": headline["e2e_ms_per_step"],
                    "h2d_bytes_per_step": headline["h2d"], "d2h_bytes_per_step": headline["d2h"]},
            "gpu_launches": headline["launches"] * steps, "clocks": sampler.stop(), "sizes": res}
