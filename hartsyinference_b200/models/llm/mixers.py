"""Token mixers and expert weights of models whose layers are described one by one.

Every mixer is a callable ``(h [T, W], batch, layer, model) -> [T, W]`` (``LayerWeights.attn_module``) that
reads and writes the decoder's page pool or state slots through the batch. Activations are bf16, or fp32
for a model run in 32 bits (``DecoderModel(dtype=torch.float32)``); weights are bf16 in both.

Sizes are the checkpoint's. Where a kernel wants a multiple (GEMM rows of 16 bytes, delta-rule heads of 32
key channels, expert tiles of 128 features) the weights are padded with zero rows / columns here, once,
so that padded channels carry zeros through the layer; the constants that depend on a size (q scale,
output-norm mean) use the true one.
"""
from __future__ import annotations

import math
from typing import Iterable, Optional

import torch

from ... import ops
from ...ops import LinearWeight
from .config import LayerSpec, MixerSpec, MoeConfig


def pad_to(n: int, m: int) -> int:
    return (n + m - 1) // m * m


def pad_cols(w: torch.Tensor, cols: int) -> torch.Tensor:
    return w if w.shape[1] == cols else torch.nn.functional.pad(w, (0, cols - w.shape[1]))


def pad_rows(w: torch.Tensor, rows: int) -> torch.Tensor:
    if w.shape[0] == rows:
        return w
    return torch.cat([w, torch.zeros(rows - w.shape[0], *w.shape[1:], dtype=w.dtype, device=w.device)])


def pad_head_rows(w: torch.Tensor, heads: int, d: int, dp: int) -> torch.Tensor:
    """[heads * d, ...] -> [heads * dp, ...] with zero rows behind every head's d."""
    if d == dp:
        return w
    w = w.reshape(heads, d, *w.shape[1:])
    z = torch.zeros(heads, dp - d, *w.shape[2:], dtype=w.dtype, device=w.device)
    return torch.cat([w, z], 1).reshape(heads * dp, *w.shape[2:])


def pad_head_cols(w: torch.Tensor, heads: int, d: int, dp: int) -> torch.Tensor:
    return w if d == dp else pad_head_rows(w.t(), heads, d, dp).t()


def _linear(parts: Iterable[torch.Tensor], device, bias: Optional[torch.Tensor] = None) -> LinearWeight:
    w = torch.cat([p.to(torch.bfloat16).to(device) for p in parts]).contiguous()
    return LinearWeight(w, None, None if bias is None else bias.to(torch.bfloat16).to(device).contiguous())


def distance_bias_table(rel: torch.Tensor, reach: int, window: int) -> torch.Tensor:
    """Per-head bias by key distance, fp32 [heads, n]: distances below half of the table's rows have a row of
    their own, longer ones share rows on a logarithmic scale that ends at ``reach``. The table stops where
    every longer distance has the last row (or at the window's edge)."""
    rows = rel.shape[0]
    half = rows / 2
    n = max(reach + 1, rows)
    if window > 0:
        n = min(n, window)
    idx = []
    for d in range(n):
        if d < half:
            idx.append(d)
        else:
            step = math.floor(math.log(d / half) / math.log(reach / half) * (rows - half))
            idx.append(min(rows - 1, int(half + step)))
    return rel.float().cpu()[idx].t().contiguous()


class BiasedAttention:
    """Grouped-query attention over the page pool with a distance bias, a window, a score cap, a sink and an
    output gate, each as the spec says. One projection GEMM (q | k | v | gate)."""

    def __init__(self, spec: MixerSpec, width: int, device, *, q: torch.Tensor, k: torch.Tensor, v: Optional[torch.Tensor],
                 o: torch.Tensor, q_bias: Optional[torch.Tensor] = None, k_bias: Optional[torch.Tensor] = None,
                 gate: Optional[torch.Tensor] = None, rel: Optional[torch.Tensor] = None):
        self.spec = spec
        hq, hk, d = spec.heads, spec.kv_heads, spec.dim
        self.d = dp = pad_to(d, 8)
        wp = pad_to(width, 8)
        head = lambda t, n: pad_head_rows(t, n, d, dp)
        parts = [head(q, hq), head(k, hk)] + ([head(v, hk)] if v is not None else []) + ([head(gate, hq)] if gate is not None else [])
        bias = None
        if q_bias is not None:
            rest = sum(p.shape[0] for p in parts[2:])
            bias = torch.cat([head(q_bias, hq), head(k_bias, hk), torch.zeros(rest, dtype=q_bias.dtype, device=q_bias.device)])
        self.proj = _linear([pad_cols(p, wp) for p in parts], device, bias)
        self.o = _linear([pad_rows(pad_head_cols(o, hq, d, dp), wp)], device)
        self.nq, self.nk = hq * dp, hk * dp
        self.shared_kv, self.gated = v is None, gate is not None
        self.bias = distance_bias_table(rel, spec.bias_reach, spec.window).to(device) if rel is not None and spec.bias_reach > 0 else None
        self.sinks = None if spec.sink is None else torch.full((hq,), float(spec.sink), dtype=torch.float32, device=device)
        self.scale = spec.scale or d ** -0.5

    def nbytes(self) -> int:
        return self.proj.nbytes() + self.o.nbytes()

    def cache_shape(self, pages: int, page: int) -> tuple:
        return ((1 if self.shared_kv else 2), pages, self.spec.kv_heads, page, self.d)

    def __call__(self, h: torch.Tensor, batch, li: int, model) -> torch.Tensor:
        p = ops.linear_act(h, self.proj)
        k0, v0 = self.nq, self.nq + self.nk
        g0 = v0 if self.shared_kv else v0 + self.nk
        cache = model.kv_cache[li]
        kc, vc = cache[0], None if self.shared_kv else cache[1]
        ops.kv_store(p[:, k0:v0], kc, batch.slot_mapping, None if self.shared_kv else p[:, v0:g0], vc)
        a = ops.attn_biased(p[:, :k0], kc, vc, batch.block_table, batch.kv_lens, None if batch.is_decode else batch.cu_q,
                            heads=self.spec.heads, max_q_len=batch.max_q_len, max_kv_len=batch.max_kv_len, scale=self.scale,
                            softcap=self.spec.softcap, window=self.spec.window, dist_bias=self.bias, sinks=self.sinks,
                            gate=p[:, g0:] if self.gated else None)
        return ops.linear_act(a, self.o)


class DeltaMixer:
    """Gated delta rule with per-channel decay. Two GEMMs before the recurrence: every projection of h at
    once (q | k | v | step size | low-rank decay | low-rank gate), then both low-rank expansions as one
    block-diagonal product."""

    def __init__(self, spec: MixerSpec, width: int, eps: float, device, *, q, k, v, b, o, conv, a_log, dt_bias, norm, a1, a2, g1, g2):
        self.spec = spec
        h, hk, d, dv = spec.heads, spec.kv_heads, spec.dim, spec.vdim
        if d > 256 or dv > 1024:
            raise ValueError(f"channel_delta heads of {d} x {dv} are not supported (at most 256 x 1024)")
        dp, dvp, wp = pad_to(d, 32), pad_to(dv, 8), pad_to(width, 8)
        ra, rg = pad_to(a1.shape[0], 8), pad_to(g1.shape[0], 8)
        parts = [pad_head_rows(q, hk, d, dp), pad_head_rows(k, hk, d, dp), pad_head_rows(v, h, dv, dvp), pad_rows(b, pad_to(h, 8)),
                 pad_rows(a1, ra), pad_rows(g1, rg)]
        self.proj = _linear([pad_cols(p, wp) for p in parts], device)
        self.b_off = 2 * hk * dp + h * dvp
        self.low = slice(self.b_off + pad_to(h, 8), self.b_off + pad_to(h, 8) + ra + rg)
        up = torch.zeros(h * dp + h * dvp, ra + rg, dtype=torch.bfloat16, device=device)
        up[:h * dp, :a2.shape[1]] = pad_head_rows(a2, h, d, dp).to(up)
        up[h * dp:, ra:ra + g2.shape[1]] = pad_head_rows(g2, h, dv, dvp).to(up)
        self.up = LinearWeight(up)
        self.o = _linear([pad_rows(pad_head_cols(o, h, dv, dvp), wp)], device)
        f32 = lambda t: t.float().to(device).contiguous()
        taps = torch.cat([pad_head_rows(conv[0], hk, d, dp), pad_head_rows(conv[1], hk, d, dp), pad_head_rows(conv[2], h, dv, dvp)])
        self.w = ops.DeltaWeights(conv=f32(taps.t()), decay_rate=f32(a_log.float().exp()), dt_bias=f32(pad_head_rows(dt_bias, h, d, dp)),
                                  norm=torch.nn.functional.pad(norm, (0, dvp - dv)).to(torch.bfloat16).to(device).contiguous(),
                                  heads=h, kv_heads=hk, dk=dp, dv=dvp, dk_true=d, dv_true=dv, eps=eps)

    def nbytes(self) -> int:
        return self.proj.nbytes() + self.up.nbytes() + self.o.nbytes()

    def state_shapes(self, slots: int) -> tuple[tuple, tuple]:
        w = self.w
        return (slots, w.conv.shape[0] - 1, w.channels), (slots, w.heads, w.dk, w.dv)

    def __call__(self, h: torch.Tensor, batch, li: int, model) -> torch.Tensor:
        p = ops.linear_act(h, self.proj)
        z = ops.linear_act(p[:, self.low], self.up)
        conv, state = model.mixer_state[li]
        y = ops.delta_mix(p, z, self.w, conv, state, batch.positions, None if batch.is_decode else batch.cu_q, batch.state_slots,
                          self.b_off)
        return ops.linear_act(y, self.o)


def build_experts(moe: MoeConfig, width: int, device, router: torch.Tensor, correction: Optional[torch.Tensor], experts):
    """Stacked expert weights for the grouped GEMMs: per expert gate | up [2F, W] and down [W, F] with F padded
    to 64 and W (as output) to 128. ``experts`` yields (gate, up, down)."""
    from .moe import MoeWeights
    wp, f, fp, wo = pad_to(width, 8), moe.expert_ffn, pad_to(moe.expert_ffn, 64), pad_to(width, 128)
    gu = torch.zeros(moe.num_experts, 2, fp, wp, dtype=torch.bfloat16, device=device)
    dn = torch.zeros(moe.num_experts, wo, fp, dtype=torch.bfloat16, device=device)
    for i, (g, u, d) in enumerate(experts):
        gu[i, 0, :f, :width] = g.to(gu)
        gu[i, 1, :f, :width] = u.to(gu)
        dn[i, :width, :f] = d.to(dn)
    return MoeWeights(router=LinearWeight(pad_cols(router, wp).to(torch.bfloat16).to(device).contiguous()),
                      router_bias=None if correction is None else correction.float().to(device).contiguous(),
                      gate_up=LinearWeight(gu.reshape(moe.num_experts * 2 * fp, wp)), down=LinearWeight(dn.reshape(moe.num_experts * wo, fp)))


def spec_param_count(ls: LayerSpec, width: int) -> int:
    m = ls.mixer
    if m.kind == "attention":
        n = width * m.dim * (m.heads * (2 + m.out_gate) + m.kv_heads * (1 if m.shared_kv else 2))
    else:
        r = m.rank or m.dim
        n = width * (2 * m.kv_heads * m.dim + 2 * m.heads * m.vdim + m.heads + 2 * r) + r * m.heads * (m.dim + m.vdim)
    if ls.moe is not None:
        n += 3 * width * ls.moe.expert_ffn * ls.moe.num_experts + width * ls.moe.choices
    return n + 4 * width
