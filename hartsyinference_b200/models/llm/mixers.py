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
from .config import DenseSpec, LayerSpec, MixerSpec, MoeConfig
from .rope import Rotary


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


def batch_parts(batch) -> list[tuple]:
    """A batch as parts that one kernel form each takes best: (rows, sequences, their ``cu_q`` or None), the runs ahead of the
    one-token runs that end a ragged batch (decoded tokens beside prompts), and those as a decode batch."""
    whole = slice(None)
    runs = None if batch.is_decode else getattr(batch, "runs", None)
    if not runs:
        return [(whole, whole, None if batch.is_decode else batch.cu_q)]
    n = len(runs)
    while n and runs[n - 1][0] == 1:
        n -= 1
    if n == len(runs):
        return [(whole, whole, batch.cu_q)]
    t = sum(r[0] for r in runs[:n])
    return ([(slice(0, t), slice(0, n), batch.cu_q[:n + 1])] if n else []) + [(slice(t, None), slice(n, None), None)]


def out_matrix(o: Optional[torch.Tensor], heads: int, v: int, vp: int, width: int, device) -> Optional[LinearWeight]:
    """A mixer's output matrix in its laid-out sizes; None when the layer holds it (:class:`ParallelBlock`)."""
    return None if o is None else _linear([pad_rows(pad_head_cols(o, heads, v, vp), pad_to(width, 8))], device)


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
    """Grouped-query attention over the page pool with a norm of q and of k (over all heads at once or per head), a rotation,
    a distance bias (a table or a slope per head), a window with kept first tokens, a score cap, a sink and an output gate (per
    value or per head), each as the spec says. One projection GEMM (q | k | v | gate). Without ``k`` and ``v`` it reads the
    pages of another layer (``spec.kv_from``), which come before it in the same pass."""

    def __init__(self, spec: MixerSpec, width: int, device, *, q: torch.Tensor, k: Optional[torch.Tensor] = None, v: Optional[torch.Tensor] = None,
                 o: Optional[torch.Tensor], q_bias: Optional[torch.Tensor] = None, k_bias: Optional[torch.Tensor] = None,
                 gate: Optional[torch.Tensor] = None, rel: Optional[torch.Tensor] = None, q_norm: Optional[torch.Tensor] = None,
                 k_norm: Optional[torch.Tensor] = None, eps: float = 0.0):
        self.spec, self.eps = spec, eps
        borrowed = spec.kv_from is not None
        self.shared_kv, self.gated = v is None and not borrowed, gate is not None
        hq, hk, d, dv = spec.heads, spec.kv_heads, spec.dim, spec.dim if self.shared_kv else spec.vdim
        if max(d, dv) > 512:
            raise ValueError(f"attention heads of {d} / {dv} values are not supported (at most 512)")
        if borrowed != (k is None) or (borrowed and (v is not None or k_norm is not None)):
            raise ValueError("attention: keys and values are a layer's own or another layer's")
        self.d, self.dv = dp, vp = pad_to(d, 8), pad_to(dv, 8)
        wp = pad_to(width, 8)
        head = lambda t, n: pad_head_rows(t, n, d, dp)
        vhead = lambda t, n: pad_head_rows(t, n, dv, vp)
        parts = [head(q, hq)] + ([head(k, hk)] if k is not None else []) + ([vhead(v, hk)] if v is not None else [])
        if gate is not None:
            parts.append(pad_rows(gate, pad_to(hq, 8)) if spec.head_gate else vhead(gate, hq))
        bias = None
        if q_bias is not None:
            rest = sum(p.shape[0] for p in parts[2:])
            bias = torch.cat([head(q_bias, hq), head(k_bias, hk), torch.zeros(rest, dtype=q_bias.dtype, device=q_bias.device)])
        self.proj = _linear([pad_cols(p, wp) for p in parts], device, bias)
        self.o = out_matrix(o, hq, dv, vp, width, device)
        self.nq, self.nk, self.nv = hq * dp, 0 if borrowed else hk * dp, 0 if borrowed or self.shared_kv else hk * vp
        self.inner = hq * vp                       # columns of what :meth:`values` returns
        norm = lambda t, n: None if t is None else head(t, n).to(torch.bfloat16).to(device).contiguous()
        self.q_norm, self.k_norm = (norm(t, 1 if spec.head_norm else n) for t, n in ((q_norm, hq), (k_norm, hk)))
        self.rotary = None if spec.rot is None else Rotary(spec.rot, device)
        if self.shared_kv and (self.rotary is not None or q_norm is not None):
            raise ValueError("attention: keys that are values are neither normed nor turned")
        self.bias = distance_bias_table(rel, spec.bias_reach, spec.window).to(device) if rel is not None and spec.bias_reach > 0 else None
        self.slopes = None
        if spec.slope_bias:
            self.slopes = torch.tensor([2.0 ** (-8.0 * (h + 1) / hq) for h in range(hq)], dtype=torch.float32, device=device)
        self.sinks = None if spec.sink is None else torch.full((hq,), float(spec.sink), dtype=torch.float32, device=device)
        self.scale = spec.scale or d ** -0.5
        if not borrowed:
            self.cache_shape = self._cache_shape

    def nbytes(self) -> int:
        return self.proj.nbytes() + (0 if self.o is None else self.o.nbytes())

    def _cache_shape(self, pages: int, page: int) -> tuple:
        """[planes, pages, kv heads, page, head size], or, with values of another size than the keys, all key pages and
        then all value pages in one row."""
        hk = self.spec.kv_heads
        if self.shared_kv or self.d == self.dv:
            return ((1 if self.shared_kv else 2), pages, hk, page, self.d)
        return (pages, hk * page * (self.d + self.dv))

    def _planes(self, cache: torch.Tensor) -> tuple[torch.Tensor, Optional[torch.Tensor]]:
        if cache.dim() > 2:
            return cache[0], None if self.shared_kv else cache[1]
        pages, hk = cache.shape[0], self.spec.kv_heads
        page = cache.shape[1] // (hk * (self.d + self.dv))
        n = pages * hk * page * self.d
        flat = cache.view(-1)
        return flat[:n].view(pages, hk, page, self.d), flat[n:].view(pages, hk, page, self.dv)

    def values(self, h: torch.Tensor, batch, li: int, model, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Gated head outputs [T, heads * value size], before the output product."""
        spec = self.spec
        p = ops.linear_act(h, self.proj)
        k0, v0 = self.nq, self.nq + self.nk
        g0 = v0 + self.nv
        kc, vc = self._planes(model.kv_cache[li if spec.kv_from is None else spec.kv_from])
        if self.rotary is not None or self.q_norm is not None:
            q = ops.qk_rope_store(p, spec.heads, kc, vc, batch.slot_mapping, table=None if self.rotary is None else self.rotary.table(batch),
                                  interleaved=self.rotary is not None and self.rotary.spec.interleaved, q_norm=self.q_norm, k_norm=self.k_norm,
                                  d_true=spec.dim, eps=self.eps, per_head=spec.head_norm, store=spec.kv_from is None)
        else:
            q = p[:, :k0]
            if self.shared_kv or self.d == self.dv:
                ops.kv_store(p[:, k0:v0], kc, batch.slot_mapping, None if self.shared_kv else p[:, v0:g0], vc)
            else:
                ops.kv_store(p[:, k0:v0], kc, batch.slot_mapping)
                ops.kv_store(p[:, v0:g0], vc, batch.slot_mapping)
        if out is None:
            out = torch.empty(h.shape[0], self.inner, dtype=h.dtype, device=h.device)
        for rows, seqs, cu in batch_parts(batch):
            ops.attn_biased(q[rows], kc, vc, batch.block_table[seqs], batch.kv_lens[seqs], cu, heads=spec.heads, max_q_len=batch.max_q_len,
                            max_kv_len=batch.max_kv_len, scale=self.scale, softcap=spec.softcap, window=spec.window, dist_bias=self.bias,
                            sinks=self.sinks, gate=p[rows, g0:] if self.gated else None, keep_first=spec.keep_first, slopes=self.slopes,
                            head_gate=spec.head_gate, out=out[rows])
        return out

    def __call__(self, h: torch.Tensor, batch, li: int, model) -> torch.Tensor:
        return ops.linear_act(self.values(h, batch, li, model), self.o)


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


class GeneralDeltaMixer:
    """Delta rule whose removal has a rate of its own per key channel: ``S = diag(w) S - (a u)(u^T S) + k v^T`` with the unit
    key u, read by r, normed per head, weighted and gated. Two GEMMs before the recurrence: every projection of h at once
    (r | k | removal rate | v | gate | low-rank decay, the last with tanh in its epilogue), then the decay's expansion."""

    def __init__(self, spec: MixerSpec, width: int, eps: float, device, *, r, k, v, a, a_bias, g, w1, w2, w0, norm, o):
        self.spec = spec
        h, d = spec.heads, spec.dim
        if d > 256:
            raise ValueError(f"general_delta heads of {d} values are not supported (at most 256)")
        dp, vp, wp = pad_to(d, 32), pad_to(d, 8), pad_to(width, 8)
        rank = pad_to(w1.shape[0], 8)
        key, val = (lambda t: pad_head_rows(t, h, d, dp)), (lambda t: pad_head_rows(t, h, d, vp))
        self.low = 3 * h * dp + 2 * h * vp
        self.proj = _linear([pad_cols(p, wp) for p in (key(r), key(k), key(a), val(v), val(g), pad_rows(w1, rank))], device)
        self.up = _linear([pad_cols(key(w2), rank)], device)
        self.o = out_matrix(o, h, d, vp, width, device)
        self.inner = h * vp
        f32 = lambda t: t.float().to(device).contiguous()
        self.w = ops.GeneralDeltaWeights(decay_bias=f32(key(w0)), rate_bias=f32(key(a_bias)), norm=val(norm).to(torch.bfloat16).to(device).contiguous(),
                                         heads=h, dk=dp, dv=vp, d_true=d, eps=eps)

    def nbytes(self) -> int:
        return self.proj.nbytes() + self.up.nbytes() + (0 if self.o is None else self.o.nbytes())

    def state_shapes(self, slots: int) -> tuple[Optional[tuple], tuple]:
        w = self.w
        return None, (slots, w.heads, w.dk, w.dv)

    def values(self, h: torch.Tensor, batch, li: int, model, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        p = ops.linear_act(h, self.proj, "tanh", act_from=self.low)
        z = ops.linear_act(p[:, self.low:], self.up)
        if out is None:
            out = torch.empty(h.shape[0], self.inner, dtype=h.dtype, device=h.device)
        for rows, seqs, cu in batch_parts(batch):
            ops.general_delta(p[rows], z[rows], self.w, model.mixer_state[li][1], batch.positions[rows], cu, batch.state_slots[seqs], out=out[rows],
                              runs=batch.runs[seqs] if cu is not None and batch.runs else None)
        return out

    def __call__(self, h: torch.Tensor, batch, li: int, model) -> torch.Tensor:
        return ops.linear_act(self.values(h, batch, li, model), self.o)


class ChannelScanMixer:
    """Selective scan (one decay per channel and state value): projection, short convolution, a second projection
    of the convolved inputs for step size, B and C, scan with the output gate in its epilogue."""

    def __init__(self, spec: MixerSpec, width: int, device, *, w_in, conv, conv_bias, x, dt, dt_bias, a_log, d, o):
        self.spec = spec
        c, n, r = spec.inner, spec.state, spec.rank
        self.n = next((s for s in (8, 16, 32, 64, 128) if s >= n), 0)
        if not self.n:
            raise ValueError(f"channel_scan with {n} state values per channel is not supported (at most 128)")
        cp, wp, self.rp = pad_to(c, 8), pad_to(width, 8), pad_to(r, 8)
        self.c = cp
        f32 = lambda t: t.float().to(device).contiguous()
        self.proj = _linear([pad_cols(pad_head_rows(w_in, 2, c, cp), wp)], device)
        self.low = _linear([pad_cols(pad_rows(p, k), cp) for p, k in ((x[:r], self.rp), (x[r:r + n], self.n), (x[r + n:], self.n))], device)
        self.dt = _linear([pad_cols(pad_rows(dt, cp), self.rp)], device)
        self.o = _linear([pad_rows(pad_cols(o, cp), wp)], device)
        self.conv, self.conv_bias = f32(pad_rows(conv, cp).t()), f32(pad_rows(conv_bias, cp))
        a = torch.zeros(cp, self.n, device=device)
        a[:c, :n] = -torch.exp(a_log.float().to(device))
        self.w = ops.ChannelScanWeights(a=a, dt_bias=f32(pad_rows(dt_bias, cp)), d=f32(pad_rows(d, cp)))

    def nbytes(self) -> int:
        return sum(w.nbytes() for w in (self.proj, self.low, self.dt, self.o))

    def state_shapes(self, slots: int) -> tuple[tuple, tuple]:
        return (slots, self.conv.shape[0] - 1, self.c), (slots, self.c, self.n)

    def __call__(self, h: torch.Tensor, batch, li: int, model) -> torch.Tensor:
        p = ops.linear_act(h, self.proj)
        conv, state = model.mixer_state[li]
        cu = None if batch.is_decode else batch.cu_q
        x = ops.short_conv(p[:, :self.c], self.conv, self.conv_bias, conv, batch.positions, cu, batch.state_slots)
        low = ops.linear_act(x, self.low)
        dt = ops.linear_act(low[:, :self.rp], self.dt)
        y = ops.channel_scan(x, dt, low, self.rp, self.rp + self.n, p[:, self.c:], self.w, state, batch.positions, cu, batch.state_slots)
        return ops.linear_act(y, self.o)


class HeadScanMixer:
    """State-space mixer with one decay per head and a matrix state: projection (z | x | B | C | step size), short
    convolution over x | B | C, scan, gate, RMS norm in equal parts."""

    def __init__(self, spec: MixerSpec, width: int, eps: float, device, *, w_in, conv, conv_bias, dt_bias, a_log, d, norm, o):
        self.spec, self.eps = spec, eps
        h, v, n, g = spec.heads, spec.vdim, spec.state, spec.groups
        np_ = next((s for s in (8, 16, 32, 64, 128, 256) if s >= n), 0)
        vp, wp = pad_to(v, 8), pad_to(width, 8)
        if not np_ or vp > 512:
            raise ValueError(f"head_scan states of {n} x {v} are not supported (at most 256 x 512)")
        if h % g or h * v % spec.norm_groups:
            raise ValueError(f"head_scan: {h} heads do not divide over {g} groups, or {h * v} channels over {spec.norm_groups} norm groups")
        f32 = lambda t: t.float().to(device).contiguous()
        inner, gn = h * v, g * n
        z, x, b, c, dt = w_in.split([inner, inner, gn, gn, h])
        head, grp = (lambda t: pad_head_rows(t, h, v, vp)), (lambda t: pad_head_rows(t, g, n, np_))
        self.proj = _linear([pad_cols(p, wp) for p in (head(z), head(x), grp(b), grp(c), pad_rows(dt, pad_to(h, 8)))], device)
        self.inner, self.channels = h * vp, h * vp + 2 * g * np_
        xbc = lambda t: torch.cat([head(t[:inner]), grp(t[inner:inner + gn]), grp(t[inner + gn:])])
        self.conv, self.conv_bias = f32(xbc(conv).t()), f32(xbc(conv_bias))
        self.norm = head(norm).to(torch.bfloat16).to(device).contiguous()
        self.o = _linear([pad_rows(pad_head_cols(o, h, v, vp), wp)], device)
        self.w = ops.HeadScanWeights(rate=f32(a_log.float().exp()), dt_bias=f32(dt_bias), d=f32(d), heads=h, groups=g, n=np_, p=vp)

    def nbytes(self) -> int:
        return self.proj.nbytes() + self.o.nbytes()

    def state_shapes(self, slots: int) -> tuple[tuple, tuple]:
        return (slots, self.conv.shape[0] - 1, self.channels), (slots, self.w.heads, self.w.n, self.w.p)

    def __call__(self, h: torch.Tensor, batch, li: int, model) -> torch.Tensor:
        p = ops.linear_act(h, self.proj)
        conv, state = model.mixer_state[li]
        cu = None if batch.is_decode else batch.cu_q
        i, s = self.inner, self.spec
        x = ops.short_conv(p[:, i:i + self.channels], self.conv, self.conv_bias, conv, batch.positions, cu, batch.state_slots)
        y = ops.head_scan(x, p[:, i + self.channels:i + self.channels + s.heads], self.w, state, batch.positions, cu, batch.state_slots,
                          batch.runs if cu is not None else None)
        y = ops.gated_norm(y, p[:, :i], self.norm, s.norm_groups, self.eps, s.heads, s.vdim)
        return ops.linear_act(y, self.o)


# ragged batches: runs of at least this many query tokens expand keys and values of their context once; shorter
# ones attend in latent space
_EXPAND_RUN = 48
# most context tokens whose keys and values are held at once
_EXPAND_TOKENS = 65536


class LatentPlan:
    """How a ragged batch is split for latent attention: groups of long runs with the part of their contexts that a
    window leaves, and the rows of the short ones. The index arrays go to the device in one copy."""

    def __init__(self, batch, expand: bool, window: int = 0):
        runs = batch.runs
        if runs is None:
            cu, kv = batch.cu_q.tolist(), batch.kv_lens.tolist()
            runs = [(b - a, n) for a, b, n in zip(cu, cu[1:], kv)]
        starts, t = [], 0
        for q, _ in runs:
            starts.append(t)
            t += q
        # first key that a run's first query sees, and keys from there on
        first = [max(0, kv - q - window + 1) if window > 0 else 0 for q, kv in runs]
        keys = [kv - f for (_, kv), f in zip(runs, first)]
        long = [i for i, (q, _) in enumerate(runs) if expand and q >= _EXPAND_RUN]
        groups: list[list[int]] = []
        for i in long:
            if not groups or sum(keys[j] for j in groups[-1]) + keys[i] > _EXPAND_TOKENS:
                groups.append([])
            groups[-1].append(i)
        flat: list[int] = []

        def put(values) -> slice:
            a = len(flat)
            flat.extend(values)
            flat.extend([0] * (-len(flat) % 4))          # every array starts on 16 bytes
            return slice(a, a + len(values))

        rows: list[tuple[int, int, int]] = []
        skip = set(long)
        for i, (q, kv) in enumerate(runs):
            if i not in skip:
                rows += [(starts[i] + j, i, kv - q + j + 1) for j in range(q)]
        at = []
        for g in groups:
            off = [0]
            for i in g:
                off.append(off[-1] + keys[i])
            at.append((put(g), put(off), put([starts[i] for i in g]), put([runs[i][0] for i in g]), put([keys[i] for i in g]),
                       put([first[i] for i in g])))
        r = [put([x[k] for x in rows]) for k in range(3)]
        dev = torch.tensor(flat, dtype=torch.int32).to(batch.tokens.device)
        self.groups = [dict(seqs=dev[a], offsets=dev[b], q_start=dev[c], q_lens=dev[d], kv_lens=dev[e], first=dev[f],
                            total=sum(keys[i] for i in g), max_kv=max(keys[i] for i in g), max_q=max(runs[i][0] for i in g))
                       for g, (a, b, c, d, e, f) in zip(groups, at)]
        # rows None: every row of the batch, in order
        self.short = len(rows)
        self.rows = dev[r[0]] if groups else None
        self.row_seq, self.row_len = dev[r[1]], dev[r[2]]


class LatentAttention:
    """Attention whose keys and values are per-head maps of one cached latent; queries through a latent of their
    own. Optional: a rotated part of queries and keys (one rotated key for all heads, cached behind the latent), a
    window, a sink per head, a sigmoid output gate (per value or per head). One projection GEMM (query latent | latent |
    rotated key | gate). The kernels turn pairs of neighbours; for a rotation of split halves the rotated rows of both
    projections are put in that order, which leaves the scores as they are."""

    def __init__(self, spec: MixerSpec, width: int, eps: float, device, *, dq, dq_norm, uq, dkv, dkv_norm, uk, uv, o, g=None, sinks=None):
        self.spec, self.eps = spec, eps
        h, d, v, t = spec.heads, spec.dim, spec.vdim, spec.rot_dim
        if spec.kv_rank > 512:
            raise ValueError(f"latent_attention with a latent of {spec.kv_rank} values is not supported (at most 512)")
        if t % 2 or t > 512 or bool(t) != (spec.rot is not None):
            raise ValueError(f"latent_attention with a rotated part of {t} values is not supported (even, at most 512, with its rotation)")
        if t and not spec.rot.interleaved:
            pairs = torch.arange(t).reshape(2, t // 2).t().reshape(-1).to(uq.device)
            uq = torch.cat([uq.reshape(h, d + t, -1)[:, :d], uq.reshape(h, d + t, -1)[:, d:][:, pairs]], 1).reshape(h * (d + t), -1)
            dkv = torch.cat([dkv[:spec.kv_rank], dkv[spec.kv_rank:][pairs.to(dkv.device)]])
        wp = pad_to(width, 8)
        self.d, self.v, self.t = dp, vp, tp = pad_to(d, 8), pad_to(v, 8), pad_to(t, 8)
        self.qr, self.r = qr, r = pad_to(spec.q_rank, 8), pad_to(spec.kv_rank, 8)
        head = lambda m, k, kp: pad_head_rows(m, h, k, kp)
        parts = [pad_rows(dq, qr), pad_rows(dkv[:spec.kv_rank], r)] + ([pad_rows(dkv[spec.kv_rank:], tp)] if t else [])
        if g is not None:
            parts.append(pad_rows(g, pad_to(h, 8)) if spec.head_gate else head(g, v, vp))
        self.proj = _linear([pad_cols(p, wp) for p in parts], device)
        self.gated = g is not None
        self.sinks = None if sinks is None else sinks.float().to(device).contiguous()
        vec = lambda m, n: pad_rows(m, n).to(torch.bfloat16).to(device).contiguous()
        self.q_norm, self.kv_norm = vec(dq_norm, qr), vec(dkv_norm, r)
        if t:                                    # both parts of every head padded on their own
            uq = uq.reshape(h, d + t, -1)
            uq = torch.cat([pad_head_rows(uq[:, :d].reshape(h * d, -1), h, d, dp).reshape(h, dp, -1),
                            pad_head_rows(uq[:, d:].reshape(h * t, -1), h, t, tp).reshape(h, tp, -1)], 1).reshape(h * (dp + tp), -1)
        else:
            uq = head(uq, d, dp)
        self.uq = _linear([pad_cols(uq, qr)], device)
        uk, uv = pad_cols(head(uk, d, dp), r), pad_cols(head(uv, v, vp), r)
        self.kv_up = _linear([uk, uv], device)
        self.uv = LinearWeight(self.kv_up.weight[h * dp:])
        self.uk_t = _linear([uk.reshape(h, dp, r).transpose(1, 2).reshape(h * r, dp)], device)     # the query's side of W_uk
        self.o = out_matrix(o, h, v, vp, width, device)
        self.inner = h * vp
        self.scale = spec.scale or (d + t) ** -0.5
        self.rotary = None if spec.rot is None else Rotary(spec.rot, device)
        if self.rotary is not None and spec.rot.dims != t:
            raise ValueError("latent_attention turns the whole rotated part")

    def nbytes(self) -> int:
        return sum(w.nbytes() for w in (self.proj, self.uq, self.kv_up, self.uk_t, self.o) if w is not None)

    def cache_shape(self, pages: int, page: int) -> tuple:
        return (1, pages, 1, page, self.r + self.t)

    def _plan(self, batch, h: torch.Tensor) -> LatentPlan:
        expand = h.is_cuda and h.dtype == torch.bfloat16 and self.d + self.t <= 192 and self.v <= 128
        if batch.plan is None:
            batch.plan = {}
        key = (expand, self.spec.window)
        if key not in batch.plan:
            batch.plan[key] = LatentPlan(batch, *key)
        return batch.plan[key]

    def values(self, h: torch.Tensor, batch, li: int, model, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Gated head outputs [T, heads * value size], before the output product."""
        heads, window, r, head_gate = self.spec.heads, self.spec.window, self.r, self.spec.head_gate
        table = None if self.rotary is None else self.rotary.table(batch)
        p = ops.linear_act(h, self.proj)
        gate = p[:, self.qr + r + self.t:] if self.gated else None
        cache = model.kv_cache[li][0]
        cq = ops.latent_prep(p, 0, self.spec.q_rank, self.q_norm, self.qr, self.spec.kv_rank, self.kv_norm, cache, batch.slot_mapping, self.eps,
                             table)
        q = ops.linear_act(cq, self.uq)
        if batch.is_decode:
            a = ops.latent_attn(ops.head_linear(q, self.uk_t, heads, tail=self.t, table=table), cache, batch.block_table, batch.kv_lens, heads,
                                self.scale, max_kv_len=batch.max_kv_len, v_dim=r, window=window, sinks=self.sinks)
            return ops.head_linear(a, self.uv, heads, gate=gate, head_gate=head_gate, out=out)
        plan = self._plan(batch, h)
        y = torch.empty(h.shape[0], heads * self.v, dtype=h.dtype, device=h.device) if out is None else out
        for g in plan.groups:
            c = ops.latent_gather(cache, batch.block_table, g["seqs"], g["offsets"], g["total"], g["max_kv"], g["first"])
            kv = ops.linear_act(c[:, :r], self.kv_up)
            ops.attn_runs(q, kv[:, :heads * self.d], kv[:, heads * self.d:], y, g["q_start"], g["q_lens"], g["offsets"], g["kv_lens"],
                          heads=heads, max_q_len=g["max_q"], scale=self.scale, gate=gate, window=window,
                          k_shared=c[:, r:] if self.t else None, table=table, sinks=self.sinks, head_gate=head_gate)
        if plan.short:
            ql = ops.head_linear(q, self.uk_t, heads, in_rows=plan.rows, tail=self.t, table=table)
            a = ops.latent_attn(ql, cache, batch.block_table, plan.row_len, heads, self.scale, row_seq=plan.row_seq,
                                max_kv_len=batch.max_kv_len, v_dim=r, window=window, sinks=self.sinks)
            ops.head_linear(a, self.uv, heads, gate=gate, head_gate=head_gate, out=y, out_rows=plan.rows)
        return y

    def __call__(self, h: torch.Tensor, batch, li: int, model) -> torch.Tensor:
        return ops.linear_act(self.values(h, batch, li, model), self.o)


class DenseFeedForward:
    """Feed-forward ``down(act(up h))`` (``coef``: the activation's numbers), or gated: ``down(silu(gate h) * up h)``.
    ``down`` None: the layer holds it (:class:`ParallelBlock`)."""

    def __init__(self, spec: DenseSpec, width: int, eps: float, device, *, up, down, coef=None, gate=None):
        if spec.act not in ("poly_norm", "relu2", "silu"):
            raise ValueError(f"unknown activation '{spec.act}'")
        self.spec, self.eps = spec, eps
        self.inner = fp = pad_to(spec.ffn, 8)
        wp = pad_to(width, 8)
        rows = [pad_rows(pad_cols(t, wp), fp) for t in (gate, up) if t is not None]
        if len(rows) != (2 if spec.act == "silu" else 1):
            raise ValueError(f"a feed-forward with activation '{spec.act}' has {'a' if spec.act == 'silu' else 'no'} gate")
        self.up = _linear(rows, device)
        self.down = None if down is None else _linear([pad_rows(pad_cols(down, fp), wp)], device)
        self.coef = None if coef is None else coef.float().to(device).contiguous()

    def nbytes(self) -> int:
        return self.up.nbytes() + (0 if self.down is None else self.down.nbytes())

    def values(self, h: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """The activation's output [T, inner], before the down product."""
        if self.spec.act == "relu2":
            return ops.linear_act(h, self.up, "relu2", out=out)
        if self.spec.act == "poly_norm":
            a = ops.poly_norm(ops.linear_act(h, self.up), self.coef, self.spec.ffn, self.eps)
        elif h.dtype == torch.float32:
            a = ops.glu_clamped(ops.linear_act(h, self.up), math.inf, 1.0, shift=0.0)
        else:
            a, _ = ops.glu(ops.linear(h, self.up, defer=h.is_cuda and h.shape[0] <= 128))
        return a if out is None else out.copy_(a)

    def __call__(self, h: torch.Tensor, model=None) -> torch.Tensor:
        return ops.linear_act(self.values(h), self.down)


class ParallelBlock:
    """Mixer and feed-forward of a layer that read the same norm and whose outputs are summed: both write what precedes
    their output product side by side into one buffer, and one product with the two output matrices side by side gives
    the sum, accumulated in 32 bits and rounded once."""

    def __init__(self, mixer, ffn: Optional[DenseFeedForward], width: int, device, *, o: torch.Tensor, down: Optional[torch.Tensor]):
        self.mixer, self.ffn = mixer, ffn
        heads = mixer.spec.heads
        vp = mixer.inner // heads
        parts = [pad_head_cols(o, heads, o.shape[1] // heads, vp).to(o.device)]
        if ffn is not None:
            parts.append(pad_cols(down.to(o.device), ffn.inner))
        self.out = _linear([pad_rows(torch.cat(parts, 1), pad_to(width, 8))], device)
        for name in ("cache_shape", "state_shapes"):       # what the cache and the state manager ask a layer for
            if hasattr(mixer, name):
                setattr(self, name, getattr(mixer, name))

    def nbytes(self) -> int:
        return self.mixer.nbytes() + self.out.nbytes() + (0 if self.ffn is None else self.ffn.nbytes())

    def __call__(self, h: torch.Tensor, hf: Optional[torch.Tensor], batch, li: int, model) -> torch.Tensor:
        """``h`` goes to the mixer, ``hf`` to the feed-forward."""
        n = self.mixer.inner
        buf = torch.empty(h.shape[0], self.out.weight.shape[1], dtype=h.dtype, device=h.device)
        self.mixer.values(h, batch, li, model, out=buf[:, :n])
        if self.ffn is not None:
            self.ffn.values(hf, out=buf[:, n:])
        return ops.linear_act(buf, self.out)


class TokenInput:
    """What a layer adds from its part of a second token embedding: ``proj(gelu_tanh(gate x) * table[token])``; the
    norm of the sum's new term is the caller's. ``table`` [vocab, dim] is the layer's columns, padded to 8."""

    def __init__(self, dim: int, width: int, device, *, table: torch.Tensor, gate: torch.Tensor, proj: torch.Tensor):
        dp, wp = pad_to(dim, 8), pad_to(width, 8)
        self.table = table
        self.gate = _linear([pad_rows(pad_cols(gate, wp), dp)], device)
        self.proj = _linear([pad_rows(pad_cols(proj, dp), wp)], device)

    def nbytes(self) -> int:
        return self.gate.nbytes() + self.proj.nbytes() + self.table.numel() * self.table.element_size()

    def __call__(self, x: torch.Tensor, tokens: torch.Tensor) -> torch.Tensor:
        return ops.linear_act(ops.side_gate(ops.linear_act(x, self.gate), tokens, self.table), self.proj)


def build_experts(moe: MoeConfig, width: int, device, router: torch.Tensor, correction: Optional[torch.Tensor], experts, shared=None):
    """Stacked expert weights for the grouped GEMMs: per expert gate | up [2F, W] (up [F, W] for experts without a gate)
    and down [W, F] with F padded to 64 and W (as output) to 128. ``experts`` yields (gate or None, up, down);
    ``shared``: (up, down, sigmoid gate [1, W]) of an ungated shared expert, whose gate becomes the router's last row."""
    from .moe import MoeWeights
    wp, f, fp, wo = pad_to(width, 8), moe.expert_ffn, pad_to(moe.expert_ffn, 64), pad_to(width, 128)
    halves = 1 if moe.expert_act == "relu2" else 2
    if halves == 1:
        fp = pad_to(f, 128)                    # the up product's own rows are tiles of 128
    gu = torch.zeros(moe.num_experts, halves, fp, wp, dtype=torch.bfloat16, device=device)
    dn = torch.zeros(moe.num_experts, wo, fp, dtype=torch.bfloat16, device=device)
    for i, (g, u, d) in enumerate(experts):
        if halves == 2:
            gu[i, 0, :f, :width] = g.to(gu)
        gu[i, halves - 1, :f, :width] = u.to(gu)
        dn[i, :width, :f] = d.to(dn)
    w = MoeWeights(router=_linear([pad_cols(router, wp)] + ([] if shared is None else [pad_cols(shared[2], wp)]), device),
                   router_bias=None if correction is None else correction.float().to(device).contiguous(),
                   gate_up=LinearWeight(gu.reshape(moe.num_experts * halves * fp, wp)), down=LinearWeight(dn.reshape(moe.num_experts * wo, fp)))
    if shared is not None:
        sp = pad_to(shared[0].shape[0], 8)
        w.shared_gate_up = _linear([pad_rows(pad_cols(shared[0], wp), sp)], device)
        w.shared_down = _linear([pad_rows(pad_cols(shared[1], sp), wp)], device)
        w.gate_in_router = True
    return w


def spec_param_count(ls: LayerSpec, width: int) -> int:
    m = ls.mixer
    if m.kind == "latent_attention":
        n = width * (m.q_rank + m.kv_rank + m.rot_dim + m.heads * ((1 + m.out_gate) * m.vdim + m.head_gate))
        n += m.heads * (m.q_rank * (m.dim + m.rot_dim) + m.kv_rank * (m.dim + m.vdim))
    elif m.kind == "channel_scan":
        n = m.inner * (3 * width + 2 * m.rank + 3 * m.state + m.conv)
    elif m.kind == "head_scan":
        n = width * (3 * m.heads * m.vdim + 2 * m.groups * m.state + m.heads) + m.conv * (m.heads * m.vdim + 2 * m.groups * m.state)
    elif m.kind == "attention":
        v = m.dim if m.shared_kv else m.vdim
        own = 0 if m.kv_from is not None else m.kv_heads * (m.dim + (0 if m.shared_kv else v))
        n = width * (m.heads * (m.dim + (1 + m.out_gate) * v + m.head_gate) + own)
    elif m.kind == "general_delta":
        n = m.heads * m.dim * (6 * width + (m.rank or m.dim)) + (m.rank or m.dim) * width
    else:
        r = m.rank or m.dim
        n = width * (2 * m.kv_heads * m.dim + 2 * m.heads * m.vdim + m.heads + 2 * r) + r * m.heads * (m.dim + m.vdim)
    if ls.moe is not None:
        mats = 2 if ls.moe.expert_act == "relu2" else 3
        n += mats * width * (ls.moe.expert_ffn * ls.moe.num_experts + ls.moe.shared_ffn * ls.moe.num_shared_experts)
        n += width * (ls.moe.choices + ls.moe.shared_gate)
    if ls.dense is not None:
        n += (3 if ls.dense.act == "silu" else 2) * width * ls.dense.ffn
    return n + 4 * width
