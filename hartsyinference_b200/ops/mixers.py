"""Ops of layers around a 32-bit residual stream: the stream's norms, attention with a distance bias and
sinks, latent attention, the gated delta rule, state-space scans, and routed experts with pass-through outputs.

Activations are bf16 (tensor-core products) or fp32 (a model run in 32 bits: plain FMA products); the
dtype of the input tensor picks the form. Same dispatch rule as the other ops: CUDA tensors go to the
kernels of ``libb200_kernels.so``, CPU tensors to the statements in :mod:`.reference`.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import _native as N
from . import reference as R
from .core import LinearWeight, linear


def _f32(t: torch.Tensor) -> int:
    assert t.dtype in (torch.float32, torch.bfloat16), t.dtype
    return 1 if t.dtype == torch.float32 else 0


def linear_act(x: torch.Tensor, w: LinearWeight) -> torch.Tensor:
    """x @ W^T (+ bias) in the dtype of ``x``: bf16 through the tensor-core GEMM, fp32 through 32-bit
    FMA tiles (the weight itself is bf16 in both)."""
    if x.dtype != torch.float32:
        return linear(x, w)
    if not x.is_cuda:
        return R.linear(x, w.host_f32(), bias=w.bias, out_dtype=torch.float32)
    m, k = x.shape
    n = w.weight.shape[0]
    assert w.weight.shape[1] == k and x.stride(1) == 1 and w.weight.stride(1) == 1 and not w.is_fp8
    out = torch.empty(m, n, dtype=torch.float32, device=x.device)
    N.check(N.lib().b200_linear_f32(x.data_ptr(), 1, w.weight.data_ptr(), N.ptr(w.bias), out.data_ptr(), m, n, k, x.stride(0),
                                    w.weight.stride(0), n, N.stream()), "b200_linear_f32")
    return out


def embedding_f32(ids: torch.Tensor, table: torch.Tensor, scale: float, dim: int) -> torch.Tensor:
    """fp32 rows ``table[ids] * scale``; columns from ``dim`` on (row padding) are zero."""
    if not table.is_cuda:
        x = table[ids.long()].float() * scale
        x[:, dim:] = 0
        return x
    t, ld = ids.numel(), table.shape[1]
    x = torch.empty(t, ld, dtype=torch.float32, device=table.device)
    N.check(N.lib().b200_embedding_f32(ids.data_ptr(), table.data_ptr(), x.data_ptr(), t, dim, ld, ld, table.shape[0],
                                       float(scale), N.stream()), "b200_embedding_f32")
    return x


@dataclass
class RoutedRows:
    """Expert outputs before they are combined: token t's value is the sum over its choices k of
    ``weights[t, k]`` times ``rows[slot_of[t, k]]`` (slot >= 0), ``source[t]`` (slot < 0 and expert index
    >= ``experts``: an expert that returns its input) or nothing."""
    rows: torch.Tensor
    slot_of: torch.Tensor
    ids: torch.Tensor
    weights: torch.Tensor
    source: Optional[torch.Tensor]
    experts: int

    def combined(self) -> torch.Tensor:
        """Plain statement of the sum (CPU tensors)."""
        t, k = self.ids.shape
        dim = self.source.shape[1] if self.source is not None else self.rows.shape[1]
        out = torch.zeros(t, dim, dtype=torch.float32)
        for j in range(k):
            s, w = self.slot_of[:, j].long(), self.weights[:, j, None]
            hit = s >= 0
            out[hit] += w[hit] * self.rows[s[hit], :dim].float()
            if self.source is not None:
                ident = ~hit & (self.ids[:, j] >= self.experts)
                out[ident] += w[ident] * self.source[ident].float()
        return out


def residual_norm(x: torch.Tensor, y, w_b: Optional[torch.Tensor], w_n: Optional[torch.Tensor], *, dim: int, eps: float,
                  layernorm: bool, dtype: torch.dtype, out: Optional[torch.Tensor] = None, plus_one: bool = False, mult: float = 1.0,
                  plain: bool = False) -> Optional[torch.Tensor]:
    """In place on the fp32 stream ``x`` [T, ld]: ``x += mult * norm(y) * w_b`` (``y`` a tensor, :class:`RoutedRows`
    or None), then returns ``norm(x) * w_n`` in ``dtype`` (without ``w_n``: the stream itself if ``plain``, else
    None). ``plus_one``: the norms multiply by 1 + w. One launch."""
    rows, ld = x.shape
    routed = y if isinstance(y, RoutedRows) else None
    if not x.is_cuda:
        def nrm(v, w):
            v = v[:, :dim]
            r, _ = R.norm(v, w.float() + 1 if plus_one else w, eps=eps, layernorm=layernorm)
            return r
        if y is not None:
            v = routed.combined() if routed is not None else y.float()
            x[:, :dim] += mult * (nrm(v, w_b) if w_b is not None else v[:, :dim])
        if w_n is None and not plain:
            return None
        h = torch.zeros(rows, ld, dtype=dtype) if out is None else out
        h[:, :dim] = (nrm(x, w_n) if w_n is not None else x[:, :dim]).to(dtype)
        return h
    assert x.dtype == torch.float32 and x.stride(1) == 1
    h = None
    if w_n is not None or plain:
        h = torch.empty(rows, ld, dtype=dtype, device=x.device) if out is None else out
        assert h.dtype == dtype and h.is_contiguous()
    yt = routed.rows if routed is not None else y
    src = routed.source if routed is not None else None
    assert yt is None or (yt.dtype == dtype and yt.stride(1) == 1)
    rc = N.lib().b200_residual_norm(
        x.data_ptr(), N.ptr(yt), N.ptr(h), N.ptr(w_b), N.ptr(w_n),
        N.ptr(routed.slot_of) if routed is not None else None, N.ptr(routed.ids) if routed is not None else None,
        N.ptr(routed.weights) if routed is not None else None, N.ptr(src), rows, dim, x.stride(0),
        yt.stride(0) if yt is not None else 0, ld, src.stride(0) if src is not None else 0,
        routed.ids.shape[1] if routed is not None else 0, routed.experts if routed is not None else 0, int(layernorm),
        int(plus_one), int(plain), float(eps), float(mult), 1 if dtype == torch.float32 else 0, N.stream())
    N.check(rc, "b200_residual_norm")
    return h


def router(x: torch.Tensor, w: LinearWeight, bias: Optional[torch.Tensor], top_k: int, *, sigmoid: bool = False,
           norm_topk: bool = False, scale: float = 1.0) -> tuple[torch.Tensor, torch.Tensor]:
    """Router logits, scores and choice in 32 bits: (expert ids int32 [T, k], weights fp32 [T, k]).
    Experts are chosen by score + ``bias``; the weights are the scores (optionally renormalised)."""
    if not x.is_cuda:
        return R.moe_route(x.float() @ w.host_f32().t(), bias, top_k, 1, 1, sigmoid, norm_topk, scale)
    t, k = x.shape
    e = w.weight.shape[0]
    assert x.stride(1) == 1 and w.weight.shape[1] == k
    ids = torch.empty(t, top_k, dtype=torch.int32, device=x.device)
    wts = torch.empty(t, top_k, dtype=torch.float32, device=x.device)
    rc = N.lib().b200_router(x.data_ptr(), _f32(x), w.weight.data_ptr(), N.ptr(bias), ids.data_ptr(), wts.data_ptr(), t, e, k,
                             x.stride(0), w.weight.stride(0), top_k, 1 if sigmoid else 0, 1 if norm_topk else 0, float(scale),
                             N.stream())
    N.check(rc, "b200_router")
    return ids, wts


def glu_clamped(x: torch.Tensor, limit: float, alpha: float, plan=None) -> torch.Tensor:
    """[rows, 2F] = gate | up -> g sigmoid(alpha g) (u + 1) with g = min(gate, limit), u = clamp(up, +-limit).
    With a dispatch plan only the rows of its blocks in use are computed (device)."""
    rows, f2 = x.shape
    if not x.is_cuda:
        return R.glu_clamped(x, limit, alpha).to(x.dtype)
    assert x.is_contiguous()
    y = torch.empty(rows, f2 // 2, dtype=x.dtype, device=x.device)
    rc = N.lib().b200_glu_clamped(x.data_ptr(), y.data_ptr(), rows, f2 // 2, float(limit), float(alpha),
                                  N.ptr(plan.dyn_blocks) if plan is not None else None, plan.cap if plan is not None else 0,
                                  _f32(x), N.stream())
    N.check(rc, "b200_glu_clamped")
    return y


def pair_linear_f32(x: torch.Tensor, w: LinearWeight, ids: torch.Tensor, experts: int, per_row: int) -> torch.Tensor:
    """fp32 rows ``x[pair // per_row] @ W[ids[pair]]^T`` of a stacked weight [experts * N, K]; rows of pairs
    whose index is not below ``experts`` are left unset."""
    pairs, k = ids.numel(), w.weight.shape[1]
    n = w.weight.shape[0] // experts
    out = torch.empty(pairs, n, dtype=torch.float32, device=x.device)
    if not x.is_cuda:
        wf = w.host_f32().reshape(experts, n, k)
        for p, e in enumerate(ids.reshape(-1).tolist()):
            if 0 <= e < experts:
                out[p] = wf[e] @ x[p // per_row].float()
        return out
    assert x.dtype == torch.float32 and x.stride(1) == 1 and x.shape[1] == k and w.weight.is_contiguous()
    rc = N.lib().b200_pair_linear_f32(x.data_ptr(), w.weight.data_ptr(), ids.data_ptr(), out.data_ptr(), pairs, per_row, experts,
                                      n, k, x.stride(0), n, N.stream())
    N.check(rc, "b200_pair_linear_f32")
    return out


def kv_store(k: torch.Tensor, k_cache: torch.Tensor, slots: torch.Tensor, v: Optional[torch.Tensor] = None,
             v_cache: Optional[torch.Tensor] = None) -> None:
    """Write key (and value) rows [T, hkv * d] (any row pitch) into pages [pages, hkv, page, d]; slot =
    page index * page + offset, negative slots are skipped."""
    _, hkv, page, d = k_cache.shape
    t = k.shape[0]
    if not k.is_cuda:
        ok = slots >= 0
        pg, off = (slots[ok] // page).long(), (slots[ok] % page).long()
        k_cache[pg, :, off] = k.reshape(t, hkv, d)[ok].to(k_cache.dtype)
        if v is not None:
            v_cache[pg, :, off] = v.reshape(t, hkv, d)[ok].to(v_cache.dtype)
        return
    assert slots.dtype == torch.int64 and k.dtype == k_cache.dtype and k.stride(1) == 1
    assert v is None or v.stride(0) == k.stride(0)
    rc = N.lib().b200_kv_store(k.data_ptr(), N.ptr(v), k_cache.data_ptr(), N.ptr(v_cache), slots.data_ptr(), t, hkv, d, page,
                               k.stride(0), k.element_size(), N.stream())
    N.check(rc, "b200_kv_store")


def attn_biased(q: torch.Tensor, k_cache: torch.Tensor, v_cache: Optional[torch.Tensor], block_table: torch.Tensor,
                kv_lens: torch.Tensor, cu_q: Optional[torch.Tensor], *, heads: int, max_q_len: int = 1, max_kv_len: int = 0,
                scale: float = 1.0, softcap: float = 0.0, window: int = 0, dist_bias: Optional[torch.Tensor] = None,
                sinks: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention over pages with, each optional, a per-head bias by key distance (``dist_bias``
    [heads, n], its last entry also stands for longer distances), a sink score per head that only enters
    the softmax denominator, and a sigmoid ``gate`` [T, heads * d] on the output. ``q`` [T, heads * d] (any
    row pitch); ``v_cache`` None: the values are the keys; ``cu_q`` None: one query token per sequence."""
    t = q.shape[0]
    _, hkv, page, d = k_cache.shape
    seqs = kv_lens.numel()
    if not q.is_cuda:
        out = torch.empty(t, heads * d, dtype=q.dtype)
        bounds = list(range(seqs + 1)) if cu_q is None else cu_q.tolist()
        for i in range(seqs):
            a, b, ln = bounds[i], bounds[i + 1], int(kv_lens[i])
            kk = R.gather_paged(k_cache, block_table[i], ln)
            vv = kk if v_cache is None else R.gather_paged(v_cache, block_table[i], ln)
            o = R.attention(q[a:b].reshape(b - a, heads, d), kk, vv, causal=True, scale=scale, softcap=softcap, window=window,
                            sinks=sinks, dist_bias=dist_bias).reshape(b - a, heads * d)
            if gate is not None:
                o = o * torch.sigmoid(gate[a:b].float())
            out[a:b] = o.to(q.dtype)
        return out
    assert block_table.dtype == torch.int32 and kv_lens.dtype == torch.int32 and q.stride(1) == 1
    assert dist_bias is None or (dist_bias.dtype == torch.float32 and dist_bias.is_contiguous())
    assert gate is None or gate.stride(1) == 1
    L = N.lib()
    f32 = _f32(q)
    exact = 1 if f32 or d > 128 or page > 64 or (cu_q is None and heads // hkv > 16) else 0
    splits, ws = 1, None
    if cu_q is None and not exact:
        dd = 64 if d <= 64 else 128
        mk = max_kv_len or block_table.shape[1] * page
        if window > 0:
            mk = min(mk, window + 63)
        splits = L.b200_attn_decode_pick_splits(seqs, hkv, mk)
        if splits > 1:
            ws = N.state(q.device).scratch(L.b200_attn_decode_workspace_bytes(seqs, heads, dd, splits)).data_ptr()
    out = torch.empty(t, heads * d, dtype=q.dtype, device=q.device)
    rc = L.b200_attn_biased(q.data_ptr(), k_cache.data_ptr(), N.ptr(v_cache), out.data_ptr(), block_table.data_ptr(),
                            kv_lens.data_ptr(), N.ptr(cu_q), t, seqs, max_q_len, heads, hkv, d, page, block_table.shape[1],
                            splits, ws, float(scale), float(softcap), int(window), N.ptr(dist_bias),
                            dist_bias.shape[1] if dist_bias is not None else 0, N.ptr(sinks), N.ptr(gate),
                            gate.stride(0) if gate is not None else 0, q.stride(0), exact, f32, N.stream())
    N.check(rc, "b200_attn_biased", 2 if splits > 1 else 1)
    return out


@dataclass
class DeltaWeights:
    """Constants of one delta-rule mixer. ``dk`` / ``dv`` are the head sizes as laid out (padded with zero
    channels), ``dk_true`` / ``dv_true`` the model's."""
    conv: torch.Tensor         # fp32 [taps, channels], channels = q heads | k heads | v heads
    decay_rate: torch.Tensor   # fp32 [heads], exp(A_log)
    dt_bias: torch.Tensor      # fp32 [heads * dk]
    norm: torch.Tensor         # bf16 [dv]
    heads: int
    kv_heads: int
    dk: int
    dv: int
    dk_true: int
    dv_true: int
    eps: float

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dk + self.heads * self.dv


def delta_mix(proj: torch.Tensor, z: torch.Tensor, w: DeltaWeights, conv_state: torch.Tensor, state: torch.Tensor,
              positions: torch.Tensor, cu_q: Optional[torch.Tensor], slots: torch.Tensor, b_off: int) -> torch.Tensor:
    """The gated delta rule between its projections. ``proj`` [T, ld] = q | k | v | ... with the step-size
    logits at column ``b_off``; ``z`` [T, heads * dk + heads * dv] = decay logits | output gate logits.
    ``conv_state`` [slots, taps - 1, channels] and ``state`` fp32 [slots, heads, dk, dv] are updated in place;
    a sequence whose first position is 0 starts from zeros, slot -1 is not stored. Returns [T, heads * dv]."""
    t = proj.shape[0]
    seqs = slots.numel()
    if not proj.is_cuda:
        return R.delta_mix(proj, z, w, conv_state, state, positions, cu_q, slots, b_off)
    assert proj.dtype == z.dtype == conv_state.dtype and state.dtype == torch.float32
    assert slots.dtype == torch.int32 and positions.dtype == torch.int32 and proj.stride(1) == 1 and z.stride(1) == 1
    L = N.lib()
    taps = w.conv.shape[0]
    ws = torch.empty(L.b200_delta_workspace_bytes(t, w.heads, w.kv_heads, w.dk, w.dv), dtype=torch.uint8, device=proj.device)
    out = torch.empty(t, w.heads * w.dv, dtype=proj.dtype, device=proj.device)
    rc = L.b200_delta(proj.data_ptr(), z.data_ptr(), w.conv.data_ptr(), w.decay_rate.data_ptr(), w.dt_bias.data_ptr(),
                      conv_state.data_ptr(), state.data_ptr(), w.norm.data_ptr(), positions.data_ptr(), N.ptr(cu_q),
                      slots.data_ptr(), ws.data_ptr(), out.data_ptr(), t, seqs, w.heads, w.kv_heads, w.dk, w.dv, w.dk_true,
                      w.dv_true, taps, proj.stride(0), b_off, z.stride(0), w.heads * w.dk, float(w.eps), _f32(proj), N.stream())
    N.check(rc, "b200_delta", L.b200_delta_launches(1 if cu_q is None else 0, taps, w.dk, w.dv))
    return out


def embedding_norm(ids: Optional[torch.Tensor], table: torch.Tensor, w: torch.Tensor, *, dim: int, eps: float, layernorm: bool = False,
                   plus_one: bool = False, scale: float = 1.0, dtype: torch.dtype = torch.bfloat16) -> tuple[torch.Tensor, torch.Tensor]:
    """(x, h): the fp32 stream ``norm(table[ids] * scale) * w`` and the same rows in ``dtype``. ``ids`` None: all
    rows of ``table`` in order. Columns from ``dim`` on (row padding) are zero."""
    ld = (dim + 7) // 8 * 8
    t = table.shape[0] if ids is None else ids.numel()
    if not table.is_cuda:
        rows = (table if ids is None else table[ids.long()])[:, :dim].float() * scale
        x = torch.zeros(t, ld)
        x[:, :dim] = R.norm(rows, w.float() + 1 if plus_one else w, eps=eps, layernorm=layernorm)[0]
        return x, x.to(dtype)
    assert table.dtype == torch.bfloat16 and table.stride(1) == 1
    x = torch.empty(t, ld, dtype=torch.float32, device=table.device)
    h = torch.empty(t, ld, dtype=dtype, device=table.device)
    N.check(N.lib().b200_embedding_norm(N.ptr(ids), table.data_ptr(), w.data_ptr(), x.data_ptr(), h.data_ptr(), t, dim, ld,
                                        table.stride(0), table.shape[0], float(scale), int(layernorm), int(plus_one), float(eps),
                                        1 if dtype == torch.float32 else 0, N.stream()), "b200_embedding_norm")
    return x, h


def poly_norm(z: torch.Tensor, coef: torch.Tensor, dim: int, eps: float) -> torch.Tensor:
    """``a N(z) + b N(z^2) + c N(z^3) + e`` per row with ``coef`` = (a, b, c, e) fp32 and N the division by the root
    mean square of the row's first ``dim`` values; columns past ``dim`` are zero."""
    rows, ld = z.shape
    if not z.is_cuda:
        return R.poly_norm(z, coef, dim, eps).to(z.dtype)
    assert z.stride(1) == 1 and coef.dtype == torch.float32
    y = torch.empty(rows, (dim + 7) // 8 * 8, dtype=z.dtype, device=z.device)
    N.check(N.lib().b200_poly_norm(z.data_ptr(), y.data_ptr(), coef.data_ptr(), rows, dim, z.stride(0), y.stride(0), float(eps), _f32(z),
                                   N.stream()), "b200_poly_norm")
    return y


# ------------------------------------------------------------------------------------------ state-space mixers
def short_conv(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor], state: torch.Tensor, positions: torch.Tensor,
               cu_q: Optional[torch.Tensor], slots: torch.Tensor) -> torch.Tensor:
    """silu of a causal convolution per channel: ``x`` [T, C] (any row pitch), ``w`` fp32 [taps, C] (last row: the
    current token). ``state`` [slots, taps - 1, C] holds the inputs before each sequence's portion and is updated in
    place; a sequence whose first position is 0 starts from zeros, slot -1 is not stored."""
    t, c = x.shape
    if not x.is_cuda:
        return R.short_conv(x, w, bias, state, positions, cu_q, slots)
    assert x.stride(1) == 1 and w.dtype == torch.float32 and w.is_contiguous() and state.dtype == x.dtype and state.is_contiguous()
    assert slots.dtype == torch.int32 and positions.dtype == torch.int32
    out = torch.empty(t, c, dtype=x.dtype, device=x.device)
    taps = w.shape[0]
    N.check(N.lib().b200_short_conv(x.data_ptr(), w.data_ptr(), N.ptr(bias), state.data_ptr(), positions.data_ptr(), N.ptr(cu_q),
                                    slots.data_ptr(), out.data_ptr(), t, slots.numel(), c, taps, x.stride(0), _f32(x), N.stream()),
            "b200_short_conv", 2 if cu_q is not None and taps > 1 else 1)
    return out


@dataclass
class ChannelScanWeights:
    """Constants of a selective scan: ``a`` fp32 [C, N] (negative), ``dt_bias``, ``d`` fp32 [C]. N is one of 8, 16, 32,
    64, 128 (padded with zero columns)."""
    a: torch.Tensor
    dt_bias: torch.Tensor
    d: torch.Tensor


def channel_scan(x: torch.Tensor, dt: torch.Tensor, bc: torch.Tensor, b_off: int, c_off: int, z: torch.Tensor, w: ChannelScanWeights,
                 state: torch.Tensor, positions: torch.Tensor, cu_q: Optional[torch.Tensor], slots: torch.Tensor) -> torch.Tensor:
    """Scan with one decay per channel c and state value n, gated:
    ``S = exp(dt a[c, n]) S + dt x B[n]``, ``y = (sum_n S C[n] + d x) silu(z)``, ``dt = softplus(logit + bias)``.
    ``x``, ``dt`` (logits), ``z`` [T, C]; B and C are columns ``b_off``.. and ``c_off``.. of ``bc``. ``state`` fp32
    [slots, C, N] is updated in place (slots and first positions as in :func:`short_conv`)."""
    t, c = x.shape
    if not x.is_cuda:
        return R.channel_scan(x, dt, bc, b_off, c_off, z, w, state, positions, cu_q, slots)
    assert x.dtype == dt.dtype == bc.dtype == z.dtype and x.stride(1) == dt.stride(1) == bc.stride(1) == z.stride(1) == 1
    assert state.dtype == torch.float32 and state.is_contiguous() and slots.dtype == torch.int32 and positions.dtype == torch.int32
    y = torch.empty(t, c, dtype=x.dtype, device=x.device)
    rc = N.lib().b200_channel_scan(x.data_ptr(), dt.data_ptr(), bc.data_ptr(), z.data_ptr(), w.dt_bias.data_ptr(), w.a.data_ptr(),
                                   w.d.data_ptr(), state.data_ptr(), positions.data_ptr(), N.ptr(cu_q), slots.data_ptr(), y.data_ptr(),
                                   slots.numel(), c, w.a.shape[1], b_off, c_off, x.stride(0), dt.stride(0), bc.stride(0), z.stride(0),
                                   y.stride(0), _f32(x), N.stream())
    N.check(rc, "b200_channel_scan")
    return y


@dataclass
class HeadScanWeights:
    """Constants of a scan with one decay per head: fp32 [heads] ``rate`` = exp(A_log), ``dt_bias``, ``d``. ``n``
    (8, 16, ..., 256) and ``p`` (a multiple of 8) are the state's sizes as laid out (padded with zeros)."""
    rate: torch.Tensor
    dt_bias: torch.Tensor
    d: torch.Tensor
    heads: int
    groups: int
    n: int
    p: int


def head_scan(x: torch.Tensor, dt: torch.Tensor, w: HeadScanWeights, state: torch.Tensor, positions: torch.Tensor,
              cu_q: Optional[torch.Tensor], slots: torch.Tensor, runs: Optional[list] = None) -> torch.Tensor:
    """Scan with a matrix state [n, p] per head: ``S = exp(-rate dt) S + B (dt x)^T``, ``y = S^T C + d x``,
    ``dt = softplus(logit + bias)``. ``x`` [T, heads p + 2 groups n] = x | B | C (head h reads group
    h // (heads / groups)), ``dt`` logits [T, heads]. ``state`` fp32 [slots, heads, n, p] is updated in place.
    ``runs`` (host list of (tokens, ..) per sequence of a ragged batch) lets long bf16 runs go through the tensor cores.
    Returns [T, heads p]."""
    t = x.shape[0]
    if not x.is_cuda:
        return R.head_scan(x, dt, w, state, positions, cu_q, slots)
    assert x.dtype == dt.dtype and x.stride(1) == 1 and dt.stride(1) == 1 and state.dtype == torch.float32 and state.is_contiguous()
    assert slots.dtype == torch.int32 and positions.dtype == torch.int32
    hp = w.heads * w.p
    y = torch.empty(t, hp, dtype=x.dtype, device=x.device)
    rc = N.lib().b200_head_scan(x.data_ptr(), dt.data_ptr(), w.dt_bias.data_ptr(), w.rate.data_ptr(), w.d.data_ptr(), state.data_ptr(),
                                positions.data_ptr(), N.ptr(cu_q), slots.data_ptr(), y.data_ptr(), slots.numel(), w.heads, w.groups, w.n,
                                w.p, hp, hp + w.groups * w.n, x.stride(0), dt.stride(0), y.stride(0), max((r[0] for r in runs or ()), default=0),
                                min((r[0] for r in runs or ()), default=0), _f32(x), N.stream())
    N.check(rc, "b200_head_scan")
    return y


def gated_norm(y: torch.Tensor, z: torch.Tensor, weight: torch.Tensor, parts: int, eps: float, heads: int, p_true: int) -> torch.Tensor:
    """``norm(y silu(z)) weight`` with the norm taken over ``parts`` equal parts of the heads * p_true values of a row
    (heads may be laid out with zero columns behind them; those stay zero)."""
    t, cols = y.shape
    pp = cols // heads
    part = heads * p_true // parts
    if not y.is_cuda:
        return R.gated_norm(y, z, weight, parts, eps, heads, p_true).to(y.dtype)
    assert y.stride(1) == 1 and z.stride(1) == 1 and y.dtype == z.dtype and weight.dtype == torch.bfloat16
    out = (torch.empty if pp == p_true else torch.zeros)(t, cols, dtype=y.dtype, device=y.device)
    N.check(N.lib().b200_gated_norm(y.data_ptr(), z.data_ptr(), weight.data_ptr(), out.data_ptr(), t, parts, part, p_true, pp,
                                    y.stride(0), z.stride(0), out.stride(0), float(eps), _f32(y), N.stream()), "b200_gated_norm")
    return out


# ------------------------------------------------------------------------------------------ latent attention
def latent_prep(x: torch.Tensor, q_off: int, q_dim: int, wq: torch.Tensor, kv_off: int, kv_dim: int, wkv: torch.Tensor,
                cache: torch.Tensor, slots: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norms of the two latents in a projection's columns ``q_off``.. and ``kv_off``..: the query's is returned
    [T, len(wq)], the key / value one is written to ``cache`` [pages, 1, page, len(wkv)]. The weights are padded to
    the laid-out widths, ``q_dim`` / ``kv_dim`` are the true ones."""
    t = x.shape[0]
    if not x.is_cuda:
        def rms(v, w, dim):
            v = v[:, :dim].float()
            out = torch.zeros(t, w.numel())
            out[:, :dim] = v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * w[:dim].float()
            return out.to(x.dtype)
        kv_store(rms(x[:, kv_off:], wkv, kv_dim), cache, slots)
        return rms(x[:, q_off:], wq, q_dim)
    assert x.stride(1) == 1 and cache.dtype == x.dtype and cache.is_contiguous() and slots.dtype == torch.int64
    cq = torch.empty(t, wq.numel(), dtype=x.dtype, device=x.device)
    N.check(N.lib().b200_latent_prep(x.data_ptr(), wq.data_ptr(), wkv.data_ptr(), cq.data_ptr(), cache.data_ptr(), slots.data_ptr(), t,
                                     x.stride(0), q_off, q_dim, wq.numel(), kv_off, kv_dim, wkv.numel(), float(eps), _f32(x), N.stream()),
            "b200_latent_prep")
    return cq


def head_linear(x: torch.Tensor, w: LinearWeight, heads: int, *, gate: Optional[torch.Tensor] = None,
                in_rows: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
                out_rows: Optional[torch.Tensor] = None) -> torch.Tensor:
    """One product per head: ``out[r, h] = W[h] x[r, h]`` with ``w`` stacked [heads * n, k], ``x`` [rows, heads * k] and
    ``out`` [rows, heads * n], optionally times ``sigmoid(gate)``. ``in_rows`` / ``out_rows`` (int32) select the rows of
    ``x`` and of ``out`` and ``gate`` that the product's rows stand for."""
    n, k = w.weight.shape[0] // heads, w.weight.shape[1]
    rows = x.shape[0] if in_rows is None else in_rows.numel()
    rows = rows if out_rows is None else out_rows.numel()
    if out is None:
        out = torch.empty(rows, heads * n, dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        xi = (x if in_rows is None else x[in_rows.long()]).float().reshape(rows, heads, -1)[:, :, :k]
        y = torch.einsum("rhk,hnk->rhn", xi, w.host_f32().reshape(heads, n, k)).reshape(rows, heads * n)
        at = slice(None) if out_rows is None else out_rows.long()
        if gate is not None:
            y = y * torch.sigmoid(gate[at].float())
        out[at] = y.to(out.dtype)
        return out
    assert x.stride(1) == 1 and out.stride(1) == 1 and w.weight.is_contiguous() and out.dtype == x.dtype
    assert x.shape[1] == heads * k and out.shape[1] == heads * n and (gate is None or gate.stride(1) == 1)
    assert all(i is None or i.dtype == torch.int32 for i in (in_rows, out_rows))
    N.check(N.lib().b200_head_linear(x.data_ptr(), w.weight.data_ptr(), out.data_ptr(), N.ptr(gate), N.ptr(in_rows), N.ptr(out_rows), rows,
                                     heads, n, k, x.stride(0), k, out.stride(0), n, gate.stride(0) if gate is not None else 0, _f32(x),
                                     N.stream()), "b200_head_linear")
    return out


def latent_attn(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, kv_lens: torch.Tensor, heads: int, scale: float,
                row_seq: Optional[torch.Tensor] = None, max_kv_len: int = 0) -> torch.Tensor:
    """Attention of queries in latent space [rows, heads * rank] over cached latents [pages, 1, page, rank], which are
    keys and values of every head: row r sees the first ``kv_lens[r]`` tokens of block-table row ``row_seq[r]`` (r when
    None). bf16 rows of at most 512 values run on the tensor cores, fp32 and wider ones as plain 32-bit arithmetic.
    Returns [rows, heads * rank]."""
    rows, rank, page = q.shape[0], cache.shape[3], cache.shape[2]
    table = block_table
    if not q.is_cuda or q.dtype == torch.float32 or rank > 512:
        if row_seq is not None:
            table = block_table[row_seq.long()].contiguous()
        return attn_biased(q, cache, None, table, kv_lens, None, heads=heads, scale=scale)
    assert q.is_contiguous() and cache.is_contiguous() and kv_lens.dtype == torch.int32 and kv_lens.numel() == rows
    assert block_table.dtype == torch.int32 and (row_seq is None or row_seq.dtype == torch.int32)
    L = N.lib()
    out = torch.empty_like(q)
    step = 32768                            # rows are the grid's second dimension
    for a in range(0, rows, step):
        b = min(a + step, rows)
        splits = L.b200_mla_pick_splits(b - a, heads, int(max_kv_len or table.shape[1] * page))
        ws = None
        if splits > 1:
            ws = torch.empty(L.b200_mla_workspace_bytes(b - a, heads, splits), dtype=torch.uint8, device=q.device)
        tab = table if row_seq is not None else table[a:b]
        rc = L.b200_latent_attn(q[a:b].data_ptr(), cache.data_ptr(), out[a:b].data_ptr(), tab.data_ptr(), kv_lens[a:b].data_ptr(),
                                N.ptr(None if row_seq is None else row_seq[a:b]), b - a, heads, rank, page, table.stride(0), splits,
                                N.ptr(ws), float(scale), N.stream())
        N.check(rc, "b200_latent_attn", 2 if splits > 1 else 1)
    return out


def latent_gather(cache: torch.Tensor, block_table: torch.Tensor, seq_ids: torch.Tensor, offsets: torch.Tensor, total: int,
                  max_len: int) -> torch.Tensor:
    """Cached latents of the sequences in ``seq_ids``, one after another: rows ``offsets[s] .. offsets[s + 1]`` of the
    result [total, rank] are the tokens of block-table row ``seq_ids[s]``."""
    page, rank = cache.shape[2], cache.shape[3]
    out = torch.empty(total, rank, dtype=cache.dtype, device=cache.device)
    if not cache.is_cuda:
        for i, s in enumerate(seq_ids.tolist()):
            a, b = int(offsets[i]), int(offsets[i + 1])
            out[a:b] = R.gather_paged(cache, block_table[s], b - a).reshape(b - a, rank)
        return out
    N.check(N.lib().b200_latent_gather(cache.data_ptr(), out.data_ptr(), block_table.data_ptr(), seq_ids.data_ptr(), offsets.data_ptr(),
                                       seq_ids.numel(), max_len, rank * cache.element_size(), page, block_table.stride(0), N.stream()),
            "b200_latent_gather")
    return out


def attn_runs(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, out: torch.Tensor, q_start: torch.Tensor, q_lens: torch.Tensor,
              kv_start: torch.Tensor, kv_lens: torch.Tensor, *, heads: int, max_q_len: int, scale: float,
              gate: Optional[torch.Tensor] = None) -> None:
    """Causal attention of runs of query rows over contiguous keys and values of their contexts: run s is rows
    ``q_start[s]`` .. + ``q_lens[s]`` of ``q`` [T, heads * d], its context rows ``kv_start[s]`` .. + ``kv_lens[s]`` of ``k``
    [.., heads * d] and ``v`` [.., heads * dv]; the last key belongs to the last query. Rows of the runs are written to
    ``out`` [T, heads * dv], times ``sigmoid(gate)``. bf16, d and dv up to 128."""
    d, dv = k.shape[1] // heads, v.shape[1] // heads
    assert q.is_cuda and q.dtype == torch.bfloat16 and out.is_contiguous() and q.stride(1) == k.stride(1) == v.stride(1) == 1
    assert out.shape[1] == heads * dv and (gate is None or gate.stride(1) == 1)
    N.check(N.lib().b200_attn_runs(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), N.ptr(gate), q_start.data_ptr(),
                                   q_lens.data_ptr(), kv_start.data_ptr(), kv_lens.data_ptr(), q_lens.numel(), max_q_len, heads, heads, d,
                                   dv, q.stride(0), k.stride(0), v.stride(0), gate.stride(0) if gate is not None else 0, float(scale),
                                   N.stream()), "b200_attn_runs")
