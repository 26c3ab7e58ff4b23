"""Ops of layers around a 32-bit residual stream: the stream's norms, attention with a distance bias and
sinks, the gated delta rule, and routed experts with pass-through outputs.

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
                  layernorm: bool, dtype: torch.dtype, out: Optional[torch.Tensor] = None) -> Optional[torch.Tensor]:
    """In place on the fp32 stream ``x`` [T, ld]: ``x += norm(y) * w_b`` (``y`` a tensor, :class:`RoutedRows`
    or None), then returns ``norm(x) * w_n`` in ``dtype`` (None without ``w_n``). One launch."""
    rows, ld = x.shape
    routed = y if isinstance(y, RoutedRows) else None
    if not x.is_cuda:
        def nrm(v, w):
            v = v[:, :dim]
            r, _ = R.norm(v, w, eps=eps, layernorm=layernorm)
            return r
        if y is not None:
            v = routed.combined() if routed is not None else y.float()
            x[:, :dim] += nrm(v, w_b) if w_b is not None else v[:, :dim]
        if w_n is None:
            return None
        h = torch.zeros(rows, ld, dtype=dtype) if out is None else out
        h[:, :dim] = nrm(x, w_n).to(dtype)
        return h
    assert x.dtype == torch.float32 and x.stride(1) == 1
    h = None
    if w_n is not None:
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
        float(eps), 1 if dtype == torch.float32 else 0, N.stream())
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
