"""Ops of layers around a 32-bit residual stream: the stream's norms, rotations, attention with a distance bias,
sinks, windows and kept first tokens, latent attention, the gated delta rule, state-space scans, and routed experts
with pass-through outputs.

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
from .core import _ACT, LinearWeight, act_code, linear


def _f32(t: torch.Tensor) -> int:
    assert t.dtype in (torch.float32, torch.bfloat16), t.dtype
    return 1 if t.dtype == torch.float32 else 0


def linear_act(x: torch.Tensor, w: LinearWeight, act: Optional[str] = None, act_from: int = 0,
               out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """act(x @ W^T (+ bias)) in the dtype of ``x``: bf16 through the tensor-core GEMM, fp32 through 32-bit
    FMA tiles (the weight itself is bf16 in both). ``act``: None, "relu2" (relu squared) or "tanh", for the output features
    from ``act_from`` on. ``out``: [M, N] of any row pitch."""
    if x.dtype != torch.float32:
        return linear(x, w, act, act_from=act_from, out=out)
    if not x.is_cuda:
        y = R.linear(x, w.host_f32(), bias=w.bias, act=act, out_dtype=torch.float32, act_from=act_from)
        return y if out is None else out.copy_(y)
    m, k = x.shape
    n = w.weight.shape[0]
    assert w.weight.shape[1] == k and x.stride(1) == 1 and w.weight.stride(1) == 1 and not w.is_fp8
    if out is None:
        out = torch.empty(m, n, dtype=torch.float32, device=x.device)
    assert out.shape == (m, n) and out.stride(1) == 1 and out.dtype == torch.float32
    N.check(N.lib().b200_linear_f32(x.data_ptr(), 1, w.weight.data_ptr(), N.ptr(w.bias), out.data_ptr(), m, n, k, x.stride(0),
                                    w.weight.stride(0), out.stride(0), act_code(act, act_from), N.stream()), "b200_linear_f32")
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
    extra: Optional[torch.Tensor] = None       # further rows [T, ..] (a shared expert) with one fp32 weight each
    extra_weight: Optional[torch.Tensor] = None

    def combined(self) -> torch.Tensor:
        """Plain statement of the sum (CPU tensors)."""
        t, k = self.ids.shape
        dim = self.source.shape[1] if self.source is not None else self.rows.shape[1]
        if self.extra is not None:
            dim = min(dim, self.extra.shape[1])
        out = torch.zeros(t, dim, dtype=torch.float32)
        for j in range(k):
            s, w = self.slot_of[:, j].long(), self.weights[:, j, None]
            hit = s >= 0
            out[hit] += w[hit] * self.rows[s[hit], :dim].float()
            if self.source is not None:
                ident = ~hit & (self.ids[:, j] >= self.experts)
                out[ident] += w[ident] * self.source[ident].float()
        if self.extra is not None:
            out += self.extra_weight[:, None] * self.extra[:, :dim].float()
        return out


@dataclass
class TanhNorm:
    """Norm without statistics: ``tanh(alpha x) * weight + bias`` (weight and bias bf16 [dim])."""
    alpha: float
    weight: torch.Tensor
    bias: torch.Tensor


def residual_norm(x: torch.Tensor, y, w_b: Optional[torch.Tensor], w_n, *, dim: int, eps: float,
                  layernorm: bool, dtype: torch.dtype, out: Optional[torch.Tensor] = None, plus_one: bool = False, mult: float = 1.0,
                  plain: bool = False, groups: int = 1, conv: Optional[tuple] = None) -> Optional[torch.Tensor]:
    """In place on the fp32 stream ``x`` [T, ld]: ``x += mult * norm(y) * w_b`` (``y`` a tensor, :class:`RoutedRows`
    or None), then returns ``norm(x) * w_n`` in ``dtype``, or :class:`TanhNorm` ``w_n`` of x (without ``w_n``: the
    stream itself if ``plain``, else None). ``plus_one``: the norms multiply by 1 + w. ``groups``: the norm on x is an RMS norm
    of that many equal parts, each on its own. ``conv`` = (w, state, positions, slots), one token per sequence: the result goes
    through :func:`input_conv` and is [n, T, ld]. One launch."""
    rows, ld = x.shape
    routed = y if isinstance(y, RoutedRows) else None
    tanh = w_n if isinstance(w_n, TanhNorm) else None
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
        if tanh is not None:
            h[:, :dim] = (torch.tanh(tanh.alpha * x[:, :dim]) * tanh.weight.float() + tanh.bias.float()).to(dtype)
        elif w_n is not None and groups > 1:
            part = x[:, :dim].reshape(rows * groups, dim // groups)
            part = part * torch.rsqrt(part.pow(2).mean(-1, keepdim=True) + eps)
            h[:, :dim] = (part.reshape(rows, dim) * (w_n.float() + 1 if plus_one else w_n.float())).to(dtype)
        else:
            h[:, :dim] = (nrm(x, w_n) if w_n is not None else x[:, :dim]).to(dtype)
        return h if conv is None else R.input_conv(h, conv[0], conv[1], conv[2], None, conv[3])
    assert x.dtype == torch.float32 and x.stride(1) == 1
    h = None
    if conv is not None:
        cw, cst, positions, slots = conv
        n, taps = cw.shape[:2]
        assert out is None and cw.dtype == torch.float32 and cw.is_contiguous() and cw.shape[2] == ld and cst.dtype == dtype
        assert cst.is_contiguous() and cst.shape[1:] == (taps - 1, ld) and slots.numel() == rows
        assert slots.dtype == torch.int32 and positions.dtype == torch.int32
        h = torch.empty(n, rows, ld, dtype=dtype, device=x.device)
    elif w_n is not None or plain:
        h = torch.empty(rows, ld, dtype=dtype, device=x.device) if out is None else out
        assert h.dtype == dtype and h.is_contiguous()
    yt = routed.rows if routed is not None else y
    src = routed.source if routed is not None else None
    extra = routed.extra if routed is not None else None
    assert extra is None or (extra.dtype == dtype and extra.stride(1) == 1 and routed.extra_weight.dtype == torch.float32)
    assert yt is None or (yt.dtype == dtype and yt.stride(1) == 1)
    rc = N.lib().b200_residual_norm(
        x.data_ptr(), N.ptr(yt), N.ptr(h), N.ptr(w_b), N.ptr(w_n if tanh is None else tanh.weight),
        N.ptr(routed.slot_of) if routed is not None else None, N.ptr(routed.ids) if routed is not None else None,
        N.ptr(routed.weights) if routed is not None else None, N.ptr(src), rows, dim, x.stride(0),
        yt.stride(0) if yt is not None else 0, ld, src.stride(0) if src is not None else 0,
        routed.ids.shape[1] if routed is not None else 0, routed.experts if routed is not None else 0, int(layernorm),
        int(plus_one), int(plain), float(eps), float(mult), 1 if dtype == torch.float32 else 0,
        N.ptr(None if tanh is None else tanh.bias), 0.0 if tanh is None else float(tanh.alpha), N.ptr(extra),
        N.ptr(routed.extra_weight) if extra is not None else None, extra.stride(0) if extra is not None else 0, int(groups),
        *((cw.data_ptr(), n, taps, cst.data_ptr(), positions.data_ptr(), slots.data_ptr()) if conv is not None else (None, 0, 0, None, None, None)),
        N.stream())
    N.check(rc, "b200_residual_norm")
    return h


def input_conv(h: torch.Tensor, w: torch.Tensor, state: torch.Tensor, positions: torch.Tensor, cu_q: Optional[torch.Tensor],
               slots: torch.Tensor, out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``h + conv_i(h)`` for every i: [n, T, C] (``out`` when given, any distance between its n matrices) from ``h`` [T, C] (any row pitch) and ``w`` fp32 [n, taps, C] (last row: the
    current token), causal over time per channel. ``state`` [slots, taps - 1, C] holds the inputs before each sequence's
    portion and is updated in place; a sequence whose first position is 0 starts from zeros, slot -1 is not stored."""
    t, c = h.shape
    if not h.is_cuda:
        y = R.input_conv(h, w, state, positions, cu_q, slots)
        return y if out is None else out.copy_(y)
    n, taps, _ = w.shape
    assert h.stride(1) == 1 and w.dtype == torch.float32 and w.is_contiguous() and w.shape[2] == c and state.dtype == h.dtype
    assert state.is_contiguous() and state.shape[1:] == (taps - 1, c) and slots.dtype == torch.int32 and positions.dtype == torch.int32
    if out is None:
        out = torch.empty(n, t, c, dtype=h.dtype, device=h.device)
    assert out.shape == (n, t, c) and out.stride(1) == c and out.stride(2) == 1 and out.dtype == h.dtype
    N.check(N.lib().b200_input_conv(h.data_ptr(), w.data_ptr(), state.data_ptr(), positions.data_ptr(), N.ptr(cu_q), slots.data_ptr(),
                                    out.data_ptr(), t, slots.numel(), c, taps, n, h.stride(0), out.stride(0), _f32(h), N.stream()),
            "b200_input_conv", 2 if cu_q is not None and taps > 1 else 1)
    return out


def cap_logits(y: torch.Tensor, scale: float, cap: float) -> torch.Tensor:
    """fp32 ``cap * tanh(y * scale / cap)`` (``cap`` 0: ``y * scale``)."""
    if not y.is_cuda:
        z = y.float() * scale
        return cap * torch.tanh(z / cap) if cap > 0 else z
    rows, n = y.shape
    assert y.is_contiguous()
    out = torch.empty(rows, n, dtype=torch.float32, device=y.device)
    N.check(N.lib().b200_cap_logits(y.data_ptr(), out.data_ptr(), y.numel(), float(scale), float(cap), _f32(y), N.stream()), "b200_cap_logits")
    return out


def side_gate(u: torch.Tensor, ids: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
    """``gelu_tanh(u) * table[ids]`` with ``u`` [T, n] and ``table`` [vocab, n] (any row pitch, bf16)."""
    t, n = u.shape
    if not u.is_cuda:
        return (R.gelu_tanh(u.float()) * table[ids.long()].float()).to(u.dtype)
    assert u.stride(1) == 1 and table.stride(1) == 1 and table.shape[1] == n and table.dtype == torch.bfloat16 and ids.dtype == torch.int32
    y = torch.empty(t, n, dtype=u.dtype, device=u.device)
    N.check(N.lib().b200_side_gate(u.data_ptr(), ids.data_ptr(), table.data_ptr(), y.data_ptr(), t, n, u.stride(0), table.stride(0),
                                   table.shape[0], _f32(u), N.stream()), "b200_side_gate")
    return y


def router(x: torch.Tensor, w: LinearWeight, bias: Optional[torch.Tensor], top_k: int, *, sigmoid: bool = False,
           norm_topk: bool = False, scale: float = 1.0, n_group: int = 1, topk_group: int = 1,
           gate: bool = False) -> tuple:
    """Router logits, scores and choice in 32 bits: (expert ids int32 [T, k], weights fp32 [T, k]).
    Experts are chosen by score + ``bias``, with ``n_group`` > 1 only among the ``topk_group`` groups of neighbours whose
    two best experts sum to most; the weights are the scores (optionally renormalised). ``gate``: the last row of ``w``
    is no expert; the sigmoid of its logit, fp32 [T], is returned as a third tensor."""
    e = w.weight.shape[0] - int(gate)
    if not x.is_cuda:
        lg = x.float() @ w.host_f32().t()
        got = R.moe_route(lg[:, :e], bias, top_k, n_group, topk_group, sigmoid, norm_topk, scale)
        return (*got, torch.sigmoid(lg[:, e])) if gate else got
    t, k = x.shape
    assert x.stride(1) == 1 and w.weight.shape[1] == k
    ids = torch.empty(t, top_k, dtype=torch.int32, device=x.device)
    wts = torch.empty(t, top_k, dtype=torch.float32, device=x.device)
    gt = torch.empty(t, dtype=torch.float32, device=x.device) if gate else None
    rc = N.lib().b200_router(x.data_ptr(), _f32(x), w.weight.data_ptr(), N.ptr(bias), ids.data_ptr(), wts.data_ptr(), t, e, k,
                             x.stride(0), w.weight.stride(0), top_k, 1 if sigmoid else 0, 1 if norm_topk else 0, float(scale),
                             n_group, topk_group, N.ptr(gt), N.stream())
    N.check(rc, "b200_router")
    return (ids, wts, gt) if gate else (ids, wts)


def glu_clamped(x: torch.Tensor, limit: float, alpha: float, plan=None, shift: float = 1.0) -> torch.Tensor:
    """[rows, 2F] = gate | up -> g sigmoid(alpha g) (u + shift) with g = min(gate, limit), u = clamp(up, +-limit).
    With a dispatch plan only the rows of its blocks in use are computed (device)."""
    rows, f2 = x.shape
    if not x.is_cuda:
        return R.glu_clamped(x, limit, alpha, shift).to(x.dtype)
    assert x.is_contiguous()
    y = torch.empty(rows, f2 // 2, dtype=x.dtype, device=x.device)
    rc = N.lib().b200_glu_clamped(x.data_ptr(), y.data_ptr(), rows, f2 // 2, float(limit), float(alpha), float(shift),
                                  N.ptr(plan.dyn_blocks) if plan is not None else None, plan.cap if plan is not None else 0,
                                  _f32(x), N.stream())
    N.check(rc, "b200_glu_clamped")
    return y


def pair_linear_f32(x: torch.Tensor, w: LinearWeight, ids: torch.Tensor, experts: int, per_row: int,
                    act: Optional[str] = None) -> torch.Tensor:
    """fp32 rows ``act(x[pair // per_row] @ W[ids[pair]]^T)`` (``act``: None or "relu2") of a stacked weight [experts * N, K]; rows of pairs
    whose index is not below ``experts`` are left unset."""
    pairs, k = ids.numel(), w.weight.shape[1]
    n = w.weight.shape[0] // experts
    out = torch.empty(pairs, n, dtype=torch.float32, device=x.device)
    if not x.is_cuda:
        wf = w.host_f32().reshape(experts, n, k)
        for p, e in enumerate(ids.reshape(-1).tolist()):
            if 0 <= e < experts:
                v = wf[e] @ x[p // per_row].float()
                out[p] = torch.relu(v) ** 2 if act == "relu2" else v
        return out
    assert x.dtype == torch.float32 and x.stride(1) == 1 and x.shape[1] == k and w.weight.is_contiguous()
    rc = N.lib().b200_pair_linear_f32(x.data_ptr(), w.weight.data_ptr(), ids.data_ptr(), out.data_ptr(), pairs, per_row, experts,
                                      n, k, x.stride(0), n, _ACT[act], N.stream())
    N.check(rc, "b200_pair_linear_f32")
    return out


def _gate_of(gate: torch.Tensor, heads: int, dv: int, head_gate: bool) -> torch.Tensor:
    """fp32 sigmoid of gate logits, one per value or (``head_gate``) the first ``heads`` columns, one per head."""
    g = torch.sigmoid(gate.float())
    return g[:, :heads].repeat_interleave(dv, 1) if head_gate else g


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
                sinks: Optional[torch.Tensor] = None, gate: Optional[torch.Tensor] = None, keep_first: int = 0,
                v_dim: int = 0, slopes: Optional[torch.Tensor] = None, head_gate: bool = False,
                out: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Causal attention over pages (with a ``window``: over the last ``window`` tokens and the ``keep_first`` first
    ones of the sequence) with, each optional, a per-head bias by key distance (``dist_bias``
    [heads, n], its last entry also stands for longer distances) or linear in it (``slopes`` fp32 [heads], taken off), a sink
    score per head that only enters the softmax denominator, and a sigmoid ``gate`` [T, heads * dv] (``head_gate``: one column
    per head) on the output. ``q`` [T, heads * d] (any
    row pitch); ``v_cache`` None: the values are the keys (their first ``v_dim`` columns when given); ``cu_q`` None:
    one query token per sequence. Returns [T, heads * dv] (``out`` when given, any row pitch)."""
    t = q.shape[0]
    _, hkv, page, d = k_cache.shape
    dv = v_cache.shape[3] if v_cache is not None else v_dim or d
    seqs = kv_lens.numel()
    if not q.is_cuda:
        out = torch.empty(t, heads * dv, dtype=q.dtype) if out is None else out
        bounds = list(range(seqs + 1)) if cu_q is None else cu_q.tolist()
        for i in range(seqs):
            a, b, ln = bounds[i], bounds[i + 1], int(kv_lens[i])
            kk = R.gather_paged(k_cache, block_table[i], ln)
            vv = kk[..., :dv] if v_cache is None else R.gather_paged(v_cache, block_table[i], ln)
            o = R.attention(q[a:b].reshape(b - a, heads, d), kk, vv, causal=True, scale=scale, softcap=softcap, window=window,
                            sinks=sinks, dist_bias=dist_bias, keep_first=keep_first, slopes=slopes).reshape(b - a, heads * dv)
            if gate is not None:
                o = o * _gate_of(gate[a:b], heads, dv, head_gate)
            out[a:b] = o.to(q.dtype)
        return out
    assert block_table.dtype == torch.int32 and kv_lens.dtype == torch.int32 and q.stride(1) == 1
    assert dist_bias is None or (dist_bias.dtype == torch.float32 and dist_bias.is_contiguous())
    assert gate is None or gate.stride(1) == 1
    assert slopes is None or (slopes.dtype == torch.float32 and dist_bias is None)
    L = N.lib()
    f32 = _f32(q)
    exact = 1 if f32 or max(d, dv) > 128 or (v_cache is None and dv != d) or page > 64 or (cu_q is None and heads // hkv > 16) else 0
    splits, ws = 1, None
    if cu_q is None and not exact:
        dd = 64 if max(d, dv) <= 64 else 128
        mk = max_kv_len or block_table.shape[1] * page
        if window > 0:
            mk = min(mk, window + 63 + (keep_first + 63) // 64 * 64)
        splits = L.b200_attn_decode_pick_splits(seqs, hkv, mk)
        if splits > 1:
            ws = N.state(q.device).scratch(L.b200_attn_decode_workspace_bytes(seqs, heads, dd, splits)).data_ptr()
    if out is None:
        out = torch.empty(t, heads * dv, dtype=q.dtype, device=q.device)
    assert out.shape == (t, heads * dv) and out.stride(1) == 1 and out.dtype == q.dtype
    rc = L.b200_attn_biased(q.data_ptr(), k_cache.data_ptr(), N.ptr(v_cache), out.data_ptr(), block_table.data_ptr(),
                            kv_lens.data_ptr(), N.ptr(cu_q), t, seqs, max_q_len, heads, hkv, d, dv, page, block_table.shape[1],
                            splits, ws, float(scale), float(softcap), int(window), int(keep_first), N.ptr(dist_bias),
                            dist_bias.shape[1] if dist_bias is not None else 0, N.ptr(sinks), N.ptr(gate),
                            gate.stride(0) if gate is not None else 0, q.stride(0), exact, f32, N.ptr(slopes), int(head_gate), out.stride(0),
                            N.stream())
    N.check(rc, "b200_attn_biased", 2 if splits > 1 else 1)
    return out


def rope_table(positions: torch.Tensor, hi: torch.Tensor, lo: torch.Tensor) -> torch.Tensor:
    """fp32 [T, n, 2] cosines and sines of ``position * (hi + lo)``: frequencies as sums of two floats, so that the
    angle keeps its precision far from the start."""
    if not positions.is_cuda:
        return R.rope_table(positions, hi, lo)
    t, n = positions.numel(), hi.numel()
    assert positions.dtype == torch.int32 and hi.dtype == lo.dtype == torch.float32
    out = torch.empty(t, n, 2, dtype=torch.float32, device=positions.device)
    N.check(N.lib().b200_rope_table(positions.data_ptr(), hi.data_ptr(), lo.data_ptr(), out.data_ptr(), t, n, N.stream()), "b200_rope_table")
    return out


def qk_rope_store(p: torch.Tensor, heads: int, k_cache: torch.Tensor, v_cache: torch.Tensor, slots: torch.Tensor, *,
                  table: Optional[torch.Tensor] = None, interleaved: bool = False, q_norm: Optional[torch.Tensor] = None,
                  k_norm: Optional[torch.Tensor] = None, d_true: int = 0, eps: float = 0.0, per_head: bool = False,
                  store: bool = True) -> torch.Tensor:
    """From a projection ``p`` [T, q | k | v] (any row pitch) to attention's inputs: RMS norm of q and of k over all their
    heads at once (``q_norm`` [heads * d], ``k_norm`` [hkv * d], or None) or, ``per_head``, of each head on its own (weights
    [d]), rotation of the first values of every q and k head
    by ``table`` (:func:`rope_table`, or None), k and v into the pages [pages, hkv, page, d] and [pages, hkv, page, dv].
    ``d_true``: the model's head size where heads are padded with zeros. ``store`` off: q only, ``p`` has no k and v.
    Returns q [T, heads * d]."""
    _, hkv, page, d = k_cache.shape
    dv = v_cache.shape[3]
    t, nq, nk = p.shape[0], heads * d, hkv * d
    dt = d_true or d
    if not p.is_cuda:
        def part(x, w, n):
            x = x.float()
            if w is not None and not per_head:
                x = x / torch.sqrt((x * x).sum(-1, keepdim=True) / (n * dt) + eps) * w.float()
            x = x.reshape(t, n, d)
            if w is not None and per_head:
                x = x / torch.sqrt((x * x).sum(-1, keepdim=True) / dt + eps) * w.float()
            return (x if table is None else R.turn(x, table, interleaved)).reshape(t, n * d).to(p.dtype)
        if store:
            kv_store(part(p[:, nq:nq + nk], k_norm, hkv), k_cache, slots)
            kv_store(p[:, nq + nk:nq + nk + hkv * dv], v_cache, slots)
        return part(p[:, :nq], q_norm, heads)
    assert p.stride(1) == 1 and slots.dtype == torch.int64 and k_cache.dtype == v_cache.dtype == p.dtype
    if per_head:
        assert q_norm.numel() == d and (not store or k_norm.numel() == d)
    else:
        assert store and (q_norm is None) == (k_norm is None) and (q_norm is None or (q_norm.numel() == nq and k_norm.numel() == nk))
    q = torch.empty(t, nq, dtype=p.dtype, device=p.device)
    if per_head:
        N.check(N.lib().b200_head_norm_store(p.data_ptr(), q_norm.data_ptr(), N.ptr(k_norm if store else None), N.ptr(table), q.data_ptr(),
                                             k_cache.data_ptr(), v_cache.data_ptr(), slots.data_ptr(), t, p.stride(0), heads, hkv if store else 0,
                                             d, dv, nq, nq + nk, page, 0 if table is None else 2 * table.shape[1], int(interleaved), dt,
                                             float(eps), _f32(p), N.stream()), "b200_head_norm_store")
        return q
    N.check(N.lib().b200_qk_rope_store(p.data_ptr(), N.ptr(q_norm), N.ptr(k_norm), N.ptr(table), q.data_ptr(), k_cache.data_ptr(),
                                       v_cache.data_ptr(), slots.data_ptr(), t, p.stride(0), heads, hkv, d, dv, nq, nq + nk, page,
                                       0 if table is None else 2 * table.shape[1], int(interleaved), heads * dt, hkv * dt, float(eps),
                                       _f32(p), N.stream()), "b200_qk_rope_store")
    return q


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


@dataclass
class GeneralDeltaWeights:
    """Constants of one general delta mixer. ``dk`` / ``dv`` are the head sizes as laid out (padded with zero channels),
    ``d_true`` the model's."""
    decay_bias: torch.Tensor   # fp32 [heads * dk]
    rate_bias: torch.Tensor    # fp32 [heads * dk]
    norm: torch.Tensor         # bf16 [heads * dv]
    heads: int
    dk: int
    dv: int
    d_true: int
    eps: float


def general_delta(proj: torch.Tensor, z: torch.Tensor, w: GeneralDeltaWeights, state: torch.Tensor, positions: torch.Tensor,
                  cu_q: Optional[torch.Tensor], slots: torch.Tensor, out: Optional[torch.Tensor] = None,
                  runs: Optional[list] = None) -> torch.Tensor:
    """Per head ``S = diag(e) S - (a u)(u^T S) + k v^T``, ``y = norm(S^T r) * weight * sigmoid(gate)`` with the unit key
    ``u = k / sqrt(k^2 + 1e-6)``, the decay ``e = exp(-exp(-1/2) sigmoid(z + decay_bias))`` and the removal rate
    ``a = sigmoid(logit + rate_bias)``, both per key channel. ``proj`` [T, ld] = r | k | a logits [heads * dk] | v | gate logits
    [heads * dv]; ``z`` [T, heads * dk] decay logits. ``state`` fp32 [slots, heads, dk, dv] is updated in place; a sequence
    whose first position is 0 starts from zeros, slot -1 is not stored. ``runs`` (host list of (tokens, ..) per sequence of a ragged
    batch) tells how the work is spread. Returns [T, heads * dv] (``out`` when given)."""
    t = proj.shape[0]
    if not proj.is_cuda:
        y = R.general_delta(proj, z, w, state, positions, cu_q, slots)
        return y if out is None else out.copy_(y)
    assert proj.dtype == z.dtype and state.dtype == torch.float32 and state.is_contiguous()
    assert slots.dtype == torch.int32 and positions.dtype == torch.int32 and proj.stride(1) == 1 and z.stride(1) == 1
    L = N.lib()
    if out is None:
        out = torch.empty(t, w.heads * w.dv, dtype=proj.dtype, device=proj.device)
    assert out.shape == (t, w.heads * w.dv) and out.stride(1) == 1 and out.dtype == proj.dtype
    decode = cu_q is None
    ws = torch.empty(L.b200_general_delta_workspace_bytes(t, w.heads, w.dk, w.dv), dtype=torch.uint8, device=proj.device)
    rc = L.b200_general_delta(proj.data_ptr(), z.data_ptr(), w.decay_bias.data_ptr(), w.rate_bias.data_ptr(), w.norm.data_ptr(), state.data_ptr(),
                              positions.data_ptr(), N.ptr(cu_q), slots.data_ptr(), ws.data_ptr(), out.data_ptr(), t, slots.numel(), w.heads, w.dk,
                              w.dv, w.d_true, proj.stride(0), z.stride(0), out.stride(0), float(w.eps),
                              max((r[0] for r in runs or ()), default=0), _f32(proj), N.stream())
    N.check(rc, "b200_general_delta", L.b200_general_delta_launches(int(decode), w.dk, w.dv))
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
                cache: torch.Tensor, slots: torch.Tensor, eps: float, table: Optional[torch.Tensor] = None) -> torch.Tensor:
    """RMS norms of the two latents in a projection's columns ``q_off``.. and ``kv_off``..: the query's is returned
    [T, len(wq)], the key / value one is written to ``cache`` [pages, 1, page, row]. The weights are padded to
    the laid-out widths, ``q_dim`` / ``kv_dim`` are the true ones. A cache row longer than ``wkv`` goes on with a rotated
    key: the projection's columns behind the latent, turned by ``table`` (pairs of neighbours; zero past it)."""
    t, r = x.shape[0], wkv.numel()
    rot_cols = cache.shape[3] - r
    if not x.is_cuda:
        def rms(v, w, dim):
            v = v[:, :dim].float()
            out = torch.zeros(t, w.numel())
            out[:, :dim] = v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * w[:dim].float()
            return out.to(x.dtype)
        row = rms(x[:, kv_off:], wkv, kv_dim)
        if rot_cols:
            k = x[:, kv_off + r:kv_off + r + rot_cols]
            row = torch.cat([row, R.turn(k[:, None], table, True)[:, 0].to(x.dtype)], 1)
        kv_store(row, cache, slots)
        return rms(x[:, q_off:], wq, q_dim)
    assert x.stride(1) == 1 and cache.dtype == x.dtype and cache.is_contiguous() and slots.dtype == torch.int64
    cq = torch.empty(t, wq.numel(), dtype=x.dtype, device=x.device)
    N.check(N.lib().b200_latent_prep(x.data_ptr(), wq.data_ptr(), wkv.data_ptr(), cq.data_ptr(), cache.data_ptr(), slots.data_ptr(), t,
                                     x.stride(0), q_off, q_dim, wq.numel(), kv_off, kv_dim, r, float(eps), N.ptr(table if rot_cols else None),
                                     2 * table.shape[1] if rot_cols else 0, rot_cols, _f32(x), N.stream()), "b200_latent_prep")
    return cq


def head_linear(x: torch.Tensor, w: LinearWeight, heads: int, *, gate: Optional[torch.Tensor] = None,
                in_rows: Optional[torch.Tensor] = None, out: Optional[torch.Tensor] = None,
                out_rows: Optional[torch.Tensor] = None, tail: int = 0, table: Optional[torch.Tensor] = None,
                head_gate: bool = False) -> torch.Tensor:
    """One product per head: ``out[r, h] = W[h] x[r, h]`` with ``w`` stacked [heads * n, k], ``x`` [rows, heads * k] and
    ``out`` [rows, heads * n], optionally times ``sigmoid(gate)`` (``head_gate``: one column per head). ``in_rows`` / ``out_rows`` (int32) select the rows of
    ``x`` and of ``out`` and ``gate`` that the product's rows stand for. ``tail`` > 0: heads of ``x`` are k + tail wide and
    heads of ``out`` n + tail; the tail is turned by the row of x in ``table`` (pairs of neighbours; zero past it)."""
    n, k = w.weight.shape[0] // heads, w.weight.shape[1]
    rows = x.shape[0] if in_rows is None else in_rows.numel()
    rows = rows if out_rows is None else out_rows.numel()
    if out is None:
        out = torch.empty(rows, heads * (n + tail), dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        pick = slice(None) if in_rows is None else in_rows.long()
        xi = x[pick].float().reshape(rows, heads, k + tail)
        y = torch.einsum("rhk,hnk->rhn", xi[..., :k], w.host_f32().reshape(heads, n, k))
        if tail:
            y = torch.cat([y, R.turn(xi[..., k:], table[pick], True)], -1)
        y = y.reshape(rows, heads * (n + tail))
        at = slice(None) if out_rows is None else out_rows.long()
        if gate is not None:
            y = y * _gate_of(gate[at], heads, n, head_gate)
        out[at] = y.to(out.dtype)
        return out
    assert x.stride(1) == 1 and out.stride(1) == 1 and w.weight.is_contiguous() and out.dtype == x.dtype
    assert x.shape[1] == heads * (k + tail) and out.shape[1] == heads * (n + tail) and (gate is None or gate.stride(1) == 1)
    assert all(i is None or i.dtype == torch.int32 for i in (in_rows, out_rows)) and (tail == 0 or gate is None)
    N.check(N.lib().b200_head_linear(x.data_ptr(), w.weight.data_ptr(), out.data_ptr(), N.ptr(gate), N.ptr(in_rows), N.ptr(out_rows), rows,
                                     heads, n, k, x.stride(0), k + tail, out.stride(0), n + tail, gate.stride(0) if gate is not None else 0,
                                     N.ptr(table if tail else None), 2 * table.shape[1] if tail else 0, tail, int(head_gate), _f32(x), N.stream()),
            "b200_head_linear")
    return out


def latent_attn(q: torch.Tensor, cache: torch.Tensor, block_table: torch.Tensor, kv_lens: torch.Tensor, heads: int, scale: float,
                row_seq: Optional[torch.Tensor] = None, max_kv_len: int = 0, v_dim: int = 0, window: int = 0,
                sinks: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention of queries in latent space [rows, heads * row] over cached rows [pages, 1, page, row], which are keys of every
    head and, in their first ``v_dim`` values (0: all), its values: row r sees the first ``kv_lens[r]`` tokens of block-table
    row ``row_seq[r]`` (r when None), with a ``window`` the last ``window`` of them; ``sinks`` fp32 [heads] are scores that only enter
    the denominators. bf16 rows of at most 512 + 64 values run on
    the tensor cores, fp32 and wider ones as plain 32-bit arithmetic. Returns [rows, heads * v_dim]."""
    rows, row, page = q.shape[0], cache.shape[3], cache.shape[2]
    lat = v_dim or row
    table = block_table
    if not q.is_cuda or q.dtype == torch.float32 or lat > 512 or row > 576:
        if row_seq is not None:
            table = block_table[row_seq.long()].contiguous()
        return attn_biased(q, cache, None, table, kv_lens, None, heads=heads, scale=scale, window=window, v_dim=lat, sinks=sinks)
    assert q.is_contiguous() and cache.is_contiguous() and kv_lens.dtype == torch.int32 and kv_lens.numel() == rows
    assert block_table.dtype == torch.int32 and (row_seq is None or row_seq.dtype == torch.int32)
    L = N.lib()
    out = torch.empty(rows, heads * lat, dtype=q.dtype, device=q.device)
    longest = int(max_kv_len or table.shape[1] * page)
    if window > 0:
        longest = min(longest, window + 63)
    step = 32768                            # rows are the grid's second dimension
    for a in range(0, rows, step):
        b = min(a + step, rows)
        splits = L.b200_mla_pick_splits(b - a, heads, longest)
        ws = None
        if splits > 1:
            ws = torch.empty(L.b200_mla_workspace_bytes(b - a, heads, splits), dtype=torch.uint8, device=q.device)
        tab = table if row_seq is not None else table[a:b]
        rc = L.b200_latent_attn(q[a:b].data_ptr(), cache.data_ptr(), out[a:b].data_ptr(), tab.data_ptr(), kv_lens[a:b].data_ptr(),
                                N.ptr(None if row_seq is None else row_seq[a:b]), b - a, heads, row, lat, page, table.stride(0), splits,
                                N.ptr(ws), float(scale), int(window), N.ptr(sinks), N.stream())
        N.check(rc, "b200_latent_attn", 2 if splits > 1 else 1)
    return out


def latent_gather(cache: torch.Tensor, block_table: torch.Tensor, seq_ids: torch.Tensor, offsets: torch.Tensor, total: int,
                  max_len: int, starts: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Cached rows of the sequences in ``seq_ids``, one after another: rows ``offsets[s] .. offsets[s + 1]`` of the
    result [total, row] are the tokens of block-table row ``seq_ids[s]`` from ``starts[s]`` (0 when None) on."""
    page, rank = cache.shape[2], cache.shape[3]
    out = torch.empty(total, rank, dtype=cache.dtype, device=cache.device)
    if not cache.is_cuda:
        for i, s in enumerate(seq_ids.tolist()):
            a, b, f = int(offsets[i]), int(offsets[i + 1]), 0 if starts is None else int(starts[i])
            out[a:b] = R.gather_paged(cache, block_table[s], f + b - a)[f:].reshape(b - a, rank)
        return out
    N.check(N.lib().b200_latent_gather(cache.data_ptr(), out.data_ptr(), block_table.data_ptr(), seq_ids.data_ptr(), offsets.data_ptr(),
                                       N.ptr(starts), seq_ids.numel(), max_len, rank * cache.element_size(), page, block_table.stride(0), N.stream()),
            "b200_latent_gather")
    return out


def attn_runs(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, out: torch.Tensor, q_start: torch.Tensor, q_lens: torch.Tensor,
              kv_start: torch.Tensor, kv_lens: torch.Tensor, *, heads: int, max_q_len: int, scale: float,
              gate: Optional[torch.Tensor] = None, window: int = 0, k_shared: Optional[torch.Tensor] = None,
              table: Optional[torch.Tensor] = None, sinks: Optional[torch.Tensor] = None, head_gate: bool = False) -> None:
    """Causal attention of runs of query rows over contiguous keys and values of their contexts: run s is rows
    ``q_start[s]`` .. + ``q_lens[s]`` of ``q`` [T, heads * d], its context rows ``kv_start[s]`` .. + ``kv_lens[s]`` of ``k``
    [.., heads * d] and ``v`` [.., heads * dv]; the last key belongs to the last query, and with a ``window`` a query sees the
    last ``window`` keys up to its own. ``k_shared`` [.., n]: the last n values of every key head, the same for all heads
    (heads of ``k`` are then d - n wide), the query's side of which is turned by ``table`` [T, pairs, 2]. Rows of the runs are
    written to ``out`` [T, heads * dv] (any row pitch), times ``sigmoid(gate)`` (``head_gate``: one column per head); ``sinks``
    fp32 [heads] are scores that only enter the denominators. bf16, d up to 192 and dv up to 128."""
    own, dv = k.shape[1] // heads, v.shape[1] // heads
    d = own + (0 if k_shared is None else k_shared.shape[1])
    assert q.is_cuda and q.dtype == torch.bfloat16 and out.stride(1) == q.stride(1) == k.stride(1) == v.stride(1) == 1
    assert q.shape[1] == heads * d and out.shape[1] == heads * dv and (gate is None or gate.stride(1) == 1)
    assert k_shared is None or (k_shared.stride(1) == 1 and k_shared.dtype == q.dtype)
    N.check(N.lib().b200_attn_runs(q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), N.ptr(gate), q_start.data_ptr(),
                                   q_lens.data_ptr(), kv_start.data_ptr(), kv_lens.data_ptr(), q_lens.numel(), max_q_len, heads, heads, d,
                                   dv, q.stride(0), k.stride(0), v.stride(0), gate.stride(0) if gate is not None else 0, float(scale),
                                   int(window), N.ptr(k_shared), own, k_shared.stride(0) if k_shared is not None else 0, N.ptr(table),
                                   table.shape[1] if table is not None else 0, N.ptr(sinks), int(head_gate), out.stride(0), N.stream()),
            "b200_attn_runs")
