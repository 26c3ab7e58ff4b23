"""Zovudra against the plain statement in ``zovudra_oracle``: every mechanism alone, then whole models through
the engine (prompts, portions, decoding, mixed batches, reused pages, generation).

Each case runs on the CPU ops and, marked ``gpu``, on the kernels in fp32 and bf16."""
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import zovudra_oracle as O  # noqa: E402
from test_lududra import BF, F32, MODES, Pages, _Holder, gen, logits_near, near, rel_err, rnd  # noqa: E402
from test_salopel import _PagedBatch, engine, play  # noqa: E402

from hartsyinference_b200 import ops  # noqa: E402
from hartsyinference_b200.engine import LLMEngine, SamplingParams  # noqa: E402
from hartsyinference_b200.exceptions import KvPoolExhaustedError  # noqa: E402
from hartsyinference_b200.models.llm import config as C  # noqa: E402
from hartsyinference_b200.models.llm import mixers as M  # noqa: E402
from hartsyinference_b200.models.llm.loader import load_llm, save_hf_checkpoint  # noqa: E402
from hartsyinference_b200.models.llm.moe import MoeFeedForward  # noqa: E402
from hartsyinference_b200.models.llm.rope import Rotary  # noqa: E402
from hartsyinference_b200.models.llm.transformer import DecoderModel  # noqa: E402
from hartsyinference_b200.models.llm.zovudra import config_from, tensor_shapes  # noqa: E402

i32 = lambda v, dev: torch.tensor(v, dtype=torch.int32, device=dev)


# ------------------------------------------------------------------------------------ norms and stream
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("dim", [40, 132, 1000, 8204])
def test_stream_tanh_norm(mode, dim):
    """Small, middling and saturated values; an RMS norm on what enters the stream beside the tanh on what leaves it."""
    dev, dt = mode
    g = gen(dim)
    rows, ld = 5, (dim + 7) // 8 * 8
    x = torch.zeros(rows, ld)
    x[:, :dim] = torch.randn(rows, dim, generator=g) * torch.tensor([1e-3, 0.1, 1.0, 5.0, 40.0])[:, None]
    y = torch.zeros(rows, ld, dtype=BF)
    y[:, :dim] = rnd(g, rows, dim, std=0.02)
    wb, wn, bn = rnd(g, dim, std=0.3) + 1, rnd(g, dim), rnd(g, dim, std=0.5)
    tn = ops.TanhNorm(0.37, wn.to(dev), bn.to(dev))
    kw = dict(dim=dim, eps=1e-4, layernorm=False, dtype=dt)
    xd = x.clone().to(dev)
    h = ops.residual_norm(xd, None, None, tn, **kw)
    for r in range(rows):                                   # row by row: they differ in size
        near(h[r, :dim], O.tanh_norm(x[r, :dim].double(), 0.37, wn.double(), bn.double()), mode, 1e-6, 4e-3)
    assert float(h[:, dim:].float().abs().sum()) == 0 and torch.equal(xd.cpu(), x)
    h = ops.residual_norm(xd, y.to(dt).to(dev), wb.to(dev), tn, **kw)
    want = x[:, :dim].double() + O.rms(y[:, :dim].double(), wb.double(), 1e-4)
    assert rel_err(xd[:, :dim], want) < 1e-6
    near(h[:, :dim], O.tanh_norm(want, 0.37, wn.double(), bn.double()), mode, 1e-6, 4e-3)


@pytest.mark.parametrize("mode", MODES)
def test_expert_rows_with_shared_rows(mode):
    dev, dt = mode
    g = gen(5)
    t, k, dim = 6, 3, 72
    rows, extra = rnd(g, 20, 128).to(dt), rnd(g, t, dim).to(dt)
    slot = torch.randperm(20, generator=g)[:t * k].reshape(t, k).to(torch.int32)
    slot[0, 1] = -1
    wts, ew = torch.rand(t, k, generator=g), torch.rand(t, generator=g)
    x = torch.randn(t, dim, generator=g)
    want = x.double() + ew[:, None].double() * extra.double()
    for i in range(t):
        for j in range(k):
            if slot[i, j] >= 0:
                want[i] += wts[i, j].double() * rows[slot[i, j].item(), :dim].double()
    xd = x.to(dev)
    ids = torch.zeros(t, k, dtype=torch.int32)
    rr = ops.RoutedRows(rows.to(dev), slot.to(dev), ids.to(dev), wts.to(dev), None, 4, extra.to(dev), ew.to(dev))
    h = ops.residual_norm(xd, rr, None, None, dim=dim, eps=1e-6, layernorm=False, dtype=dt, plain=True)
    assert rel_err(xd, want) < 1e-6 and torch.equal(h, xd.to(dt))


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("dim,width", [(16, 96), (5, 40), (24, 20), (256, 136)])
def test_token_input(mode, dim, width):
    """The layer's own columns of the table, repeated tokens, large gates on either side of zero."""
    dev, dt = mode
    g = gen(dim)
    wp, dp = (width + 7) // 8 * 8, (dim + 7) // 8 * 8
    x = torch.zeros(9, wp, dtype=BF)
    x[:, :width] = rnd(g, 9, width)
    w = {"s.gate": rnd(g, dim, width, std=3 * width ** -0.5), "s.proj": rnd(g, width, dim, std=dim ** -0.5), "s.norm": rnd(g, width, std=0.3) + 1}
    table = rnd(g, 7, 3 * dim)
    ids = [3, 0, 6, 3, 3, 1, 5, 2, 0]
    want = O.side_input(x[:, :width].double(), table[ids, dim:2 * dim].double(), {n: v.double() for n, v in w.items()}, "s.", 1e-4)
    cols = torch.zeros(7, 3 * dp, dtype=BF)
    for i in range(3):
        cols[:, i * dp:i * dp + dim] = table[:, i * dim:(i + 1) * dim]
    m = M.TokenInput(dim, width, dev, table=cols.to(dev)[:, dp:2 * dp], gate=w["s.gate"], proj=w["s.proj"])
    s = torch.zeros(9, wp, device=dev)
    ops.residual_norm(s, m(x.to(dt).to(dev), i32(ids, dev)), w["s.norm"].to(dev), None, dim=width, eps=1e-4, layernorm=False, dtype=dt)
    near(s[:, :width], want, mode, 2e-6, 1e-2)


# ------------------------------------------------------------------------------------ rotation
ROTS = {"plain": dict(dims=32, base=10000.0), "part": dict(dims=12, base=500.0), "one": dict(dims=2, base=7.0),
        "scaled": dict(dims=64, base=1e6, scaling=dict(factor=8.0, low=1.0, high=4.0, original=256)),
        "edges": dict(dims=24, base=300.0, scaling=dict(factor=2.0, low=2.0, high=2.5, original=100))}


def rot_spec(rot, interleaved=False):
    s = rot.get("scaling")
    sc = C.RopeScaling() if not s else C.RopeScaling("llama3", s["factor"], s["low"], s["high"], s["original"])
    return C.RotarySpec(rot["dims"], rot["base"], interleaved, sc)


@pytest.mark.parametrize("mode", MODES[:2])
@pytest.mark.parametrize("rot", list(ROTS))
def test_rotation_table(mode, rot):
    """Frequencies on each side of the scaling's borders, and angles far from the start."""
    dev = mode[0]
    r = Rotary(rot_spec(ROTS[rot]), dev)
    f = torch.tensor(O.frequencies(ROTS[rot]), dtype=torch.float64)
    assert float(((r.hi.double() + r.lo.double()).cpu() / f - 1).abs().max()) < 1e-13
    pos = [0, 1, 2, 63, 1000, 131071, 1000003]
    b = _Holder()
    b.positions, b.plan = i32(pos, dev), None
    t = r.table(b)
    assert r.table(b) is t and Rotary(rot_spec(ROTS[rot]), dev).table(b) is t       # one table for all layers that turn alike
    ang = torch.tensor(pos, dtype=torch.float64)[:, None] * f
    assert float((t.cpu().double() - torch.stack([ang.cos(), ang.sin()], -1)).abs().max()) < 4e-7


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,hkv,d,dv,rot,inter,norm,page", [(4, 2, 32, 32, "plain", False, True, 16), (3, 1, 16, 40, "part", False, True, 8),
                                                                (2, 2, 64, 24, "scaled", True, False, 16), (5, 5, 24, 8, "edges", False, True, 64),
                                                                (2, 1, 160, 16, "one", True, True, 16), (6, 3, 8, 8, None, False, True, 16)])
def test_norm_rotation_and_store(mode, heads, hkv, d, dv, rot, inter, norm, page):
    """Norms over all heads at once (large heads beside small ones), partial rotations, pairs inside one vector and
    across vectors, tokens that are not stored."""
    dev, dt = mode
    g = gen(d + dv)
    n = 70
    size = torch.logspace(-1, 1, heads + hkv).repeat_interleave(d)
    p = torch.cat([rnd(g, n, (heads + hkv) * d) * size, rnd(g, n, hkv * dv)], 1).to(BF)
    qw, kw = rnd(g, heads * d, std=0.4) + 1, rnd(g, hkv * d, std=0.4) + 1
    pd = p.double()
    q, k, v = pd[:, :heads * d], pd[:, heads * d:(heads + hkv) * d], pd[:, (heads + hkv) * d:]
    if norm:
        q, k = O.rms(q, qw.double(), 0.01), O.rms(k, kw.double(), 0.01)
    turn = lambda x: x if rot is None else O.rotate(x, ROTS[rot], inter)
    wq = torch.cat([turn(q[:, h * d:(h + 1) * d]) for h in range(heads)], 1)
    wk = torch.cat([turn(k[:, h * d:(h + 1) * d]) for h in range(hkv)], 1)
    pk, pv = Pages(gen(1), [n], hkv, d, page, dt, dev), Pages(gen(1), [n], hkv, dv, page, dt, dev)
    before = pk.cache.clone()
    slots = pk.slots(0, 0, n)
    slots[7] = -1
    table = None
    if rot is not None:
        b = _Holder()
        b.positions, b.plan = i32(list(range(n)), dev), None
        table = Rotary(rot_spec(ROTS[rot], inter), dev).table(b)
    got = ops.qk_rope_store(p.to(dt).to(dev), heads, pk.cache, pv.cache, slots.to(dev), table=table, interleaved=inter,
                            q_norm=qw.to(dev) if norm else None, k_norm=kw.to(dev) if norm else None, eps=0.01)
    near(got, wq, mode, 1e-6, 4e-3)
    ok = slots >= 0
    at = slots[ok]
    rows = lambda c: c.cpu()[at // page, :, at % page].reshape(n - 1, -1)
    near(rows(pk.cache), wk[ok], mode, 1e-6, 4e-3)
    assert torch.equal(rows(pv.cache).to(BF), p[ok][:, (heads + hkv) * d:])
    seven = pk.slots(0, 7, 1)
    assert torch.equal(pk.cache[seven // page, :, seven % page], before[seven // page, :, seven % page])


# ------------------------------------------------------------------------------------ attention
def plant(q, k, rows, spots, head, group, gain=4.0):
    """Make one key stand out for one query of one head."""
    u = torch.nn.functional.normalize(q[rows, head].float(), dim=0)
    k[spots, group] += (u * gain).to(BF)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("hq,hkv,d,dv,page,window,keep,tail", [
    (6, 2, 64, 64, 16, 50, 7, 1), (6, 2, 64, 64, 16, 50, 7, 70), (6, 2, 40, 24, 8, 17, 1, 3), (8, 8, 128, 64, 16, 65, 70, 130), (3, 1, 16, 104, 64, 1, 3, 5),
    (20, 1, 24, 24, 16, 130, 65, 1), (2, 1, 160, 32, 16, 33, 9, 9), (16, 1, 96, 128, 32, 64, 64, 1), (4, 4, 8, 8, 16, 1000, 5, 2), (2, 1, 32, 32, 16, 20, 0, 40),
    (4, 1, 64, 64, 16, 0, 9, 50), (2, 2, 64, 128, 16, 16, 200, 40), (2, 1, 48, 200, 16, 70, 2, 33)])
def test_window_with_kept_tokens(mode, hq, hkv, d, dv, page, window, keep, tail):
    """Four sequences whose last ``tail`` tokens are the queries. Keys just inside and just outside the window, the last kept
    token, the first that is not kept, and tokens at page and tile edges each stand out for some query."""
    dev, dt = mode
    g = gen(hq * 100 + d + keep)
    lens = [tail + 300, tail + 2, max(tail, 5), tail + 130]
    scale, group = 0.8, hq // hkv
    q = [rnd(g, n, hq, d, std=d ** -0.5) for n in lens]
    k, v = [rnd(g, n, hkv, d) for n in lens], [rnd(g, n, hkv, dv) for n in lens]
    for i, n in enumerate(lens):
        for r in range(n - tail, n, max(1, tail // 7)):
            spots = [r - window + 1, r - window, keep - 1, keep, 0, r // page * page, r // page * page - 1, 63, 64, r]
            for h, spot in enumerate(spots):
                if 0 <= spot <= r:
                    plant(q[i], k[i], r, spot, (h + r) % hq, (h + r) % hq // group)
    pk, pv = Pages(gen(3), lens, hkv, d, page, dt, dev), Pages(gen(3), lens, hkv, dv, page, dt, dev)
    for i, n in enumerate(lens):
        ops.kv_store(k[i].reshape(n, -1).to(dt).to(dev), pk.cache, pk.slots(i, 0, n).to(dev))
        ops.kv_store(v[i].reshape(n, -1).to(dt).to(dev), pv.cache, pv.slots(i, 0, n).to(dev))
    mask = dict(size=window, keep_first=keep)
    want = torch.cat([torch.cat([O.masked_attention(q[i][:, h].double(), k[i][:, h // group].double(), v[i][:, h // group].double(), scale, mask, lens[i] - tail)
                                 for h in range(hq)], 1) for i in range(len(lens))])
    rows = torch.cat([x[-tail:].reshape(tail, -1) for x in q]).to(dt).to(dev)
    run = lambda cu: ops.attn_biased(rows, pk.cache, pv.cache, pk.table.to(dev), i32(lens, dev), cu, heads=hq, max_q_len=tail,
                                     max_kv_len=max(lens), scale=scale, window=window, keep_first=keep)
    near(run(i32([tail * i for i in range(len(lens) + 1)], dev)), want, mode, 1e-5, 1e-2)
    if tail == 1:
        near(run(None), want, mode, 1e-5, 1e-2)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,rank,rot,page,window", [(5, 64, 48, 16, 40), (6, 40, 8, 8, 0), (17, 128, 64, 16, 70), (1, 96, 32, 64, 1), (33, 24, 104, 16, 130),
                                                        (3, 512, 64, 32, 65), (20, 264, 16, 16, 9), (2, 200, 56, 16, 64), (2, 160, 200, 16, 33), (2, 448, 64, 16, 50)])
def test_latent_rows_with_rotated_part(mode, heads, rank, rot, page, window):
    """Queries in latent space: rows of the cache are keys, their first part the values; keys at the window's edge stand
    out through the latent for some heads and through the rotated part for others."""
    dev, dt = mode
    g = gen(heads * 10 + rank)
    lens = [300, 1, 65, 128, page + 1]
    row = rank + rot
    pg = Pages(g, lens, 1, row, page, dt, dev)
    lat = [rnd(g, n, row) for n in lens]
    rows = [(i, m) for i, n in enumerate(lens) for m in sorted({n, max(1, n // 2)}, reverse=True)]
    q = rnd(g, len(rows), heads, row, std=row ** -0.5)
    for r, (i, n) in enumerate(rows):
        for h, spot in enumerate((n - window, n - window - 1, n - 1, 0, page - 1, page, 63, 64)):
            if 0 <= spot < n:
                part = slice(0, rank) if h % 2 else slice(rank, row)
                lat[i][spot, part] += (torch.nn.functional.normalize(q[r, h % heads, part].float(), dim=0) * 5).to(BF)
    for i, n in enumerate(lens):
        ops.kv_store(lat[i].to(dt).to(dev), pg.cache, pg.slots(i, 0, n).to(dev))
    want = []
    for r, (i, n) in enumerate(rows):
        c = lat[i][max(0, n - window) if window else 0:n].double()
        want.append(torch.cat([torch.softmax(c @ q[r, h].double() * 1.7, 0) @ c[:, :rank] for h in range(heads)]))
    qd = q.reshape(len(rows), -1).to(dt).to(dev)
    out = ops.latent_attn(qd, pg.cache, pg.table.to(dev), i32([n for _, n in rows], dev), heads, 1.7, row_seq=i32([i for i, _ in rows], dev),
                          max_kv_len=max(lens), v_dim=rank, window=window)
    near(out, torch.stack(want), mode, 1e-5, 6e-3)
    ends = [r for r, (i, n) in enumerate(rows) if n == lens[i]]
    out = ops.latent_attn(qd[ends].contiguous(), pg.cache, pg.table.to(dev), i32(lens[:-1] + [0], dev), heads, 1.7, max_kv_len=4096, v_dim=rank,
                          window=window)                     # one row per sequence (decode), the last one empty
    near(out[:-1], torch.stack(want)[ends][:-1], mode, 1e-5, 6e-3)
    assert float(out[-1].float().abs().max()) == 0


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,n,k,tail,rot,rows", [(3, 40, 24, 8, 6, 5), (6, 72, 64, 32, 32, 130), (2, 512, 128, 64, 64, 64), (16, 8, 200, 16, 10, 1)])
def test_head_linear_with_turned_tail(mode, heads, n, k, tail, rot, rows):
    dev, dt = mode
    g = gen(n + k)
    x, w = rnd(g, rows + 4, heads, k + tail), rnd(g, heads * n, k, std=k ** -0.5)
    x[..., k + rot:] = 0
    b = _Holder()
    b.positions, b.plan = i32(list(range(rows + 4)), dev), None
    table = Rotary(C.RotarySpec(rot, 100.0, True), dev).table(b)
    full = torch.cat([torch.cat([x[:, h, :k].double() @ w[h * n:(h + 1) * n].double().T, O.rotate(x[:, h, k:].double(), dict(dims=rot, base=100.0), True)], 1)
                      for h in range(heads)], 1)
    pick = torch.randperm(rows + 4, generator=g)[:rows]
    xd = x.reshape(rows + 4, -1).to(dt).to(dev)
    near(ops.head_linear(xd, ops.LinearWeight(w.to(dev)), heads, tail=tail, table=table), full, mode, 1e-6, 4e-3)
    few = ops.head_linear(xd, ops.LinearWeight(w.to(dev)), heads, tail=tail, table=table, in_rows=pick.to(torch.int32).to(dev))
    near(few, full[pick], mode, 1e-6, 4e-3)


@pytest.mark.gpu
@pytest.mark.parametrize("heads,own,rot,dv,window", [(3, 64, 48, 72, 130), (3, 40, 16, 24, 1), (2, 64, 64, 128, 64), (5, 16, 8, 104, 65), (2, 32, 32, 32, 0),
                                                     (3, 128, 64, 128, 70), (2, 104, 40, 64, 0)])
def test_runs_with_shared_rotated_keys(heads, own, rot, dv, window):
    """Runs that are not adjacent, contexts cut at the first visible key, keys at the window's edges stand out."""
    g = gen(own + dv)
    d = own + rot
    runs = [(70, 70), (3, 200), (129, 130), (64, 321)]           # (queries, keys)
    starts = [10, 100, 105, 240]
    t = 310
    q = rnd(g, t, heads, d, std=d ** -0.5)
    b = _Holder()
    b.positions, b.plan = i32([7 * i % 1000 for i in range(t)], "cuda"), None
    table = Rotary(C.RotarySpec(rot, 50.0, True), "cuda").table(b)
    qt = q.double().clone()
    tc = table.cpu().double()
    u, v = qt[..., own::2].clone(), qt[..., own + 1::2].clone()
    qt[..., own::2], qt[..., own + 1::2] = u * tc[:, None, :, 0] - v * tc[:, None, :, 1], v * tc[:, None, :, 0] + u * tc[:, None, :, 1]
    ks, ss, vs, want = [], [], [], torch.full((t, heads * dv), 7.0, dtype=torch.float64)
    for (nq, nk), a in zip(runs, starts):
        k, sh, vv = rnd(g, nk, heads, own), rnd(g, nk, rot), rnd(g, nk, heads, dv)
        for i in range(0, nq, 5):
            p = nk - nq + i
            for h, spot in enumerate((p, p + 1, p - window + 1, p - window, 64)):
                if 0 <= spot < nk:
                    e = torch.nn.functional.normalize(qt[a + i, h % heads].float(), dim=0) * 3
                    k[spot, h % heads] += e[:own].to(BF)
                    sh[spot] += e[own:].to(BF)
        for h in range(heads):
            full = torch.cat([k[:, h], sh], 1).double()
            for i in range(nq):
                n = nk - nq + i + 1
                lo = max(0, n - window) if window else 0
                s = torch.softmax(full[lo:n] @ qt[a + i, h] * 2.5, 0)
                want[a + i, h * dv:(h + 1) * dv] = s @ vv[lo:n, h].double()
        ks.append(k.reshape(nk, -1)), ss.append(sh), vs.append(vv.reshape(nk, -1))
    out = torch.full((t, heads * dv), 7.0, dtype=BF, device="cuda")
    at = [0]
    for _, nk in runs:
        at.append(at[-1] + nk)
    kv, sh = torch.cat([torch.cat(ks), torch.cat(vs)], 1).cuda(), torch.cat([rnd(g, at[-1], 16), torch.cat(ss)], 1).cuda()
    c = lambda v: i32(v, "cuda")
    ops.attn_runs(q.reshape(t, -1).cuda(), kv[:, :heads * own], kv[:, heads * own:], out, c(starts), c([r[0] for r in runs]), c(at),
                  c([r[1] for r in runs]), heads=heads, max_q_len=129, scale=2.5, window=window, k_shared=sh[:, 16:], table=table)
    near(out, want, ("cuda", BF), bf16=1e-2)
    others = torch.ones(t, dtype=torch.bool)
    for (nq, _), a in zip(runs, starts):
        others[a:a + nq] = False
    assert bool((out.cpu()[others] == 7.0).all())


# ------------------------------------------------------------------------------------ mixers
WIDTH = 24


def run_portions(m, hs, pages, cache, cuts, order, dt, dev):
    """Portions of the given sizes beside each other, in the given order, then single tokens together."""
    holder = _Holder()
    holder.kv_cache = [cache]
    got = [torch.zeros(len(h), WIDTH) for h in hs]
    done = [0] * len(hs)
    cuts = list(cuts)
    while any(d < len(h) for d, h in zip(done, hs)):
        c = cuts.pop(0) if cuts else (1,) * len(hs)
        runs = [(i, done[i], min(c[i], len(hs[i]) - done[i])) for i in order if min(c[i], len(hs[i]) - done[i]) > 0]
        rows = torch.cat([hs[i][a:a + n] for i, a, n in runs]).to(dt).to(dev)
        y = m(rows, _PagedBatch(dev, pages, runs, c == (1,) * len(hs)), 0, holder).float().cpu()
        for i, a, n in runs:
            got[i][a:a + n], y = y[:n, :WIDTH], y[n:]
            done[i] += n
    return got


CUTS = [(60, 2, 0), (2, 50, 1), (49, 1, 2), (1, 0, 1), (47, 1, 1), (64, 2, 1), (3, 1, 0)]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,kv,dim,vdim,rot,window,keep,scale", [(4, 2, 16, 16, 16, 20, 3, 1.0), (6, 3, 40, 24, 24, 33, 1, 0.3), (3, 1, 20, 12, 8, 50, 70, 0.5),
                                                                     (2, 2, 64, 80, 64, 17, 0, 0.2), (5, 1, 12, 136, 12, 9, 4, 0.7), (2, 1, 8, 8, 2, 0, 0, 0.9)])
def test_attention_mixer(mode, heads, kv, dim, vdim, rot, window, keep, scale):
    dev, dt = mode
    g = gen(dim + vdim)
    mix = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, rot=dict(dims=rot, base=200.0, scaling=dict(factor=4.0, low=1.0, high=4.0, original=64)),
               scale=scale, mask=dict(size=window, keep_first=keep))
    shapes = {"q": (heads * dim, WIDTH), "k": (kv * dim, WIDTH), "v": (kv * vdim, WIDTH), "o": (WIDTH, heads * vdim)}
    t = {n: rnd(g, *s, std=s[1] ** -0.5) for n, s in shapes.items()}
    t["q.norm"], t["k.norm"] = rnd(g, heads * dim, std=0.4) + 1, rnd(g, kv * dim, std=0.4) + 1
    hs = [rnd(g, 250, WIDTH), rnd(g, 60, WIDTH), rnd(g, 9, WIDTH)]
    wd = {"mix." + n: v.double() for n, v in t.items()}
    want = [O.attention_mixer(h.double(), mix, wd, "mix.", 1e-3) for h in hs]
    spec = C.MixerSpec(kind="attention", heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, window=window, keep_first=keep, qk_norm=True,
                       rot=rot_spec(mix["rot"]))
    m = M.BiasedAttention(spec, WIDTH, dev, q=t["q"], k=t["k"], v=t["v"], o=t["o"], q_norm=t["q.norm"], k_norm=t["k.norm"], eps=1e-3)
    pages = Pages(g, [len(h) for h in hs], 1, 8, 16, dt, dev)
    cache = torch.full(m.cache_shape(pages.cache.shape[0], 16), 5.0, dtype=dt, device=dev)
    for a, b in zip(run_portions(m, hs, pages, cache, CUTS, [1, 0, 2], dt, dev), want):
        near(a, b, mode, 5e-5, 2e-2)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,dim,rot,vdim,kv_rank,q_rank,window,scale", [(3, 16, 8, 24, 32, 20, 40, 1.5), (6, 40, 6, 8, 72, 12, 0, 0.7), (2, 64, 32, 64, 20, 48, 70, 1.0),
                                                                            (18, 8, 16, 12, 16, 9, 1, 2.0), (2, 20, 10, 136, 24, 16, 30, 1.0), (2, 128, 64, 128, 96, 32, 65, 0.5),
                                                                            (1, 200, 8, 16, 40, 8, 20, 0.5)])
def test_latent_attention_mixer(mode, heads, dim, rot, vdim, kv_rank, q_rank, window, scale):
    """Long runs (expanded keys, contexts cut at the window) beside short ones, then decoding."""
    dev, dt = mode
    g = gen(dim + vdim)
    mix = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale, rot=dict(dims=rot, base=90.0),
               mask=dict(size=window))
    shapes = {"dq": (q_rank, WIDTH), "uq": (heads * (dim + rot), q_rank), "dkv": (kv_rank + rot, WIDTH), "uk": (heads * dim, kv_rank),
              "uv": (heads * vdim, kv_rank), "o": (WIDTH, heads * vdim)}
    t = {n: rnd(g, *s, std=s[1] ** -0.5) for n, s in shapes.items()}
    t["dq.norm"], t["dkv.norm"] = rnd(g, q_rank, std=0.3) + 1, rnd(g, kv_rank, std=0.3) + 1
    hs = [rnd(g, 250, WIDTH), rnd(g, 60, WIDTH), rnd(g, 9, WIDTH)]
    wd = {"mix." + n: v.double() for n, v in t.items()}
    want = [O.latent_attention_mixer(h.double(), mix, wd, "mix.", 1e-4) for h in hs]
    spec = C.MixerSpec(kind="latent_attention", heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale, window=window, rot_dim=rot,
                       rot=rot_spec(mix["rot"], True))
    m = M.LatentAttention(spec, WIDTH, 1e-4, dev, **{n.replace(".", "_"): v for n, v in t.items()})
    pages = Pages(g, [len(h) for h in hs], 1, m.r + m.t, 16, dt, dev)
    for a, b in zip(run_portions(m, hs, pages, pages.cache[None], CUTS, [1, 0, 2], dt, dev), want):
        near(a, b, mode, 5e-5, 3e-2)


# ------------------------------------------------------------------------------------ feed-forwards
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("width,ff,rows", [(24, 20, 3), (64, 256, 150), (2048, 72, 5)])
def test_gated_dense(mode, width, ff, rows):
    dev, dt = mode
    g = gen(ff)
    w = {"gate": rnd(g, ff, width, std=2 * width ** -0.5), "up": rnd(g, ff, width, std=width ** -0.5), "down": rnd(g, width, ff, std=ff ** -0.5)}
    h = rnd(g, rows, width)
    m = M.DenseFeedForward(C.DenseSpec(ff, "silu"), width, 1e-6, dev, **w)
    near(m(h.to(dt).to(dev))[:, :width], O.dense_ff(h.double(), {"f." + n: v.double() for n, v in w.items()}, "f."), mode, 2e-6, 1e-2)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("m,n,k", [(3, 40, 24), (5, 256, 4096), (300, 128, 64)])
def test_relu_squared_product(mode, m, n, k):
    """Also where the product is cut along its inner dimension: the square comes after the sum."""
    dev, dt = mode
    g = gen(n + k)
    x, w = rnd(g, m, k), rnd(g, n, k, std=k ** -0.5)
    near(ops.linear_act(x.to(dt).to(dev), ops.LinearWeight(w.to(dev)), "relu2"), O.relu2(x.double() @ w.double().T), mode, 2e-6, 5e-3)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("experts,groups,keep,top,width,rows", [(20, 4, 3, 4, 40, 9), (12, 6, 2, 2, 64, 30), (8, 8, 3, 2, 24, 7), (10, 1, 1, 4, 32, 700), (64, 8, 2, 6, 136, 700),
                                                                (40, 5, 5, 5, 72, 20), (160, 4, 1, 8, 64, 650), (96, 32, 4, 1, 64, 3)])
def test_router_in_groups(mode, experts, groups, keep, top, width, rows):
    """Groups whose single best expert is not in the best groups, against the choice token by token; the shared gate."""
    dev, dt = mode
    g = gen(experts + rows)
    x, w = rnd(g, rows, width), rnd(g, experts + 1, width, std=1.5 * width ** -0.5)
    scores = O.sigmoid(x.double() @ w.double().T)
    ids, wts, gate = ops.router(x.to(dt).to(dev), ops.LinearWeight(w.to(dev)), None, top, sigmoid=True, norm_topk=True, scale=1.7, n_group=groups,
                                topk_group=keep, gate=True)
    assert rel_err(gate, scores[:, -1]) < 1e-5
    cut = 0
    for t in range(rows):
        row = scores[t, :-1].tolist()
        want = O.choose(row, dict(top=top, groups=dict(count=groups, keep=keep)))
        cut += want != O.choose(row, dict(top=top))
        assert ids[t].tolist() == want
        ref = scores[t, want] / (scores[t, want].sum() + 1e-20) * 1.7
        assert rel_err(wts[t], ref) < 1e-5
    assert cut > 0 or keep == groups or experts == groups
    plain, _ = ops.router(x.to(dt).to(dev), ops.LinearWeight(w[:experts].to(dev)), None, top, sigmoid=True)
    assert plain[0].tolist() == O.choose(scores[0, :-1].tolist(), dict(top=top))


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("experts,groups,keep,top,ff,shared,width,rows", [(8, 4, 2, 3, 24, 40, 40, 5), (6, 1, 1, 1, 136, None, 64, 33), (16, 2, 1, 4, 64, 16, 136, 300),
                                                                          (5, 5, 4, 4, 8, 8, 24, 1)])
def test_experts(mode, experts, groups, keep, top, ff, shared, width, rows):
    """Ungated experts, idle ones included, with and without a gated shared expert of another size."""
    dev, dt = mode
    g = gen(ff + rows)
    w = {"router": rnd(g, experts, width, std=2 * width ** -0.5)}
    for e in [f"e{i}" for i in range(experts)] + (["shared"] if shared else []):
        f = shared if e == "shared" else ff
        w[e + ".up"], w[e + ".down"] = rnd(g, f, width, std=width ** -0.5), rnd(g, width, f, std=f ** -0.5)
    if shared:
        w["shared.sg"] = rnd(g, 1, width, std=2 * width ** -0.5)
    h = rnd(g, rows, width)
    mlp = {"kind": "moe", "expert": {"ff": ff}, "router": dict(experts=experts, top=top, scale=1.3, groups=dict(count=groups, keep=keep)),
           "shared": {"ff": shared} if shared else None}
    want = O.moe_ff(h.double(), mlp, {"m." + n: v.double() for n, v in w.items()}, "m.")
    cfg = config_from(model_cfg(20, width, [att(2, 1, 8, 8, 8, 4, 1, mlp=mlp)]))
    moe = cfg.layer_specs[0].moe
    parts = M.build_experts(moe, width, dev, w["router"], None, ((None, w[f"e{i}.up"], w[f"e{i}.down"]) for i in range(experts)),
                            (w["shared.up"], w["shared.down"], w["shared.sg"]) if shared else None)
    m = MoeFeedForward(cfg, parts, moe=moe, hidden=width)
    x = torch.zeros(rows, width, device=dev)
    ops.residual_norm(x, m.routed_rows(h.to(dt).to(dev)), None, None, dim=width, eps=1e-6, layernorm=False, dtype=dt)
    near(x, want, mode, 3e-6, 1.5e-2)
    near(m(h.to(dt).to(dev))[:, :width], want, mode, 3e-6, 1.5e-2)


# ------------------------------------------------------------------------------------ whole models
def att(heads, kv, dim, vdim, rot, window, keep, scale=None, mlp=None, scaling=None, base=5000.0):
    return {"type": "attention", "mlp": mlp,
            "mixer": dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale or 0.8 * dim ** -0.5, mask=dict(size=window, keep_first=keep),
                          rot=dict(dims=rot, base=base, **({"scaling": scaling} if scaling else {})))}


def lat(heads, dim, rot, vdim, kv_rank, q_rank, window, scale=None, mlp=None, base=3000.0):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale or 1.3 * (dim + rot) ** -0.5,
                          mask=dict(size=window), rot=dict(dims=rot, base=base))}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, groups, keep, scale, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": dict(experts=experts, top=top, groups=dict(count=groups, keep=keep), scale=scale),
            "shared": {"ff": shared}}


def model_cfg(vocab, width, layers, side=8, eps=1e-5, scale=0.7):
    return {"architecture": "Zovudra", "embedding": {"scale": scale}, "norm": {"eps": eps}, "token_side": {"dim": side}, "vocab": vocab, "width": width,
            "layers": layers}


LONG = dict(factor=8.0, low=1.0, high=4.0, original=64)
CASES = {
    # every kind of layer, a layer without feed-forward, odd sizes, windows shorter and longer than a page
    "mixed": model_cfg(301, 136, [att(6, 3, 40, 24, 16, 21, 5, mlp=moe(12, 3, 40, 3, 2, 1.6, 72), scaling=LONG), lat(5, 40, 12, 24, 56, 30, 33, mlp=dense(100)),
                                  att(4, 1, 16, 32, 16, 70, 1), lat(3, 24, 20, 16, 40, 22, 50, mlp=moe(8, 2, 24, 4, 3, 0.8, 16))], side=12),
    "attention": model_cfg(97, 64, [att(2, 2, 32, 32, 32, 17, 70, mlp=dense(60)), att(9, 3, 8, 136, 6, 40, 3, scaling=LONG, mlp=dense(24))], side=5, eps=1e-4, scale=1.0),
    "latent": model_cfg(130, 100, [lat(18, 16, 8, 12, 32, 24, 16), lat(2, 64, 32, 64, 136, 48, 64, mlp=moe(6, 1, 88, 1, 1, 2.0, 40)), lat(4, 128, 64, 96, 64, 40, 20)],
                        side=24, eps=1e-6),
}


def rand_weights(cfg, seed=0):
    g = gen(seed)
    w = {}
    for n, s in tensor_shapes(config_from(cfg)).items():
        leaf = n.rsplit(".", 1)[-1]
        if leaf == "alpha":
            w[n] = (torch.rand((), generator=g) * 0.4 + 0.3).to(BF)
        elif leaf == "b":
            w[n] = rnd(g, *s, std=0.2)
        elif "norm" in leaf:
            w[n] = rnd(g, *s, std=0.3) + 1
        elif n in ("embed", "side.embed"):
            w[n] = rnd(g, *s)
        else:
            w[n] = rnd(g, *s, std=s[-1] ** -0.5)
    return w


_BUILT, _WANT = {}, {}


def built(case, mode):
    if (case, mode) not in _BUILT:
        cfg, w = CASES[case], rand_weights(CASES[case])
        model = DecoderModel(config_from(cfg), mode[0], dtype=mode[1])
        model.load_state_dict(w.get)
        _BUILT[case, mode] = (cfg, w, model)
    return _BUILT[case, mode]


def _expected(case, tokens):
    key = (case, tuple(tokens))
    if key not in _WANT:
        clear = []
        y = O.forward(tokens, CASES[case], rand_weights(CASES[case]), clear=clear)
        _WANT[key] = y, torch.tensor(clear).amin(0) if clear else torch.ones(len(tokens))
    return _WANT[key]


def expected(case, tokens):
    return _expected(case, tokens)[0]


def check(got, case, tokens, mode):
    """Logits of all positions. In bf16 a token for which two experts or groups are as good as tied may take the other
    one: such positions are left out there."""
    want, clear = _expected(case, tokens)
    sure = clear > (0.0 if mode[1] == F32 else 0.005)
    assert int(sure.sum()) >= 0.6 * len(tokens) or len(tokens) < 10
    logits_near(got.cpu()[sure], want[sure], mode)


def prompt(case, n, seed):
    return torch.randint(0, CASES[case]["vocab"], (n,), generator=gen(seed)).tolist()


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("case", list(CASES))
def test_model_cuts(mode, case):
    """Whole prompt, token by token, and portions: the same logits at every position."""
    _, _, model = built(case, mode)
    toks = prompt(case, 110, 1)
    eng = engine(model)
    for cuts in ([110], [1] * 110, [2] * 55, [16, 1, 1, 15, 2, 75], [3, 5, 7, 11, 13, 17, 54], [50, 48] + [1] * 12):
        check(play(eng, toks, cuts), case, toks, mode)
        assert eng.kv.num_free == eng.num_pages


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("case", list(CASES))
def test_model_mixed_batches(mode, case):
    """Unequal requests in one batch, portions beside single tokens, requests that pause, and pages that change hands,
    against each request alone."""
    _, _, model = built(case, mode)
    seqs = {k: prompt(case, n, 10 + i) for i, (k, n) in enumerate((("a", 105), ("b", 70), ("c", 1), ("d", 23), ("e", 110), ("f", 9)))}
    eng = engine(model, tokens=320)
    at = {k: 0 for k in seqs}
    got = {k: [] for k in seqs}
    steps = [dict(a=20, b=3), dict(a=1, c=1, b=1), dict(b=60, d=2), dict(a=1, b=1, d=1), dict(a=1, b=1, d=1), dict(a=47, d=19), dict(b=4, e=31),
             dict(a=1, e=1), dict(e=1, a=34), dict(e=1, f=7), dict(f=1, e=76), dict(f=1)]
    for st in steps:
        ents, ends = [], []
        for k, n in st.items():
            ents.append((k, seqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
            if at[k] == len(seqs[k]):
                ends.append(k)
        y = eng.replay(ents, ends)
        for k, n in st.items():
            got[k].append(y[:n])
            y = y[n:]
    assert all(at[k] == len(seqs[k]) for k in seqs) and eng.kv.num_free == eng.num_pages
    for k in seqs:
        check(torch.cat(got[k]), case, seqs[k], mode)


@pytest.mark.parametrize("mode", MODES)
def test_model_stream_per_layer(mode):
    cfg, w, model = built("mixed", mode)
    toks = prompt("mixed", 30, 3)
    want, got = [], []
    O.forward(toks, cfg, w, layers_out=want)
    eng = engine(model)
    model._forward_mixers = lambda b: type(model)._forward_mixers(model, b, got)
    try:
        eng.replay([("a", toks, [])], ["a"])
    finally:
        del model.__dict__["_forward_mixers"]
    assert len(got) == len(want) == len(cfg["layers"])
    for a, b in zip(got, want):
        e = (a.cpu().double() - b).norm(dim=1) / b.norm(dim=1)
        assert float(e.max()) < (2e-5 if mode[1] == F32 else 5e-2), float(e.max())


@pytest.mark.parametrize("mode", MODES)
def test_long_decode(mode):
    _, _, model = built("mixed", mode)
    toks = prompt("mixed", 150, 4)
    check(play(engine(model), toks, [4] + [1] * 146), "mixed", toks, mode)


@pytest.mark.parametrize("mode", MODES)
def test_pool_is_bounded(mode):
    _, _, model = built("mixed", mode)
    eng = engine(model, tokens=64, batch=2)
    assert not model.cfg.recurrent and not eng.kv.state_slots
    eng.replay([("a", prompt("mixed", 33, 0), []), ("b", [1], [])])
    with pytest.raises(KvPoolExhaustedError):
        eng.replay([("c", [1], []), ("b", [2] * 16, [])])
    eng.replay([], ["a", "b", "c"])
    assert eng.kv.num_free == eng.num_pages


# ------------------------------------------------------------------------------------ generation
def greedy(case, toks, n):
    out = list(toks)
    for _ in range(n):
        out.append(int(expected(case, out)[-1].argmax()))
    return out[len(toks):]


@pytest.mark.parametrize("mode", [MODES[0], MODES[1]])
@pytest.mark.parametrize("case", ["mixed", "latent"])
def test_greedy_generation(mode, case):
    """The engine's scheduler: chunked prompts beside decoding requests, then decode steps alone; then a pool so
    small that requests are pre-empted and recomputed."""
    _, _, model = built(case, mode)
    prompts = [prompt(case, n, 20 + n) for n in (37, 5, 18)]
    want = [greedy(case, p, 10) for p in prompts]
    params = SamplingParams(greedy=True, ignore_eos=True, max_tokens=10)
    eng = LLMEngine(model, num_pages=32, page_size=8, max_batch=4, prefill_chunk=16, max_model_len=96)
    assert eng.generate(prompts, params) == want
    assert eng.kv.num_free == 32
    tight = LLMEngine(model, num_pages=9, page_size=8, max_batch=4, prefill_chunk=64, max_model_len=72)
    assert tight.generate(prompts, params) == want
    assert tight.stats()["preemptions"] > 0 and tight.kv.num_free == 9


@pytest.mark.gpu
def test_generation_bf16_graph_equals_eager():
    _, _, model = built("mixed", ("cuda", BF))
    prompts = [prompt("mixed", n, 40 + n) for n in (30, 9, 14, 2, 100)]
    params = SamplingParams(greedy=True, ignore_eos=True, max_tokens=16)
    run = lambda graphs: LLMEngine(model, num_pages=64, page_size=16, max_batch=8, prefill_chunk=64, max_model_len=128,
                                   use_cuda_graphs=graphs).generate(prompts, params)
    assert run(True) == run(False)


@pytest.mark.parametrize("mode", [MODES[0], MODES[2]])
def test_sampled_generation(mode):
    _, _, model = built("mixed", mode)
    eng = engine(model)
    params = SamplingParams(temperature=0.8, top_k=20, top_p=0.9, seed=3, ignore_eos=True, max_tokens=6)
    p = prompt("mixed", 11, 2)
    a, b = eng.generate([p], params), eng.generate([p], params)
    assert a == b and len(a[0]) == 6


# ------------------------------------------------------------------------------------ framework entry points
@pytest.fixture
def checkpoint(tmp_path):
    save_hf_checkpoint(CASES["mixed"], rand_weights(CASES["mixed"]), tmp_path / "m")
    return tmp_path / "m"


def test_checkpoint_loads_by_config(checkpoint):
    llm = load_llm(checkpoint, "cpu", dtype=F32)
    assert llm.config.arch == "zovudra" and llm.model.dtype == F32
    toks = prompt("mixed", 12, 8)
    y = engine(llm.model).replay([("x", toks, [11])], ["x"])
    logits_near(y, expected("mixed", toks)[11:], ("cpu", F32))
    with pytest.raises(ValueError):
        llm.config.validate_tp(2)
    total = sum(v.numel() for v in rand_weights(CASES["mixed"]).values())
    assert abs(llm.config.param_count() / total - 1) < 0.02 and llm.model.weight_bytes() > 2 * total


@pytest.mark.parametrize("bad", [lat(2, 8, 8, 8, 520, 8, 4), lat(2, 8, 5, 8, 16, 8, 4), att(3, 2, 8, 8, 8, 4, 1), att(2, 1, 8, 8, 10, 4, 1), att(2, 1, 520, 8, 8, 4, 1),
                                 att(2, 1, 8, 8, 8, 4, 1, mlp=moe(10, 2, 8, 4, 2, 1.0, 8)), att(2, 1, 8, 8, 8, 4, 1, mlp=moe(8, 3, 8, 4, 1, 1.0, 8)),
                                 {**att(2, 1, 8, 8, 8, 4, 1), "type": "other"}, att(2, 1, 8, 8, 8, 4, 1, mlp={"kind": "other"})])
def test_sizes_without_a_kernel_are_refused(bad):
    cfg = model_cfg(20, 16, [bad])
    with pytest.raises(ValueError):
        DecoderModel(config_from(cfg), "cpu").load_state_dict(rand_weights(cfg).get)


def test_absent_options():
    """No mask, no groups, no shared expert, no token input: the plain forms."""
    layers = [att(2, 1, 16, 16, 16, 0, 0, mlp=moe(4, 2, 16, 1, 1, 1.0, 8)), lat(2, 16, 8, 8, 24, 16, 0, mlp=dense(16))]
    for layer in layers:
        del layer["mixer"]["mask"]
    del layers[0]["mlp"]["shared"], layers[0]["mlp"]["router"]["groups"]
    cfg = model_cfg(40, 32, layers)
    del cfg["token_side"]
    w = rand_weights(cfg)
    assert not any("side" in n or "shared" in n for n in w)
    model = DecoderModel(config_from(cfg), "cpu", dtype=F32)
    model.load_state_dict(w.get)
    toks = torch.randint(0, 40, (40,), generator=gen(1)).tolist()
    logits_near(play(engine(model), toks, [20, 1, 1, 18]), O.forward(toks, cfg, w), ("cpu", F32))


def test_checkpoint_is_recognised(checkpoint):
    from hartsyinference_b200.assets.registry import detect
    from hartsyinference_b200.engine.planner import shape_of_checkpoint
    d = detect(checkpoint)
    assert (d.family, d.arch) == ("llm", "zovudra")
    assert shape_of_checkpoint(checkpoint) is None          # stays on one GPU


def test_service_generates_and_embeds(checkpoint):
    """Through the text service: token ids in, greedy ids out as the engine gives them; embedding a text in between
    leaves the running requests' pages alone."""
    from hartsyinference_b200.engine.requests import EngineOptions, Modality, ModelSpec, TextRequest
    from hartsyinference_b200.engine.text_service import TextService
    svc = TextService(EngineOptions(max_batch=2, max_model_len=64), device="cpu")
    spec = ModelSpec("m", Modality.TEXT, local_path=str(checkpoint))
    req = TextRequest(messages=[], prompt_token_ids=prompt("mixed", 20, 5), max_tokens=6, greedy=True, ignore_eos=True)
    try:
        a = svc.generate(spec, req).token_ids
        e = svc.embed(spec, ["abc", "abcd"])
        assert e.shape == (2, CASES["mixed"]["width"]) and torch.isfinite(e).all()
        assert svc.generate(spec, req).token_ids == a and len(a) == 6
    finally:
        svc.release()


@pytest.mark.parametrize("mode", [MODES[0], MODES[1]])
def test_trace_run(checkpoint, tmp_path, monkeypatch, capsys, mode):
    from hartsyinference_b200.cli import trace
    toks = prompt("mixed", 40, 6)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": toks[:30], "want": [0, 29]}, {"id": "b", "tokens": toks[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": toks[3:4], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": toks[30:], "want": [9]}, {"id": "c", "tokens": toks[:2], "want": [1]}], "end": ["a", "c"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(x) for x in lines) + "\n"))
    out = tmp_path / "o"
    assert trace.main(["--model", str(checkpoint), "--dtype", "float32", "--out", str(out), "--max-tokens", "128", "--device", mode[0]]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    read = lambda n: torch.frombuffer(bytearray((out / n).read_bytes()), dtype=F32).reshape(-1, CASES["mixed"]["vocab"])
    want = expected("mixed", toks)
    logits_near(read("0.f32"), want[[0, 29]], mode)
    logits_near(read("2.f32"), want[[39, 1]], mode)


def test_text_command(checkpoint):
    from click.testing import CliRunner
    from hartsyinference_b200.cli.main import cli
    r = CliRunner().invoke(cli, ["text", str(checkpoint), "hello", "--raw", "--greedy", "--max-tokens", "4", "--device", "cpu"])
    assert r.exit_code == 0, r.output
