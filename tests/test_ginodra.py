"""Ginodra against the plain statement in ``ginodra_oracle``: every mechanism alone, then whole models through the
engine (prompts, portions, decoding, mixed batches, reused pages and slots, generation).

Each case runs on the CPU ops and, marked ``gpu``, on the kernels in fp32 and bf16."""
import io
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import ginodra_oracle as O  # noqa: E402
from test_lududra import BF, F32, MODES, Pages, _Holder, gen, logits_near, near, rel_err, rnd  # noqa: E402
from test_salopel import _Batch, _PagedBatch, check_slots_left_alone, engine, play, run_cuts  # noqa: E402
from test_zovudra import plant, run_portions  # noqa: E402

from hartsyinference_b200 import ops  # noqa: E402
from hartsyinference_b200.engine import LLMEngine, SamplingParams  # noqa: E402
from hartsyinference_b200.exceptions import KvPoolExhaustedError  # noqa: E402
from hartsyinference_b200.models.llm import config as C  # noqa: E402
from hartsyinference_b200.models.llm import mixers as M  # noqa: E402
from hartsyinference_b200.models.llm.ginodra import config_from, tensor_shapes  # noqa: E402
from hartsyinference_b200.models.llm.loader import load_llm, save_hf_checkpoint  # noqa: E402
from hartsyinference_b200.models.llm.rope import Rotary  # noqa: E402
from hartsyinference_b200.models.llm.transformer import DecoderModel  # noqa: E402

i32 = lambda v, dev: torch.tensor(v, dtype=torch.int32, device=dev)
up8 = lambda n: (n + 7) // 8 * 8
WIDTH = 24


# ------------------------------------------------------------------------------------ norms, convolutions, logits
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("dim,groups", [(40, 5), (132, 3), (96, 32), (1000, 8), (120, 1), (2048, 16), (8192, 2), (9000, 9), (60, 60)])
def test_stream_norm_in_groups(mode, dim, groups):
    """Parts of very different size beside each other, parts that begin inside a vector, with and without a new term."""
    dev, dt = mode
    g = gen(dim)
    rows, ld = 5, up8(dim)
    size = torch.logspace(-2, 2, groups).repeat_interleave(dim // groups)
    x, y = torch.zeros(rows, ld), torch.zeros(rows, ld, dtype=BF)
    x[:, :dim] = torch.randn(rows, dim, generator=g) * size
    y[:, :dim] = rnd(g, rows, dim)
    w = rnd(g, dim, std=0.3) + 1
    kw = dict(dim=dim, eps=1e-3, layernorm=False, dtype=dt, mult=0.6, groups=groups)
    xd = x.clone().to(dev)
    h = ops.residual_norm(xd, None, None, w.to(dev), **kw)
    near(h[:, :dim], O.group_norm(x[:, :dim].double(), w.double(), groups, 1e-3), mode, 1e-6, 4e-3)
    h = ops.residual_norm(xd, y.to(dt).to(dev), None, w.to(dev), **kw)
    want = x[:, :dim].double() + 0.6 * y[:, :dim].double()
    assert rel_err(xd[:, :dim], want) < 1e-6 and float(h[:, dim:].float().abs().sum()) == 0
    near(h[:, :dim], O.group_norm(want, w.double(), groups, 1e-3), mode, 1e-6, 4e-3)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("taps,sets,dim,groups", [(4, 2, 40, 5), (1, 2, 24, 1), (2, 1, 264, 3), (3, 2, 1040, 8), (6, 2, 44, 4), (4, 1, 9000, 2), (8, 1, 16, 2)])
def test_input_convolutions(mode, taps, sets, dim, groups):
    """Portions down to one and two tokens beside another sequence, then decoding behind the norm in the same launch; the
    slots hold what earlier sequences left."""
    dev, dt = mode
    g = gen(taps * dim)
    ld, lens = up8(dim), [47, 21, 30]
    x = [torch.nn.functional.pad(torch.randn(n, dim, generator=g), (0, ld - dim)) for n in lens]
    nw, cw = rnd(g, dim, std=0.3) + 1, rnd(g, sets, dim, taps, std=0.5)
    want = []
    for v in x:
        h = O.group_norm(v[:, :dim].double(), nw.double(), groups, 1e-4)
        h = h.to(dt).double()                      # what the state holds is in the activation type
        want.append(torch.stack([O.input_conv(h, cw[i].double()) for i in range(sets)]))
    w = torch.zeros(sets, taps, ld)
    w[:, :, :dim] = cw.float().transpose(1, 2)
    w, state, slots = w.to(dev).contiguous(), torch.full((4, taps - 1, ld), 3.0, dtype=dt, device=dev), [2, 0, 3]
    kw = dict(dim=dim, eps=1e-4, layernorm=False, dtype=dt, groups=groups)
    got = [torch.zeros(sets, n, dim) for n in lens]
    done = [0, 0, 0]

    def step(counts, decode=False):
        use = [(i, n) for i, n in enumerate(counts) if n]
        pos, cu = [], [0]
        for i, n in use:
            pos += range(done[i], done[i] + n)
            cu.append(cu[-1] + n)
        rows = torch.cat([x[i][done[i]:done[i] + n] for i, n in use]).to(dev).contiguous()
        p, s = i32(pos, dev), i32([slots[i] for i, _ in use], dev)
        if decode:
            y = ops.residual_norm(rows, None, None, nw.to(dev), conv=(w, state, p, s), **kw)
        else:
            y = ops.input_conv(ops.residual_norm(rows, None, None, nw.to(dev), **kw), w, state, p, i32(cu, dev), s)
        assert y.shape == (sets, cu[-1], ld) and float(y[..., dim:].float().abs().sum()) == 0
        for (i, n), a in zip(use, cu):
            got[i][:, done[i]:done[i] + n] = y[:, a:a + n, :dim].float().cpu()
            done[i] += n

    for counts in ((17, 2, 0), (2, 1, 9), (1, 5, 1), (9, 0, 2), (3, 3, 10)):
        step(counts)
    while any(d < n for d, n in zip(done, lens)):
        step([int(d < n) for d, n in zip(done, lens)], True)
    for a, b in zip(got, want):
        near(a, b, mode, 1e-6, 4e-3)
        near(a[:, :taps], b[:, :taps], mode, 1e-6, 4e-3)      # the first tokens see zeros before them
    before = state.clone()
    p, s, rows = i32([5], dev), i32([-1], dev), x[0][:1].to(dev).contiguous()
    ops.residual_norm(rows, None, None, nw.to(dev), conv=(w, state, p, s), **kw)
    ops.input_conv(ops.residual_norm(rows, None, None, nw.to(dev), **kw), w, state, p, i32([0, 1], dev), s)
    assert torch.equal(state, before) and (taps == 1 or float(state[1].float().min()) == 3.0)


@pytest.mark.parametrize("mode", MODES[1:])
def test_long_input_convolution(mode):
    """Enough tokens for many per warp, an empty run between two sequences, against the same tokens in pieces."""
    dev, dt = mode
    g = gen(4)
    h, w = rnd(g, 3000, 1040).to(dt).to(dev), (torch.randn(2, 4, 1040, generator=g) * 0.5).to(dev)
    state = torch.full((3, 3, 1040), 2.0, dtype=dt, device=dev)
    whole = ops.input_conv(h, w, state, i32(list(range(1203)) + list(range(1797)), dev), i32([0, 1203, 1203, 3000], dev), i32([0, 1, 2], dev))
    after = state.clone()
    for a, b, slot in ((0, 1203, 0), (1203, 3000, 2)):
        for c in range(a, b, 101):
            e = min(c + 101, b)
            y = ops.input_conv(h[c:e], w, state, i32(list(range(c - a, e - a)), dev), i32([0, e - c], dev), i32([slot], dev))
            assert torch.equal(y, whole[:, c:e])
    assert torch.equal(state, after)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("scale,cap", [(0.3, 5.0), (2.0, 0.7), (1.5, 0.0)])
def test_capped_logits(mode, scale, cap):
    dev, dt = mode
    y = (torch.randn(7, 101, generator=gen(1)) * 9).to(BF)
    z = y.double() * scale
    got = ops.cap_logits(y.to(dt).to(dev), scale, cap)
    assert got.dtype == F32 and rel_err(got, cap * torch.tanh(z / cap) if cap else z) < 1e-6


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("m,n,k,start", [(3, 40, 24, 16), (5, 264, 4096, 200), (300, 136, 64, 128), (20, 64, 72, 0)])
def test_tanh_of_the_last_columns(mode, m, n, k, start):
    """Also where the product is cut along its inner dimension, and into a wider buffer."""
    dev, dt = mode
    g = gen(n + k)
    x, w = rnd(g, m, k), rnd(g, n, k, std=2 * k ** -0.5)
    want = x.double() @ w.double().T
    want[:, start:] = torch.tanh(want[:, start:])
    buf = torch.full((m, n + 24), 7.0, dtype=dt, device=dev)
    ops.linear_act(x.to(dt).to(dev), ops.LinearWeight(w.to(dev)), "tanh", act_from=start, out=buf[:, 16:16 + n])
    near(buf[:, 16:16 + n], want, mode, 2e-6, 5e-3)
    assert bool((buf[:, :16] == 7.0).all()) and bool((buf[:, 16 + n:] == 7.0).all())


# ------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,hkv,d,dt_,dv,page,rot", [(4, 2, 32, 32, 32, 16, None), (3, 1, 16, 12, 40, 8, None), (6, 3, 104, 100, 24, 16, None),
                                                         (5, 5, 200, 200, 8, 64, None), (2, 1, 320, 320, 16, 16, None), (17, 1, 64, 64, 64, 16, (24, False)),
                                                         (2, 2, 48, 48, 8, 16, (16, True))])
def test_head_norms_and_store(mode, heads, hkv, d, dt_, dv, page, rot):
    """Large heads beside small ones, padded heads, tokens that are not stored; queries alone."""
    dev, dt = mode
    g = gen(d + dv)
    n = 70
    size = torch.logspace(-2, 1, heads + hkv)[:, None].expand(-1, d).reshape(-1)
    p = torch.cat([rnd(g, n, (heads + hkv) * d) * size, rnd(g, n, hkv * dv)], 1).to(BF)
    p[:, :(heads + hkv) * d].view(n, heads + hkv, d)[..., dt_:] = 0
    qw, kw = rnd(g, d, std=0.4) + 1, rnd(g, d, std=0.4) + 1
    x = p[:, :(heads + hkv) * d].double().view(n, heads + hkv, d)
    table = None
    if rot:
        b = _Holder()
        b.positions, b.plan = i32(list(range(n)), dev), None
        table = Rotary(C.RotarySpec(rot[0], 300.0, rot[1]), dev).table(b)

    def head(h):
        w = (qw if h < heads else kw).double()
        y = torch.zeros(n, d, dtype=torch.float64)
        y[:, :dt_] = O.rms(x[:, h, :dt_], w[:dt_], 0.01)
        if rot:
            r = rot[0]
            part = y[:, :r]
            if rot[1]:                                        # pairs of neighbours as split halves
                part = torch.cat([part[:, 0::2], part[:, 1::2]], 1)
            part = O.rotate(part, 300.0)
            y[:, :r] = torch.stack([part[:, :r // 2], part[:, r // 2:]], 2).reshape(n, r) if rot[1] else part
        return y

    want_q, want_k = torch.cat([head(h) for h in range(heads)], 1), torch.cat([head(heads + h) for h in range(hkv)], 1)
    pk, pv = Pages(gen(1), [n], hkv, d, page, dt, dev), Pages(gen(1), [n], hkv, dv, page, dt, dev)
    before = pk.cache.clone()
    slots = pk.slots(0, 0, n)
    slots[7] = -1
    kwargs = dict(table=table, interleaved=bool(rot and rot[1]), eps=0.01, d_true=dt_, per_head=True)
    got = ops.qk_rope_store(p.to(dt).to(dev), heads, pk.cache, pv.cache, slots.to(dev), q_norm=qw.to(dev), k_norm=kw.to(dev), **kwargs)
    near(got, want_q, mode, 1e-6, 4e-3)
    at = slots[slots >= 0]
    rows = lambda c: c.cpu()[at // page, :, at % page].reshape(n - 1, -1)
    near(rows(pk.cache), want_k[slots >= 0], mode, 1e-6, 4e-3)
    assert torch.equal(rows(pv.cache).to(BF), p[slots >= 0][:, (heads + hkv) * d:])
    seven = pk.slots(0, 7, 1)
    assert torch.equal(pk.cache[seven // page, :, seven % page], before[seven // page, :, seven % page])
    held = pk.cache.clone()
    alone = ops.qk_rope_store(p[:, :heads * d].to(dt).to(dev), heads, pk.cache, pv.cache, slots.to(dev), q_norm=qw.to(dev), store=False, **kwargs)
    assert torch.equal(alone, got) and torch.equal(pk.cache, held)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("hq,hkv,d,dv,page,window,tail", [
    (6, 2, 64, 64, 16, 50, 1), (6, 2, 64, 64, 16, 50, 70), (6, 2, 40, 24, 8, 17, 3), (8, 8, 128, 64, 16, 65, 130), (3, 1, 16, 104, 64, 1, 5),
    (20, 1, 24, 24, 16, 130, 1), (2, 1, 160, 32, 16, 33, 9), (16, 1, 96, 128, 32, 64, 1), (4, 4, 8, 8, 16, 1000, 2), (4, 2, 32, 32, 16, 0, 40),
    (9, 3, 64, 128, 16, 16, 1), (2, 1, 48, 200, 16, 70, 33)])
def test_window_with_slopes_and_head_gates(mode, hq, hkv, d, dv, page, window, tail):
    """Four sequences whose last ``tail`` tokens are the queries. Keys just inside and just outside the window, at page and
    tile edges and the first one each stand out for some query, by enough to outweigh the distance."""
    dev, dt = mode
    g = gen(hq * 100 + d + window)
    lens = [tail + 300, tail + 2, max(tail, 5), tail + 130]
    scale, group = 0.8, hq // hkv
    slopes = torch.tensor([O.slope(h, hq) for h in range(hq)], dtype=torch.float32)
    q = [rnd(g, n, hq, d, std=d ** -0.5) for n in lens]
    k, v = [rnd(g, n, hkv, d) for n in lens], [rnd(g, n, hkv, dv) for n in lens]
    for i, n in enumerate(lens):
        for r in range(n - tail, n, max(1, tail // 7)):
            spots = [r - window + 1, r - window, 0, r // page * page, r // page * page - 1, 63, 64, r]
            for h, spot in enumerate(spots):
                if 0 <= spot <= r:
                    at = (h + r) % hq
                    lift = float(slopes[at]) * (r - spot) / scale / float(q[i][r, at].float().norm())
                    plant(q[i], k[i], r, spot, at, at // group, 4.0 + (lift if lift < 40 else 0.0))
    gates = rnd(g, tail * len(lens), up8(hq), std=2.0)
    pk, pv = Pages(gen(3), lens, hkv, d, page, dt, dev), Pages(gen(3), lens, hkv, dv, page, dt, dev)
    for i, n in enumerate(lens):
        ops.kv_store(k[i].reshape(n, -1).to(dt).to(dev), pk.cache, pk.slots(i, 0, n).to(dev))
        ops.kv_store(v[i].reshape(n, -1).to(dt).to(dev), pv.cache, pv.slots(i, 0, n).to(dev))
    want = torch.cat([torch.cat([O.causal_attention(q[i][:, h].double(), k[i][:, h // group].double(), v[i][:, h // group].double(), scale, window,
                                                    O.slope(h, hq))[-tail:] for h in range(hq)], 1) for i in range(len(lens))])
    want = want * O.sigmoid(gates[:, :hq].double()).repeat_interleave(dv, 1)
    rows, gd = torch.cat([x[-tail:].reshape(tail, -1) for x in q]).to(dt).to(dev), gates.to(dt).to(dev)
    buf = torch.full((len(rows), hq * dv + 16), 7.0, dtype=dt, device=dev)

    def run(cu):
        ops.attn_biased(rows, pk.cache, pv.cache, pk.table.to(dev), i32(lens, dev), cu, heads=hq, max_q_len=tail, max_kv_len=max(lens), scale=scale,
                        window=window, slopes=slopes.to(dev), gate=gd, head_gate=True, out=buf[:, 8:8 + hq * dv])
        assert bool((buf[:, :8] == 7.0).all()) and bool((buf[:, 8 + hq * dv:] == 7.0).all())
        return buf[:, 8:8 + hq * dv]
    near(run(i32([tail * i for i in range(len(lens) + 1)], dev)), want, mode, 1e-5, 1e-2)
    if tail == 1:
        near(run(None), want, mode, 1e-5, 1e-2)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,rank,rot,page", [(5, 64, 48, 16), (6, 40, 8, 8), (17, 128, 64, 16), (33, 24, 104, 16), (3, 512, 64, 32), (2, 160, 200, 16), (1, 8, 8, 64)])
def test_latent_rows_with_sinks(mode, heads, rank, rot, page):
    """Sinks from far below to far above the scores: what each leaves of the output is told apart; also a context that is
    cut into several ranges, and an empty one."""
    dev, dt = mode
    g = gen(heads * 10 + rank)
    lens = [900, 1, 65, 128, page + 1]
    row = rank + rot
    pg = Pages(g, lens, 1, row, page, dt, dev)
    lat = [rnd(g, n, row) for n in lens]
    sinks = torch.linspace(-3, 8, heads)[torch.randperm(heads, generator=g)].to(BF).float()
    rows = [(i, m) for i, n in enumerate(lens) for m in sorted({n, max(1, n // 2)}, reverse=True)]
    q = rnd(g, len(rows), heads, row, std=row ** -0.5)
    for r, (i, n) in enumerate(rows):
        for h, spot in enumerate((n - 1, 0, page - 1, page, 63, 64)):
            if 0 <= spot < n:
                part = slice(0, rank) if h % 2 else slice(rank, row)
                lat[i][spot, part] += (torch.nn.functional.normalize(q[r, h % heads, part].float(), dim=0) * 5).to(BF)
    for i, n in enumerate(lens):
        ops.kv_store(lat[i].to(dt).to(dev), pg.cache, pg.slots(i, 0, n).to(dev))
    want = []
    for r, (i, n) in enumerate(rows):
        c = lat[i][:n].double()
        out = []
        for h in range(heads):
            s = torch.cat([c @ q[r, h].double() * 1.7, sinks[h:h + 1].double()])
            out.append(torch.softmax(s, 0)[:-1] @ c[:, :rank])
        want.append(torch.cat(out))
    qd = q.reshape(len(rows), -1).to(dt).to(dev)
    out = ops.latent_attn(qd, pg.cache, pg.table.to(dev), i32([n for _, n in rows], dev), heads, 1.7, row_seq=i32([i for i, _ in rows], dev),
                          max_kv_len=max(lens), v_dim=rank, sinks=sinks.to(dev))
    near(out, torch.stack(want), mode, 1e-5, 6e-3)
    ends = [r for r, (i, n) in enumerate(rows) if n == lens[i]]
    out = ops.latent_attn(qd[ends].contiguous(), pg.cache, pg.table.to(dev), i32(lens[:-1] + [0], dev), heads, 1.7, max_kv_len=4096, v_dim=rank,
                          sinks=sinks.to(dev))               # one row per sequence (decode), the last one empty
    near(out[:-1], torch.stack(want)[ends][:-1], mode, 1e-5, 6e-3)
    assert float(out[-1].float().abs().max()) == 0


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,n,k,rows", [(3, 40, 24, 5), (6, 72, 64, 130), (16, 128, 512, 64), (9, 8, 200, 1)])
def test_head_linear_with_head_gates(mode, heads, n, k, rows):
    dev, dt = mode
    g = gen(n + k)
    x, w, gates = rnd(g, rows, heads, k), rnd(g, heads * n, k, std=k ** -0.5), rnd(g, rows + 3, up8(heads), std=2.0)
    at = torch.randperm(rows + 3, generator=g)[:rows]
    y = torch.stack([x[:, h].double() @ w[h * n:(h + 1) * n].double().T for h in range(heads)], 1)
    want = (y * O.sigmoid(gates[at, :heads].double())[:, :, None]).reshape(rows, -1)
    buf = torch.full((rows + 3, heads * n + 8), 7.0, dtype=dt, device=dev)
    ops.head_linear(x.reshape(rows, -1).to(dt).to(dev), ops.LinearWeight(w.to(dev)), heads, gate=gates.to(dt).to(dev), head_gate=True,
                    out=buf[:, :heads * n], out_rows=at.to(torch.int32).to(dev))
    near(buf.cpu()[at][:, :heads * n], want, mode, 1e-6, 5e-3)
    rest = torch.ones(rows + 3, dtype=torch.bool)
    rest[at] = False
    assert bool((buf.cpu()[rest] == 7.0).all()) and bool((buf[:, heads * n:] == 7.0).all())


@pytest.mark.gpu
@pytest.mark.parametrize("heads,own,rot,dv", [(3, 64, 48, 72), (5, 40, 16, 24), (2, 64, 64, 128), (9, 16, 8, 104), (3, 128, 64, 128), (2, 104, 0, 64)])
def test_runs_with_sinks_and_head_gates(heads, own, rot, dv):
    """Runs that are not adjacent, over whole contexts, into a wider buffer."""
    g = gen(own + dv)
    d = own + rot
    runs, starts, t = [(70, 70), (3, 200), (129, 130), (64, 321)], [10, 100, 105, 240], 310           # (queries, keys)
    q, gates = rnd(g, t, heads, d, std=d ** -0.5), rnd(g, t, up8(heads), std=2.0)
    sinks = torch.linspace(-2, 7, heads)
    table, qt = None, q.double().clone()
    if rot:
        b = _Holder()
        b.positions, b.plan = i32([7 * i % 1000 for i in range(t)], "cuda"), None
        table = Rotary(C.RotarySpec(rot, 50.0, True), "cuda").table(b)
        tc = table.cpu().double()
        u, v = qt[..., own::2].clone(), qt[..., own + 1::2].clone()
        qt[..., own::2], qt[..., own + 1::2] = u * tc[:, None, :, 0] - v * tc[:, None, :, 1], v * tc[:, None, :, 0] + u * tc[:, None, :, 1]
    ks, ss, vs, want = [], [], [], torch.zeros(t, heads * dv, dtype=torch.float64)
    for (nq, nk), a in zip(runs, starts):
        k, sh, vv = rnd(g, nk, heads, own), rnd(g, nk, rot), rnd(g, nk, heads, dv)
        for h in range(heads):
            full = torch.cat([k[:, h], sh], 1).double()
            for i in range(nq):
                n = nk - nq + i + 1
                s = torch.softmax(torch.cat([full[:n] @ qt[a + i, h] * 2.5, sinks[h:h + 1].double()]), 0)[:-1]
                want[a + i, h * dv:(h + 1) * dv] = s @ vv[:n, h].double() * O.sigmoid(gates[a + i, h].double())
        ks.append(k.reshape(nk, -1)), ss.append(sh), vs.append(vv.reshape(nk, -1))
    buf = torch.full((t, heads * dv + 16), 7.0, dtype=BF, device="cuda")
    at = [0]
    for _, nk in runs:
        at.append(at[-1] + nk)
    kv, sh = torch.cat([torch.cat(ks), torch.cat(vs)], 1).cuda(), torch.cat(ss).cuda()
    c = lambda v: i32(v, "cuda")
    ops.attn_runs(q.reshape(t, -1).cuda(), kv[:, :heads * own], kv[:, heads * own:], buf[:, 8:8 + heads * dv], c(starts), c([r[0] for r in runs]), c(at),
                  c([r[1] for r in runs]), heads=heads, max_q_len=129, scale=2.5, k_shared=sh if rot else None, table=table, sinks=sinks.cuda(),
                  gate=gates.cuda(), head_gate=True)
    mine = torch.zeros(t, dtype=torch.bool)
    for (nq, _), a in zip(runs, starts):
        mine[a:a + nq] = True
    near(buf.cpu()[mine][:, 8:8 + heads * dv], want[mine], ("cuda", BF), bf16=1e-2)
    assert bool((buf.cpu()[~mine] == 7.0).all()) and bool((buf[:, :8] == 7.0).all()) and bool((buf[:, -8:] == 7.0).all())


# ------------------------------------------------------------------------------------ mixers
CUTS = [(60, 2, 0), (2, 50, 1), (49, 1, 2), (1, 0, 1), (47, 1, 1), (64, 2, 1), (3, 1, 0)]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,kv,dim,vdim,window,scale", [(4, 2, 16, 16, 20, 1.0), (6, 3, 40, 24, 33, 0.3), (3, 1, 20, 12, 50, 0.5),
                                                            (2, 2, 64, 80, 17, 0.2), (5, 1, 12, 136, 9, 0.7), (8, 8, 8, 8, 0, 0.9), (16, 4, 16, 8, 64, 1.0)])
def test_attention_mixers_on_shared_keys(mode, heads, kv, dim, vdim, window, scale):
    """A layer with keys and values of its own and, behind it, one that reads them with another window and scale."""
    dev, dt = mode
    g = gen(dim + vdim)
    mix = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale, mask=dict(size=window))
    mix2 = {**mix, "scale": scale * 0.5, "mask": dict(size=window // 2 + 1)}
    shapes = {"q": (heads * dim, WIDTH), "k": (kv * dim, WIDTH), "v": (kv * vdim, WIDTH), "o": (WIDTH, heads * vdim), "g": (heads, WIDTH)}
    t = {n: rnd(g, *s, std=s[1] ** -0.5) for n, s in shapes.items()}
    t2 = {n: rnd(g, *shapes[n], std=shapes[n][1] ** -0.5) for n in "qog"}
    for x in (t, t2):
        x["q.norm"], x["g"] = rnd(g, dim, std=0.4) + 1, x["g"] * 2
    t["k.norm"] = rnd(g, dim, std=0.4) + 1
    hs = [rnd(g, 250, WIDTH), rnd(g, 60, WIDTH), rnd(g, 9, WIDTH)]
    wd = {"a." + n: v.double() for n, v in t.items()} | {"b." + n: v.double() for n, v in t2.items()}
    kvs = [O.keys_values(h.double(), mix, wd, "a.", 1e-3) for h in hs]
    want = [O.attention_mixer(h.double(), mix, wd, "a.", 1e-3, x) + O.attention_mixer(h.double(), mix2, wd, "b.", 1e-3, x) for h, x in zip(hs, kvs)]
    spec = lambda m, src: C.MixerSpec(kind="attention", heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=m["scale"], window=m["mask"]["size"],
                                      head_norm=True, slope_bias=True, head_gate=True, kv_from=src)
    own = M.BiasedAttention(spec(mix, None), WIDTH, dev, q=t["q"], k=t["k"], v=t["v"], o=t["o"], gate=t["g"], q_norm=t["q.norm"], k_norm=t["k.norm"], eps=1e-3)
    other = M.BiasedAttention(spec(mix2, 0), WIDTH, dev, q=t2["q"], o=t2["o"], gate=t2["g"], q_norm=t2["q.norm"], eps=1e-3)
    assert hasattr(own, "cache_shape") and not hasattr(other, "cache_shape")

    class Both:
        def __call__(self, h, batch, li, holder):
            holder.kv_cache = holder.kv_cache[:1] + [None]
            return own(h, batch, 0, holder).float() + other(h, batch, 1, holder).float()
    pages = Pages(g, [len(h) for h in hs], 1, 8, 16, dt, dev)
    cache = torch.full(own.cache_shape(pages.cache.shape[0], 16), 5.0, dtype=dt, device=dev)
    for a, b in zip(run_portions(Both(), hs, pages, cache, CUTS, [1, 0, 2], dt, dev), want):
        near(a, b, mode, 5e-5, 2e-2)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,dim,rot,vdim,kv_rank,q_rank,scale", [(3, 16, 8, 24, 32, 20, 1.5), (6, 40, 6, 8, 72, 12, 0.7), (2, 64, 32, 64, 20, 48, 1.0),
                                                                     (18, 8, 16, 12, 16, 9, 2.0), (2, 20, 10, 136, 24, 16, 1.0), (2, 128, 64, 128, 96, 32, 0.5),
                                                                     (1, 200, 8, 16, 40, 8, 0.5), (9, 24, 0, 16, 32, 8, 1.0)])
def test_latent_attention_mixer(mode, heads, dim, rot, vdim, kv_rank, q_rank, scale):
    """Split halves turned, sinks that matter, one gate per head: long runs (expanded keys) beside short ones, then
    decoding."""
    dev, dt = mode
    g = gen(dim + vdim)
    mix = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale, rot=dict(dims=rot, base=90.0))
    shapes = {"dq": (q_rank, WIDTH), "uq": (heads * (dim + rot), q_rank), "dkv": (kv_rank + rot, WIDTH), "uk": (heads * dim, kv_rank),
              "uv": (heads * vdim, kv_rank), "o": (WIDTH, heads * vdim), "g": (heads, WIDTH)}
    t = {n: rnd(g, *s, std=s[1] ** -0.5) for n, s in shapes.items()}
    t["g"] = t["g"] * 2
    t["dq.norm"], t["dkv.norm"], t["sink"] = rnd(g, q_rank, std=0.3) + 1, rnd(g, kv_rank, std=0.3) + 1, rnd(g, heads, std=3.0)
    hs = [rnd(g, 250, WIDTH), rnd(g, 60, WIDTH), rnd(g, 9, WIDTH)]
    wd = {"mix." + n: v.double() for n, v in t.items()}
    want = [O.latent_attention_mixer(h.double(), mix, wd, "mix.", 1e-4) for h in hs]
    spec = C.MixerSpec(kind="latent_attention", heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale, rot_dim=rot, head_gate=True,
                       rot=C.RotarySpec(rot, 90.0) if rot else None)
    t["sinks"] = t.pop("sink")
    m = M.LatentAttention(spec, WIDTH, 1e-4, dev, **{n.replace(".", "_"): v for n, v in t.items()})
    pages = Pages(g, [len(h) for h in hs], 1, m.r + m.t, 16, dt, dev)
    for a, b in zip(run_portions(m, hs, pages, pages.cache[None], CUTS, [1, 0, 2], dt, dev), want):
        near(a, b, mode, 5e-5, 3e-2)


def delta_case(g, heads, dim, rank):
    mix, n = dict(heads=heads, dim=dim), heads * dim
    shapes = {"w1": (rank, WIDTH), "w2": (n, rank), "o": (WIDTH, n), **{x: (n, WIDTH) for x in "rkvga"}}
    t = {x: rnd(g, *s, std=s[1] ** -0.5) for x, s in shapes.items()}
    t["w0"], t["a.b"], t["norm"] = rnd(g, n) - 5.0, rnd(g, n), rnd(g, n, std=0.3) + 1         # slow decay: early writes still count
    t["k"] = t["k"] * torch.logspace(-0.5, 0.5, heads).repeat_interleave(dim)[:, None].to(BF)     # keys that are not near unit length
    return mix, t


def build_delta(mix, t, dev, eps=1e-3):
    spec = C.MixerSpec(kind="general_delta", heads=mix["heads"], kv_heads=mix["heads"], dim=mix["dim"], vdim=mix["dim"])
    return M.GeneralDeltaMixer(spec, WIDTH, eps, dev, a_bias=t["a.b"], **{n: v for n, v in t.items() if n != "a.b"})


def used_slots(m, dev, slots=3):
    """State slots that hold what an earlier sequence left there."""
    conv, rec = m.state_shapes(slots)
    assert conv is None
    return [(torch.zeros(0, device=dev), torch.full(rec, -2.0, dtype=F32, device=dev))]


DELTA_SIZES = [(2, 32, 8), (4, 24, 5), (3, 64, 16), (2, 128, 12), (1, 160, 9), (2, 256, 20), (6, 40, 3), (1, 96, 40), (2, 192, 8), (5, 8, 1), (1, 224, 8)]
DELTA_CUTS = ((17, 0), (2, 5), (1, 2), (16, 1), (3, 9), (0, 2), (64, 3), (65, 1), (7, 0))


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", DELTA_SIZES, ids=str)
def test_general_delta_mixer(mode, sizes):
    """Portions down to one and two tokens beside another sequence, then decoding; every cut gives what the whole sequence
    gives, whatever the slots held before."""
    dev, dt = mode
    g = gen(sum(sizes))
    mix, t = delta_case(g, *sizes)
    hs = [rnd(g, 190, WIDTH), rnd(g, 29, WIDTH)]
    wd = {"mix." + n: v.double() for n, v in t.items()}
    m = build_delta(mix, t, dev)
    state = used_slots(m, dev)
    for got, h in zip(run_cuts(m, state, hs, [2, 0], DELTA_CUTS, dt, dev), hs):
        near(got, O.general_delta_mixer(h.double(), mix, wd, "mix.", 1e-3), mode, 3e-5, 2.5e-2)
    check_slots_left_alone(m, state, hs[0], dt, dev)


@pytest.mark.parametrize("mode", MODES)
def test_delta_far_write(mode):
    """What is written at position 0 is read back 400 tokens later: slow decays, small inputs in between; a key of length
    zero removes and writes nothing."""
    dev, dt = mode
    g = gen(9)
    mix, t = delta_case(g, 2, 32, 8)
    t["w0"], t["a.b"] = torch.full((64,), -9.0).to(BF), torch.full((64,), -4.0).to(BF)
    h = rnd(g, 400, WIDTH, std=0.02)
    h[0], h[200] = rnd(g, WIDTH, std=3.0), 0
    h[399] = h[0]
    want = O.general_delta_mixer(h.double(), mix, {"mix." + n: v.double() for n, v in t.items()}, "mix.", 1e-3)
    m = build_delta(mix, t, dev)
    for cuts in (((400,),), ((1,), (2,), (250,), (100,))):
        y = run_cuts(m, used_slots(m, dev), [h], [1], cuts, dt, dev)[0]
        near(y[:5], want[:5], mode, 3e-5, 2e-2)
        near(y[395:], want[395:], mode, 5e-5, 3e-2)


@pytest.mark.parametrize("mode", MODES[1:])
@pytest.mark.parametrize("heads,dim", [(16, 32), (60, 64), (40, 128), (20, 192)])
def test_delta_long_portion_equals_short_ones(mode, heads, dim):
    """Many columns, so that a column's rows lie in fewer lanes, against pieces with few columns; two sequences and an empty
    run between them."""
    dev, dt = mode
    g = gen(77)
    m = build_delta(*delta_case(g, heads, dim, 8), dev)
    n = 11                                                    # sequences
    hs = rnd(g, 100 * n, WIDTH).to(dt).to(dev)
    state = used_slots(m, dev, n + 1)
    holder = _Holder()
    holder.mixer_state = state
    cu = [100 * i for i in range(n + 1)]
    whole = m(hs, _Batch(dev, list(range(100)) * n, list(range(n)) + [n], cu[:4] + cu[3:]), 0, holder)
    after = state[0][1].clone()
    assert float(after[3].max()) == -2.0                      # the slot of the empty run
    for i, slot in ((0, 0), (5, 6)):
        parts = []
        for a, b in ((0, 1), (1, 3), (3, 40), (40, 100)):
            rows = hs[100 * i + a:100 * i + b]
            parts.append(m(rows, _Batch(dev, range(a, b), [slot], [0, b - a]), 0, holder))
        assert rel_err(torch.cat(parts), whole[100 * i:100 * i + 100].cpu()) < (1e-6 if dt == F32 else 3e-3)
        assert rel_err(state[0][1][slot], after[slot].cpu()) < (1e-6 if dt == F32 else 3e-3)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("width,ff,dim,rows", [(24, 20, 8, 3), (40, 256, 24, 150), (136, None, 16, 5), (2048, 72, 32, 5)])
def test_parallel_block(mode, width, ff, dim, rows):
    """Mixer and feed-forward on inputs of their own, one output product; a layer without feed-forward."""
    dev, dt = mode
    g = gen(width)
    mix = dict(heads=2, dim=dim)
    n = 2 * dim
    t = {"w1": rnd(g, 8, width, std=width ** -0.5), "w2": rnd(g, n, 8), "o": rnd(g, width, n, std=n ** -0.5), "w0": rnd(g, n), "a.b": rnd(g, n),
         "norm": rnd(g, n, std=0.3) + 1, **{x: rnd(g, n, width, std=width ** -0.5) for x in "rkvga"}}
    w = {"up": rnd(g, ff or 8, width, std=width ** -0.5), "down": rnd(g, width, ff or 8, std=(ff or 8) ** -0.5)}
    h, hf = rnd(g, rows, width), rnd(g, rows, width)
    want = O.general_delta_mixer(h.double(), mix, {"m." + k: v.double() for k, v in t.items()}, "m.", 1e-3)
    if ff:
        want = want + O.feed_forward(hf.double(), {"m." + k: v.double() for k, v in w.items()}, "m.")
    spec = C.MixerSpec(kind="general_delta", heads=2, kv_heads=2, dim=dim, vdim=dim)
    mixer = M.GeneralDeltaMixer(spec, width, 1e-3, dev, a_bias=t["a.b"], **{k: v for k, v in t.items() if k not in ("a.b", "o")}, o=None)
    ffn = M.DenseFeedForward(C.DenseSpec(ff, "relu2"), width, 1e-3, dev, up=w["up"], down=None) if ff else None
    b = M.ParallelBlock(mixer, ffn, width, dev, o=t["o"], down=w["down"] if ff else None)
    assert hasattr(b, "state_shapes") and not hasattr(b, "cache_shape")
    holder = _Holder()
    holder.mixer_state = [(None, torch.zeros(mixer.state_shapes(1)[1], device=dev))]
    y = b(h.to(dt).to(dev), hf.to(dt).to(dev), _Batch(dev, range(rows), [0], [0, rows]), 0, holder)
    near(y[:, :width], want, mode, 3e-5, 1.5e-2)


def test_one_token_runs_at_the_end_are_a_part_of_their_own():
    b = _Holder()
    b.is_decode, b.cu_q = False, torch.tensor([0, 3, 4, 9, 10, 11])
    b.runs = [(3, 3), (1, 8), (5, 9), (1, 2), (1, 40)]
    (r1, s1, c1), (r2, s2, c2) = M.batch_parts(b)
    assert (r1, s1, c1.tolist()) == (slice(0, 9), slice(0, 3), [0, 3, 4, 9]) and (r2, s2, c2) == (slice(9, None), slice(3, None), None)
    b.runs = [(1, 3), (1, 1)]
    assert M.batch_parts(b) == [(slice(0, None), slice(0, None), None)]
    for runs in ([(1, 1), (2, 5)], None):
        b.runs = runs
        assert M.batch_parts(b) == [(slice(None), slice(None), b.cu_q)]
    b.is_decode = True
    assert M.batch_parts(b) == [(slice(None), slice(None), None)]


# ------------------------------------------------------------------------------------ whole models
def att(heads, kv, dim, vdim, window, scale=None, ff=None, source=None):
    m = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, scale=scale or 0.8 * dim ** -0.5, mask=dict(size=window))
    return {"type": "attention", "mlp": None if ff is None else dict(kind="dense", ff=ff), "mixer": m if source is None else {**m, "kv_from": source}}


def lat(heads, dim, rot, vdim, kv_rank, q_rank, scale=None, ff=None, base=3000.0):
    return {"type": "latent_attention", "mlp": None if ff is None else dict(kind="dense", ff=ff),
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale or 1.3 * (dim + rot) ** -0.5,
                          rot=dict(dims=rot, base=base))}


def dlt(heads, dim, ff=None):
    return {"type": "general_delta", "mlp": None if ff is None else dict(kind="dense", ff=ff), "mixer": dict(heads=heads, dim=dim)}


def model_cfg(vocab, width, layers, eps=1e-5, groups=4, taps=4, mult=0.6, scale=0.4, cap=15.0):
    return {"architecture": "Ginodra", "vocab": vocab, "width": width, "norm": dict(eps=eps, groups=groups), "canon": dict(taps=taps), "residual_mult": mult,
            "logit_scale": scale, "logit_softcap": cap, "layers": layers}


CASES = {
    # every kind of layer, layers without feed-forward, odd sizes, norm parts that begin inside a vector, keys used by two
    # later layers with windows of their own
    "mixed": model_cfg(301, 132, [lat(5, 40, 12, 24, 56, 30, ff=100), att(6, 3, 40, 24, 21, ff=72), dlt(3, 24), att(6, 3, 40, 24, 33, 0.2, source=1),
                                  att(12, 3, 40, 24, 9, ff=60, source=1), lat(3, 24, 20, 16, 40, 22)], groups=3),
    "attention": model_cfg(97, 64, [att(2, 2, 32, 32, 17, ff=60), att(9, 3, 8, 136, 70), att(9, 3, 8, 136, 16, ff=24, source=1)], eps=1e-4, groups=8, taps=2,
                           mult=1.0, scale=1.0, cap=4.0),
    "latent": model_cfg(130, 100, [lat(18, 16, 8, 12, 32, 24, ff=88), lat(2, 64, 32, 64, 136, 48), lat(4, 128, 64, 96, 64, 40, ff=40)], eps=1e-6, groups=1, taps=3,
                        mult=0.5),
    "recurrent": model_cfg(75, 80, [dlt(2, 64, ff=48), dlt(5, 16), dlt(1, 136, ff=8)], groups=10, taps=6, mult=0.8, scale=0.25),
}


def rand_weights(cfg, seed=0):
    g = gen(seed)
    w = {}
    for n, s in tensor_shapes(config_from(cfg)).items():
        leaf = n.rsplit(".", 1)[-1]
        if "norm" in leaf:
            w[n] = rnd(g, *s, std=0.3) + 1
        elif leaf == "w0":
            w[n] = rnd(g, *s) - 4.0
        elif leaf == "sink":
            w[n] = rnd(g, *s, std=2.0)
        elif leaf == "b":
            w[n] = rnd(g, *s)
        elif n == "embed":
            w[n] = rnd(g, *s)
        else:
            w[n] = rnd(g, *s, std=0.4 if leaf.startswith("canon") else s[-1] ** -0.5)
    return w


_BUILT, _WANT = {}, {}


def built(case, mode):
    if (case, mode) not in _BUILT:
        cfg, w = CASES[case], rand_weights(CASES[case])
        model = DecoderModel(config_from(cfg), mode[0], dtype=mode[1])
        model.load_state_dict(w.get)
        _BUILT[case, mode] = (cfg, w, model)
    return _BUILT[case, mode]


def expected(case, tokens):
    key = (case, tuple(tokens))
    if key not in _WANT:
        _WANT[key] = O.forward(tokens, CASES[case], rand_weights(CASES[case]))
    return _WANT[key]


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
        logits_near(play(eng, toks, cuts), expected(case, toks), mode)
        assert eng.kv.num_free == eng.num_pages and eng.kv.num_free_slots == 4


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("case", list(CASES))
def test_model_mixed_batches(mode, case):
    """Unequal requests in one batch, portions beside single tokens, requests that pause, and pages and slots that change
    hands, against each request alone."""
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
        logits_near(torch.cat(got[k]), expected(case, seqs[k]), mode)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("case", ["mixed", "recurrent"])
def test_model_stream_per_layer(mode, case):
    cfg, w, model = built(case, mode)
    toks = prompt(case, 30, 3)
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
@pytest.mark.parametrize("case", ["mixed", "recurrent"])
def test_long_decode(mode, case):
    _, _, model = built(case, mode)
    toks = prompt(case, 150, 4)
    logits_near(play(engine(model), toks, [4] + [1] * 146), expected(case, toks), mode)


@pytest.mark.parametrize("mode", MODES)
def test_pool_and_slots_are_bounded(mode):
    """Every layer's inputs are state: also a model without a recurrent mixer holds a slot per sequence."""
    _, _, model = built("attention", mode)
    eng = engine(model, tokens=64, batch=2)
    assert model.cfg.recurrent and eng.kv.state_slots == 2 and model.kv_cache[2] is None and model.kv_cache[1] is not None
    taps, width = 2, 64
    es = 4 if mode[1] == F32 else 2
    assert model.state_bytes_per_slot() == 3 * (taps - 1) * width * es
    eng.replay([("a", prompt("attention", 33, 0), []), ("b", [1], [])])
    with pytest.raises(KvPoolExhaustedError):              # both slots are taken
        eng.replay([("c", [1], [])])
    eng.replay([], ["a", "b", "c"])
    with pytest.raises(ValueError):
        eng.replay([("d", [1] * 100, [])])
    assert eng.kv.num_free == eng.num_pages


# ------------------------------------------------------------------------------------ generation
def greedy(case, toks, n):
    out = list(toks)
    for _ in range(n):
        out.append(int(expected(case, out)[-1].argmax()))
    return out[len(toks):]


@pytest.mark.parametrize("mode", [MODES[0], MODES[1]])
@pytest.mark.parametrize("case", ["mixed", "recurrent"])
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
    assert tight.stats()["preemptions"] > 0 and tight.kv.num_free == 9 and tight.kv.num_free_slots == 4


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
    assert llm.config.arch == "ginodra" and llm.model.dtype == F32
    toks = prompt("mixed", 12, 8)
    y = engine(llm.model).replay([("x", toks, [11])], ["x"])
    logits_near(y, expected("mixed", toks)[11:], ("cpu", F32))
    with pytest.raises(ValueError):
        llm.config.validate_tp(2)
    total = sum(v.numel() for v in rand_weights(CASES["mixed"]).values())
    assert abs(llm.config.param_count() / total - 1) < 0.02 and llm.model.weight_bytes() > 2 * total


@pytest.mark.parametrize("bad", [[lat(2, 8, 8, 8, 520, 8)], [lat(2, 8, 5, 8, 16, 8)], [att(3, 2, 8, 8, 4)], [att(2, 1, 520, 8, 4)], [dlt(2, 264)],
                                 [att(2, 1, 8, 8, 4, source=0)], [att(2, 1, 8, 8, 4), att(2, 2, 8, 8, 4, source=0)], [dlt(2, 8), att(2, 1, 8, 8, 4, source=0)],
                                 [att(2, 1, 8, 8, 4, source=1), att(2, 1, 8, 8, 4)], [att(2, 1, 8, 8, 4), att(2, 1, 8, 16, 4, source=0)],
                                 [{**att(2, 1, 8, 8, 4), "type": "other"}], [{**dlt(2, 8), "mlp": {"kind": "other", "ff": 8}}]])
def test_what_has_no_kernel_is_refused(bad):
    cfg = model_cfg(20, 16, bad)
    with pytest.raises(ValueError):
        DecoderModel(config_from(cfg), "cpu").load_state_dict(rand_weights(cfg).get)


def test_uneven_norm_parts_are_refused():
    with pytest.raises(ValueError):
        config_from(model_cfg(20, 20, [dlt(1, 8)], groups=3))


@pytest.mark.parametrize("mode", MODES)
def test_absent_options(mode):
    """No mask, no feed-forward, no cap, no convolution, one norm part: the plain forms."""
    layers = [att(2, 1, 16, 16, 0), lat(2, 16, 8, 8, 24, 16, ff=16), att(4, 1, 16, 16, 0, ff=8, source=0), dlt(1, 8)]
    for i in (0, 2):
        del layers[i]["mixer"]["mask"]
    cfg = model_cfg(40, 32, layers, groups=1, taps=1, mult=1.0, scale=1.0, cap=1e4)
    w = rand_weights(cfg)
    for n in w:
        if ".canon" in n:
            w[n] = torch.zeros_like(w[n])
    toks = torch.randint(0, 40, (40,), generator=gen(1)).tolist()
    want = O.forward(toks, cfg, w)
    plain = {k: v for k, v in cfg.items() if k not in ("canon", "residual_mult", "logit_scale", "logit_softcap")}
    plain["norm"] = {"eps": cfg["norm"]["eps"]}
    model = DecoderModel(config_from(plain), mode[0], dtype=mode[1])
    model.load_state_dict({n: v for n, v in w.items() if ".canon" not in n}.get)
    logits_near(play(engine(model), toks, [20, 1, 1, 18]), want, mode)


def test_checkpoint_is_recognised(checkpoint):
    from hartsyinference_b200.assets.registry import detect
    from hartsyinference_b200.engine.planner import shape_of_checkpoint
    d = detect(checkpoint)
    assert (d.family, d.arch) == ("llm", "ginodra")
    assert shape_of_checkpoint(checkpoint) is None          # stays on one GPU


def test_service_generates_and_embeds(checkpoint):
    """Through the text service: token ids in, greedy ids out as the engine gives them; embedding a text in between
    leaves the running requests' pages and state alone."""
    from hartsyinference_b200.engine.requests import EngineOptions, Modality, ModelSpec, TextRequest
    from hartsyinference_b200.engine.text_service import TextService
    svc = TextService(EngineOptions(max_batch=2, max_model_len=64), device="cpu")
    spec = ModelSpec("m", Modality.TEXT, local_path=str(checkpoint))
    req = TextRequest(messages=[], prompt_token_ids=prompt("mixed", 20, 5), max_tokens=6, greedy=True, ignore_eos=True)
    try:
        a = svc.generate(spec, req).token_ids
        model = svc._host(spec).llm.model
        held = [t for t in (*model.kv_cache, *model.input_state, *(x for st in model.mixer_state if st for x in st)) if t is not None]
        before = [t.clone() for t in held]
        e = svc.embed(spec, ["abc", "abcd"])
        now = [t for t in (*model.kv_cache, *model.input_state, *(x for st in model.mixer_state if st for x in st)) if t is not None]
        assert all(x is y and torch.equal(x, z) for x, y, z in zip(now, held, before, strict=True))
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


def test_random_weights_run():
    """Synthetic weights of a configuration, as the benchmark uses them."""
    model = DecoderModel(config_from(CASES["mixed"]), "cpu", dtype=F32)
    model.random_init(seed=1)
    y = engine(model).replay([("a", prompt("mixed", 9, 1), [8])], ["a"])
    assert torch.isfinite(y).all() and float(y.abs().max()) < 15.0 and not math.isclose(float(y.std()), 0.0)
