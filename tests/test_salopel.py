"""Salopel against the plain statement in ``salopel_oracle``: every mechanism alone, then whole models through
the engine (prompts, portions, decoding, mixed batches, reused pages and slots, generation).

Each case runs on the CPU ops and, marked ``gpu``, on the kernels in fp32 and bf16."""
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import salopel_oracle as O  # noqa: E402
from test_lududra import BF, F32, MODES, Pages, _Holder, gen, logits_near, near, rel_err, rnd  # noqa: E402
from test_lududra import _Batch as _PlainBatch  # noqa: E402

from hartsyinference_b200 import ops  # noqa: E402
from hartsyinference_b200.engine import LLMEngine, SamplingParams  # noqa: E402
from hartsyinference_b200.exceptions import KvPoolExhaustedError  # noqa: E402
from hartsyinference_b200.models.llm import config as C  # noqa: E402
from hartsyinference_b200.models.llm import mixers as M  # noqa: E402
from hartsyinference_b200.models.llm.loader import load_llm, save_hf_checkpoint  # noqa: E402
from hartsyinference_b200.models.llm.salopel import config_from, tensor_shapes  # noqa: E402
from hartsyinference_b200.models.llm.transformer import DecoderModel  # noqa: E402


class _Batch(_PlainBatch):
    def __init__(self, dev, positions, slots, cu=None):
        super().__init__(dev, positions, slots, cu)
        self.runs = None if cu is None else [(b - a, None) for a, b in zip(cu, cu[1:])]


# ------------------------------------------------------------------------------------ norms and stream
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("dim", [40, 136, 1000, 8204])
def test_stream_norms_around_zero(mode, dim):
    """Weights stored around zero, a factor on the sublayer's output, and the stream itself as the next input."""
    dev, dt = mode
    g = gen(dim)
    rows, ld = 5, (dim + 7) // 8 * 8
    x = torch.zeros(rows, ld)
    x[:, :dim] = torch.randn(rows, dim, generator=g) * 3 + 1.5
    y = torch.zeros(rows, ld, dtype=BF)
    y[:, :dim] = rnd(g, rows, dim, std=0.02)
    wb, wn = rnd(g, dim, std=0.3), rnd(g, dim, std=0.3)
    want = x[:, :dim].double() - 0.3 * O.rms_plus_one(y[:, :dim].double(), wb.double(), 1e-4)
    kw = dict(dim=dim, eps=1e-4, layernorm=False, dtype=dt, plus_one=True, mult=-0.3)
    xd = x.to(dev)
    h = ops.residual_norm(xd, y.to(dt).to(dev), wb.to(dev), None, plain=True, **kw)
    assert rel_err(xd[:, :dim], want) < 1e-6                # the stream is fp32 whatever the activations are
    assert torch.equal(h, xd.to(dt)) and float(h[:, dim:].float().abs().sum()) == 0
    h = ops.residual_norm(xd, None, None, wn.to(dev), plain=True, **kw)
    near(h[:, :dim], O.rms_plus_one(want, wn.double(), 1e-4), mode, 1e-6, 4e-3)
    assert ops.residual_norm(xd, None, None, None, **kw) is None


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("dim", [44, 1160, 9000])
def test_normed_embedding(mode, dim):
    dev, dt = mode
    g = gen(dim)
    ld = (dim + 7) // 8 * 8
    table = torch.zeros(11, ld, dtype=BF)
    table[:, :dim] = rnd(g, 11, dim, std=0.01)
    w = rnd(g, dim, std=0.3)
    ids = torch.tensor([3, 0, 10, 3], dtype=torch.int32)
    kw = dict(dim=dim, eps=1e-5, plus_one=True, dtype=dt)
    x, h = ops.embedding_norm(ids.to(dev), table.to(dev), w.to(dev), **kw)
    want = O.rms_plus_one(table[ids.long(), :dim].double(), w.double(), 1e-5)
    assert x.dtype == F32 and rel_err(x[:, :dim], want) < 1e-6 and torch.equal(h, x.to(dt))
    x2, _ = ops.embedding_norm(None, table[ids.long()].to(dev), w.to(dev), **kw)       # rows given instead of ids
    assert torch.equal(x2, x) and x.shape[1] == ld and float(x[:, dim:].abs().sum()) == 0


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("ff,rows", [(20, 3), (256, 70), (1000, 5), (9000, 4), (1544, 1100)])
def test_poly_norm(mode, ff, rows):
    """Each power's weight matters, small rows feel eps."""
    dev, dt = mode
    g = gen(ff)
    z = torch.zeros(rows, (ff + 7) // 8 * 8, dtype=BF)
    z[:, :ff] = rnd(g, rows, ff) * torch.tensor([0.02, 0.3, 2.0, 9.0, 1.0]).repeat(rows // 5 + 1)[:rows, None].to(BF)
    for act in ([0.7, -0.4, 0.3, 0.2], [0, 0, 1, 0], [0, 1, 0, 0], [1, 0, 0, 0]):
        got = ops.poly_norm(z.to(dt).to(dev), torch.tensor(act, dtype=F32, device=dev), ff, 1e-3)
        near(got[:, :ff], O.poly_norm(z[:, :ff].double(), torch.tensor(act, dtype=torch.float64), 1e-3), mode, 2e-6, 4e-3)
        assert float(got[:, ff:].float().abs().sum()) == 0


# ------------------------------------------------------------------------------------ recurrent mixers
WIDTH = 24


def channel_case(g, inner, state, rank, conv):
    mix = dict(inner=inner, state=state, dt_rank=rank, conv=conv)
    shapes = {"in": (2 * inner, WIDTH), "x": (rank + 2 * state, inner), "dt": (inner, rank), "o": (WIDTH, inner)}
    t = {n: rnd(g, *s, std=s[1] ** -0.5) for n, s in shapes.items()}
    t["conv"], t["conv.b"] = rnd(g, inner, conv, std=0.6), rnd(g, inner, std=0.3)
    t["dt.b"], t["A_log"], t["D"] = rnd(g, inner) - 2.0, rnd(g, inner, state), rnd(g, inner)
    return mix, t


def build_channel(mix, t, dev):
    spec = C.MixerSpec(kind="channel_scan", inner=mix["inner"], state=mix["state"], rank=mix["dt_rank"], conv=mix["conv"])
    return M.ChannelScanMixer(spec, WIDTH, dev, w_in=t["in"], conv=t["conv"], conv_bias=t["conv.b"], x=t["x"], dt=t["dt"], dt_bias=t["dt.b"],
                              a_log=t["A_log"], d=t["D"], o=t["o"])


def head_case(g, heads, groups, state, vdim, parts, conv):
    mix = dict(heads=heads, groups=groups, state=state, vdim=vdim, norm_groups=parts, conv=conv)
    inner, gn = heads * vdim, groups * state
    t = {"in": rnd(g, 2 * inner + 2 * gn + heads, WIDTH, std=WIDTH ** -0.5), "o": rnd(g, WIDTH, inner, std=inner ** -0.5)}
    t["conv"], t["conv.b"] = rnd(g, inner + 2 * gn, conv, std=0.6), rnd(g, inner + 2 * gn, std=0.3)
    t["dt_bias"], t["A_log"], t["D"], t["norm"] = rnd(g, heads) - 1.0, rnd(g, heads) - 1.0, rnd(g, heads), rnd(g, inner, std=0.3) + 1
    return mix, t


def build_head(mix, t, dev, eps=1e-3):
    spec = C.MixerSpec(kind="head_scan", heads=mix["heads"], groups=mix["groups"], state=mix["state"], vdim=mix["vdim"],
                       norm_groups=mix["norm_groups"], conv=mix["conv"])
    return M.HeadScanMixer(spec, WIDTH, eps, dev, w_in=t["in"], conv=t["conv"], conv_bias=t["conv.b"], dt_bias=t["dt_bias"], a_log=t["A_log"],
                           d=t["D"], norm=t["norm"], o=t["o"])


def used_slots(m, dt, dev, slots=3):
    """State slots that hold what an earlier sequence left there."""
    conv, rec = m.state_shapes(slots)
    return [(torch.full(conv, 3.0, dtype=dt, device=dev), torch.full(rec, -2.0, dtype=F32, device=dev))]


def run_cuts(m, state, hs, slots, cuts, dt, dev):
    """Portions of the given sizes beside each other, then single tokens together while sequences last."""
    holder = _Holder()
    holder.mixer_state = state
    got = [torch.zeros(h.shape[0], WIDTH) for h in hs]
    done = [0] * len(hs)

    def step(counts, decode):
        use = [(i, n) for i, n in enumerate(counts) if n]
        pos, cu = [], [0]
        for i, n in use:
            pos += range(done[i], done[i] + n)
            cu.append(cu[-1] + n)
        rows = torch.cat([hs[i][done[i]:done[i] + n] for i, n in use]).to(dt).to(dev)
        y = m(rows, _Batch(dev, pos, [slots[i] for i, _ in use], None if decode else cu), 0, holder).float().cpu()
        for (i, n), a in zip(use, cu):
            got[i][done[i]:done[i] + n] = y[a:a + n, :WIDTH]
            done[i] += n

    for c in cuts:
        step(c, False)
    while any(d < h.shape[0] for d, h in zip(done, hs)):
        step([int(d < h.shape[0]) for d, h in zip(done, hs)], True)
    return got


CUTS = ((17, 0), (2, 5), (1, 2), (16, 1), (3, 9), (0, 2), (64, 3), (65, 1), (48, 0), (130, 2))
CHANNEL_SIZES = [(32, 16, 4, 4), (20, 5, 1, 1), (72, 32, 9, 3), (40, 8, 16, 2), (33, 64, 3, 6), (8, 100, 2, 4), (100, 12, 5, 5)]
HEAD_SIZES = [(4, 2, 16, 16, 2, 4), (3, 1, 32, 20, 1, 3), (6, 3, 8, 8, 4, 2), (2, 2, 128, 64, 2, 4), (5, 1, 40, 12, 3, 1), (2, 1, 200, 136, 1, 6),
              (1, 1, 64, 256, 1, 4), (8, 4, 12, 24, 8, 5), (6, 2, 20, 40, 6, 4)]


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", CHANNEL_SIZES, ids=str)
def test_channel_scan_mixer(mode, sizes):
    """Portions down to one and two tokens, beside another sequence, then decoding; every cut gives what the whole
    sequence gives, whatever the slots held before."""
    dev, dt = mode
    g = gen(sum(sizes))
    mix, t = channel_case(g, *sizes)
    hs = [rnd(g, 352, WIDTH), rnd(g, 29, WIDTH)]
    wd = {"mix." + n: v.double() for n, v in t.items()}
    m = build_channel(mix, t, dev)
    state = used_slots(m, dt, dev)
    for got, h in zip(run_cuts(m, state, hs, [2, 0], CUTS, dt, dev), hs):
        near(got, O.mamba1_mixer(h.double(), mix, wd, "mix."), mode, 3e-5, 2e-2)
    check_slots_left_alone(m, state, hs[0], dt, dev)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("sizes", HEAD_SIZES, ids=str)
def test_head_scan_mixer(mode, sizes):
    """As above, with groups that share B and C and norm parts that begin inside a head."""
    dev, dt = mode
    g = gen(sum(sizes))
    mix, t = head_case(g, *sizes)
    hs = [rnd(g, 352, WIDTH), rnd(g, 29, WIDTH)]
    wd = {"mix." + n: v.double() for n, v in t.items()}
    m = build_head(mix, t, dev)
    state = used_slots(m, dt, dev)
    for got, h in zip(run_cuts(m, state, hs, [2, 0], CUTS, dt, dev), hs):
        near(got, O.mamba2_mixer(h.double(), mix, wd, "mix.", 1e-3), mode, 3e-5, 2e-2)
    check_slots_left_alone(m, state, hs[0], dt, dev)


def check_slots_left_alone(m, state, h, dt, dev):
    """Slot 1 belongs to nobody: untouched; a row without a slot stores nothing, in a portion or alone."""
    holder = _Holder()
    holder.mixer_state = state
    before = [s.clone() for s in state[0]]
    m(h[:1].to(dt).to(dev), _Batch(dev, [0], [-1]), 0, holder)
    m(h[:7].to(dt).to(dev), _Batch(dev, range(7), [-1], [0, 7]), 0, holder)
    assert all(torch.equal(a, b) for a, b in zip(before, state[0]))
    assert float(state[0][1][1].min()) == float(state[0][1][1].max()) == -2.0


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("kind", ["channel", "head"])
def test_first_tokens_and_far_write(mode, kind):
    """The convolution sees zeros before the start, and what is written at position 0 is read back 400 tokens
    later: slow decays, small inputs in between."""
    dev, dt = mode
    g = gen(9)
    h = rnd(g, 400, WIDTH, std=0.02)
    h[0] = rnd(g, WIDTH, std=3.0)
    h[399] = h[0]
    if kind == "channel":
        mix, t = channel_case(g, 32, 16, 4, 4)
        t["A_log"] = torch.full((32, 16), -7.0).to(BF)
        m, want = build_channel(mix, t, dev), lambda w: O.mamba1_mixer(h.double(), mix, w, "mix.")
    else:
        mix, t = head_case(g, 2, 1, 32, 16, 2, 4)
        t["A_log"] = torch.full((2,), -7.0).to(BF)
        m, want = build_head(mix, t, dev), lambda w: O.mamba2_mixer(h.double(), mix, w, "mix.", 1e-3)
    want = want({"mix." + n: v.double() for n, v in t.items()})
    for cuts in (((400,),), ((1,), (2,), (250,), (100,))):
        y = run_cuts(m, used_slots(m, dt, dev), [h], [1], cuts, dt, dev)[0]
        near(y[:5], want[:5], mode, 3e-5, 2e-2)
        near(y[395:], want[395:], mode, 5e-5, 3e-2)


@pytest.mark.parametrize("mode", MODES[1:])
@pytest.mark.parametrize("kind", ["channel", "head"])
def test_long_portion_equals_short_ones(mode, kind):
    """A portion long enough for many tokens per warp, two sequences and an empty run between them, against the
    same tokens in pieces."""
    dev, dt = mode
    g = gen(77)
    mix, t = channel_case(g, 1040, 16, 8, 4) if kind == "channel" else head_case(g, 32, 2, 16, 32, 2, 4)
    m = build_channel(mix, t, dev) if kind == "channel" else build_head(mix, t, dev)
    hs = rnd(g, 2200, WIDTH).to(dt).to(dev)
    state = used_slots(m, dt, dev)
    holder = _Holder()
    holder.mixer_state = state
    whole = m(hs, _Batch(dev, list(range(1203)) + list(range(997)), [0, 1, 2], [0, 1203, 1203, 2200]), 0, holder)
    after = [s.clone() for s in state[0]]
    parts = []
    for a, b, slot in ((0, 1203, 0), (1203, 2200, 2)):
        for c in range(a, b, 101):
            e = min(c + 101, b)
            parts.append(m(hs[c:e], _Batch(dev, range(c - a, e - a), [slot], [0, e - c]), 0, holder))
    assert rel_err(torch.cat(parts), whole.cpu()) < (1e-6 if dt == F32 else 3e-3)
    for x, y in zip(after, state[0]):
        for slot in (0, 2):
            assert rel_err(y[slot].float(), x[slot].float().cpu()) < (1e-6 if dt == F32 else 3e-3)


# ------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,rank,page", [(4, 64, 16), (6, 40, 8), (17, 128, 16), (1, 96, 64), (33, 24, 16), (3, 512, 32), (20, 264, 16)])
def test_latent_rows(mode, heads, rank, page):
    """Queries in latent space over pages in shuffled order: the first key, the last one, keys at page and tile edges
    and one that has just been left out each stand out for some head of some row."""
    dev, dt = mode
    g = gen(heads * 10 + rank)
    lens = [300, 1, 65, 128, page + 1]
    pg = Pages(g, lens, 1, rank, page, dt, dev)
    lat = [rnd(g, n + 1, rank) for n in lens]
    q = rnd(g, 2 * len(lens), heads, rank, std=rank ** -0.5)
    rows = []                                        # (sequence, keys): every sequence at its end and somewhere before
    for i, n in enumerate(lens):
        rows += [(i, n), (i, max(1, n // 2))]
    for r, (i, n) in enumerate(rows):
        for h, spot in enumerate((0, n - 1, n, page - 1, page, 63, 64, n // 2)):
            if spot < n:
                u = torch.nn.functional.normalize(q[r, h % heads].float(), dim=0)
                lat[i][spot] += (u * 4).to(BF)
    for i, n in enumerate(lens):
        ops.kv_store(lat[i][:n].to(dt).to(dev), pg.cache, pg.slots(i, 0, n).to(dev))
    want = []
    for r, (i, n) in enumerate(rows):
        c = lat[i][:n].double()
        want.append(torch.cat([torch.softmax(c @ q[r, h].double() * 1.7, 0) @ c for h in range(heads)]))
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    qd = q.reshape(len(rows), -1).to(dt).to(dev)
    out = ops.latent_attn(qd, pg.cache, pg.table.to(dev), i32([n for _, n in rows]), heads, 1.7, row_seq=i32([i for i, _ in rows]),
                          max_kv_len=max(lens))
    near(out, torch.stack(want), mode, 1e-5, 6e-3)
    # one row per sequence (decode), the last one empty
    ends = qd[::2].contiguous()
    out = ops.latent_attn(ends, pg.cache, pg.table.to(dev), i32(lens[:-1] + [0]), heads, 1.7, max_kv_len=4096)
    near(out[:-1], torch.stack(want[::2])[:-1], mode, 1e-5, 6e-3)
    assert float(out[-1].float().abs().max()) == 0


@pytest.mark.gpu
@pytest.mark.parametrize("heads,d,dv", [(4, 64, 64), (3, 40, 24), (2, 128, 128), (5, 16, 104)])
def test_runs_over_expanded_contexts(heads, d, dv):
    """Runs that are not adjacent and start inside their contexts; keys just seen and just not yet seen stand out."""
    g = gen(d + dv)
    runs = [(70, 70), (3, 200), (129, 130), (64, 321)]           # (queries, keys)
    t = sum(r[0] for r in runs) + 40
    starts = [10, 100, 105, 240]
    q, gate = rnd(g, t, heads * d, std=d ** -0.5), rnd(g, t, heads * dv)
    ks, vs, want = [], [], torch.full((t, heads * dv), 7.0, dtype=torch.float64)
    for (nq, nk), a in zip(runs, starts):
        k, v = rnd(g, nk, heads * d), rnd(g, nk, heads * dv)
        for i in range(0, nq, 5):
            for h, spot in enumerate((nk - nq + i, nk - nq + i + 1, 0, nk - nq - 1, 64)):
                if 0 <= spot < nk and h < heads:
                    u = torch.nn.functional.normalize(q[a + i, h * d:(h + 1) * d].float(), dim=0)
                    k[spot, h * d:(h + 1) * d] += (u * 3).to(BF)
        for h in range(heads):
            for i in range(nq):
                n = nk - nq + i + 1
                s = torch.softmax(k[:n, h * d:(h + 1) * d].double() @ q[a + i, h * d:(h + 1) * d].double() * 2.5, 0)
                want[a + i, h * dv:(h + 1) * dv] = s @ v[:n, h * dv:(h + 1) * dv].double() * torch.sigmoid(gate[a + i, h * dv:(h + 1) * dv].double())
        ks.append(k)
        vs.append(v)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    out = torch.full((t, heads * dv), 7.0, dtype=BF, device="cuda")
    at = [0]
    for _, nk in runs:
        at.append(at[-1] + nk)
    kv = torch.cat([torch.cat(ks), torch.cat(vs)], 1).cuda()
    ops.attn_runs(q.cuda(), kv[:, :heads * d], kv[:, heads * d:], out, i32(starts), i32([r[0] for r in runs]), i32(at), i32([r[1] for r in runs]),
                  heads=heads, max_q_len=129, scale=2.5, gate=gate.cuda())
    near(out, want, ("cuda", BF), bf16=6e-3)
    others = torch.ones(t, dtype=torch.bool)
    for (nq, _), a in zip(runs, starts):
        others[a:a + nq] = False
    assert bool((out.cpu()[others] == 7.0).all())                # rows of no run are left alone


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,n,k,rows", [(3, 40, 24, 5), (6, 64, 64, 130), (2, 512, 128, 64), (16, 8, 200, 1), (1, 72, 8, 300)])
def test_head_linear(mode, heads, n, k, rows):
    dev, dt = mode
    g = gen(n + k)
    x, w, gate = rnd(g, rows + 4, heads * k), rnd(g, heads * n, k, std=k ** -0.5), rnd(g, rows + 4, heads * n + 8)
    full = torch.cat([x[:, h * k:(h + 1) * k].double() @ w[h * n:(h + 1) * n].double().T for h in range(heads)], 1)
    lw = ops.LinearWeight(w.to(dev))
    xd = x.to(dt).to(dev)
    near(ops.head_linear(xd, lw, heads), full, mode, 1e-6, 4e-3)
    pick = torch.randperm(rows + 4, generator=g)[:rows]
    pd = pick.to(torch.int32).to(dev)
    few = ops.head_linear(xd, lw, heads, in_rows=pd)
    near(few, full[pick], mode, 1e-6, 4e-3)
    out = torch.full((rows + 4, heads * n), 5.0, dtype=dt, device=dev)
    ops.head_linear(xd[:rows], lw, heads, gate=gate.to(dt).to(dev)[:, :heads * n], out=out, out_rows=pd)
    near(out[pick.to(dev)], full[:rows] * torch.sigmoid(gate[pick, :heads * n].double()), mode, 1e-6, 4e-3)
    rest = torch.ones(rows + 4, dtype=torch.bool)
    rest[pick] = False
    assert bool((out.cpu()[rest] == 5.0).all())


class _PagedBatch(_Batch):
    def __init__(self, dev, pages, runs, decode):
        """``runs``: (sequence, start, count)."""
        pos, cu = [], [0]
        for _, a, n in runs:
            pos += range(a, a + n)
            cu.append(cu[-1] + n)
        super().__init__(dev, pos, [0] * len(runs), None if decode else cu)
        self.tokens = self.positions
        self.slot_mapping = torch.cat([pages.slots(s, a, n) for s, a, n in runs]).to(dev)
        self.block_table = pages.table[[s for s, _, _ in runs]].to(dev)
        self.kv_lens = torch.tensor([a + n for _, a, n in runs], dtype=torch.int32, device=dev)
        self.max_kv_len, self.max_q_len = max(a + n for _, a, n in runs), max(n for _, _, n in runs)
        self.runs, self.plan = [(n, a + n) for _, a, n in runs], None


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,dim,vdim,kv_rank,q_rank,scale", [(3, 16, 24, 32, 20, 1.5), (6, 40, 8, 72, 12, 0.7), (2, 64, 64, 20, 48, 1.0),
                                                                 (18, 8, 12, 16, 9, 2.0), (2, 20, 136, 24, 16, 1.0)])
def test_latent_attention_mixer(mode, heads, dim, vdim, kv_rank, q_rank, scale):
    """Prompts in portions of many sizes beside each other (long runs, runs of one and two, in any order), then
    decoding, with scores large enough that few keys count."""
    dev, dt = mode
    g = gen(dim + vdim)
    mix = dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale)
    hd, hv = heads * dim, heads * vdim
    shapes = {"dq": (q_rank, WIDTH), "uq": (hd, q_rank), "dkv": (kv_rank, WIDTH), "uk": (hd, kv_rank), "uv": (hv, kv_rank), "g": (hv, WIDTH),
              "o": (WIDTH, hv)}
    t = {n: rnd(g, *s, std=s[1] ** -0.5) for n, s in shapes.items()}
    t["dq.norm"], t["dkv.norm"] = rnd(g, q_rank, std=0.3) + 1, rnd(g, kv_rank, std=0.3) + 1
    hs = [rnd(g, 170, WIDTH), rnd(g, 60, WIDTH), rnd(g, 9, WIDTH)]
    wd = {"mix." + n: v.double() for n, v in t.items()}
    want = [O.latent_attention_mixer(h.double(), mix, wd, "mix.", 1e-4) for h in hs]
    spec = C.MixerSpec(kind="latent_attention", heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale, out_gate=True)
    m = M.LatentAttention(spec, WIDTH, 1e-4, dev, dq=t["dq"], dq_norm=t["dq.norm"], uq=t["uq"], dkv=t["dkv"], dkv_norm=t["dkv.norm"], uk=t["uk"],
                          uv=t["uv"], g=t["g"], o=t["o"])
    pages = Pages(g, [len(h) for h in hs], 1, m.r, 16, dt, dev)
    holder = _Holder()
    holder.kv_cache = [pages.cache[None]]
    got = [torch.zeros(len(h), WIDTH) for h in hs]
    done = [0, 0, 0]
    order = [1, 0, 2]
    cuts = [(60, 2, 0), (2, 50, 1), (49, 1, 2), (1, 0, 1), (47, 1, 1)]
    while any(d < len(h) for d, h in zip(done, hs)):
        c = cuts.pop(0) if cuts else (1, 1, 1)
        runs = [(i, done[i], min(c[i], len(hs[i]) - done[i])) for i in order if min(c[i], len(hs[i]) - done[i]) > 0]
        rows = torch.cat([hs[i][a:a + n] for i, a, n in runs]).to(dt).to(dev)
        y = m(rows, _PagedBatch(dev, pages, runs, c == (1, 1, 1)), 0, holder).float().cpu()
        for i, a, n in runs:
            got[i][a:a + n], y = y[:n, :WIDTH], y[n:]
            done[i] += n
    for a, b in zip(got, want):
        near(a, b, mode, 5e-5, 3e-2)


# ------------------------------------------------------------------------------------ whole models
def sel(inner, state, rank, conv=4):
    return {"type": "mamba1", "mlp": None, "mixer": dict(inner=inner, state=state, dt_rank=rank, conv=conv)}


def ssd(heads, groups, state, vdim, parts=1, conv=4):
    return {"type": "mamba2", "mlp": None, "mixer": dict(heads=heads, groups=groups, state=state, vdim=vdim, norm_groups=parts, conv=conv)}


def lat(heads, dim, vdim, kv_rank, q_rank, scale=0.5, ff=None):
    return {"type": "latent_attention", "mlp": None if ff is None else {"kind": "dense", "ff": ff},
            "mixer": dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, q_rank=q_rank, scale=scale)}


def ff(layer, n):
    return {**layer, "mlp": {"kind": "dense", "ff": n}}


def model_cfg(vocab, width, layers, eps=1e-5, mult=0.6):
    layers = [{**layers[x], "weights_of": x} if isinstance(x, int) else x for x in layers]
    return {"architecture": "Salopel", "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width, "layers": layers}


CASES = {
    # every kind, feed-forwards on any of them, layers used twice and three times, odd sizes
    "mixed": model_cfg(301, 136, [lat(5, 40, 24, 56, 30, ff=100), ff(sel(72, 16, 5, 3), 60), ssd(4, 2, 24, 20, 2, 2), 0, 1, 0, 2]),
    "recurrent": model_cfg(97, 64, [ssd(6, 3, 16, 8, 3), sel(40, 5, 1, 1), ff(ssd(2, 1, 64, 32, 1, 5), 72), 1], eps=1e-4, mult=1.0),
    "attention": model_cfg(130, 100, [lat(18, 16, 12, 32, 24, 1.0), lat(2, 64, 64, 136, 48, 0.3, ff=88), 0], eps=1e-6, mult=0.35),
}


def rand_weights(cfg, seed=0):
    g = gen(seed)
    w = {}
    for n, s in tensor_shapes(config_from(cfg)).items():
        leaf = n.rsplit(".", 1)[-1]
        mix = ".mix." in n
        if leaf in ("norm1", "norm2") or (leaf == "norm" and not mix):
            w[n] = rnd(g, *s, std=0.3)
        elif leaf == "norm":
            w[n] = rnd(g, *s, std=0.2) + 1
        elif leaf == "A_log":
            w[n] = rnd(g, *s) - 2
        elif leaf == "dt_bias" or n.endswith(".dt.b"):
            w[n] = rnd(g, *s) - 1
        elif leaf == "D" or leaf == "b":
            w[n] = rnd(g, *s, std=0.5)
        elif leaf == "conv":
            w[n] = rnd(g, *s, std=0.6)
        elif leaf == "act":
            w[n] = torch.tensor([0.6, -0.4, 0.5, 0.1]).to(BF)
        else:
            w[n] = rnd(g, *s, std=(2.0 if leaf == "uk" else 1.0) * s[-1] ** -0.5)
    return w


# seeds at which no compared position is so ill-conditioned that bf16 rounding alone (the CPU ops in bf16) moves its
# logits by more than a few percent: an output norm blows up a sublayer's result where that happens to be near zero
SEEDS = {"mixed": 1, "recurrent": 11, "attention": 0}


def weights(case):
    return rand_weights(CASES[case], SEEDS[case])


_BUILT, _WANT = {}, {}


def built(case, mode):
    if (case, mode) not in _BUILT:
        cfg, w = CASES[case], weights(case)
        model = DecoderModel(config_from(cfg), mode[0], dtype=mode[1])
        model.load_state_dict(w.get)
        _BUILT[case, mode] = (cfg, w, model)
    return _BUILT[case, mode]


def expected(case, tokens):
    key = (case, tuple(tokens))
    if key not in _WANT:
        _WANT[key] = O.forward(tokens, CASES[case], weights(case))
    return _WANT[key]


def prompt(case, n, seed):
    return torch.randint(0, CASES[case]["vocab"], (n,), generator=gen(seed)).tolist()


def engine(model, tokens=256, batch=4, page=16, **kw):
    return LLMEngine(model, num_pages=(tokens + page - 1) // page, page_size=page, max_batch=batch, prefill_chunk=tokens,
                     max_model_len=tokens, **kw)


def play(eng, tokens, cuts, key="a"):
    out, at = [], 0
    for n in cuts:
        out.append(eng.replay([(key, tokens[at:at + n], range(n))], [key] if at + n == len(tokens) else []))
        at += n
    assert at == len(tokens)
    return torch.cat(out)


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("case", list(CASES))
def test_model_cuts(mode, case):
    """Whole prompt, token by token, and portions: the same logits at every position."""
    _, _, model = built(case, mode)
    toks = prompt(case, 110, 1)
    want = expected(case, toks)
    eng = engine(model)
    for cuts in ([110], [1] * 110, [2] * 55, [16, 1, 1, 15, 2, 75], [3, 5, 7, 11, 13, 17, 54], [50, 48] + [1] * 12):
        logits_near(play(eng, toks, cuts), want, mode)
        assert eng.kv.num_free == eng.num_pages
    if model.cfg.recurrent:
        assert eng.kv.num_free_slots == 4


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("case", list(CASES))
def test_model_mixed_batches(mode, case):
    """Unequal requests in one batch, portions beside single tokens, requests that pause, and pages and slots that
    change hands, against each request alone."""
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
def test_model_stream_per_layer(mode):
    cfg, w, model = built("mixed", mode)
    toks = prompt("mixed", 30, 3)
    want, got = [], []
    O.forward(toks, cfg, w, layers_out=want)
    eng = engine(model)
    inner, model._forward_mixers = model._forward_mixers, lambda b: type(model)._forward_mixers(model, b, got)
    try:
        eng.replay([("a", toks, [])], ["a"])
    finally:
        model._forward_mixers = inner
        del model.__dict__["_forward_mixers"]
    assert len(got) == len(want) == len(cfg["layers"])
    for a, b in zip(got, want):
        e = (a.cpu().double() - b).norm(dim=1) / b.norm(dim=1)
        assert float(e.max()) < (2e-5 if mode[1] == F32 else 5e-2), float(e.max())


@pytest.mark.parametrize("mode", MODES)
def test_long_decode(mode):
    _, _, model = built("mixed", mode)
    toks = prompt("mixed", 150, 4)
    logits_near(play(engine(model), toks, [4] + [1] * 146), expected("mixed", toks), mode)


def test_shared_layers_keep_their_own_state():
    """Layers that use another one's weights have caches and states of their own, and their weights count once."""
    cfg, _, model = built("mixed", MODES[0].values[0])
    eng = engine(model)
    assert model.layers[3] is model.layers[0] and model.layers[6] is model.layers[2]
    eng.replay([("a", prompt("mixed", 20, 1), [])])
    assert model.kv_cache[0].data_ptr() != model.kv_cache[3].data_ptr() and not torch.equal(model.kv_cache[0], model.kv_cache[3])
    assert not torch.equal(model.mixer_state[2][1], model.mixer_state[6][1])
    alone = DecoderModel(config_from({**cfg, "layers": cfg["layers"][:3]}), "cpu", dtype=F32)
    alone.load_state_dict(weights("mixed").get)
    assert alone.weight_bytes() == model.weight_bytes() and model.cfg.param_count() == alone.cfg.param_count()


def test_weights_can_come_from_a_later_layer():
    a, b = ssd(2, 1, 16, 8), sel(16, 8, 2)
    cfg = {**model_cfg(50, 32, [a, b, a, b]), "layers": [{**a, "weights_of": 2}, b, a, {**b, "weights_of": 1}]}
    w = rand_weights(cfg)
    model = DecoderModel(config_from(cfg), "cpu", dtype=F32)
    model.load_state_dict(w.get)
    toks = torch.randint(0, 50, (30,), generator=gen(1)).tolist()
    logits_near(play(engine(model), toks, [10, 1, 1, 18]), O.forward(toks, cfg, w), ("cpu", F32))
    with pytest.raises(ValueError):
        config_from({**cfg, "layers": [{**a, "weights_of": 1}, {**a, "weights_of": 0}]})


@pytest.mark.parametrize("mode", MODES)
def test_pool_and_slots_are_bounded(mode):
    _, _, model = built("mixed", mode)
    eng = engine(model, tokens=64, batch=2)
    eng.replay([("a", prompt("mixed", 33, 0), []), ("b", [1], [])])
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
    save_hf_checkpoint(CASES["mixed"], weights("mixed"), tmp_path / "m")
    return tmp_path / "m"


def test_checkpoint_loads_by_config(checkpoint):
    llm = load_llm(checkpoint, "cpu", dtype=F32)
    assert llm.config.arch == "salopel" and llm.config.recurrent and llm.model.dtype == F32
    toks = prompt("mixed", 12, 8)
    y = engine(llm.model).replay([("x", toks, [11])], ["x"])
    logits_near(y, expected("mixed", toks)[11:], ("cpu", F32))
    with pytest.raises(ValueError):
        llm.config.validate_tp(2)


@pytest.mark.parametrize("bad", [sel(16, 129, 2), ssd(2, 1, 257, 8), ssd(3, 2, 8, 8), ssd(2, 1, 8, 9, 4), lat(2, 8, 8, 520, 8)])
def test_sizes_without_a_kernel_are_refused(bad):
    cfg = model_cfg(20, 16, [bad])
    with pytest.raises(ValueError):
        DecoderModel(config_from(cfg), "cpu").load_state_dict(rand_weights(cfg).get)


def test_checkpoint_is_recognised(checkpoint):
    from hartsyinference_b200.assets.registry import detect
    from hartsyinference_b200.engine.planner import shape_of_checkpoint
    d = detect(checkpoint)
    assert (d.family, d.arch) == ("llm", "salopel")
    assert shape_of_checkpoint(checkpoint) is None          # stays on one GPU


def test_service_generates_and_embeds(checkpoint):
    """Through the text service: token ids in, greedy ids out as the engine gives them; embedding a text in between
    leaves the running requests' pages and states alone."""
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
