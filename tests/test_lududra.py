"""Lududra against the plain statement in ``lududra_oracle``: every mechanism alone, then whole models
through the engine (prompts, portions, decoding, mixed batches, reused pages and slots, generation).

Each case runs on the CPU ops and, marked ``gpu``, on the kernels in fp32 and bf16."""
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import lududra_oracle as O  # noqa: E402

from hartsyinference_b200 import ops, runtime  # noqa: E402
from hartsyinference_b200.engine import LLMEngine, SamplingParams  # noqa: E402
from hartsyinference_b200.exceptions import KvPoolExhaustedError  # noqa: E402
from hartsyinference_b200.models.llm import config as C  # noqa: E402
from hartsyinference_b200.models.llm.loader import load_llm, save_hf_checkpoint  # noqa: E402
from hartsyinference_b200.models.llm.lududra import lududra_config, tensor_shapes  # noqa: E402
from hartsyinference_b200.models.llm.mixers import distance_bias_table  # noqa: E402
from hartsyinference_b200.models.llm.transformer import DecoderModel  # noqa: E402

BF, F32 = torch.bfloat16, torch.float32
MODES = [pytest.param(("cpu", F32), id="cpu-f32"), pytest.param(("cuda", F32), id="cuda-f32", marks=pytest.mark.gpu),
         pytest.param(("cuda", BF), id="cuda-bf16", marks=pytest.mark.gpu)]


def rel_err(got, want):
    got, want = got.detach().cpu().double(), want.double()
    return float((got - want).norm() / want.norm().clamp_min(1e-30))


def near(got, want, mode, f32=2e-5, bf16=1e-2):
    e = rel_err(got, want)
    assert e < (f32 if mode[1] == F32 else bf16), e


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rnd(g, *shape, std=1.0):
    return (torch.randn(*shape, generator=g) * std).to(BF)


# ------------------------------------------------------------------------------------ norms and stream
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("dim,layernorm", [(40, True), (136, True), (136, False), (1000, True), (8200, True)])
def test_stream_norms(mode, dim, layernorm):
    dev, dt = mode
    g = gen(dim)
    rows, ld = 5, (dim + 7) // 8 * 8
    x = torch.zeros(rows, ld)
    x[:, :dim] = torch.randn(rows, dim, generator=g) * 3 + 1.5
    y = torch.zeros(rows, ld, dtype=BF)
    y[:, :dim] = rnd(g, rows, dim, std=0.2) + 0.7
    wb, wn = rnd(g, dim), rnd(g, dim)
    norm = (lambda v, w: O.layer_norm(v, w, 1e-5)) if layernorm else (lambda v, w: O.rms_unit(v, 1e-5) * w)
    want_x = x[:, :dim].double() + norm(y[:, :dim].double(), wb.double())
    want_h = norm(want_x, wn.double())
    xd = x.to(dev)
    h = ops.residual_norm(xd, y.to(dt).to(dev), wb.to(dev), wn.to(dev), dim=dim, eps=1e-5, layernorm=layernorm, dtype=dt)
    assert rel_err(xd[:, :dim], want_x) < 1e-6            # the stream is fp32 whatever the activations are
    near(h[:, :dim], want_h, mode, 1e-6, 4e-3)
    assert h.dtype == dt and float(h[:, dim:].float().abs().sum()) == 0
    h2 = ops.residual_norm(xd, None, None, wn.to(dev), dim=dim, eps=1e-5, layernorm=layernorm, dtype=dt)
    assert torch.equal(h2.cpu(), h.cpu())


@pytest.mark.parametrize("mode", MODES)
def test_embedding_stream(mode):
    dev, _ = mode
    table = torch.zeros(11, 48, dtype=BF)
    table[:, :44] = rnd(gen(0), 11, 44)
    ids = torch.tensor([3, 0, 10, 3], dtype=torch.int32)
    x = ops.embedding_f32(ids.to(dev), table.to(dev), 1.7, 44)
    assert x.dtype == F32 and rel_err(x, table[ids.long()].double() * 1.7) < 1e-7


# ------------------------------------------------------------------------------------ attention
def test_distance_buckets():
    for rows, reach, window in ((8, 50, 17), (16, 100, 4000), (4, 9, 30), (32, 128, 0), (10, 77, 78)):
        rel = torch.arange(rows).float()[:, None].repeat(1, 2)
        t = distance_bias_table(rel, reach, window)
        for n in range(3 * reach):
            if window and n >= window:
                break
            assert int(t[1, min(n, t.shape[1] - 1)]) == O.distance_bucket(n, rows, reach), (rows, reach, n)


class Pages:
    """Keys of several sequences laid out in shuffled pages."""

    def __init__(self, g, lens, hkv, d, page, dtype, dev):
        counts = [(n + page - 1) // page for n in lens]
        order = torch.randperm(sum(counts) + 3, generator=g)
        self.table = torch.zeros(len(lens), max(counts), dtype=torch.int32)
        self.cache = torch.full((sum(counts) + 3, hkv, page, d), 7.0, dtype=dtype, device=dev)    # what freed pages left behind
        a = 0
        for i, c in enumerate(counts):
            self.table[i, :c] = order[a:a + c].to(torch.int32)
            a += c
        self.page, self.dev = page, dev

    def slots(self, seq, start, count):
        pos = torch.arange(start, start + count)
        return self.table[seq][pos // self.page].long() * self.page + pos % self.page


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("hq,hkv,d,page,window,tail", [(4, 1, 64, 16, 24, 1), (6, 2, 40, 8, 17, 3), (8, 8, 128, 16, 65, 70),
                                                       (3, 3, 96, 64, 1, 5), (20, 1, 24, 16, 130, 1), (2, 1, 160, 16, 33, 9),
                                                       (16, 1, 128, 32, 64, 1), (4, 2, 8, 16, 1000, 2)])
def test_window_attention(mode, hq, hkv, d, page, window, tail):
    """Three sequences whose last ``tail`` tokens are the queries. A key just inside the window, one just
    outside, one at a page's edge and the first one each stand out for some query."""
    dev, dt = mode
    g = gen(hq * 100 + d)
    lens = [tail + 150, tail + 2, max(tail, 5)]
    rows, reach, cap, scale = 8, 60, 20.0, 0.3
    q = [rnd(g, n, hq, d, std=d ** -0.5) for n in lens]
    k = [rnd(g, n, hkv, d) for n in lens]
    for i, n in enumerate(lens):
        for j, spot in enumerate((n - window, n - 1 - window, page - 1, page, 0, n - 1)):
            if 0 <= spot < n:
                h = j % hq
                u = torch.nn.functional.normalize(q[i][n - 1, h].float(), dim=0)
                k[i][spot, h // (hq // hkv)] += (u * 6).to(BF)
    for x in q:
        x *= 4
    rel = rnd(g, rows, hq)
    table = distance_bias_table(rel, reach, window)
    gate = [rnd(g, n, hq * d) for n in lens]
    sinks = torch.zeros(hq)
    want = []
    for i, n in enumerate(lens):
        o = torch.zeros(tail, hq, d, dtype=torch.float64)
        for h in range(hq):
            kk = k[i][:, h // (hq // hkv)].double()
            bias = lambda m, h=h: rel.double()[O.distance_bucket(m, rows, reach), h]
            o[:, h] = O.attention_weights(q[i][:, h].double(), kk, bias, scale, cap, window, n - tail) @ kk
        want.append(o.reshape(tail, -1) * torch.sigmoid(gate[i][n - tail:].double()))
    pg = Pages(g, lens, hkv, d, page, dt, dev)
    for i, n in enumerate(lens):
        ops.kv_store(k[i].reshape(n, -1).to(dt).to(dev), pg.cache, pg.slots(i, 0, n).to(dev))
    packed = torch.cat([torch.cat([x[n - tail:].reshape(tail, -1) for x, n in zip(q, lens)]),
                        torch.cat([x[n - tail:] for x, n in zip(gate, lens)])], 1).to(dt).to(dev)
    cu = None if tail == 1 else torch.arange(0, 3 * tail + 1, tail, dtype=torch.int32).to(dev)
    out = ops.attn_biased(packed[:, :hq * d], pg.cache, None, pg.table.to(dev), torch.tensor(lens, dtype=torch.int32).to(dev), cu,
                          heads=hq, max_q_len=tail, max_kv_len=max(lens), scale=scale, softcap=cap, window=window,
                          dist_bias=table.to(dev), sinks=sinks.to(dev), gate=packed[:, hq * d:])
    near(out, torch.cat(want), mode, 1e-5, 6e-3)


@pytest.mark.parametrize("mode", MODES)
def test_attention_options_alone(mode):
    """Separate values, no window, no cap, no bias, no sink: the ordinary attention; then a sink of its own
    value per head."""
    dev, dt = mode
    g = gen(5)
    n, hq, hkv, d, tail = 90, 4, 2, 32, 6
    q, k, v = rnd(g, n, hq, d), rnd(g, n, hkv, d), rnd(g, n, hkv, d)
    kp, vp = Pages(g, [n], hkv, d, 16, dt, dev), None
    vp = torch.zeros_like(kp.cache)
    flat = lambda x: x.reshape(n, -1).to(dt).to(dev)
    ops.kv_store(flat(k), kp.cache, kp.slots(0, 0, n).to(dev), flat(v), vp)
    for sinks in (None, torch.tensor([0.5, -1.0, 2.0, 0.0])):
        want = torch.zeros(tail, hq, d, dtype=torch.float64)
        for h in range(hq):
            for r in range(tail):
                i = n - tail + r
                s = k[:i + 1, h // 2].double() @ q[i, h].double() * d ** -0.5
                e = torch.exp(s)
                want[r, h] = (e @ v[:i + 1, h // 2].double()) / (e.sum() + (torch.exp(sinks[h].double()) if sinks is not None else 0))
        got = ops.attn_biased(flat(q)[n - tail:], kp.cache, vp, kp.table.to(dev), torch.tensor([n], dtype=torch.int32).to(dev),
                              torch.tensor([0, tail], dtype=torch.int32).to(dev), heads=hq, max_q_len=tail, scale=d ** -0.5,
                              sinks=None if sinks is None else sinks.to(dev))
        near(got, want.reshape(tail, -1), mode, 1e-5, 6e-3)


# ------------------------------------------------------------------------------------ delta rule
def delta_case(g, heads, groups, dk, dv, taps, rank=None):
    mix = dict(heads=heads, kv_heads=groups, dim=dk, vdim=dv, conv=taps)
    w = 24
    rank = rank or 10
    shapes = {"q": (groups * dk, w), "k": (groups * dk, w), "v": (heads * dv, w), "b": (heads, w), "a1": (rank, w), "a2": (heads * dk, rank),
              "g1": (rank + 3, w), "g2": (heads * dv, rank + 3), "o": (w, heads * dv)}
    t = {n: rnd(g, *s, std=s[1] ** -0.5) for n, s in shapes.items()}
    for n in "qkv":
        t[n + ".conv"] = rnd(g, shapes[n][0], taps, std=0.6)
    t["A_log"] = rnd(g, heads) - 3.0              # slow decay: what was written long ago still counts
    t["dt_bias"] = rnd(g, heads * dk)
    t["norm"] = rnd(g, dv) + 1
    return mix, w, t


def build_delta(mix, w, t, dev, dt):
    from hartsyinference_b200.models.llm.mixers import DeltaMixer
    spec = C.MixerSpec(kind="channel_delta", heads=mix["heads"], kv_heads=mix["kv_heads"], dim=mix["dim"], vdim=mix["vdim"], conv=mix["conv"])
    m = DeltaMixer(spec, w, 1e-5, dev, q=t["q"], k=t["k"], v=t["v"], b=t["b"], o=t["o"], conv=(t["q.conv"], t["k.conv"], t["v.conv"]),
                   a_log=t["A_log"], dt_bias=t["dt_bias"], norm=t["norm"], a1=t["a1"], a2=t["a2"], g1=t["g1"], g2=t["g2"])
    conv, rec = m.state_shapes(3)
    # slots hold what an earlier sequence left there
    return m, [(torch.full(conv, 3.0, dtype=dt, device=dev), torch.full(rec, -2.0, dtype=F32, device=dev))]


class _Batch:
    def __init__(self, dev, positions, slots, cu=None):
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
        self.positions, self.state_slots, self.is_decode = i32(positions), i32(slots), cu is None
        self.cu_q = None if cu is None else i32(cu)


class _Holder:
    pass


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("heads,groups,dk,dv,taps", [(2, 2, 32, 32, 4), (4, 2, 24, 40, 3), (3, 1, 64, 16, 2), (2, 1, 128, 128, 4),
                                                     (1, 1, 160, 72, 1), (2, 2, 256, 256, 5), (6, 3, 40, 8, 6)])
def test_delta_mixer(mode, heads, groups, dk, dv, taps):
    """Portions down to one and two tokens, beside another sequence, then decoding; every cut gives what the
    whole sequence gives."""
    dev, dt = mode
    g = gen(dk + dv)
    mix, w, t = delta_case(g, heads, groups, dk, dv, taps)
    hs = [rnd(g, 45, w), rnd(g, 23, w)]
    wd = {"mix." + n: v.double() for n, v in t.items()}
    want = [O.delta_mixer(h.double(), mix, wd, "mix.", 1e-5) for h in hs]
    m, state = build_delta(mix, w, t, dev, dt)
    holder = _Holder()
    holder.mixer_state = state
    got = [torch.zeros(45, w), torch.zeros(23, w)]
    done = [0, 0]
    slots = [2, 0]
    for cut in ((17, 0), (2, 5), (1, 2), (16, 1), (3, 9), (0, 2)):
        pos, cu, rows, use = [], [0], [], []
        for i, n in enumerate(cut):
            if n:
                pos += range(done[i], done[i] + n)
                cu.append(cu[-1] + n)
                rows.append(hs[i][done[i]:done[i] + n])
                use.append((i, n))
        y = m(torch.cat(rows).to(dt).to(dev), _Batch(dev, pos, [slots[i] for i, _ in use], cu), 0, holder).float().cpu()
        for (i, n), a in zip(use, cu):
            got[i][done[i]:done[i] + n] = y[a:a + n, :w]
            done[i] += n
    while done[0] < 45 or done[1] < 23:            # decode what is left, together while both last
        use = [i for i in (0, 1) if done[i] < hs[i].shape[0]]
        rows = torch.stack([hs[i][done[i]] for i in use]).to(dt).to(dev)
        y = m(rows, _Batch(dev, [done[i] for i in use], [slots[i] for i in use]), 0, holder).float().cpu()
        for j, i in enumerate(use):
            got[i][done[i]] = y[j, :w]
            done[i] += 1
    for i in (0, 1):
        near(got[i], want[i], mode, 3e-5, 2e-2)
    # slot 1 belongs to nobody: untouched; a row without a slot stores nothing
    before = [s.clone() for s in state[0]]
    m(hs[0][:1].to(dt).to(dev), _Batch(dev, [0], [-1]), 0, holder)
    assert all(torch.equal(a, b) for a, b in zip(before, state[0]))
    assert float(state[0][1][1].min()) == float(state[0][1][1].max()) == -2.0


@pytest.mark.parametrize("mode", MODES)
def test_delta_first_tokens_and_far_write(mode):
    """The convolution sees zeros before the start, and a value written at position 0 is read back 400
    tokens later."""
    dev, dt = mode
    g = gen(9)
    mix, w, t = delta_case(g, 2, 2, 32, 32, 4)
    t["A_log"] = torch.full((2,), -9.0).to(BF)
    h = rnd(g, 400, w, std=0.02)
    h[0] = rnd(g, w, std=3.0)
    h[399] = h[0]
    wd = {"mix." + n: v.double() for n, v in t.items()}
    want = O.delta_mixer(h.double(), mix, wd, "mix.", 1e-5)
    m, state = build_delta(mix, w, t, dev, dt)
    holder = _Holder()
    holder.mixer_state = state
    y = m(h.to(dt).to(dev), _Batch(dev, range(400), [1], [0, 400]), 0, holder)[:, :w]
    near(y[:5], want[:5], mode, 3e-5, 2e-2)
    near(y[395:], want[395:], mode, 3e-5, 3e-2)


@pytest.mark.parametrize("mode", MODES[1:])
def test_delta_long_portion_equals_short_ones(mode):
    """A portion long enough for several tokens per warp, spanning two sequences, against the same tokens in
    pieces: the recurrence runs the same operations wherever it is cut."""
    dev, dt = mode
    g = gen(77)
    mix, w, t = delta_case(g, 16, 16, 32, 32, 4)
    hs = rnd(g, 2200, w).to(dt).to(dev)
    m, state = build_delta(mix, w, t, dev, dt)
    holder = _Holder()
    holder.mixer_state = state
    whole = m(hs, _Batch(dev, list(range(1203)) + list(range(997)), [0, 2], [0, 1203, 2200]), 0, holder)
    after = [s.clone() for s in state[0]]
    parts = []
    for a, b, slot in ((0, 1203, 0), (1203, 2200, 2)):
        for c in range(a, b, 101):
            e = min(c + 101, b)
            parts.append(m(hs[c:e], _Batch(dev, range(c - a, e - a), [slot], [0, e - c]), 0, holder))
    assert rel_err(torch.cat(parts), whole.cpu()) < (1e-6 if dt == F32 else 2e-3)
    for x, y in zip(after, state[0]):
        for slot in (0, 2):
            assert rel_err(y[slot].float(), x[slot].float().cpu()) < (1e-6 if dt == F32 else 2e-3)


# ------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("experts,identity,top,ff,limit,tokens", [(5, 2, 3, 40, 0.7, 37), (3, 0, 1, 64, 1.5, 300), (4, 6, 5, 24, 0.3, 1),
                                                                  (33, 7, 4, 136, 1.0, 21), (20, 5, 6, 32, 1.0, 700), (150, 3, 2, 16, 0.8, 650)])
def test_experts(mode, experts, identity, top, ff, limit, tokens):
    from hartsyinference_b200.models.llm.mixers import build_experts
    from hartsyinference_b200.models.llm.moe import MoeFeedForward
    dev, dt = mode
    g = gen(experts)
    w = 88
    mlp = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top}}
    t = {}
    for e in range(experts):
        t.update({f"e{e}.gate": rnd(g, ff, w, std=0.3), f"e{e}.up": rnd(g, ff, w, std=0.3), f"e{e}.down": rnd(g, w, ff, std=0.3)})
    t["router"] = rnd(g, experts + identity, w, std=0.2)
    t["correction"] = rnd(g, experts + identity, std=0.3)      # large enough to change who is chosen
    h = rnd(g, tokens, w)
    wd = {"m." + n: v.double() for n, v in t.items()}
    want = O.expert_ff(h.double(), mlp, wd, "m.")
    moe = C.MoeConfig(num_experts=experts, identity_experts=identity, top_k=top, expert_ffn=ff, glu_limit=limit, exact_router=True)
    weights = build_experts(moe, w, dev, t["router"], t["correction"], ((t[f"e{e}.gate"], t[f"e{e}.up"], t[f"e{e}.down"]) for e in range(experts)))
    m = MoeFeedForward(C.TransformerConfig(hidden_size=w), weights, moe=moe, hidden=w)
    hd = h.to(dt).to(dev)
    ids, wts = m.route(hd)
    wi, ww = O.router(h.double(), t["router"].double(), t["correction"].double(), top)
    same = (ids.cpu().long() == wi).all(1)
    assert same.float().mean() > 0.98                           # near-ties may fall either way
    assert rel_err(wts.cpu()[same], ww[same]) < 1e-5            # scores are 32-bit in both activation types
    near(m(hd)[same.to(dev)], want[same], mode, 2e-5, 1e-2)
    x = torch.zeros(tokens, w, device=dev)
    nb = rnd(g, w)
    ops.residual_norm(x, m.routed_rows(hd), nb.to(dev), None, dim=w, eps=1e-6, layernorm=True, dtype=dt)
    near(x[same.to(dev)], O.layer_norm(want, nb.double(), 1e-6)[same], mode, 2e-5, 1e-2)


# ------------------------------------------------------------------------------------ whole models
def att(heads, kv, dim, window, reach=30, rows=8, scale=0.2, cap=15.0):
    return {"type": "attention", "_rows": rows, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim, "bias_max": reach,
                                                           "mask": {"size": window}, "scale": scale, "softcap": cap}}


def dlt(heads, kv, dim, vdim, conv=4):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def moe(experts, identity, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "identity": identity, "top": top}}


def model_cfg(vocab, width, layers, eps=1e-5, scale=2.0):
    return {"architecture": "Lududra", "embedding": {"scale": scale}, "norm": {"eps": eps}, "vocab": vocab, "width": width,
            "layers": [{**layer, "mlp": mlp} for layer, mlp in layers]}


CASES = {
    # window over page edges, grouped heads of both kinds, a layer without feed-forward, odd sizes
    "mixed": model_cfg(301, 136, [(att(6, 2, 40, 21), moe(5, 2, 3, 40, 0.7)), (dlt(4, 2, 24, 40, 3), None),
                                  (dlt(2, 2, 32, 48), moe(3, 0, 2, 72, 1.2)), (att(4, 4, 16, 7, reach=20, rows=4), moe(4, 3, 1, 24, 0.5))]),
    "delta_only": model_cfg(97, 64, [(dlt(2, 1, 64, 32, 2), moe(4, 1, 2, 32, 1.0)), (dlt(3, 3, 16, 8, 4), moe(2, 2, 2, 16, 2.0))], eps=1e-6),
    "attention_only": model_cfg(130, 96, [(att(20, 1, 24, 33), moe(6, 2, 2, 48, 0.9)), (att(2, 1, 128, 64, reach=90, rows=16), None)],
                                eps=1e-4, scale=1.0),
}


def rand_weights(cfg, calm=False, seed=0):
    """``calm`` weights for comparisons in bf16: routers whose choice no rounding can change (the scores are
    nearly equal, the corrections well apart) and attention scores of ordinary size."""
    g = gen(seed)
    shapes = dict(tensor_shapes(lududra_config(cfg)))
    for i, layer in enumerate(cfg["layers"]):        # sizes that only a tensor's shape gives
        if layer["type"] == "attention":
            shapes[f"l{i}.mix.rel"] = (layer["_rows"], layer["mixer"]["heads"])
        else:
            m = layer["mixer"]
            for n, out in (("a", m["heads"] * m["dim"]), ("g", m["heads"] * m["vdim"])):
                r = 12 if n == "a" else 20
                shapes[f"l{i}.mix.{n}1"], shapes[f"l{i}.mix.{n}2"] = (r, cfg["width"]), (out, r)
    w = {}
    for n, s in shapes.items():
        leaf = n.rsplit(".", 1)[-1]
        if "norm" in leaf:
            w[n] = rnd(g, *s, std=0.2) + 1
        elif leaf == "A_log":
            w[n] = rnd(g, *s) - 3
        elif leaf == "conv":
            w[n] = rnd(g, *s, std=0.6)
        elif leaf in ("b", "dt_bias", "rel") and len(s) < 2 or leaf == "rel":
            w[n] = rnd(g, *s)
        elif leaf == "correction":
            w[n] = (torch.randperm(s[0], generator=g) * 0.2).to(BF) if calm else rnd(g, *s, std=0.2)
        elif leaf == "router":
            w[n] = rnd(g, *s, std=(0.1 if calm else 1.0) * s[1] ** -0.5)
        else:
            gain = 3.0 if not calm and leaf in ("q", "k") and cfg["layers"][int(n[1])]["type"] == "attention" else 1.0    # scores that stand out
            w[n] = rnd(g, *s, std=gain * (s[-1] ** -0.5 if len(s) == 2 else 1.0))
    return w


_BUILT = {}


def built(case, mode):
    key = (case, mode)
    if key not in _BUILT:
        cfg = CASES[case]
        w = rand_weights(cfg, mode[1] == BF)
        model = DecoderModel(lududra_config(cfg), mode[0], dtype=mode[1])
        model.load_state_dict(w.get)
        _BUILT[key] = (cfg, w, model)
    return _BUILT[key]


_WANT = {}


def expected(case, tokens, mode=("cpu", F32)):
    key = (case, tuple(tokens), mode[1])
    if key not in _WANT:
        _WANT[key] = O.forward(tokens, CASES[case], rand_weights(CASES[case], mode[1] == BF))
    return _WANT[key]


def prompt(case, n, seed):
    return torch.randint(0, CASES[case]["vocab"], (n,), generator=gen(seed)).tolist()


def engine(model, tokens=256, batch=4, page=16, **kw):
    return LLMEngine(model, num_pages=(tokens + page - 1) // page, page_size=page, max_batch=batch, prefill_chunk=tokens,
                     max_model_len=tokens, **kw)


def logits_near(got, want, mode):
    """Root mean square of the difference over the vocabulary against the logits' own spread, at every
    position."""
    d = got.detach().cpu().double() - want
    e = d.pow(2).mean(-1).sqrt() / want.std()
    assert float(e.max()) < (2e-4 if mode[1] == F32 else 8e-2), float(e.max())


def play(eng, case, tokens, cuts, key="a"):
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
    toks = prompt(case, 75, 1)
    want = expected(case, toks, mode)
    eng = engine(model)
    for cuts in ([75], [1] * 75, [2] * 37 + [1], [16, 1, 1, 15, 2, 40], [3, 5, 7, 11, 13, 17, 19], [33] + [1] * 42):
        logits_near(play(eng, case, toks, cuts), want, mode)
        assert eng.kv.num_free == eng.num_pages
    if model.cfg.recurrent:
        assert eng.kv.num_free_slots == 4


@pytest.mark.parametrize("mode", MODES)
@pytest.mark.parametrize("case", list(CASES))
def test_model_mixed_batches(mode, case):
    """Unequal requests in one batch, portions beside single tokens, requests that pause, and pages and slots
    that change hands, against each request alone."""
    _, _, model = built(case, mode)
    seqs = {k: prompt(case, n, 10 + i) for i, (k, n) in enumerate((("a", 75), ("b", 40), ("c", 1), ("d", 23), ("e", 60), ("f", 9)))}
    eng = engine(model, tokens=224)
    at = {k: 0 for k in seqs}
    got = {k: [] for k in seqs}
    steps = [dict(a=20, b=3), dict(a=1, c=1, b=1), dict(b=30, d=2), dict(a=1, b=1, d=1), dict(a=1, b=1, d=1), dict(a=17, d=19), dict(b=4, e=31),
             dict(a=1, e=1), dict(a=34, e=1), dict(e=1, f=7), dict(e=26, f=1), dict(f=1)]
    for st in steps:
        ents, ends = [], []
        for k, n in st.items():
            ents.append((k, seqs[k][at[k]:at[k] + n], list(range(n))))
            at[k] += n
            if at[k] == len(seqs[k]):
                ends.append(k)
        y = eng.replay(ents, ends)
        r = 0
        for k, n in st.items():
            got[k].append(y[r:r + n])
            r += n
    assert all(at[k] == len(seqs[k]) for k in seqs) and eng.kv.num_free == eng.num_pages
    for k in seqs:
        logits_near(torch.cat(got[k]), expected(case, seqs[k], mode), mode)


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
    assert len(got) == len(want)
    for a, b in zip(got, want):
        e = (a.cpu().double() - b).norm(dim=1) / b.norm(dim=1)
        assert float(e.max()) < (2e-5 if mode[1] == F32 else 3e-2), float(e.max())


@pytest.mark.parametrize("mode", MODES)
def test_long_decode(mode):
    """Most of a sequence decoded token by token, far past every window."""
    _, _, model = built("mixed", mode)
    toks = prompt("mixed", 150, 4)
    logits_near(play(engine(model), "mixed", toks, [4] + [1] * 146), expected("mixed", toks, mode), mode)


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
@pytest.mark.parametrize("case", ["mixed", "delta_only"])
def test_greedy_generation(mode, case):
    """The engine's scheduler: chunked prompts beside decoding requests, then decode steps alone; then a pool so
    small that requests are pre-empted and recomputed."""
    _, _, model = built(case, mode)
    prompts = [prompt(case, n, 20 + n) for n in (37, 5, 18)]
    want = [greedy(case, p, 12) for p in prompts]
    params = SamplingParams(greedy=True, ignore_eos=True, max_tokens=12)
    eng = LLMEngine(model, num_pages=32, page_size=8, max_batch=4, prefill_chunk=16, max_model_len=96)
    assert eng.generate(prompts, params) == want
    assert eng.kv.num_free == 32
    tight = LLMEngine(model, num_pages=9, page_size=8, max_batch=4, prefill_chunk=64, max_model_len=72)
    assert tight.generate(prompts, params) == want
    assert tight.stats()["preemptions"] > 0 and tight.kv.num_free == 9
    if model.cfg.recurrent:
        assert tight.kv.num_free_slots == 4


@pytest.mark.gpu
def test_generation_bf16_graph_equals_eager():
    _, _, model = built("mixed", ("cuda", BF))
    prompts = [prompt("mixed", n, 40 + n) for n in (30, 9, 14, 2, 50)]
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
    cfg = json.loads(json.dumps(CASES["mixed"]))
    for layer in cfg["layers"]:
        layer.pop("_rows", None)
    w = rand_weights(CASES["mixed"])
    save_hf_checkpoint(cfg, w, tmp_path / "m")
    return tmp_path / "m"


def test_checkpoint_loads_by_config(checkpoint):
    llm = load_llm(checkpoint, "cpu", dtype=F32)
    assert llm.config.arch == "lududra" and llm.config.recurrent and llm.model.dtype == F32
    toks = prompt("mixed", 12, 8)
    y = engine(llm.model).replay([("x", toks, [11])], ["x"])
    logits_near(y, expected("mixed", toks)[11:], ("cpu", F32))
    with pytest.raises(ValueError):
        DecoderModel(C.tiny(), "cpu", dtype=F32)           # other architectures run in bf16
    with pytest.raises(ValueError):
        llm.config.validate_tp(2)


def test_checkpoint_is_recognised(checkpoint):
    from hartsyinference_b200.assets.registry import detect
    from hartsyinference_b200.engine.planner import shape_of_checkpoint
    d = detect(checkpoint)
    assert (d.family, d.arch) == ("llm", "lududra")
    assert shape_of_checkpoint(checkpoint) is None          # stays on one GPU


def test_service_generates_and_embeds(checkpoint):
    """Through the text service: token ids in, greedy ids out as the engine gives them; embedding a text in
    between leaves the running requests' pages and states alone."""
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
    assert sorted(p.name for p in out.iterdir()) == ["0.f32", "2.f32"]
    read = lambda n: torch.frombuffer(bytearray((out / n).read_bytes()), dtype=F32).reshape(-1, CASES["mixed"]["vocab"])
    want = expected("mixed", toks)
    logits_near(read("0.f32"), want[[0, 29]], mode)
    logits_near(read("2.f32"), want[[39, 1]], mode)


def test_text_command(checkpoint):
    from click.testing import CliRunner
    from hartsyinference_b200.cli.main import cli
    r = CliRunner().invoke(cli, ["text", str(checkpoint), "hello", "--raw", "--greedy", "--max-tokens", "4", "--device", "cpu"])
    assert r.exit_code == 0, r.output
    assert "4 tokens" in r.output + (r.stderr if r.stderr_bytes else "")


def test_state_slots_follow_sequences():
    kv = runtime.KvAllocator(8, 4, state_slots=2)
    kv.append(1, 3)
    kv.append(2, 1)
    assert {kv.seq_slot(1), kv.seq_slot(2)} == {0, 1} and not kv.can_append(3, 1)
    with pytest.raises(KvPoolExhaustedError):
        kv.append(3, 1)
    assert kv.num_free == 6 and kv.truncate(1, 2) == -1     # state cannot be rolled back
    s = kv.seq_slot(1)
    kv.append(1, 9)
    assert kv.seq_slot(1) == s
    kv.free(1)
    kv.append(3, 1)
    assert kv.seq_slot(3) == s and kv.seq_slot(1) == -1 and kv.fork_prefix(2, 9, 1) == -1
