"""Parallel decoder on the GPU against the plain statement (parallel_oracle): the mechanisms alone at kernel level, then whole models -
prompts, decoding, portions, unequal batches, reused slots, chunk edges, long decoding, greedy generation."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ctorch_b200 as B
import parallel_cases as P
import parallel_oracle as O
from ctorch_b200.workloads import bf16_bits, bf16_to_f32
from test_hybrid_gpu import Pass, all_places, dev, joined, planes, ratio

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOLERANCE = {"f32": 2e-5, "bf16": 2e-2}

_models = {}


def model_of(name, dtype, seed=0):
    key = (name, dtype, seed)
    if key not in _models:
        weights = P.make_weights(P.CASES[name], seed)
        _models[key] = (B.LanguageModel(P.CASES[name], weights, dtype=dtype), weights)
    return _models[key]


def rounded(a):
    return bf16_to_f32(bf16_bits(np.asarray(a, dtype=np.float32)))


# ---- mechanisms alone -------------------------------------------------------------------------------------------
class Chunked:
    """One chunked-attention layer's kernels over torch memory; the slots start full of junk."""

    def __init__(self, heads, kv_heads, dim, vdim, chunk, dtype, slots=4, capacity=400, dims=None, base=100.0, scale=0.3, eps=1e-5, extra=5, seed=0):
        rng = np.random.default_rng(seed)
        self.n = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, chunk=chunk, dims=dims if dims is not None else dim, base=base, scale=scale, eps=eps)
        self.bf16, self.capacity, self.extra = dtype == "bf16", capacity, extra
        self.stride = heads * (dim + 1) + kv_heads * (dim + vdim) + extra
        entries = min(chunk, capacity) if chunk else capacity
        self.q_norm, self.k_norm = rng.uniform(0.5, 1.5, heads * dim), rng.uniform(0.5, 1.5, kv_heads * dim)
        half = self.n["dims"] // 2
        angle = np.arange(capacity)[:, None] * float(base) ** (-2.0 * np.arange(half) / max(1, self.n["dims"]))
        kind = torch.bfloat16 if self.bf16 else torch.float32
        self.keys = torch.full((slots, kv_heads, entries, dim), float("nan"), dtype=kind, device="cuda")
        self.values = torch.full((slots, kv_heads, entries, vdim), float("nan"), dtype=kind, device="cuda")
        self.keep = [dev(np.cos(angle)), dev(np.sin(angle)), dev(self.q_norm), dev(self.k_norm)]
        k = self.keep
        self.kind = kind
        self.a = B.ChunkArgs(heads, kv_heads, dim, vdim, self.n["dims"], slots, chunk, entries, scale, eps, k[0].data_ptr(), k[1].data_ptr(), capacity,
                             k[2].data_ptr(), k[3].data_ptr(), B.BF16 if self.bf16 else B.F32, self.keys.data_ptr(), self.values.data_ptr())

    def kernels(self):
        self.a.projected, self.a.stride, self.a.query = 16, self.stride, 16
        return [B.lib().b200_chunk_attention_kernel(C.byref(self.a), count, self.n["heads"] * self.n["vdim"]).decode() for count in (1, 2)]

    def attend(self, p, rows, max_length, units=None, route=None, out_stride=None):
        n, count = self.n, rows.shape[0]
        projected = dev(rows)
        new = lambda *s: torch.full(s, float("nan"), dtype=self.kind, device="cuda")
        q, k, v = new(count, n["heads"], n["dim"]), new(count, n["kv_heads"], n["dim"]), new(count, n["kv_heads"], n["vdim"])
        width = n["heads"] * n["vdim"]
        stride = out_stride or width
        out = torch.full((count, stride), float("nan"), device="cuda")
        hi, lo = planes(count, stride)
        a = self.a
        a.projected, a.stride, a.query, a.key, a.value = projected.data_ptr(), self.stride, q.data_ptr(), k.data_ptr(), v.data_ptr()
        need = B.lib().b200_chunk_scratch_bytes(C.byref(a), count, p.c.sequences, p.c.max_count, max_length)
        scratch = torch.full((need // 4 + 1,), float("nan"), device="cuda")
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_chunk_prepare(C.byref(a), C.byref(p.c), C.byref(units) if units else None, C.byref(route) if route else None, None))
        B.kcheck(B.lib().b200_chunk_attention(C.byref(a), C.byref(p.c), max_length, scratch.data_ptr(), need, out.data_ptr(), hi.data_ptr(), lo.data_ptr(),
                                              stride, None))
        torch.cuda.synchronize()
        got = out.cpu().numpy()[:, :width]
        assert ratio(joined(hi, lo)[:, :width], got) < 3e-5
        self.split = need > 0
        return got

    def want(self, rows):
        """Gated attention of one whole sequence of projected rows."""
        n, T = self.n, len(rows)
        H, G, d, e = n["heads"], n["kv_heads"], n["dim"], n["vdim"]
        q, k, v, g = np.split(rows[:, :self.stride - self.extra].astype(np.float64), np.cumsum([H * d, G * d, G * e]), axis=1)
        pos = np.arange(T)
        q = O.rotate_half(O.rms_norm(q, self.q_norm, n["eps"]).reshape(T, H, d).transpose(1, 0, 2), pos, n["dims"], n["base"])
        k = O.rotate_half(O.rms_norm(k, self.k_norm, n["eps"]).reshape(T, G, d).transpose(1, 0, 2), pos, n["dims"], n["base"])
        o = O.chunked_attention(q, k, v.reshape(T, G, e).transpose(1, 0, 2), n["scale"], n["chunk"] or None)
        return (o * O.sigmoid(g)[:, :, None]).reshape(T, H * e)


CHUNKED = [dict(heads=4, kv_heads=2, dim=16, vdim=24, chunk=13), dict(heads=3, kv_heads=3, dim=10, vdim=14, chunk=20, dims=6),
           dict(heads=1, kv_heads=1, dim=64, vdim=64, chunk=1), dict(heads=20, kv_heads=1, dim=32, vdim=16, chunk=65),
           dict(heads=6, kv_heads=2, dim=128, vdim=128, chunk=0), dict(heads=2, kv_heads=1, dim=128, vdim=40, chunk=128),
           dict(heads=8, kv_heads=8, dim=48, vdim=128, chunk=1000), dict(heads=2, kv_heads=2, dim=192, vdim=96, chunk=64, dims=20),
           dict(heads=70, kv_heads=1, dim=8, vdim=8, chunk=63), dict(heads=2, kv_heads=1, dim=256, vdim=256, chunk=100),
           dict(heads=4, kv_heads=2, dim=16, vdim=16, chunk=64, dims=0)]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("spec", CHUNKED, ids=lambda s: "h{heads}_{kv_heads}_d{dim}_{vdim}_c{chunk}".format(**s))
def test_chunked_attention_layer(spec, dtype):
    """Norms over all heads, rotation of halves, append and attention: a prompt of unequal sequences, single rows, portions of two and
    more, in shuffled slots."""
    k = Chunked(**spec, dtype=dtype, seed=spec["dim"])
    assert k.kernels() == (["chunk_step_kernel", "chunk_mma_kernel"] if dtype == "bf16" and spec["dim"] % 8 == 0 else ["chunk_generic_kernel"] * 2)
    tol = 5e-6 if dtype == "f32" else 1.5e-2
    rng = np.random.default_rng(9)
    slots, totals = [2, 0, 3], [209, 76, 14]
    data = [rng.normal(size=(t, k.stride)) for t in totals]
    want = [k.want(r) for r in data]
    done, lengths = [0, 0, 0], [0] * 4
    for counts in ([150, 64, 1], [1, 1, 1], [1, 1, 1], [1, 0, 1], [2, 2, 2], [1, 1, 1], [3, 1, 3], [50, 6, 4]):
        live = [i for i in range(3) if counts[i]]
        p = Pass([counts[i] for i in live], [slots[i] for i in live], lengths)
        got = k.attend(p, np.concatenate([data[i][done[i]:done[i] + counts[i]] for i in live]), 300, out_stride=spec["heads"] * spec["vdim"] + 8)
        at = 0
        for i in live:
            assert ratio(got[at:at + counts[i]], want[i][done[i]:done[i] + counts[i]]) < tol, (counts, i)
            at += counts[i]
            done[i] += counts[i]
        p.advance()
        torch.cuda.synchronize()
        lengths = p.lengths.cpu().tolist()
    assert done == totals


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("heads, kv_heads, chunk", [(2, 2, 64), (4, 1, 37), (24, 1, 130), (2, 1, 0)])
def test_one_key_stands_out(heads, kv_heads, chunk, dtype):
    """Every query asks for one key: the first of its chunk, its own, tile borders, and - what must go unanswered - the last of the
    chunk before and the next position.  A chunk that is one position off shows as another value."""
    T, d, e = 300, 64, 16
    k = Chunked(heads, kv_heads, d, e, chunk, dtype, slots=2, capacity=T, dims=0, scale=1.0, seed=1, extra=3)
    k.q_norm[:], k.k_norm[:] = 1.0, 1.0
    k.keep[2].fill_(1.0)
    k.keep[3].fill_(1.0)
    rng = np.random.default_rng(2)
    keys, values = rng.normal(size=(T, kv_heads, d)), rng.normal(size=(T, kv_heads, e))
    rows = np.zeros((T, k.stride))
    H, G = heads, kv_heads
    rows[:, H * d:(H + G) * d], rows[:, (H + G) * d:(H + G) * d + G * e] = keys.reshape(T, -1), values.reshape(T, -1)
    size = chunk or T
    answered = np.zeros((T, H, e))
    asked_outside = np.zeros((T, H), dtype=bool)
    for t in range(T):
        begin = t - t % size
        inside = [x for x in (begin, begin + 1, begin + 63, begin + 64, t - 1, t) if begin <= x <= t]
        outside = [x for x in (begin - 1, t + 1) if 0 <= x < T]
        for h in range(H):
            asked_outside[t, h] = bool(outside) and rng.random() < 0.3
            target = rng.choice(outside if asked_outside[t, h] else inside)
            rows[t, h * d:(h + 1) * d] = keys[target, h // (H // G)]
            answered[t, h] = values[target, h // (H // G)]
    want = k.want(rows).reshape(T, H, e)
    if not asked_outside.all():   # the score of the asked key (64 against about 8) decides
        assert np.abs(want - 0.5 * answered)[~asked_outside].max() < 0.05 and np.abs(want - 0.5 * answered)[asked_outside].mean() > 0.3
    at, lengths = 0, [0, 0]
    for count in (1, 35, 1, 1, 1, 25, 1, 1, 62, 1, 1, 1, 2, 2, 61, 1, 1, 1, T - 200):
        p = Pass([count], [1], lengths)
        got = k.attend(p, rows[at:at + count], T)
        assert np.abs(got.reshape(count, H, e) - want[at:at + count]).max() < (1e-4 if dtype == "f32" else 0.05), (at, count)
        p.advance()
        torch.cuda.synchronize()
        lengths, at = p.lengths.cpu().tolist(), at + count
    assert at <= T


@pytest.mark.parametrize("group, dim, vdim", [(4, 64, 64), (1, 128, 128), (20, 64, 48)])
def test_split_keys_of_a_step(group, dim, vdim):
    """Few sequences with a long chunk: the keys of a step are split over CTAs; one of the sequences has just entered a new chunk."""
    k = Chunked(group, 1, dim, vdim, 1000, "bf16", slots=3, capacity=2100, seed=group)
    rng = np.random.default_rng(3)
    lengths = [0, 0, 0]
    slots, totals = [2, 0, 1], [990, 1003, 70]
    data = [rng.normal(size=(t, k.stride)) for t in totals]
    p = Pass([t - 1 for t in totals], slots, lengths)
    k.attend(p, np.concatenate([r[:-1] for r in data]), 2100)
    p.advance()
    torch.cuda.synchronize()
    p = Pass([1, 1, 1], slots, p.lengths.cpu().tolist())
    got = k.attend(p, np.concatenate([r[-1:] for r in data]), 2100)
    assert k.split
    for i, r in enumerate(data):
        assert ratio(got[i], k.want(r)[-1]) < 1.5e-2


@pytest.mark.parametrize("rows, experts, top, units, kind", [(1, 1, 1, 1, 2), (5, 7, 3, 40, 1), (33, 64, 8, 2100, 2), (300, 40, 40, 13, 1), (9, 1024, 5, 0, 0)])
def test_router_and_units(rows, experts, top, units, kind):
    """Choice, scores and places of the router; activation of the units beside the attention."""
    k = Chunked(2, 1, 8, 8, 4, "f32", extra=experts + units * 2 + 3, seed=rows, slots=rows, capacity=8)
    rng = np.random.default_rng(rows)
    data = rng.normal(0, 2, (rows, k.stride))
    column = k.stride - k.extra
    chosen, rank = torch.full((2, rows, top), -1, dtype=torch.int32, device="cuda")
    weight, counts = torch.zeros(rows, top, device="cuda"), torch.zeros(experts, dtype=torch.int32, device="cuda")
    out = torch.full((rows, units + 4), 7.0, device="cuda")
    hi, lo = planes(rows, units + 4)
    route = B.Route(experts, top, column, chosen.data_ptr(), weight.data_ptr(), rank.data_ptr(), counts.data_ptr())
    u = B.Units(kind, column + experts + 1, units, out.data_ptr(), hi.data_ptr(), lo.data_ptr(), units + 4)
    p = Pass([1] * rows, list(range(rows)), [0] * rows)
    got = k.attend(p, data, 8, u, route)
    assert ratio(got[:1], k.want(data[:1])) < 5e-6
    logits = data[:, column:column + experts].astype(np.float32)
    want = np.argsort(-logits, axis=1, kind="stable")[:, :top]
    assert np.array_equal(chosen.cpu(), want)
    assert ratio(weight.cpu(), O.sigmoid(np.take_along_axis(logits, want, 1).astype(np.float64))) < 1e-6
    assert np.array_equal(counts.cpu(), np.bincount(want.ravel(), minlength=experts))
    ranks = rank.cpu().numpy()
    for e in np.unique(want):
        assert sorted(ranks[want == e]) == list(range((want == e).sum()))
    part = data[:, column + experts + 1:]
    if kind == 1:
        activated = O.silu(part[:, 0:2 * units:2]) * part[:, 1:2 * units:2]
    else:
        activated = O.gelu_exact(part[:, :units]) if units else part[:, :0]
    if units:
        assert ratio(out.cpu()[:, :units], activated) < 2e-6 and ratio(joined(hi, lo)[:, :units], activated) < 3e-5
    assert bool((out[:, units:] == 7.0).all())


def test_router_ties_take_the_lower_index():
    k = Chunked(1, 1, 8, 8, 4, "f32", extra=70, slots=1, capacity=8)
    data = np.ones((1, k.stride))
    data[0, -70:] = 0.0
    data[0, -70 + 40] = 1.0
    chosen, weight = torch.zeros(1, 3, dtype=torch.int32, device="cuda"), torch.zeros(1, 3, device="cuda")
    k.attend(Pass([1], [0], [0]), data, 8, None, B.Route(70, 3, k.stride - 70, chosen.data_ptr(), weight.data_ptr(), None, None))
    assert chosen.cpu().tolist() == [[40, 0, 1]]


def run_experts(rows, experts, top, width, ff, dtype, form, load, seed=0, parts=2):
    rng = np.random.default_rng(seed)
    up, down = rounded(rng.normal(0, 1.5 * width ** -0.5, (experts, ff, width))), rounded(rng.normal(0, ff ** -0.5, (experts, width, ff)))
    x, res = rng.normal(size=(rows, width)).astype(np.float32), rng.normal(0, 2, (rows, width)).astype(np.float32)
    if load == "one":       # every row takes the last experts
        chosen = np.tile(np.arange(experts - top, experts), (rows, 1))
    else:                   # few experts take most rows, some none
        chosen = np.stack([rng.permutation(np.unique(np.concatenate([rng.geometric(0.3, 40) % experts, np.arange(top)])))[:top] for _ in range(rows)])
    weight = rng.uniform(0.2, 1.0, (rows, top))
    norm = rng.uniform(0.5, 2.0, rows) if form != "f32" else np.ones(rows)     # factor that a split norm leaves to the consumer
    h = x.astype(np.float64) * norm[:, None]
    want = res.astype(np.float64)
    for k in range(top):
        for e in np.unique(chosen[:, k]):
            at = chosen[:, k] == e
            want[at] += O.gelu_exact((weight[at, k, None] * h[at]) @ up[e].T) @ down[e].T
    kind = torch.bfloat16 if dtype == "bf16" else torch.float32
    t = lambda a, d=torch.float32: torch.tensor(np.ascontiguousarray(a), device="cuda").to(d)
    tup, tdown, tx, tres = t(up, kind), t(down, kind), t(x), t(res)
    tc, tw = t(chosen.astype(np.int32), torch.int32), t(weight.astype(np.float32))
    hi, lo = planes(rows, width)
    hi.copy_(tx)
    lo.copy_(tx - hi.float())
    total = (norm ** -2 - 1e-3) * width
    sq = t(np.stack([total * s for s in np.full(parts, 1.0 / parts)]).astype(np.float32))
    y = torch.full_like(tres, float("nan"))
    a = B.Experts(experts=experts, top=top, rows=rows, inner=width, ff=ff, weight_dtype=B.BF16 if dtype == "bf16" else B.F32, up=tup.data_ptr(),
                  down=tdown.data_ptr(), chosen=tc.data_ptr(), weight=tw.data_ptr(), residual=tres.data_ptr(), y=y.data_ptr())
    if form == "f32":
        a.x = tx.data_ptr()
    else:
        a.x_hi, a.x_lo, a.sumsq_in, a.parts_in, a.eps = hi.data_ptr(), lo.data_ptr(), sq.data_ptr(), parts, 1e-3
    torch.cuda.synchronize()
    if form == "grouped":
        ranks, counts = np.zeros((rows, top), dtype=np.int32), np.zeros(experts, dtype=np.int32)
        for s in np.random.default_rng(5).permutation(rows * top):    # the places come in no order
            e = chosen.ravel()[s]
            ranks.ravel()[s] = counts[e]
            counts[e] += 1
        tr, tcounts = t(ranks, torch.int32), t(counts, torch.int32)
        need = B.lib().b200_experts_grouped_bytes(C.byref(a))
        scratch = torch.full((need // 4,), float("nan"), device="cuda")
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_experts_grouped(C.byref(a), tr.data_ptr(), tcounts.data_ptr(), scratch.data_ptr(), need, None))
    else:
        act = torch.full((rows * top, ff), float("nan"), device="cuda")
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_experts_streamed(C.byref(a), act.data_ptr(), None))
    torch.cuda.synchronize()
    status = C.c_int32()
    B.kcheck(B.lib().b200_take_device_status(0, None, C.byref(status)))
    assert status.value == 0
    return ratio(y.cpu(), want)


@pytest.mark.parametrize("rows, experts, top, width, ff", [(1, 1, 1, 8, 8), (3, 5, 2, 36, 21), (17, 12, 4, 184, 104), (40, 3, 3, 100, 264)])
@pytest.mark.parametrize("dtype, form", [("f32", "f32"), ("bf16", "f32"), ("bf16", "planes")])
def test_streamed_experts(rows, experts, top, width, ff, dtype, form):
    assert run_experts(rows, experts, top, width, ff, dtype, form, "some") < (3e-6 if form == "f32" else 3e-5)


@pytest.mark.parametrize("rows, experts, top, width, ff", [(1, 2, 1, 8, 8), (25, 8, 1, 64, 72), (60, 70, 5, 200, 136), (90, 6, 2, 136, 200), (700, 5, 2, 136, 264), (300, 300, 3, 64, 32)])
@pytest.mark.parametrize("load", ["some", "one"])
def test_grouped_experts(rows, experts, top, width, ff, load):
    assert run_experts(rows, experts, top, width, ff, "bf16", "grouped", load) < 5e-5


@pytest.mark.parametrize("rows, inner, units", [(1, 64, 40), (16, 256, 130), (40, 136, 64), (300, 128, 100), (270, 64, 33)])
def test_gated_units_beside_other_columns(rows, inner, units):
    """SwiGLU epilogue into a column range of wider rows, every linear kernel family."""
    rng = np.random.default_rng(units)
    x, w = rng.normal(size=(rows, inner)), rounded(rng.normal(0, 1.5 * inner ** -0.5, (2 * units, inner)))
    hi, lo = planes(rows, inner)
    tx = dev(x)
    hi.copy_(tx)
    lo.copy_(tx - hi.float())
    tw = torch.tensor(w, device="cuda").bfloat16()
    for column, stride in ((6, units + 14), (0, 0), (3, units + 5)):
        oh, ol = planes(rows, stride or units)
        a = B.ShadowLinearArgs(x_hi=hi.data_ptr(), x_lo=lo.data_ptr(), rows=rows, inner=inner, weight=tw.data_ptr(), out=2 * units, epilogue=2,
                               out_hi=oh.data_ptr() + 2 * column, out_lo=ol.data_ptr() + 2 * column, out_stride=stride)
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_linear_shadow(C.byref(a), None))
        torch.cuda.synchronize()
        z = x @ w.T.astype(np.float64)
        got = joined(oh, ol)
        assert ratio(got[:, column:column + units], O.silu(z[:, 0::2]) * z[:, 1::2]) < 5e-5
        assert np.all(got[:, :column] == 0) and np.all(got[:, column + units:] == 0)


# ---- whole models -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", P.CASES)
def test_prompt_matches_the_statement_layer_by_layer(name, dtype):
    model, w = model_of(name, dtype)
    c = P.CASES[name]
    for count in (71, 9):    # tiles of one expert; slots that stream their experts
        ids = P.decided_tokens(c, w, count)
        trail = []
        want = O.forward(c, w, ids, trail)
        model.new_cache(2, 80)
        got_trail = model.trail(1, ids)
        for i, rows in enumerate(trail):
            assert ratio(got_trail[i], rows) < TOLERANCE[dtype], f"layer run {i}"
        assert ratio(model.run([(0, ids, all_places(count))]), want) < TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", P.CASES)
def test_decoding_and_portions_equal_the_whole_prompt(name, dtype):
    """Token by token, portions of two, unequal portions: the logits of every position equal those of one pass."""
    model, w = model_of(name, dtype)
    c = P.CASES[name]
    ids = P.decided_tokens(c, w, 70, seed=3)
    model.new_cache(1, 70)
    whole = model.run([(0, ids, all_places(70))])
    tol = 1e-5 if dtype == "f32" else 1e-2
    for portions in ([1] * 70, [2] * 35, [3, 1, 5, 1, 1, 54, 1, 2, 1, 1], [63, 1, 1, 5], [64, 6], [65, 2, 2, 1]):
        model.cache.release(0)
        at, out = 0, []
        for n in portions:
            out.append(model.run([(0, ids[at:at + n], all_places(n))]))
            at += n
        assert ratio(np.concatenate(out), whole) < tol, portions[:4]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", ["mixed", "wide", "odd", "ones"])
def test_unequal_batches_equal_each_alone_and_slots_are_reused(name, dtype):
    model, w = model_of(name, dtype)
    c = P.CASES[name]
    counts, tails = [1, 67, 20, 3, 130], [4, 6, 1, 9, 5]
    full = [P.decided_tokens(c, w, n + t, seed=n) for n, t in zip(counts, tails)]
    prompts = [ids[:n] for ids, n in zip(full, counts)]
    model.new_cache(1, 140)
    alone = []
    for ids in full:
        alone.append(model.run([(0, ids, all_places(len(ids)))]))
        model.cache.release(0)
    tol = 1e-5 if dtype == "f32" else 1e-2
    model.new_cache(6, 140)
    # the second time round the requests sit in other slots, which hold what the first batch left
    for slots in ([0, 1, 2, 3, 4], [4, 5, 0, 1, 3]):
        got = [[] for _ in full]

        def step(parts):
            out = model.run([(slots[i], full[i][a:b], all_places(b - a)) for i, a, b in parts])
            for i, a, b in parts:
                got[i].append(out[:b - a])
                out = out[b - a:]
        step([(i, 0, len(p)) for i, p in enumerate(prompts)])
        for t in range(max(tails)):
            parts = [(i, len(p) + t, len(p) + t + 1) for i, p in enumerate(prompts) if t < tails[i]]
            step(parts[::-1] if t % 2 else parts)   # the order of the rows in a batch does not matter either
            for i, n in enumerate(tails):
                if t + 1 == n:
                    model.cache.release(slots[i])
        for i in range(len(full)):
            assert ratio(np.concatenate(got[i]), alone[i]) < tol, (slots, i)


def test_prompts_and_single_tokens_in_one_pass():
    """A pass in which one request brings a prompt, one goes on by a token and one by three."""
    for dtype in ("f32", "bf16"):
        model, w = model_of("mixed", dtype)
        c = P.CASES["mixed"]
        full = [P.decided_tokens(c, w, n, seed=n) for n in (40, 33, 50)]
        model.new_cache(3, 60)
        alone = [model.run([(i, ids, all_places(len(ids)))]) for i, ids in enumerate(full)]
        model.cache.clear()
        model.run([(1, full[1][:32], []), (2, full[2][:47], [])])
        got = model.run([(0, full[0], all_places(40)), (1, full[1][32:], [0]), (2, full[2][47:], [0, 1, 2])])
        want = np.concatenate([alone[0], alone[1][32:], alone[2][47:]])
        assert ratio(got, want) < (1e-5 if dtype == "f32" else 1e-2)


def test_long_pass_is_cut_and_joined():
    """More rows than one pass over the layers takes: the cut falls inside a sequence and between sequences."""
    model, _ = model_of("ones", "f32")
    c = P.CASES["ones"]
    ids = [P.tokens(c, n, seed=n) for n in (5000, 6000, 40)]
    model.new_cache(3, 6000)
    places = [[0, 4999], [3190, 3191, 3192, 5999], [39]]
    got = model.run([(i, t, p) for i, (t, p) in enumerate(zip(ids, places))])
    at = 0
    for i, (t, wanted) in enumerate(zip(ids, places)):
        model.cache.release(i)
        alone = []
        for a in range(0, len(t), 2500):
            part = t[a:a + 2500]
            alone.append(model.run([(i, part, [p - a for p in wanted if a <= p < a + len(part)])]))
        assert ratio(got[at:at + len(wanted)], np.concatenate(alone)) < 2e-5
        at += len(wanted)


@pytest.mark.parametrize("name, dtype", [("mixed", "f32"), ("plain", "bf16")])   # (plain: every expert is chosen, no call is close)
def test_long_decoding_stays_with_the_statement(name, dtype):
    model, w = model_of(name, dtype)
    c = P.CASES[name]
    ids = P.tokens(c, 300, seed=8)
    want = O.forward(c, w, ids)
    model.new_cache(1, 300)
    model.run([(0, ids[:5], [])])
    got = np.concatenate([model.run([(0, [t], [0])]) for t in ids[5:]])
    assert ratio(got, want[5:]) < TOLERANCE[dtype]


@pytest.mark.parametrize("name", ["mixed", "odd", "plain", "deep"])
def test_greedy_generation_equals_the_statement(name):
    """The framework's own loop: prompts of unequal length in one batch, the token loop in a captured graph."""
    model, w = model_of(name, "f32")
    c = P.CASES[name]
    prompts, steps = [P.tokens(c, n, seed=n) for n in (9, 2, 31)], 12
    got = model.generate(prompts, steps)
    for row, prompt in zip(got, prompts):
        want, margin = O.greedy(c, w, prompt, steps)
        assert margin > 1e-4 and list(row) == want


@pytest.mark.parametrize("name, batch", [("mixed", 1), ("mixed", 20), ("wide", 40), ("plain", 150), ("uneven", 3), ("deep", 30)])
def test_bf16_generation_feeds_back_its_own_choice(name, batch):
    """bf16 loop (fused logits + choice; streaming and dense projections; streamed and grouped experts): replaying its tokens gives
    logits whose best is the token chosen next, and the logits asked for on demand are those."""
    model, _ = model_of(name, "bf16")
    c = P.CASES[name]
    steps, prompts = 8, np.stack([P.tokens(c, 10, seed=b) for b in range(batch)])
    model.new_cache(batch, 10 + steps)
    gen = B.Generation(model, batch, steps)
    gen.prefill(prompts)
    gen.step(steps - 1)
    tokens, last = gen.tokens(), gen.logits()
    assert gen.launches_per_step() > 0 and tokens.shape == (batch, steps)
    model.new_cache(1, 10 + steps)
    for b in range(0, batch, max(1, batch // 20)):
        ids = np.concatenate([prompts[b], tokens[b]])
        logits = model.run([(0, ids, all_places(len(ids)))])
        model.cache.release(0)
        for s in range(steps):
            row = logits[9 + s]
            assert row.max() - row[tokens[b, s]] < 1e-2 * np.abs(row).max()
        assert ratio(last[b], logits[9 + steps - 1]) < 1e-2


def test_sampling_and_host_steps():
    model, _ = model_of("mixed", "f32")
    c = P.CASES["mixed"]
    prompts = np.stack([P.tokens(c, 7, seed=b) for b in range(3)])
    greedy = model.generate(list(prompts), 6)
    assert np.array_equal(model.generate(list(prompts), 6, temperature=1e-4), greedy)   # cold sampling is the greedy choice
    model.new_cache(3, 13)
    gen = B.Generation(model, 3, 6)
    gen.prefill(prompts)
    first = gen.tokens()[:, 0].copy()
    assert np.array_equal(gen.run_host(first, 5).T, greedy[:, 1:])


def test_cache_errors_leave_the_model_usable():
    model, _ = model_of("mixed", "f32")
    c = P.CASES["mixed"]
    model.new_cache(2, 10)
    ids = P.tokens(c, 10)
    want = model.run([(1, ids, [9])])
    model.cache.release(1)
    for entries, message in (([(0, P.tokens(c, 11), [])], "capacity"), ([(2, ids, [])], "slot out of range"), ([(0, ids[:2], []), (0, ids[:2], [])], "twice"),
                             ([(0, [c["vocab"]], [])], "out of range"), ([(0, ids[:2], [2])], "wanted place")):
        with pytest.raises(B.B200Error, match=message):
            model.run(entries)
    assert ratio(model.run([(1, ids, [9])]), want) < 1e-6


def test_module_forward_equals_the_statement():
    model, w = model_of("mixed", "f32")
    ids = np.stack([P.tokens(P.CASES["mixed"], 12, seed=1), P.tokens(P.CASES["mixed"], 12, seed=2)])
    got = model.module(B.Tensor.from_numpy(ids.astype(np.int64))).numpy()
    for b in range(2):
        assert ratio(got[b], O.forward(P.CASES["mixed"], w, ids[b])) < TOLERANCE["f32"]


def test_single_plane_activations():
    """The bf16-activation option (one plane in passes over more than 16 rows) stays near the statement.  (Every expert is chosen, so
    that no router's choice can turn.)"""
    c = P.CASES["plain"]
    weights = P.make_weights(c, 0)
    model = B.LanguageModel(c, weights)
    model.set_activation_dtype("bf16")
    ids = P.tokens(c, 60)
    model.new_cache(1, 60)
    assert ratio(model.run([(0, ids, all_places(60))]), O.forward(c, weights, ids)) < 4e-2


def test_argument_errors_are_refused_before_a_launch():
    k = Chunked(2, 1, 8, 8, 4, "f32", slots=1, capacity=8)
    rows = torch.zeros(2, k.stride, device="cuda")
    k.a.projected, k.a.stride, k.a.query = rows.data_ptr(), k.stride, rows.data_ptr()
    p = Pass([2], [0], [0])
    assert B.lib().b200_chunk_prepare(C.byref(k.a), C.byref(p.c), None, None, None) == -1 and b"workspaces" in B.lib().b200_last_error()
    p = Pass([1], [0], [0])
    r = B.Route(4, 5, 0, rows.data_ptr(), rows.data_ptr(), None, None)
    assert B.lib().b200_chunk_prepare(C.byref(k.a), C.byref(p.c), None, C.byref(r), None) == -1 and b"router" in B.lib().b200_last_error()
    e = B.Experts(experts=2, top=3, rows=1, inner=8, ff=8, weight_dtype=B.F32)
    assert B.lib().b200_experts_streamed(C.byref(e), rows.data_ptr(), None) == -1


def test_command_lines(tmp_path):
    """The generation command and the trace runner as a user starts them."""
    c = P.CASES["mixed"]
    w = P.make_weights(c, 2)
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir()
    out.mkdir()
    P.write_folder(folder, c, w)
    prompts = [P.tokens(c, 5, seed=1).tolist(), P.tokens(c, 3, seed=2).tolist()]
    run = subprocess.run([sys.executable, "-m", "ctorch_b200.generate", "--model", str(folder), "--dtype", "f32", "--steps", "4",
                          *[",".join(map(str, p)) for p in prompts]], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [[int(t) for t in line.split(",")] for line in run.stdout.split()] == [O.greedy(c, w, p, 4)[0] for p in prompts]
    a, b = P.decided_tokens(c, w, 22, seed=5).tolist(), P.decided_tokens(c, w, 4, seed=6).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": b[:3], "want": []}, {"id": "y", "tokens": a[:20], "want": [0, 15, 16, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": a[20:21], "want": []}, {"id": "x", "tokens": b[3:], "want": []}], "end": ["x"]},
             {"step": 2, "entries": [{"id": "y", "tokens": a[21:], "want": [0]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "z", "tokens": b, "want": [3]}], "end": ["z"]}]
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 2e-2)):
        run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "40"],
                             input="".join(json.dumps(s) + "\n" for s in steps), cwd=ROOT, capture_output=True, text=True, timeout=600)
        assert run.returncode == 0, run.stderr
        assert [line for line in run.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        full_a, full_b = O.forward(c, w, a), O.forward(c, w, b)
        for step, want in ((0, full_a[[0, 15, 16, 19]]), (2, full_a[[21]]), (3, full_b[[3]])):
            assert ratio(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(-1, c["vocab"]), want) < tol
