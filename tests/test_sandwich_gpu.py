"""Sandwich decoder on the GPU against the plain statement (sandwich_oracle): the mechanisms alone at kernel level, then whole models -
prompts, decoding, portions, unequal batches, reused slots, far keys, long decoding, greedy generation."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ctorch_b200 as B
import sandwich_cases as S
import sandwich_oracle as O
from hybrid_oracle import rotate
from test_hybrid_gpu import Pass, all_places, dev, joined, planes, ratio
from test_parallel_gpu import rounded

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOLERANCE = {"f32": 2e-5, "bf16": 2e-2}

_models = {}


def model_of(name, dtype, seed=0):
    key = (name, dtype, seed)
    if key not in _models:
        weights = S.make_weights(S.CASES[name], seed)
        _models[key] = (B.LanguageModel(S.CASES[name], weights, dtype=dtype), weights)
    return _models[key]


def status_is_clear():
    status = C.c_int32()
    B.kcheck(B.lib().b200_take_device_status(0, None, C.byref(status)))
    return status.value == 0


# ---- attention alone --------------------------------------------------------------------------------------------
class Grouped:
    """One attention layer's kernels over torch memory, in one of the forms of this design (`kind`: 1 biased keys as values with a sink of
    score 0 and gates, 2 head norms with learned sinks, 3 projection norms with learned sinks and gates); the slots start full of junk."""

    def __init__(self, kind, heads, kv_heads, dim, vdim, dtype, slots=4, capacity=400, dims=None, base=100.0, scale=0.3, cap=0.0, eps=1e-5, factor=1.0,
                 sinks=None, extra=5, seed=0):
        rng = np.random.default_rng(seed)
        dims = 0 if kind == 3 else dims if dims is not None else dim
        self.kind, self.bf16, self.capacity, self.extra = kind, dtype == "bf16", capacity, extra
        self.n = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, dims=dims, base=base, scale=scale, cap=cap, eps=eps, factor=factor)
        self.columns = heads * dim + kv_heads * dim + (0 if kind == 1 else kv_heads * vdim) + (0 if kind == 2 else heads)
        self.stride = self.columns + extra
        self.q_bias, self.k_bias = rng.normal(0, 0.5, heads * dim), rng.normal(0, 0.5, kv_heads * dim)
        self.q_norm, self.k_norm = rng.uniform(0.5, 1.5, heads * dim), rng.uniform(0.5, 1.5, kv_heads * dim)
        self.sinks = np.zeros(heads) if kind == 1 else np.asarray(sinks if sinks is not None else rng.uniform(-1.0, 3.0, heads))
        angle = np.arange(capacity)[:, None] * float(base) ** (-2.0 * np.arange(dims // 2) / max(1, dims))
        self.type = torch.bfloat16 if self.bf16 else torch.float32
        self.keys = torch.full((slots, kv_heads, capacity, dim), float("nan"), dtype=self.type, device="cuda")
        self.values = torch.full((slots, kv_heads, capacity, vdim), float("nan"), dtype=self.type, device="cuda")
        self.keep = [dev(a) for a in (np.cos(angle), np.sin(angle), self.q_norm, self.k_norm, self.q_bias, self.k_bias, self.sinks)]
        k = [t.data_ptr() for t in self.keep]
        a = self.a = B.ChunkArgs(heads, kv_heads, dim, vdim, dims, slots, 0, capacity, scale, eps, k[0], k[1], capacity, None, None, B.BF16 if self.bf16 else B.F32,
                                 self.keys.data_ptr(), self.values.data_ptr())
        a.rotate_pairs, a.softcap, a.sink, a.scaled, a.out_scale = 1, cap, k[6], 1, factor
        if kind == 1:
            a.norm, a.q_bias, a.k_bias, a.keys_as_values = B.HEAD_NORM_NONE, k[4], k[5], 1
        elif kind == 2:
            a.norm, a.no_gate = B.HEAD_NORM_HEAD, 1
        else:
            a.norm, a.q_norm, a.k_norm = B.HEAD_NORM_PROJECTION, k[2], k[3]

    def attend(self, p, rows, max_length):
        n, count = self.n, rows.shape[0]
        projected = dev(rows)
        q = torch.full((count, n["heads"], n["dim"]), float("nan"), dtype=self.type, device="cuda")
        width = n["heads"] * n["vdim"]
        out = torch.full((count, width + 8), float("nan"), device="cuda")
        hi, lo = planes(count, width + 8)
        a = self.a
        a.projected, a.stride, a.query = projected.data_ptr(), rows.shape[1], q.data_ptr()
        need = B.lib().b200_chunk_scratch_bytes(C.byref(a), count, p.c.sequences, p.c.max_count, max_length)
        scratch = torch.full((need // 4 + 1,), float("nan"), device="cuda")
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_chunk_prepare(C.byref(a), C.byref(p.c), None, None, None))
        B.kcheck(B.lib().b200_chunk_attention(C.byref(a), C.byref(p.c), max_length, scratch.data_ptr(), need, out.data_ptr(), hi.data_ptr(), lo.data_ptr(), width + 8, None))
        torch.cuda.synchronize()
        got = out.cpu().numpy()[:, :width]
        assert ratio(joined(hi, lo)[:, :width], got) < 3e-5
        self.split = need > 0
        return got

    def parts(self, rows):
        """Queries, keys, values [heads, T, size] and gates [T, heads] of a sequence's projected rows."""
        n, T = self.n, len(rows)
        H, G, d, e = n["heads"], n["kv_heads"], n["dim"], n["vdim"]
        sizes = np.cumsum([H * d, G * d, 0 if self.kind == 1 else G * e])
        q, k, v, g = np.split(rows[:, :self.columns].astype(np.float64), sizes, axis=1)
        turn = lambda x: rotate(x, np.arange(T), n["dims"], n["base"]) if n["dims"] else x
        if self.kind == 1:
            q, k = O.heads_of(q + self.q_bias, H), O.heads_of(k + self.k_bias, G)
            return turn(q), turn(k), k, O.sigmoid(g)
        if self.kind == 2:
            return O.rms(turn(O.heads_of(q, H)), n["eps"]), O.rms(turn(O.heads_of(k, G)), n["eps"]), O.heads_of(v, G), np.ones((T, H))
        return O.heads_of(O.rms(q, n["eps"]) * self.q_norm, H), O.heads_of(O.rms(k, n["eps"]) * self.k_norm, G), O.heads_of(v, G), O.sigmoid(g)

    def want(self, rows):
        q, k, v, gate = self.parts(rows)
        o = O.attend(q, k, v, self.n["scale"], self.n["cap"] or None, self.sinks) * gate[:, :, None]
        return self.n["factor"] * o.reshape(len(rows), -1)


GROUPED = [dict(kind=1, heads=4, kv_heads=2, dim=16, vdim=16), dict(kind=1, heads=3, kv_heads=1, dim=10, vdim=10, dims=6), dict(kind=1, heads=40, kv_heads=1, dim=96, vdim=96, factor=0.5),
           dict(kind=1, heads=2, kv_heads=2, dim=256, vdim=256, dims=20), dict(kind=1, heads=6, kv_heads=2, dim=20, vdim=20, dims=6),
           dict(kind=2, heads=4, kv_heads=2, dim=24, vdim=16, cap=4.0), dict(kind=2, heads=3, kv_heads=3, dim=10, vdim=14, cap=2.0, dims=2),
           dict(kind=2, heads=1, kv_heads=1, dim=64, vdim=64), dict(kind=2, heads=20, kv_heads=1, dim=128, vdim=64, cap=1.0, scale=1.0), dict(kind=2, heads=2, kv_heads=1, dim=192, vdim=96, cap=45.0),
           dict(kind=3, heads=8, kv_heads=2, dim=64, vdim=64, factor=0.7), dict(kind=3, heads=3, kv_heads=1, dim=10, vdim=6, factor=-1.5), dict(kind=3, heads=4, kv_heads=4, dim=72, vdim=128)]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("spec", GROUPED, ids=lambda s: "k{kind}_h{heads}_{kv_heads}_d{dim}_{vdim}".format(**s))
def test_attention_layer(spec, dtype):
    """Biases, norms, rotation of pairs, append, capped scores, sinks and gates: a prompt of unequal sequences, single rows, portions of two
    and more, in shuffled slots."""
    k = Grouped(**spec, dtype=dtype, seed=spec["dim"])
    tol = 5e-6 if dtype == "f32" else 1.5e-2
    rng = np.random.default_rng(9)
    slots, totals = [2, 0, 3], [209, 76, 14]
    data = [rng.normal(size=(t, k.stride)) for t in totals]
    want = [k.want(r) for r in data]
    done, lengths = [0, 0, 0], [0] * 4
    for counts in ([150, 64, 1], [1, 1, 1], [1, 1, 1], [1, 0, 1], [2, 2, 2], [1, 1, 1], [3, 1, 3], [50, 6, 4]):
        live = [i for i in range(3) if counts[i]]
        p = Pass([counts[i] for i in live], [slots[i] for i in live], lengths)
        got = k.attend(p, np.concatenate([data[i][done[i]:done[i] + counts[i]] for i in live]), 300)
        at = 0
        for i in live:
            assert ratio(got[at:at + counts[i]], want[i][done[i]:done[i] + counts[i]]) < tol, (counts, i)
            at += counts[i]
            done[i] += counts[i]
        p.advance()
        torch.cuda.synchronize()
        lengths = p.lengths.cpu().tolist()
    assert done == totals and status_is_clear()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("kind, heads, kv_heads", [(1, 2, 2), (1, 24, 1), (2, 4, 1), (3, 2, 1)])
def test_one_key_stands_out(kind, heads, kv_heads, dtype):
    """Every query asks for one key - the first, its own, tile borders, one far back - or for the next position, which must go unanswered;
    a missing sink, a key too many or too few shows as another value."""
    T, d = 300, 64
    e = d if kind == 1 else 16
    k = Grouped(kind, heads, kv_heads, d, e, dtype, slots=2, capacity=T, dims=0, scale=1.0, seed=1, extra=3, sinks=np.linspace(50.0, 68.0, heads))
    for a in (k.q_norm, k.k_norm):
        a[:] = 1.0
    for a in (k.q_bias, k.k_bias):
        a[:] = 0.0
    for i, v in ((2, 1.0), (3, 1.0), (4, 0.0), (5, 0.0)):
        k.keep[i].fill_(v)
    rng = np.random.default_rng(2)
    H, G = heads, kv_heads
    keys = rng.normal(size=(T, G, d))
    keys *= 8.0 / np.linalg.norm(keys, axis=2, keepdims=True)      # |key|^2 = 64
    values = keys if kind == 1 else rng.normal(size=(T, G, e))
    rows = np.zeros((T, k.stride))
    rows[:, H * d:(H + G) * d] = keys.reshape(T, -1)
    if kind != 1:
        rows[:, (H + G) * d:(H + G) * d + G * e] = values.reshape(T, -1)
    answered, ahead = np.zeros((T, H, e)), np.zeros((T, H), dtype=bool)
    for t in range(T):
        inside = [x for x in (0, 1, 63, 64, 127, 128, t - 64, t - 1, t) if 0 <= x <= t]
        for h in range(H):
            ahead[t, h] = t + 1 < T and rng.random() < 0.3
            target = t + 1 if ahead[t, h] else rng.choice(inside)
            rows[t, h * d:(h + 1) * d] = keys[target, h // (H // G)]
            answered[t, h] = values[target, h // (H // G)]
    want = k.want(rows).reshape(T, H, e)
    share = {1: 1.0, 2: None, 3: None}[kind]
    if share is not None:      # the asked key's score, 64, decides (gates are 1/2)
        assert np.abs(want - 0.5 * answered)[~ahead].max() < 0.05 and np.abs(want - 0.5 * answered)[ahead].mean() > 0.3
    else:                      # sinks from far below to above the asked key's score
        assert np.abs(want[:, 0] - (1.0 if kind == 2 else 0.5) * answered[:, 0])[~ahead[:, 0]].max() < 0.05 and np.abs(want[:, -1]).max() < 0.2
    at, lengths = 0, [0, 0]
    for count in (1, 35, 1, 1, 1, 25, 1, 1, 62, 1, 1, 1, 2, 2, 61, 1, 1, 1, T - 200):
        p = Pass([count], [1], lengths)
        got = k.attend(p, rows[at:at + count], T)
        assert np.abs(got.reshape(count, H, e) - want[at:at + count]).max() < (1e-4 if dtype == "f32" else 0.06), (at, count)
        p.advance()
        torch.cuda.synchronize()
        lengths, at = p.lengths.cpu().tolist(), at + count
    assert at <= T


@pytest.mark.parametrize("kind, group, dim, vdim, cap", [(1, 4, 64, 64, 0.0), (2, 1, 128, 128, 3.0), (3, 20, 64, 48, 0.0), (2, 6, 40, 56, 45.0)])
def test_split_keys_of_a_step(kind, group, dim, vdim, cap):
    """Few long sequences: the keys of a step are split over CTAs, the sink joins once."""
    k = Grouped(kind, group, 1, dim, vdim, "bf16", slots=3, capacity=2100, cap=cap, sinks=np.full(group, 6.0), seed=group)
    rng = np.random.default_rng(3)
    slots, totals = [2, 0, 1], [990, 1003, 70]
    data = [rng.normal(size=(t, k.stride)) for t in totals]
    p = Pass([t - 1 for t in totals], slots, [0, 0, 0])
    k.attend(p, np.concatenate([r[:-1] for r in data]), 2100)
    p.advance()
    torch.cuda.synchronize()
    p = Pass([1, 1, 1], slots, p.lengths.cpu().tolist())
    got = k.attend(p, np.concatenate([r[-1:] for r in data]), 2100)
    assert k.split
    for i, r in enumerate(data):
        assert ratio(got[i], k.want(r)[-1]) < 1.5e-2


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_keys_of_another_layer(dtype):
    """A layer with queries only over the slots that another one fills: prompt, portion, single rows."""
    source, reader = (Grouped(2, heads, 2, 24, 16, dtype, slots=2, capacity=150, cap=5.0, seed=heads) for heads in (4, 6))
    rng = np.random.default_rng(4)
    T = 140
    made, asked = rng.normal(size=(T, source.stride)), rng.normal(size=(T, 6 * 24 + 3))
    _, keys, values, _ = source.parts(made)
    q = O.rms(rotate(O.heads_of(asked[:, :6 * 24], 6), np.arange(T), 24, 100.0), 1e-5)
    want = O.attend(q, keys, values, 0.3, 5.0, reader.sinks).reshape(T, -1)
    reader.a.key_cache, reader.a.value_cache, reader.a.keys_elsewhere = source.a.key_cache, source.a.value_cache, 1
    at, lengths = 0, [0, 0]
    for count in (70, 1, 1, 2, 65, 1):
        p = Pass([count], [1], lengths)
        source.attend(p, made[at:at + count], T)
        assert ratio(reader.attend(p, asked[at:at + count], T), want[at:at + count]) < (5e-6 if dtype == "f32" else 1.5e-2), at
        p.advance()
        torch.cuda.synchronize()
        lengths, at = p.lengths.cpu().tolist(), at + count


# ---- lightning attention alone ----------------------------------------------------------------------------------
@pytest.mark.parametrize("heads, dim, vdim, batch", [(2, 64, 32, 3), (1, 16, 16, 1), (5, 9, 7, 2), (3, 130, 24, 2), (4, 300, 64, 1), (8, 128, 128, 3), (16, 64, 64, 200)])
def test_lightning_recurrence(heads, dim, vdim, batch):
    """Prompts of unequal lengths, single rows and portions in shuffled slots full of junk; decays from almost nothing to one."""
    rng = np.random.default_rng(dim)
    decay = np.resize([0.999, 0.3, 1.0, 0.9, 1e-3], heads)
    inner, channels, lead = heads * vdim, heads * vdim + 2 * heads * dim, 8
    stride = lead + inner + channels + 4
    slots = rng.permutation(batch + 2)[:batch].tolist()
    state = torch.full((batch + 2, heads, dim, vdim), float("nan"), device="cuda")
    tdecay = dev(decay)
    plan = [[30 + 7 * (b % 5) for b in range(batch)], [1] * batch, [1] * batch, [2] * batch, [17] * batch, [1] * batch] if batch < 100 else [[2] * batch, [1] * batch, [1] * batch]
    totals = [sum(step[b] for step in plan) for b in range(batch)]
    data = [rng.normal(size=(t, stride)) for t in totals]

    def want(rows):
        part = O.silu(rows[:, lead + inner:lead + inner + channels].astype(np.float32).astype(np.float64))
        v, k, q = np.split(part, np.cumsum([inner, heads * dim]), axis=1)
        shaped = lambda x: x.reshape(len(rows), heads, -1)
        return O.lightning_recurrence(shaped(q), shaped(k), shaped(v), decay.astype(np.float32)).reshape(len(rows), inner)
    check = range(batch) if batch < 100 else range(0, batch, 37)
    expected = {b: want(data[b]) for b in check}
    done, lengths = [0] * batch, [0] * (batch + 2)
    for step in plan:
        p = Pass(step, slots, lengths)
        rows = dev(np.concatenate([data[b][done[b]:done[b] + step[b]] for b in range(batch)]))
        y, mixed = torch.full((rows.shape[0], inner), float("nan"), device="cuda"), torch.empty(rows.shape[0], channels, device="cuda")
        a = B.SsmArgs(heads=heads, vdim=vdim, state=dim, groups=heads, taps=1, ssm_state=state.data_ptr(), projected=rows.data_ptr() + 4 * lead, mixed=mixed.data_ptr(),
                      y=y.data_ptr(), decay=tdecay.data_ptr(), stride=stride)
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_ssm_forward(C.byref(a), C.byref(p.c), None))
        p.advance()
        torch.cuda.synchronize()
        first = p.first_host
        for b in check:
            assert ratio(y[first[b]:first[b + 1]].cpu(), expected[b][done[b]:done[b] + step[b]]) < 1e-5, (step[b], b)
        done = [d + s for d, s in zip(done, step)]
        lengths = p.lengths.cpu().tolist()
    assert done == totals and status_is_clear()


@pytest.mark.parametrize("rows, width, parts", [(1, 16, 1), (5, 64, 2), (33, 35, 5), (3, 4096, 1)])
def test_norm_before_the_gate(rows, width, parts):
    rng = np.random.default_rng(width)
    y, z, w = rng.normal(size=(rows, width)), rng.normal(size=(rows, width + 4)), rng.uniform(0.5, 1.5, width)
    ty, tz, tw = dev(y), dev(z), dev(w)
    out = torch.full((rows, width + 12), 7.0, device="cuda")
    hi, lo = planes(rows, width + 12)
    torch.cuda.synchronize()
    B.kcheck(B.lib().b200_norm_gated(ty.data_ptr(), tz.data_ptr(), width + 4, tw.data_ptr(), rows, width, parts, 1e-3, 0.7, out.data_ptr() + 32, hi.data_ptr() + 16,
                                     lo.data_ptr() + 16, width + 12, None))
    torch.cuda.synchronize()
    want = 0.7 * O.rms(y.reshape(rows, parts, -1), 1e-3).reshape(rows, width) * w * O.sigmoid(z[:, :width])
    assert ratio(out.cpu()[:, 8:8 + width], want) < 2e-6 and ratio(joined(hi, lo)[:, 8:8 + width], want) < 3e-5
    assert bool((out[:, :8] == 7.0).all()) and bool((out[:, 8 + width:] == 7.0).all())


# ---- residual stream, embedding, logits -------------------------------------------------------------------------
@pytest.mark.parametrize("rows, width", [(1, 8), (5, 36), (40, 53), (700, 1024), (3, 4097), (2, 9000)])
@pytest.mark.parametrize("last", [False, True])
def test_norms_around_a_sublayer(rows, width, last):
    rng = np.random.default_rng(width)
    y, x, after, following = rng.normal(0, 3, (rows, width)), rng.normal(size=(rows, width)), rng.normal(1, 0.3, width), rng.normal(1, 0.3, width)
    ty, tx, ta, tn = map(dev, (y, x, after, following))
    normed = torch.full_like(tx, 7.0)
    hi, lo = planes(rows, width)
    a = B.Sandwich(ta.data_ptr(), None if last else tn.data_ptr(), 1e-3, tx.data_ptr(), tx.data_ptr(), normed.data_ptr(), hi.data_ptr(), lo.data_ptr())
    torch.cuda.synchronize()
    B.kcheck(B.lib().b200_sandwich_rows(ty.data_ptr(), rows, width, C.byref(a), None))
    torch.cuda.synchronize()
    total = x + O.rms(y, 1e-3) * after
    assert ratio(tx.cpu(), total) < 1e-6
    if last:
        assert bool((normed == 7.0).all())
    else:
        want = O.rms(total, 1e-3) * following
        assert ratio(normed.cpu(), want) < 2e-6 and ratio(joined(hi, lo), want) < 3e-5


@pytest.mark.parametrize("dtype, width", [("f32", 64), ("bf16", 64), ("bf16", 37), ("bf16", 5000)])
def test_pair_embedding(dtype, width):
    """Rows of pairs inside a pass, across passes, and the row of a sequence's first token; slots hold other sequences' tokens before."""
    vocab, spec = 50, dict(buckets=23, mul_prev=131, mul_cur=7)
    rng = np.random.default_rng(1)
    table, pairs, following = rounded(rng.normal(size=(vocab, width))), rounded(rng.normal(size=(24, width))), rng.normal(1, 0.3, width)
    kind = torch.bfloat16 if dtype == "bf16" else torch.float32
    (tt, tp), tn = (torch.tensor(a, device="cuda").to(kind) for a in (table, pairs)), dev(following)
    last = torch.full((4,), 49, dtype=torch.int32, device="cuda")
    ids = [rng.integers(0, vocab, 40) for _ in range(3)]
    want = [O.embedding({"embed": table.astype(np.float64), "bigram": pairs.astype(np.float64)}, i, {"embedding": {"bigram": spec}}) for i in ids]
    slots, done, lengths = [3, 0, 2], [0, 0, 0], [0] * 4
    for counts in ([5, 1, 9], [1, 1, 1], [1, 1, 1], [2, 1, 3], [1, 1, 1]):
        p = Pass(counts, slots, lengths)
        tokens = torch.tensor(np.concatenate([ids[b][done[b]:done[b] + counts[b]] for b in range(3)]), device="cuda")
        rows = tokens.shape[0]
        x, normed = torch.empty(rows, width, device="cuda"), torch.empty(rows, width, device="cuda")
        hi, lo = planes(rows, width)
        e = B.PairEmbedding(tt.data_ptr(), tp.data_ptr(), B.BF16 if dtype == "bf16" else B.F32, vocab, width, 23, 131, 7, last.data_ptr(), tn.data_ptr(), 1e-3, x.data_ptr(),
                            normed.data_ptr(), hi.data_ptr(), lo.data_ptr())
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_embed_pairs(C.byref(e), tokens.data_ptr(), C.byref(p.c), None))
        B.kcheck(B.lib().b200_rows_advance_tokens(C.byref(p.c), tokens.data_ptr(), last.data_ptr(), None))
        torch.cuda.synchronize()
        expected = np.concatenate([want[b][done[b]:done[b] + counts[b]] for b in range(3)])
        assert ratio(x.cpu(), expected) < 1e-6, counts
        expected = O.rms(expected, 1e-3) * following
        assert ratio(normed.cpu(), expected) < 2e-6 and ratio(joined(hi, lo), expected) < 3e-5
        done = [d + n for d, n in zip(done, counts)]
        lengths = p.lengths.cpu().tolist()
        assert [lengths[s] for s in slots] == done and [int(last[s]) for s in slots] == [int(ids[b][done[b] - 1]) for b in range(3)]
    assert int(last[1]) == 49


def test_capped_logits():
    x = np.random.default_rng(0).normal(0, 40, 70001)
    t = dev(x)
    B.kcheck(B.lib().b200_soft_cap(t.data_ptr(), x.size, 35.0, None))
    torch.cuda.synchronize()
    assert ratio(t.cpu(), O.soft_cap(x, 35.0)) < 1e-6


# ---- feed-forwards ----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows, inner, units", [(1, 64, 40), (16, 256, 130), (40, 136, 64), (300, 128, 100), (270, 64, 33), (3, 30, 21), (9, 100, 7)])
def test_clamped_units(rows, inner, units):
    """The epilogue of every linear kernel family, and of the f32 rows."""
    rng = np.random.default_rng(units)
    x, w = rng.normal(size=(rows, inner)), rounded(rng.normal(0, 1.5 * inner ** -0.5, (2 * units, inner)))
    z = x @ w.T.astype(np.float64)
    tx, unit = dev(x), B.ClampedUnit(1.702, 1.3)
    want = O.clamped_units(z[:, 0::2], z[:, 1::2], 1.3)
    assert (np.abs(z) > 1.3).any()
    for kind, code, tol in ((torch.float32, B.F32, 2e-6), (torch.bfloat16, B.BF16, 1e-4)):
        tw, y = torch.tensor(w, device="cuda").to(kind), torch.empty(rows, units, device="cuda")
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_linear_units(tx.data_ptr(), rows, inner, tw.data_ptr(), code, 2 * units, C.byref(unit), y.data_ptr(), None))
        torch.cuda.synchronize()
        assert ratio(y.cpu(), want) < tol
    if inner % 8:
        return
    hi, lo = planes(rows, inner)
    hi.copy_(tx)
    lo.copy_(tx - hi.float())
    oh, ol = planes(rows, units)
    a = B.ShadowLinearArgs(x_hi=hi.data_ptr(), x_lo=lo.data_ptr(), rows=rows, inner=inner, weight=tw.data_ptr(), out=2 * units, epilogue=2, out_hi=oh.data_ptr(), out_lo=ol.data_ptr(),
                           unit=C.pointer(unit))
    torch.cuda.synchronize()
    B.kcheck(B.lib().b200_linear_shadow(C.byref(a), None))
    torch.cuda.synchronize()
    assert ratio(joined(oh, ol), want) < 5e-5


@pytest.mark.parametrize("rows, experts, identity, top, corrected", [(1, 1, 0, 1, True), (5, 7, 3, 3, True), (33, 64, 16, 8, False), (300, 4, 6, 10, True), (9, 1000, 24, 5, True)])
def test_router_choice(rows, experts, identity, top, corrected):
    outputs = experts + identity
    rng = np.random.default_rng(rows)
    logits, correction = rng.normal(0, 2, (rows, outputs + 3)), rng.normal(0, 0.5, outputs)
    tl, tc = dev(logits), dev(correction)
    chosen, rank = torch.full((2, rows, top), -1, dtype=torch.int32, device="cuda")
    weight, counts = torch.zeros(rows, top, device="cuda"), torch.zeros(experts, dtype=torch.int32, device="cuda")
    route = B.Route(outputs, top, 0, chosen.data_ptr(), weight.data_ptr(), rank.data_ptr(), counts.data_ptr(), 1, tc.data_ptr() if corrected else None, identity)
    torch.cuda.synchronize()
    B.kcheck(B.lib().b200_route_rows(tl.data_ptr(), rows, outputs + 3, C.byref(route), None))
    torch.cuda.synchronize()
    want, score = O.route(logits[:, :outputs].astype(np.float32).astype(np.float64), correction.astype(np.float32) if corrected else 0.0, top)
    assert np.array_equal(chosen.cpu(), want) and ratio(weight.cpu(), score) < 2e-6
    real = want[want < experts]
    assert np.array_equal(counts.cpu(), np.bincount(real, minlength=experts))
    ranks = rank.cpu().numpy()
    for e in np.unique(real):
        assert sorted(ranks[want == e]) == list(range((want == e).sum()))


def run_experts(rows, experts, identity, top, width, ff, dtype, form, finish=False, only=None, seed=0):
    """`only`: every row chooses these outputs."""
    rng = np.random.default_rng(seed)
    up = rounded(rng.normal(0, 1.5 * width ** -0.5, (experts, 2 * ff, width)))      # gate and up rows interleaved
    down = rounded(rng.normal(0, ff ** -0.5, (experts, width, ff)))
    h = rng.normal(size=(rows, width)).astype(np.float32)
    chosen = np.stack([rng.permutation(experts + identity)[:top] for _ in range(rows)]) if only is None else np.tile(only, (rows, 1))
    weight = rng.uniform(0.2, 1.0, (rows, top))
    want = np.zeros((rows, width))
    for k in range(top):
        for e in np.unique(chosen[:, k]):
            at = chosen[:, k] == e
            x = h[at].astype(np.float64)
            y = x if e >= experts else (O.silu(x @ up[e, 0::2].T) * (x @ up[e, 1::2].T)) @ down[e].T
            want[at] += weight[at, k, None] * y
    kind = torch.bfloat16 if dtype == "bf16" else torch.float32
    t = lambda a, d=torch.float32: torch.tensor(np.ascontiguousarray(a), device="cuda").to(d)
    tup, tdown, th, tc, tw = t(up, kind), t(down, kind), t(h), t(chosen.astype(np.int32), torch.int32), t(weight.astype(np.float32))
    hi, lo = planes(rows, width)
    hi.copy_(th)
    lo.copy_(th - hi.float())
    y = torch.full((rows, width), float("nan"), device="cuda")
    a = B.Experts(experts=experts, top=top, rows=rows, inner=width, ff=ff, weight_dtype=B.BF16 if dtype == "bf16" else B.F32, up=tup.data_ptr(), down=tdown.data_ptr(),
                  chosen=tc.data_ptr(), weight=tw.data_ptr(), y=y.data_ptr(), gated=1, weigh_results=1, identity=identity, eps=1e-3)
    if form == "f32":
        a.x = th.data_ptr()
    else:
        a.x_hi, a.x_lo = hi.data_ptr(), lo.data_ptr()
    stream, after, following = (rng.normal(size=s) for s in ((rows, width), width, width))
    ts, ta, tf = map(dev, (stream, after, following))
    nh, nl = planes(rows, width)
    sandwich = B.Sandwich(ta.data_ptr(), tf.data_ptr(), 1e-3, ts.data_ptr(), ts.data_ptr(), None, nh.data_ptr(), nl.data_ptr())
    if finish:
        a.after, a.y = C.pointer(sandwich), None
    torch.cuda.synchronize()
    if form == "grouped":
        ranks, counts = np.zeros((rows, top), dtype=np.int32), np.zeros(experts, dtype=np.int32)
        for s in np.random.default_rng(5).permutation(rows * top):    # the places come in no order
            e = chosen.ravel()[s]
            if e < experts:
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
    assert status_is_clear()
    if not finish:
        return ratio(y.cpu(), want)
    total = stream + O.rms(want, 1e-3) * after
    return max(ratio(ts.cpu(), total), ratio(joined(nh, nl), O.rms(total, 1e-3) * following))


@pytest.mark.parametrize("rows, experts, identity, top, width, ff", [(1, 1, 1, 1, 8, 8), (3, 5, 2, 2, 36, 21), (17, 12, 0, 4, 184, 104), (40, 3, 3, 5, 100, 264)])
@pytest.mark.parametrize("dtype, form", [("f32", "f32"), ("bf16", "f32"), ("bf16", "planes")])
def test_streamed_experts(rows, experts, identity, top, width, ff, dtype, form):
    assert run_experts(rows, experts, identity, top, width, ff, dtype, form) < (4e-6 if form == "f32" else 3e-5)


@pytest.mark.parametrize("rows, experts, identity, top, width, ff", [(25, 8, 2, 1, 64, 72), (60, 70, 6, 5, 200, 136), (90, 6, 6, 2, 136, 200), (700, 5, 1, 2, 136, 264), (300, 300, 20, 3, 64, 32)])
@pytest.mark.parametrize("finish", [False, True])
def test_grouped_experts(rows, experts, identity, top, width, ff, finish):
    assert run_experts(rows, experts, identity, top, width, ff, "bf16", "grouped", finish) < 6e-5


@pytest.mark.parametrize("only", [[4, 5], [3, 4], [0, 1]])
def test_rows_that_choose_identity_experts_alone_or_never(only):
    for form, finish in (("planes", False), ("grouped", False), ("grouped", True)):
        assert run_experts(40, 4, 2, 2, 64, 48, "bf16", form, finish, only) < 6e-5


# ---- whole models -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", S.CASES)
def test_prompt_matches_the_statement_layer_by_layer(name, dtype):
    model, w = model_of(name, dtype)
    c = S.CASES[name]
    for count in (71, 9, 2):
        ids = S.decided_tokens(c, w, count)
        trail = []
        want = O.forward(c, w, ids, trail)
        model.new_cache(2, 80)
        got_trail = model.trail(1, ids)
        for i, rows in enumerate(trail):
            assert ratio(got_trail[i], rows) < TOLERANCE[dtype], f"layer {i}"
        assert ratio(model.run([(0, ids, all_places(count))]), want) < TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", S.CASES)
def test_decoding_and_portions_equal_the_whole_prompt(name, dtype):
    """Token by token, portions of two, unequal portions: the logits of every position equal those of one pass."""
    model, w = model_of(name, dtype)
    c = S.CASES[name]
    ids = S.decided_tokens(c, w, 70, seed=3)
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
    c = S.CASES[name]
    counts, tails = [1, 67, 20, 3, 130], [4, 6, 1, 9, 5]
    full = [S.decided_tokens(c, w, n + t, seed=n) for n, t in zip(counts, tails)]
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
        c = S.CASES["mixed"]
        full = [S.decided_tokens(c, w, n, seed=n) for n in (40, 33, 50)]
        model.new_cache(3, 60)
        alone = [model.run([(i, ids, all_places(len(ids)))]) for i, ids in enumerate(full)]
        model.cache.clear()
        model.run([(1, full[1][:32], []), (2, full[2][:47], [])])
        got = model.run([(0, full[0], all_places(40)), (1, full[1][32:], [0]), (2, full[2][47:], [0, 1, 2])])
        want = np.concatenate([alone[0], alone[1][32:], alone[2][47:]])
        assert ratio(got, want) < (1e-5 if dtype == "f32" else 1e-2)


def test_long_pass_is_cut_and_joined():
    """More rows than one pass over the layers takes: the cut falls inside a sequence (its pair, state and keys cross it) and between
    sequences."""
    model, _ = model_of("ones", "f32")
    c = S.CASES["ones"]
    ids = [S.tokens(c, n, seed=n) for n in (5000, 6000, 40)]
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
        assert ratio(got[at:at + len(wanted)], np.concatenate(alone)) < 1e-4
        at += len(wanted)


@pytest.mark.parametrize("name, dtype", [("mixed", "f32"), ("plain", "bf16")])   # (plain: every expert is chosen, no call is close)
def test_long_decoding_stays_with_the_statement(name, dtype):
    model, w = model_of(name, dtype)
    c = S.CASES[name]
    ids = S.tokens(c, 300, seed=8)
    want = O.forward(c, w, ids)
    model.new_cache(1, 300)
    model.run([(0, ids[:5], [])])
    got = np.concatenate([model.run([(0, [t], [0])]) for t in ids[5:]])
    assert ratio(got, want[5:]) < TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_far_tokens_reach_the_last_logits(dtype):
    """The last position's logits follow tokens far back through the slot's keys, whole and decoded."""
    model, w = model_of("plain", dtype)
    c = S.CASES["plain"]
    ids = S.tokens(c, 260, seed=4)
    model.new_cache(2, 260)
    for place in (0, 1, 63, 64, 127, 128, 200, 258):
        other = ids.copy()
        other[place] = (other[place] + 77) % c["vocab"]
        want = O.forward(c, w, other)[-1]
        model.cache.clear()
        whole = model.run([(0, other, [259])])
        model.run([(1, other[:250], [])])
        single = [model.run([(1, [t], [0])]) for t in other[250:]][-1]
        assert ratio(whole[0], want) < TOLERANCE[dtype] and ratio(single[0], want) < TOLERANCE[dtype], place


@pytest.mark.parametrize("name", ["mixed", "odd", "plain", "deep"])
def test_greedy_generation_equals_the_statement(name):
    """The framework's own loop: prompts of unequal length in one batch, the token loop in a captured graph."""
    model, w = model_of(name, "f32")
    c = S.CASES[name]
    prompts, steps = [S.tokens(c, n, seed=n) for n in (9, 2, 31)], 12
    got = model.generate(prompts, steps)
    for row, prompt in zip(got, prompts):
        want, margin = O.greedy(c, w, prompt, steps)
        assert margin > 1e-4 and list(row) == want


@pytest.mark.parametrize("name, batch", [("mixed", 1), ("mixed", 20), ("wide", 40), ("plain", 150), ("uneven", 3), ("deep", 30)])
def test_bf16_generation_feeds_back_its_own_choice(name, batch):
    """bf16 loop (fused logits + choice; streaming and dense projections; streamed and grouped experts): replaying its tokens gives
    logits whose best is the token chosen next, and the logits asked for on demand are those."""
    model, _ = model_of(name, "bf16")
    c = S.CASES[name]
    steps, prompts = 8, np.stack([S.tokens(c, 10, seed=b) for b in range(batch)])
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
    c = S.CASES["mixed"]
    prompts = np.stack([S.tokens(c, 7, seed=b) for b in range(3)])
    greedy = model.generate(list(prompts), 6)
    assert np.array_equal(model.generate(list(prompts), 6, temperature=1e-4), greedy)   # cold sampling is the greedy choice
    model.new_cache(3, 13)
    gen = B.Generation(model, 3, 6)
    gen.prefill(prompts)
    first = gen.tokens()[:, 0].copy()
    assert np.array_equal(gen.run_host(first, 5).T, greedy[:, 1:])


def test_cache_errors_leave_the_model_usable():
    model, _ = model_of("mixed", "f32")
    c = S.CASES["mixed"]
    model.new_cache(2, 10)
    ids = S.tokens(c, 10)
    want = model.run([(1, ids, [9])])
    model.cache.release(1)
    for entries, message in (([(0, S.tokens(c, 11), [])], "capacity"), ([(2, ids, [])], "slot out of range"), ([(0, ids[:2], []), (0, ids[:2], [])], "twice"),
                             ([(0, [c["vocab"]], [])], "out of range"), ([(0, ids[:2], [2])], "wanted place")):
        with pytest.raises(B.B200Error, match=message):
            model.run(entries)
    assert ratio(model.run([(1, ids, [9])]), want) < 1e-6


def test_module_forward_equals_the_statement():
    model, w = model_of("mixed", "f32")
    ids = np.stack([S.tokens(S.CASES["mixed"], 12, seed=1), S.tokens(S.CASES["mixed"], 12, seed=2)])
    got = model.module(B.Tensor.from_numpy(ids.astype(np.int64))).numpy()
    for b in range(2):
        assert ratio(got[b], O.forward(S.CASES["mixed"], w, ids[b])) < TOLERANCE["f32"]


def test_single_plane_activations():
    """The bf16-activation option (one plane in passes over more than 16 rows) stays near the statement.  (Every output is chosen, so
    that no router's choice can turn.)"""
    c = S.CASES["plain"]
    weights = S.make_weights(c, 0)
    model = B.LanguageModel(c, weights)
    model.set_activation_dtype("bf16")
    ids = S.tokens(c, 60)
    model.new_cache(1, 60)
    assert ratio(model.run([(0, ids, all_places(60))]), O.forward(c, weights, ids)) < 4e-2


def test_argument_errors_are_refused_before_a_launch():
    k = Grouped(1, 2, 1, 8, 8, "f32", slots=1, capacity=8)
    rows = torch.zeros(2, k.stride, device="cuda")
    k.a.projected, k.a.stride, k.a.query = rows.data_ptr(), k.columns - 1, rows.data_ptr()
    p = Pass([1], [0], [0])
    refused = lambda: B.lib().b200_chunk_prepare(C.byref(k.a), C.byref(p.c), None, None, None) == -1
    assert refused() and b"shorter" in B.lib().b200_last_error()
    k.a.stride = k.stride
    for field, wrong in (("norm", 3), ("norm", 0), ("vdim", 4), ("softcap", -1.0)):
        kept = getattr(k.a, field)
        setattr(k.a, field, wrong)
        assert refused(), field
        setattr(k.a, field, kept)
    a = B.SsmArgs(heads=1, vdim=4, state=4, groups=1, taps=2, ssm_state=rows.data_ptr(), projected=rows.data_ptr(), mixed=rows.data_ptr(), y=rows.data_ptr(), decay=rows.data_ptr())
    assert B.lib().b200_ssm_forward(C.byref(a), C.byref(p.c), None) == -1
    r = B.Route(4, 5, 0, rows.data_ptr(), rows.data_ptr(), None, None)
    assert B.lib().b200_route_rows(rows.data_ptr(), 1, 8, C.byref(r), None) == -1
    e = B.Experts(experts=2, top=4, rows=1, inner=8, ff=8, weight_dtype=B.F32, identity=1)
    assert B.lib().b200_experts_streamed(C.byref(e), rows.data_ptr(), None) == -1
    assert B.lib().b200_soft_cap(rows.data_ptr(), 1, 0.0, None) == -1


def test_command_lines(tmp_path):
    """The generation command and the trace runner as a user starts them."""
    c = S.CASES["mixed"]
    w = S.make_weights(c, 2)
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir()
    out.mkdir()
    S.write_folder(folder, c, w)
    prompts = [S.tokens(c, 5, seed=1).tolist(), S.tokens(c, 3, seed=2).tolist()]
    run = subprocess.run([sys.executable, "-m", "ctorch_b200.generate", "--model", str(folder), "--dtype", "f32", "--steps", "4",
                          *[",".join(map(str, p)) for p in prompts]], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [[int(t) for t in line.split(",")] for line in run.stdout.split()] == [O.greedy(c, w, p, 4)[0] for p in prompts]
    a, b = S.decided_tokens(c, w, 22, seed=5).tolist(), S.decided_tokens(c, w, 4, seed=6).tolist()
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
