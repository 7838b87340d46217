"""Post-norm decoder on the GPU against the plain statement (postnorm_oracle): the mechanisms alone at kernel level, then whole models -
prompts, decoding, portions, unequal batches, reused slots, far keys, window and block edges, long decoding, greedy generation."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ctorch_b200 as B
import postnorm_cases as S
import postnorm_oracle as O
from test_hybrid_gpu import Pass, all_places, dev, joined, planes, ratio

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
class Windowed:
    """One attention layer's kernels over torch memory: `kind` 1 pooled blocks (projection norms, normed values, a gate per value), 2 kept
    tokens (weighted head norms, stretched positions, mixed heads unless `mixing` is off); the slots start full of junk."""

    def __init__(self, kind, heads, kv_heads, dim, vdim, dtype, size, pool=0, keep=0, slots=4, capacity=400, dims=None, base=100.0, factor=1.0, scale=0.3,
                 eps=1e-5, mixing=True, talk=None, extra=5, seed=0):
        rng = np.random.default_rng(seed)
        dims = dim // 2 // 2 * 2 if dims is None else dims
        self.kind, self.bf16, self.capacity, self.extra, self.mixing = kind, dtype == "bf16", capacity, extra, mixing and kind == 2
        self.n = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, dims=dims, base=base, factor=factor, scale=scale, eps=eps, size=size, pool=pool, keep=keep)
        self.columns = heads * dim + kv_heads * (dim + vdim) + (heads * vdim if kind == 1 else 0)
        self.stride = self.columns + extra
        whole = kind == 1
        self.q_norm, self.k_norm = rng.uniform(0.5, 1.5, heads * dim if whole else dim), rng.uniform(0.5, 1.5, kv_heads * dim if whole else dim)
        self.talk = np.asarray(talk) if talk is not None else np.eye(heads) * 0.7 + rng.normal(0, 0.4, (heads, heads))
        angle = np.arange(capacity)[:, None] * float(base) ** (-2.0 * np.arange(dims // 2) / max(1, dims)) / factor
        self.type = torch.bfloat16 if self.bf16 else torch.float32
        windowed = size > 0 and size + keep < capacity
        entries = keep + size + (capacity // pool if pool else 0) if windowed else capacity
        self.keys = torch.full((slots, kv_heads, entries, dim), float("nan"), dtype=self.type, device="cuda")
        self.values = torch.full((slots, kv_heads, entries, vdim), float("nan"), dtype=self.type, device="cuda")
        self.pool_state = torch.full((slots, kv_heads, dim + vdim), float("nan"), device="cuda")
        self.keep_alive = [dev(a) for a in (np.cos(angle), np.sin(angle), self.q_norm, self.k_norm, self.talk)]
        k = [t.data_ptr() for t in self.keep_alive]
        a = self.a = B.ChunkArgs(heads, kv_heads, dim, vdim, dims, slots, 0, entries, scale, eps, k[0], k[1], capacity, k[2], k[3], B.BF16 if self.bf16 else B.F32,
                                 self.keys.data_ptr(), self.values.data_ptr())
        a.no_gate = 1
        if windowed:
            a.window, a.keep, a.pool = size, keep, pool
            if pool:
                a.pool_state = self.pool_state.data_ptr()
        if kind == 1:
            a.norm, a.norm_values, a.gate_values = B.HEAD_NORM_PROJECTION, 1, 1
        else:
            a.norm = B.HEAD_NORM_HEAD
        if self.mixing:
            a.talk = k[4]

    def attend(self, p, rows, max_length):
        n, count = self.n, rows.shape[0]
        projected = dev(rows)
        work = [torch.full((count, h, d), float("nan"), dtype=self.type, device="cuda")
                for h, d in ((n["heads"], n["dim"]), (n["kv_heads"], n["dim"]), (n["kv_heads"], n["vdim"]))]
        width = n["heads"] * n["vdim"]
        out = torch.full((count, width + 8), float("nan"), device="cuda")
        hi, lo = planes(count, width + 8)
        a = self.a
        a.projected, a.stride, a.query, a.key, a.value = projected.data_ptr(), rows.shape[1], *(t.data_ptr() for t in work)
        need = B.lib().b200_chunk_scratch_bytes(C.byref(a), count, p.c.sequences, p.c.max_count, max_length)
        scratch = torch.full((need // 4 + 1,), float("nan"), device="cuda")
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_chunk_prepare(C.byref(a), C.byref(p.c), None, None, None))
        B.kcheck(B.lib().b200_chunk_attention(C.byref(a), C.byref(p.c), max_length, scratch.data_ptr(), need, out.data_ptr(), hi.data_ptr(), lo.data_ptr(), width + 8, None))
        torch.cuda.synchronize()
        got = out.cpu().numpy()[:, :width]
        assert ratio(joined(hi, lo)[:, :width], got) < 3e-5
        self.scratch = need
        return got

    def parts(self, rows):
        """Queries, keys, values [heads, T, size] and gates [T, heads * vdim] of a sequence's projected rows."""
        n, T = self.n, len(rows)
        H, G, d, e = n["heads"], n["kv_heads"], n["dim"], n["vdim"]
        q, k, v, g = np.split(rows[:, :self.columns].astype(np.float32).astype(np.float64), np.cumsum([H * d, G * d, G * e]), axis=1)
        turn = lambda x: O.rotate_halves(x, np.arange(T), n["dims"], n["base"], n["factor"])
        if self.kind == 1:
            return (turn(O.heads_of(O.rms(q, n["eps"]) * self.q_norm, H)), turn(O.heads_of(O.rms(k, n["eps"]) * self.k_norm, G)),
                    O.rms(O.heads_of(v, G), n["eps"]), O.sigmoid(g))
        return turn(O.rms(O.heads_of(q, H), n["eps"]) * self.q_norm), turn(O.rms(O.heads_of(k, G), n["eps"]) * self.k_norm), O.heads_of(v, G), 1.0

    def want(self, rows):
        n, T = self.n, len(rows)
        q, k, v, gate = self.parts(rows)
        group, size = n["heads"] // n["kv_heads"], n["size"] or T
        if n["pool"]:
            weights = O.pooled_window_weights(q, k, n["scale"], size, n["pool"])
            v = np.concatenate([v, O.block_means(v, n["pool"])], axis=1)
        else:
            score = np.einsum("htd,hjd->htj", q, np.repeat(k, group, axis=0)) * n["scale"]
            weights = O.softmax(np.where(O.seen_tokens(T, size, n["keep"]), score, -np.inf))
        if self.mixing:
            weights = O.mixed_heads(weights, self.talk)
        return np.einsum("htj,hje->the", weights, np.repeat(v, group, axis=0)).reshape(T, -1) * gate


WINDOWS = [dict(kind=1, heads=4, kv_heads=2, dim=16, vdim=24, size=40, pool=8), dict(kind=1, heads=3, kv_heads=1, dim=10, vdim=14, size=9, pool=13),
           dict(kind=1, heads=40, kv_heads=1, dim=96, vdim=96, size=65, pool=3), dict(kind=1, heads=2, kv_heads=2, dim=256, vdim=256, size=64, pool=64, scale=0.1),
           dict(kind=1, heads=6, kv_heads=2, dim=20, vdim=12, size=1, pool=1), dict(kind=1, heads=2, kv_heads=1, dim=64, vdim=64, size=127, pool=5),
           dict(kind=1, heads=2, kv_heads=1, dim=64, vdim=128, size=50, pool=0), dict(kind=1, heads=2, kv_heads=1, dim=64, vdim=64, size=1000, pool=5),
           dict(kind=2, heads=4, kv_heads=2, dim=24, vdim=16, size=40, keep=5, factor=3.0), dict(kind=2, heads=3, kv_heads=3, dim=10, vdim=14, size=6, keep=11),
           dict(kind=2, heads=1, kv_heads=1, dim=64, vdim=64, size=64, keep=1), dict(kind=2, heads=20, kv_heads=1, dim=128, vdim=64, size=63, keep=70),
           dict(kind=2, heads=8, kv_heads=8, dim=192, vdim=256, size=33, keep=0), dict(kind=2, heads=64, kv_heads=2, dim=64, vdim=40, size=100, keep=3),
           dict(kind=2, heads=72, kv_heads=2, dim=8, vdim=8, size=30, keep=2), dict(kind=2, heads=6, kv_heads=2, dim=40, vdim=128, size=0),
           dict(kind=2, heads=6, kv_heads=3, dim=64, vdim=64, size=45, keep=4, mixing=False), dict(kind=2, heads=3, kv_heads=1, dim=10, vdim=6, size=1, keep=1, mixing=False)]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("spec", WINDOWS, ids=lambda s: "k{kind}_h{heads}_{kv_heads}_d{dim}_{vdim}_w{size}".format(**s))
def test_attention_layer(spec, dtype):
    """Norms, rotation, append, windows, blocks, kept tokens, mixed heads, gates: a prompt of unequal sequences, single rows, portions of two
    and more, in shuffled slots."""
    k = Windowed(**spec, dtype=dtype, seed=spec["dim"])
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
@pytest.mark.parametrize("size, pool, keep, heads, kv_heads", [(40, 8, 0, 2, 1), (64, 16, 0, 2, 2), (7, 30, 0, 3, 1), (129, 1, 0, 2, 1), (40, 0, 6, 2, 1), (64, 0, 70, 4, 2), (65, 0, 1, 20, 1)])
def test_one_key_stands_out(size, pool, keep, heads, kv_heads, dtype):
    """Every query asks for one key: its own, the window's last and the one that has just left it, kept tokens and the next ones, tile borders;
    where blocks of one token or of equal keys are pooled, also for those.  What is not seen must go unanswered."""
    T, d, e = 300, 64, 16
    k = Windowed(1 if pool else 2, heads, kv_heads, d, e, dtype, size, pool, keep, slots=2, capacity=T, dims=0, scale=1.0, talk=np.eye(heads), extra=3, seed=1)
    for i in (2, 3):
        k.keep_alive[i].fill_(1.0)
    k.q_norm[:] = k.k_norm[:] = 1.0
    rng = np.random.default_rng(2)
    H, G, group = heads, kv_heads, heads // kv_heads
    keys = rng.normal(size=(T, G, d))
    if pool:                                     # equal keys in a block: its mean is the key
        keys = np.repeat(keys[::pool], pool, axis=0)[:T]
    keys /= np.sqrt((keys ** 2).mean(axis=(1, 2) if pool else 2, keepdims=True))
    values = rng.normal(size=(T, G, e))
    rows = np.zeros((T, k.stride))
    rows[:, H * d:(H + G) * d] = keys.reshape(T, -1)
    rows[:, (H + G) * d:(H + G) * d + G * e] = values.reshape(T, -1)
    for t in range(T):
        inside = [x for x in (0, 1, keep - 1, keep, 63, 64, 127, t - size - pool, t - size - 1, t - size, t - size + 1, t - size + pool, t - 1, t) if 0 <= x <= t]
        for h in range(H):
            rows[t, h * d:(h + 1) * d] = keys[rng.choice(inside), h // group]
    want = k.want(rows)
    # every key that is answered or not shows: moving the window by one, or leaving out a kept token, changes answers a lot
    for planted in (dict(size=size - 1), dict(size=size + 1), *([dict(keep=keep - 1), dict(keep=keep + 1)] if keep else [])):
        if pool == 1:
            break      # a block of one token is that token: the window has no edge
        kept = dict(k.n)
        k.n.update(planted)
        assert np.abs(k.want(rows) - want).max() > 0.3, planted
        k.n.update(kept)
    at, lengths = 0, [0, 0]
    for count in (1, 35, 1, 1, 1, 25, 1, 1, 62, 1, 1, 1, 2, 2, 61, 1, 1, 1, T - 200):
        p = Pass([count], [1], lengths)
        got = k.attend(p, rows[at:at + count], T)
        assert np.abs(got - want[at:at + count]).max() < (2e-4 if dtype == "f32" else 0.06), (at, count)
        p.advance()
        torch.cuda.synchronize()
        lengths, at = p.lengths.cpu().tolist(), at + count
    assert at <= T


@pytest.mark.parametrize("kind, group, kv_heads, dim, vdim, size, pool, keep", [(1, 4, 1, 64, 64, 500, 3, 0), (1, 6, 1, 128, 40, 130, 1, 0), (2, 4, 1, 64, 128, 600, 0, 90), (2, 2, 3, 40, 64, 700, 0, 0)])
def test_split_keys_of_a_step(kind, group, kv_heads, dim, vdim, size, pool, keep):
    """Few long sequences: the keys of a step are split over CTAs."""
    k = Windowed(kind, group * kv_heads, kv_heads, dim, vdim, "bf16", size, pool, keep, slots=3, capacity=2100, seed=group)
    rng = np.random.default_rng(3)
    slots, totals = [2, 0, 1], [990, 1003, 70]
    data = [rng.normal(size=(t, k.stride)) for t in totals]
    p = Pass([t - 1 for t in totals], slots, [0, 0, 0])
    k.attend(p, np.concatenate([r[:-1] for r in data]), 2100)
    p.advance()
    torch.cuda.synchronize()
    p = Pass([1, 1, 1], slots, p.lengths.cpu().tolist())
    got = k.attend(p, np.concatenate([r[-1:] for r in data]), 2100)
    assert k.scratch > 0
    for i, r in enumerate(data):
        assert ratio(got[i], k.want(r)[-1]) < 1.5e-2


def test_mixed_heads_in_portions_of_the_tables():
    """A pass whose tables of scores exceed what is kept at a time: portions of positions, and of sequences."""
    k = Windowed(2, 32, 4, 16, 16, "bf16", 300, 0, 5, slots=40, capacity=800, seed=4)
    rng = np.random.default_rng(5)
    k.a.table_bytes = 24 << 20
    for totals in ([700, 431, 640], [40] * 36):
        data = [rng.normal(size=(t, k.stride)) for t in totals]
        slots = rng.permutation(40)[:len(totals)].tolist()
        got = k.attend(Pass(totals, slots, [0] * 40), np.concatenate(data), 800)
        assert k.scratch < 26 << 20
        at = 0
        for i, r in enumerate(data):
            if len(totals) < 9 or i % 7 == 0:
                assert ratio(got[at:at + len(r)], k.want(r)) < 1.5e-2, i
            at += len(r)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_blocks_hold_the_means_of_what_the_cache_holds(dtype):
    """However a prompt is cut, a block is the mean of its cached keys and values; the open block's sum waits in its own place."""
    pool, size, T = 6, 8, 50
    k = Windowed(1, 2, 2, 8, 4, dtype, size, pool, 0, slots=3, capacity=T, seed=3)
    rows = np.random.default_rng(1).normal(size=(T, k.stride))
    _, keys, values, _ = k.parts(rows)
    if dtype == "bf16":
        keys, values = (torch.tensor(x).to(torch.bfloat16).double().numpy() for x in (keys, values))
    tol = 1e-6 if dtype == "f32" else 1e-2
    for slot, cuts in ((2, [T]), (0, [1] * T), (1, [3, 1, 1, 7, 1, 2, 20, 1, 1, 1, 12])):
        lengths, at = [0] * 3, 0
        for count in cuts:
            p = Pass([count], [slot], lengths)
            k.attend(p, rows[at:at + count], T)
            p.advance()
            torch.cuda.synchronize()
            lengths, at = p.lengths.cpu().tolist(), at + count
        assert at == T
        for cache, x in ((k.keys, keys), (k.values, values)):
            got = cache[slot].float().cpu().numpy()
            assert ratio(got[:, size:size + T // pool], O.block_means(x, pool)) < tol
            assert ratio(got[:, np.arange(T - size, T) % size], x[:, T - size:]) < tol
        open_rows = T % pool
        want = np.concatenate([x[:, T - open_rows:].sum(axis=1) for x in (keys, values)], axis=1)
        assert ratio(k.pool_state[slot].cpu(), want) < tol


# ---- the delta rule alone ---------------------------------------------------------------------------------------
@pytest.mark.parametrize("heads, groups, dim, vdim, taps, batch", [(2, 1, 64, 32, 4, 3), (1, 1, 16, 16, 1, 1), (6, 3, 9, 7, 2, 2), (4, 2, 130, 24, 3, 2), (2, 2, 300, 64, 4, 1), (8, 4, 128, 128, 4, 3),
                                                                   (3, 1, 96, 1040, 5, 1), (2, 1, 20, 300, 4, 2), (1, 1, 512, 8, 2, 2), (16, 8, 32, 64, 4, 200), (8, 8, 128, 128, 4, 90)])
def test_delta_recurrence(heads, groups, dim, vdim, taps, batch):
    """Prompts of unequal lengths, single rows and portions in shuffled slots full of junk; decays from almost nothing to almost one; large
    batches stream their states."""
    rng = np.random.default_rng(dim)
    inner, channels = heads * vdim, heads * vdim + 2 * groups * dim
    stride = inner + channels + 2 * heads + 3
    stride += -stride % 4
    conv, a_log, dt_bias = rng.normal(0, 0.6, (channels, taps)), np.resize([-6.0, 0.5, 2.0, -2.0], heads), rng.normal(-1, 1, heads)
    slots = rng.permutation(batch + 2)[:batch].tolist()
    ring = torch.full((batch + 2, taps, channels), float("nan"), device="cuda")
    state = torch.full((batch + 2, heads, dim, vdim), float("nan"), device="cuda")
    tconv, tbias, ta, tdt = map(dev, (conv, np.zeros(channels), a_log, dt_bias))
    plan = [[30 + 7 * (b % 5) for b in range(batch)], [1] * batch, [1] * batch, [2] * batch, [17] * batch, [1] * batch] if batch < 50 else [[2] * batch, [1] * batch, [1] * batch, [1] * batch]
    totals = [sum(step[b] for step in plan) for b in range(batch)]
    data = [rng.normal(size=(t, stride)) for t in totals]

    def want(rows):
        T = len(rows)
        r = rows.astype(np.float32).astype(np.float64)
        v, k, q = np.split(O.short_conv(r[:, inner:inner + channels], conv.astype(np.float32).astype(np.float64)), np.cumsum([inner, groups * dim]), axis=1)
        spread = lambda x: np.repeat(O.unit(x.reshape(T, groups, dim)), heads // groups, axis=1)
        g = np.exp(-np.exp(a_log.astype(np.float32)) * O.softplus(r[:, inner + channels:inner + channels + heads] + dt_bias.astype(np.float32)))
        beta = O.sigmoid(r[:, inner + channels + heads:inner + channels + 2 * heads])
        return O.delta_rule(spread(q) * dim ** -0.5, spread(k), v.reshape(T, heads, vdim), beta, g)[0].reshape(T, inner)
    check = range(batch) if batch < 50 else range(0, batch, 37)
    expected = {b: want(data[b]) for b in check}
    done, lengths = [0] * batch, [0] * (batch + 2)
    for step in plan:
        p = Pass(step, slots, lengths)
        rows = dev(np.concatenate([data[b][done[b]:done[b] + step[b]] for b in range(batch)]))
        y, mixed = torch.full((rows.shape[0], inner), float("nan"), device="cuda"), torch.empty(rows.shape[0], channels, device="cuda")
        a = B.SsmArgs(heads=heads, vdim=vdim, state=dim, groups=groups, taps=taps, conv_weight=tconv.data_ptr(), conv_bias=tbias.data_ptr(), dt_bias=tdt.data_ptr(),
                      a_log=ta.data_ptr(), conv_state=ring.data_ptr(), ssm_state=state.data_ptr(), projected=rows.data_ptr(), mixed=mixed.data_ptr(), y=y.data_ptr(),
                      stride=stride, delta=1)
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_ssm_forward(C.byref(a), C.byref(p.c), None))
        p.advance()
        torch.cuda.synchronize()
        first = p.first_host
        for b in check:
            assert ratio(y[first[b]:first[b + 1]].cpu(), expected[b][done[b]:done[b] + step[b]]) < 2e-5, (step[b], b)
        done = [d + s for d, s in zip(done, step)]
        lengths = p.lengths.cpu().tolist()
    assert done == totals and status_is_clear()


@pytest.mark.parametrize("rows, heads, size", [(1, 1, 16), (5, 3, 64), (33, 5, 7), (3, 2, 1030), (700, 4, 128)])
def test_head_norm_and_gate(rows, heads, size):
    rng = np.random.default_rng(size)
    width = heads * size
    y, z, w = rng.normal(size=(rows, width)), rng.normal(size=(rows, width + 4)), rng.uniform(0.5, 1.5, size)
    ty, tz, tw = dev(y), dev(z), dev(w)
    out = torch.full((rows, width + 12), 7.0, device="cuda")
    hi, lo = planes(rows, width + 12)
    torch.cuda.synchronize()
    B.kcheck(B.lib().b200_head_norm_gated(ty.data_ptr(), tz.data_ptr(), width + 4, tw.data_ptr(), rows, heads, size, 1e-3, out.data_ptr() + 32, hi.data_ptr() + 16,
                                          lo.data_ptr() + 16, width + 12, None))
    torch.cuda.synchronize()
    want = ((O.rms(y.reshape(rows, heads, size), 1e-3) * w).reshape(rows, width)) * O.silu(z[:, :width])
    assert ratio(out.cpu()[:, 8:8 + width], want) < 2e-6 and ratio(joined(hi, lo)[:, 8:8 + width], want) < 3e-5
    assert bool((out[:, :8] == 7.0).all()) and bool((out[:, 8 + width:] == 7.0).all())


# ---- residual stream, router ------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows, width", [(1, 8), (5, 36), (40, 53), (300, 1024), (3, 4097), (2, 9000)])
def test_norm_behind_a_sublayer_and_the_stream_itself(rows, width):
    rng = np.random.default_rng(width)
    y, x, after = rng.normal(0, 3, (rows, width)), rng.normal(size=(rows, width)), rng.normal(1, 0.3, width)
    ty, tx, ta = map(dev, (y, x, after))
    plain = torch.full_like(tx, 7.0)
    hi, lo = planes(rows, width)
    a = B.Sandwich(ta.data_ptr(), None, 1e-3, tx.data_ptr(), tx.data_ptr(), plain.data_ptr(), hi.data_ptr(), lo.data_ptr(), 1)
    torch.cuda.synchronize()
    B.kcheck(B.lib().b200_sandwich_rows(ty.data_ptr(), rows, width, C.byref(a), None))
    torch.cuda.synchronize()
    total = x + O.rms(y, 1e-3) * after
    assert ratio(tx.cpu(), total) < 1e-6 and bool((plain == tx).all()) and ratio(joined(hi, lo), total) < 3e-5


@pytest.mark.parametrize("rows, experts, top, biased", [(1, 1, 1, True), (40, 6, 2, True), (9, 33, 33, False), (70, 300, 40, True), (500, 16, 4, True)])
def test_router_weighs_the_chosen_alone(rows, experts, top, biased):
    rng = np.random.default_rng(experts)
    logits, bias = rng.normal(0, 2.0, (rows, experts + 3)), rng.normal(0, 2.0, experts)
    tl, tb = dev(logits), dev(bias)
    chosen, rank = (torch.full((rows, top), -7, dtype=torch.int32, device="cuda") for _ in range(2))
    counts, weight = torch.zeros(experts, dtype=torch.int32, device="cuda"), torch.full((rows, top), float("nan"), device="cuda")
    route = B.Route(experts=experts, top=top, chosen=chosen.data_ptr(), weight=weight.data_ptr(), rank=rank.data_ptr(), counts=counts.data_ptr(),
                    bias=tb.data_ptr() if biased else None, chosen_softmax=1)
    torch.cuda.synchronize()
    B.kcheck(B.lib().b200_route_rows(tl.data_ptr(), rows, experts + 3, C.byref(route), None))
    torch.cuda.synchronize()
    z = logits[:, :experts].astype(np.float32) + (bias.astype(np.float32) if biased else np.float32(0))
    want, score = O.route(z.astype(np.float64), top)
    assert np.array_equal(chosen.cpu(), want) and ratio(weight.cpu(), score) < 2e-6
    assert np.array_equal(counts.cpu(), np.bincount(want.ravel(), minlength=experts))


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
@pytest.mark.parametrize("name", ["mixed", "wide", "odd", "uneven"])
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
    """More rows than one pass over the layers takes: the cut falls inside a sequence (its states, windows and blocks cross it) and between
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


@pytest.mark.parametrize("name, batch", [("mixed", 1), ("mixed", 20), ("wide", 40), ("plain", 150), ("uneven", 3), ("deep", 30), ("ones", 2), ("recurrent", 9), ("attending", 3)])
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
    k = Windowed(1, 2, 1, 8, 8, "f32", 4, 2, slots=1, capacity=16)
    rows = torch.zeros(2, k.stride, device="cuda")
    k.a.projected, k.a.stride, k.a.query = rows.data_ptr(), k.columns - 1, rows.data_ptr()
    p = Pass([1], [0], [0])
    refused = lambda: B.lib().b200_chunk_prepare(C.byref(k.a), C.byref(p.c), None, None, None) == -1
    assert refused() and b"shorter" in B.lib().b200_last_error()
    k.a.stride = k.stride
    for field, wrong in (("window", -1), ("window", 0), ("keep", 2), ("chunk", 4), ("entries", 3), ("pool_state", None), ("no_gate", 0), ("keys_elsewhere", 1), ("q_norm", None)):
        kept = getattr(k.a, field)
        setattr(k.a, field, wrong)
        assert refused(), field
        setattr(k.a, field, kept)
    p2 = Pass([2], [0], [0])
    assert B.lib().b200_chunk_prepare(C.byref(k.a), C.byref(p2.c), None, None, None) == -1 and b"workspaces" in B.lib().b200_last_error()
    r = rows.data_ptr()
    a = B.SsmArgs(heads=1, vdim=4, state=4, groups=1, taps=1, ssm_state=r, projected=r, mixed=r, y=r, dt_bias=r, a_log=r, delta=1)
    assert B.lib().b200_ssm_forward(C.byref(a), C.byref(p.c), None) == -1      # no convolution
    route = B.Route(4, 2, 0, r, r, None, None)
    route.chosen_softmax = route.softmax = 1
    assert B.lib().b200_route_rows(r, 1, 8, C.byref(route), None) == -1
    s = B.Sandwich(r, r, 1e-5, r, r, r, None, None, 1)
    assert B.lib().b200_sandwich_rows(r, 1, 4, C.byref(s), None) == -1
    assert B.lib().b200_head_norm_gated(r, r, 4, r, 1, 1, 0, 1e-5, r, None, None, 4, None) == -1


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
