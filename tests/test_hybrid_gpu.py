"""Hybrid decoder on the GPU against the plain statement (hybrid_oracle): the mechanisms alone at kernel level, then whole models -
prompts, decoding, portions, unequal batches, reused slots, far keys, long decoding, greedy generation."""
import ctypes as C
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import ctorch_b200 as B
import hybrid_cases as H
import hybrid_oracle as O

torch = pytest.importorskip("torch")
pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOLERANCE = {"f32": 2e-5, "bf16": 2e-2}


def ratio(got, want):
    """Largest difference over the largest reference magnitude."""
    return float(np.abs(np.asarray(got, dtype=np.float64) - want).max() / np.abs(want).max())


_models = {}


def model_of(name, dtype, seed=0):
    key = (name, dtype, seed)
    if key not in _models:
        weights = H.make_weights(H.CASES[name], seed)
        _models[key] = (B.LanguageModel(H.CASES[name], weights, dtype=dtype), weights)
    return _models[key]


def all_places(n):
    return list(range(n))


# ---- mechanisms alone -------------------------------------------------------------------------------------------
class Pass:
    """A packed pass in device memory: counts of new rows per sequence, the slots they live in, lengths of all slots."""

    def __init__(self, counts, slots, lengths):
        first = np.concatenate([[0], np.cumsum(counts)])
        self.slot = torch.tensor(slots, dtype=torch.int32, device="cuda")
        self.first = torch.tensor(first, dtype=torch.int32, device="cuda")
        self.sequence = torch.tensor(np.repeat(np.arange(len(counts)), counts), dtype=torch.int32, device="cuda")
        self.lengths = torch.tensor(lengths, dtype=torch.int32, device="cuda")
        self.first_host = first
        self.c = B.Rows(int(first[-1]), len(counts), int(max(counts)), self.slot.data_ptr(), self.first.data_ptr(), self.sequence.data_ptr(),
                        self.lengths.data_ptr())

    def advance(self):
        B.kcheck(B.lib().b200_rows_advance(C.byref(self.c), None))


def dev(a):
    return torch.tensor(np.ascontiguousarray(a, dtype=np.float32), device="cuda")


def planes(rows, width):
    return torch.zeros(rows, width, dtype=torch.bfloat16, device="cuda"), torch.zeros(rows, width, dtype=torch.bfloat16, device="cuda")


def joined(hi, lo):
    return (hi.float() + lo.float()).cpu().numpy()


@pytest.mark.parametrize("rows, width", [(1, 8), (5, 100), (700, 1030)])
def test_dynamic_tanh(rows, width):
    rng = np.random.default_rng(rows)
    x, more, vec, w, b = (rng.normal(0, 2, s) for s in ((rows, width), (rows, width), width, width, width))
    tx, tm, tv, tw, tb = map(dev, (x, more, vec, w, b))
    norm = B.ElementwiseNorm(0.37, tw.data_ptr(), tb.data_ptr())
    total, out = torch.empty_like(tx), torch.empty_like(tx)
    hi, lo = planes(rows, width)
    B.kcheck(B.lib().b200_dynamic_tanh(tx.data_ptr(), tm.data_ptr(), tv.data_ptr(), rows, width, C.byref(norm), total.data_ptr(), out.data_ptr(),
                                       hi.data_ptr(), lo.data_ptr(), None))
    torch.cuda.synchronize()
    want = O.dynamic_tanh(x + more + vec, 0.37, w, b)
    assert ratio(total.cpu(), x + more + vec) < 1e-6 and ratio(out.cpu(), want) < 1e-6 and ratio(joined(hi, lo), want) < 3e-5


@pytest.mark.parametrize("rows, inner, out", [(1, 64, 40), (3, 128, 130), (16, 256, 512), (20, 136, 200), (100, 512, 256), (300, 256, 384), (40, 4096, 64)])
def test_projection_writes_the_next_norm(rows, inner, out):
    """Residual epilogue of every linear kernel family with a Dynamic Tanh norm behind it."""
    rng = np.random.default_rng(out)
    x, w = rng.normal(size=(rows, inner)), H.bf16_to_f32(H.bf16_bits(rng.normal(0, inner ** -0.5, (out, inner)).astype(np.float32)))
    res, nw, nb = rng.normal(0, 2, (rows, out)), rng.normal(1, 0.3, out), rng.normal(0, 0.3, out)
    hi, lo = planes(rows, inner)
    tx = dev(x)
    hi.copy_(tx)
    lo.copy_(tx - hi.float())
    tw, tres, tnw, tnb = torch.tensor(w, device="cuda").bfloat16(), dev(res), dev(nw), dev(nb)
    y = torch.empty_like(tres)
    oh, ol = planes(rows, out)
    norm = B.ElementwiseNorm(0.6, tnw.data_ptr(), tnb.data_ptr())
    a = B.ShadowLinearArgs(x_hi=hi.data_ptr(), x_lo=lo.data_ptr(), rows=rows, inner=inner, weight=tw.data_ptr(), out=out, epilogue=1,
                           residual=tres.data_ptr(), y=y.data_ptr(), out_hi=oh.data_ptr(), out_lo=ol.data_ptr(), out_norm=C.pointer(norm))
    torch.cuda.synchronize()
    B.kcheck(B.lib().b200_linear_shadow(C.byref(a), None))
    torch.cuda.synchronize()
    total = res + x @ w.T.astype(np.float64)
    assert ratio(y.cpu(), total) < 3e-5
    assert ratio(joined(oh, ol), O.dynamic_tanh(total, 0.6, nw, nb)) < 5e-5


SSM = [dict(heads=4, vdim=16, state=24, groups=2, taps=4), dict(heads=1, vdim=1, state=1, groups=1, taps=1), dict(heads=3, vdim=10, state=7, groups=1, taps=5),
       dict(heads=2, vdim=70, state=128, groups=2, taps=3), dict(heads=4, vdim=36, state=96, groups=2, taps=2), dict(heads=2, vdim=20, state=200, groups=1, taps=4),
       dict(heads=1, vdim=300, state=300, groups=1, taps=4), dict(heads=8, vdim=64, state=50, groups=4, taps=4)]


@pytest.mark.parametrize("spec", SSM, ids=lambda s: "h{heads}_p{vdim}_n{state}_g{groups}_t{taps}".format(**s))
def test_state_space_recurrence(spec):
    """Prompt of unequal sequences through the scan, then single rows, then a portion of two, in shuffled slots with junk in
    them: outputs and final states against the recurrence, token by token."""
    s = spec
    heads, P, N, G, taps = s["heads"], s["vdim"], s["state"], s["groups"], s["taps"]
    channels, inner = heads * P + 2 * G * N, heads * P
    rng = np.random.default_rng(N)
    totals, slots = [37, 1 + 3 + 2, 20], [3, 0, 2]
    conv_w, conv_b = rng.normal(0, 0.5, (channels, taps)), rng.normal(0, 0.3, channels)
    dt_bias, a_log, d = rng.uniform(-2, 1, heads), rng.uniform(-1, 1.5, heads), rng.uniform(0.5, 1.5, heads)
    rows = [rng.normal(size=(t, inner + channels + heads)) for t in totals]
    want, states = [], []
    for r in rows:
        mixed = O.silu(O.short_conv(r[:, inner:inner + channels], conv_w, conv_b))
        y, S = O.ssm_recurrence(mixed[:, :inner].reshape(-1, heads, P), mixed[:, inner:inner + G * N].reshape(-1, G, N),
                                mixed[:, inner + G * N:].reshape(-1, G, N), O.softplus(r[:, inner + channels:] + dt_bias), a_log, d, return_state=True)
        want.append(y.reshape(-1, inner))
        states.append(S)
    params = [dev(v) for v in (conv_w, conv_b, dt_bias, a_log, d)]
    conv_state = torch.full((4, taps, channels), 7.0, device="cuda")
    ssm_state = torch.full((4, heads, N, P), 5.0, device="cuda")
    lengths = [0] * 4
    done = [0, 0, 0]
    # the first pass brings unequal prompts, then single rows, then portions of two
    for counts in ([32, 1, 15], [1, 1, 1], [1, 1, 1], [1, 1, 1], [2, 2, 2]):
        p = Pass(counts, slots, lengths)
        chunk = dev(np.concatenate([r[a:a + n] for r, a, n in zip(rows, done, counts)]))
        mixed, y = torch.empty(chunk.shape[0], channels, device="cuda"), torch.empty(chunk.shape[0], inner, device="cuda")
        a = B.SsmArgs(heads, P, N, G, taps, *[t.data_ptr() for t in params], conv_state.data_ptr(), ssm_state.data_ptr(), chunk.data_ptr(),
                      mixed.data_ptr(), y.data_ptr())
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_ssm_forward(C.byref(a), C.byref(p.c), None))
        p.advance()
        torch.cuda.synchronize()
        for i, n in enumerate(counts):
            got = y[p.first_host[i]:p.first_host[i + 1]].cpu()
            assert ratio(got, want[i][done[i]:done[i] + n]) < 2e-5, (counts, i)
            done[i] += n
        lengths = p.lengths.cpu().tolist()
    assert done == totals
    for i, slot in enumerate(slots):
        assert ratio(ssm_state[slot].cpu(), states[i]) < 2e-5
    assert float(ssm_state[1].min()) == 5.0 == float(ssm_state[1].max())   # the slot nobody used


def test_streamed_state_space_step():
    """Many sequences: the persistent streaming form of a step, some sequences at their first token, slots in another order than rows."""
    heads, P, N, G, taps, count = 16, 64, 36, 2, 4, 520
    channels, inner = heads * P + 2 * G * N, heads * P
    rng = np.random.default_rng(0)
    conv_w, conv_b = rng.normal(0, 0.5, (channels, taps)), rng.normal(0, 0.3, channels)
    dt_bias, a_log, d = rng.uniform(-2, 1, heads), rng.uniform(-1, 1.5, heads), rng.uniform(0.5, 1.5, heads)
    params = [dev(v) for v in (conv_w, conv_b, dt_bias, a_log, d)]
    slots = rng.permutation(count)
    lengths = np.where(np.arange(count) % 3 == 0, 0, 5)   # every third slot starts afresh
    conv_state, ssm_state = dev(rng.normal(size=(count, taps, channels))), dev(rng.normal(size=(count, heads, N, P)))
    old_conv, old_state = conv_state.cpu().numpy().astype(np.float64), ssm_state.cpu().numpy().astype(np.float64)
    x = rng.normal(size=(count, inner + channels + heads))
    p = Pass([1] * count, slots.tolist(), lengths.tolist())
    tx, mixed, y = dev(x), torch.empty(count, channels, device="cuda"), torch.empty(count, inner, device="cuda")
    a = B.SsmArgs(heads, P, N, G, taps, *[t.data_ptr() for t in params], conv_state.data_ptr(), ssm_state.data_ptr(), tx.data_ptr(), mixed.data_ptr(),
                  y.data_ptr())
    torch.cuda.synchronize()
    B.kcheck(B.lib().b200_ssm_forward(C.byref(a), C.byref(p.c), None))
    torch.cuda.synchronize()
    got, state = y.cpu().numpy(), ssm_state.cpu().numpy()
    for r in range(0, count, 7):
        slot = slots[r]
        length = lengths[slot]
        past = np.stack([old_conv[slot, (length - b) % taps] if length - b >= 0 else np.zeros(channels) for b in (3, 2, 1)])
        if length == 0:
            past[:] = 0.0
        m = O.silu((np.concatenate([past, x[r:r + 1, inner:inner + channels]]) * conv_w.T).sum(0) + conv_b)
        dt = O.softplus(x[r, inner + channels:] + dt_bias)
        for h in range(heads):
            g = h // (heads // G)
            xs, Bm, Cm = m[h * P:(h + 1) * P], m[inner + g * N:inner + (g + 1) * N], m[inner + (G + g) * N:inner + (G + g + 1) * N]
            S = np.exp(-np.exp(a_log[h]) * dt[h]) * (old_state[slot, h] if length else 0.0) + dt[h] * np.outer(Bm, xs)
            assert ratio(state[slot, h], S) < 1e-5
            assert np.abs(got[r, h * P:(h + 1) * P] - (S.T @ Cm + d[h] * xs)).max() < 1e-4
        assert np.allclose(conv_state[slot, length % taps].cpu().numpy(), x[r, inner:inner + channels], atol=1e-5)


@pytest.mark.parametrize("rows, width, parts", [(3, 64, 1), (2, 96, 4), (1, 30, 3), (5, 6000, 2), (4, 16, 16)])
def test_gated_group_norm(rows, width, parts):
    rng = np.random.default_rng(width)
    y, z, w = rng.normal(size=(rows, width)), rng.normal(0, 2, (rows, width + 5)), rng.normal(1, 0.3, width)
    y[:, :width // parts] *= 100.0   # parts of very different size: one shared root mean square would show
    ty, tz, tw = dev(y), dev(z), dev(w)
    out = torch.empty_like(ty)
    hi, lo = planes(rows, width)
    B.kcheck(B.lib().b200_gated_group_norm(ty.data_ptr(), tz.data_ptr(), width + 5, tw.data_ptr(), rows, width, parts, 1e-3, out.data_ptr(),
                                           hi.data_ptr(), lo.data_ptr(), None))
    torch.cuda.synchronize()
    want = O.gated_norm(y, z[:, :width], w, parts, 1e-3)
    assert ratio(out.cpu(), want) < 3e-6 and ratio(joined(hi, lo), want) < 3e-5


class Latent:
    """One latent-attention layer's kernels over torch memory."""

    def __init__(self, heads, dim, rot, vdim, rank, q_rank, dtype, slots=3, capacity=300, dims=None, base=100.0, scale=0.2, seed=0, eps=1e-5):
        rng = np.random.default_rng(seed)
        self.n = dict(heads=heads, dim=dim, rot=rot, vdim=vdim, rank=rank, q_rank=q_rank, dims=dims or rot, base=base, scale=scale, eps=eps)
        self.bf16, self.slots = dtype == "bf16", slots
        q = (lambda a: H.bf16_to_f32(H.bf16_bits(a.astype(np.float32)))) if self.bf16 else (lambda a: a.astype(np.float32))
        self.uk, self.uv = q(rng.normal(0, rank ** -0.5, (heads, dim, rank))), q(rng.normal(0, rank ** -0.5, (heads, vdim, rank)))
        self.q_norm, self.kv_norm = rng.uniform(0.5, 1.5, q_rank), rng.uniform(0.5, 1.5, rank)
        angle = np.arange(capacity)[:, None] * base ** (-2.0 * np.arange(self.n["dims"] // 2) / self.n["dims"])
        to = (lambda a: torch.tensor(np.ascontiguousarray(a), device="cuda").bfloat16()) if self.bf16 else dev
        self.lengths = torch.zeros(slots, dtype=torch.int32, device="cuda")
        self.keep = [dev(np.cos(angle)), dev(np.sin(angle)), dev(self.q_norm), dev(self.kv_norm), to(self.uk.transpose(0, 2, 1)), to(self.uv)]
        self.cache = C.c_void_p()
        code = B.BF16 if self.bf16 else B.F32
        B.kcheck(B.lib().b200_latent_cache_create(0, code, slots, rank + rot, capacity, 64, self.lengths.data_ptr(), C.byref(self.cache)))
        k = self.keep
        self.a = B.LatentArgs(heads, dim, rot, vdim, rank, q_rank, self.n["dims"], scale, eps, k[0].data_ptr(), k[1].data_ptr(), capacity, k[2].data_ptr(),
                              k[3].data_ptr(), self.cache, code, k[4].data_ptr(), k[5].data_ptr())

    def shuffle_pages(self, seed):
        pages = B.lib().b200_kv_cache_pages_per_sequence(self.cache) * self.slots
        table = np.random.default_rng(seed).permutation(pages).astype(np.int32)
        B.kcheck(B.lib().b200_kv_cache_set_page_table(self.cache, table.ctypes.data_as(C.POINTER(C.c_int32)), None))

    def kernel(self):
        return B.lib().b200_latent_attention_kernel(C.byref(self.a)).decode()

    def prepare(self, p, projected):
        out = torch.empty(projected.shape[0], self.n["q_rank"], device="cuda")
        hi, lo = planes(*out.shape)
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_latent_prepare(C.byref(self.a), C.byref(p.c), projected.data_ptr(), out.data_ptr(), hi.data_ptr(), lo.data_ptr(), None))
        torch.cuda.synchronize()
        assert ratio(joined(hi, lo), out.cpu().numpy()) < 3e-5
        return out.cpu().numpy()

    def attend(self, p, query, max_length):
        n = self.n
        rows = query.shape[0]
        tq = dev(query)
        absorbed = torch.full((rows, n["heads"], n["rank"] + n["rot"]), float("nan"), device="cuda")
        out = torch.full((rows, n["heads"], n["rank"]), float("nan"), device="cuda")
        bytes_ = B.lib().b200_latent_scratch_bytes(C.byref(self.a), rows, p.c.sequences, p.c.max_count, max_length)
        scratch = torch.full((bytes_ // 4 + 1,), float("nan"), device="cuda")
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_latent_query(C.byref(self.a), C.byref(p.c), tq.data_ptr(), absorbed.data_ptr(), None))
        B.kcheck(B.lib().b200_latent_attention(C.byref(self.a), C.byref(p.c), absorbed.data_ptr(), max_length, scratch.data_ptr(), bytes_, out.data_ptr(), None))
        torch.cuda.synchronize()
        return absorbed.cpu().numpy(), out.cpu().numpy()

    def value(self, latent, gate):
        n = self.n
        rows = latent.shape[0]
        tl, tg = dev(latent), dev(gate)
        out = torch.empty(rows, n["heads"] * n["vdim"], device="cuda")
        hi, lo = planes(*out.shape)
        torch.cuda.synchronize()
        B.kcheck(B.lib().b200_latent_value(C.byref(self.a), rows, tl.data_ptr(), tg.data_ptr(), tg.shape[1], out.data_ptr(), hi.data_ptr(), lo.data_ptr(), None))
        torch.cuda.synchronize()
        assert ratio(joined(hi, lo), out.cpu().numpy()) < 3e-5
        return out.cpu().numpy()

    def close(self):
        B.lib().b200_kv_cache_release(self.cache)


LATENT = [dict(heads=4, dim=16, rot=8, vdim=24, rank=32, q_rank=40), dict(heads=3, dim=10, rot=6, vdim=14, rank=22, q_rank=13, dims=4),
          dict(heads=16, dim=32, rot=64, vdim=40, rank=512, q_rank=96), dict(heads=20, dim=24, rot=16, vdim=16, rank=144, q_rank=48),
          dict(heads=40, dim=8, rot=24, vdim=72, rank=264, q_rank=24), dict(heads=1, dim=72, rot=8, vdim=8, rank=128, q_rank=8)]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("spec", LATENT, ids=lambda s: "h{heads}_r{rank}_{rot}".format(**s))
def test_latent_attention_layer(spec, dtype):
    """norms + rotation + append, absorbed query, attention and value up-projection: a prompt of unequal sequences, then single
    rows (split over CTAs) and a portion of three, on shuffled pages."""
    k = Latent(**spec, dtype=dtype, seed=spec["rank"])
    n = k.n
    k.shuffle_pages(4)
    even = spec["rank"] % 8 == 0
    assert k.kernel() == ("latent_mma_kernel" if dtype == "bf16" and even else "latent_generic_kernel")
    tol = 3e-6 if dtype == "f32" else 1e-2   # bf16: the cached latents
    rng = np.random.default_rng(9)
    Hn, d, r, K, e = n["heads"], n["dim"], n["rot"], n["rank"], n["vdim"]
    slots, totals = [2, 0, 1], [205, 70, 8]
    data = [rng.normal(size=(t, n["q_rank"] + K + r + Hn * e)) for t in totals]
    queries = [rng.normal(size=(t, Hn, d + r)) for t in totals]
    want = []
    for rows, q in zip(data, queries):
        T = len(rows)
        pos = np.arange(T)
        c = O.rms(rows[:, n["q_rank"]:n["q_rank"] + K], n["eps"]) * k.kv_norm
        rot = O.rotate(rows[:, n["q_rank"] + K:n["q_rank"] + K + r], pos, n["dims"], n["base"])
        keys = np.concatenate([np.einsum("hdk,tk->htd", k.uk, c), np.broadcast_to(rot, (Hn, T, r))], -1)
        qr = np.concatenate([q[..., :d].transpose(1, 0, 2), O.rotate(q[..., d:].transpose(1, 0, 2), pos, n["dims"], n["base"])], -1)
        # weights over the latents themselves, then the value up-projection
        want.append(O.causal_softmax_attention(qr, keys, np.broadcast_to(c, (Hn, T, K)), n["scale"]))
    done, lengths = [0, 0, 0], [0, 0, 0]
    for counts in ([150, 64, 1], [1, 1, 1], [1, 1, 1], [1, 1, 1], [3, 3, 3], [49, 0, 1]):
        live = [i for i in range(3) if counts[i]]
        p = Pass([counts[i] for i in live], [slots[i] for i in live], lengths)
        k.lengths.copy_(p.lengths)
        rows = np.concatenate([data[i][done[i]:done[i] + counts[i]] for i in live])
        q = np.concatenate([queries[i][done[i]:done[i] + counts[i]] for i in live])
        q_latent = k.prepare(p, dev(rows))
        assert ratio(q_latent, O.rms(rows[:, :n["q_rank"]], n["eps"]) * k.q_norm) < 3e-6
        absorbed, out = k.attend(p, q, 256)
        assert ratio(absorbed[..., :K], np.einsum("thd,hdk->thk", q[..., :d], k.uk)) < (3e-6 if dtype == "f32" else 3e-5)
        expect = np.concatenate([want[i][done[i]:done[i] + counts[i]] for i in live])
        assert ratio(out, expect) < tol, counts
        gate = rng.normal(size=(len(rows), Hn * e + 3))
        v = np.einsum("hek,thk->the", k.uv, expect).reshape(len(rows), -1) * O.sigmoid(gate[:, :Hn * e])
        assert ratio(k.value(expect, gate), v) < (3e-6 if dtype == "f32" else 3e-5)
        p.advance()
        torch.cuda.synchronize()
        lengths = p.lengths.cpu().tolist()
        for i in live:
            done[i] += counts[i]
    k.close()


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("heads", [2, 24])
def test_one_key_stands_out(heads, dtype):
    """Every query asks for one latent, far away, at page borders, its own or the first: an edge that is one token off, a wrong
    page or a key seen too early shows as another latent."""
    k = Latent(heads=heads, dim=64, rot=8, vdim=8, rank=64, q_rank=8, dtype=dtype, capacity=420, scale=1.0, seed=1, slots=2)
    k.shuffle_pages(1)
    T, K = 400, 64
    rng = np.random.default_rng(2)
    latents = rng.normal(size=(T, K))
    rows = np.zeros((T, 8 + K + 8 + heads * 8))
    rows[:, :8], rows[:, 8:8 + K] = 1.0, latents
    c = O.rms(latents, k.n["eps"]) * k.kv_norm
    targets = lambda t: [x for x in (0, 1, 62, 63, 64, 65, 127, 128, 191, 192, 319, 320, t - 1, t) if 0 <= x <= t]
    rng2 = np.random.default_rng(3)
    aim = np.array([[rng2.choice(targets(t)) for _ in range(heads)] for t in range(T)])
    # the query's unrotated part solves uk^T q = 40 c_target as well as it can (uk is square here), so that score stands out
    q = np.zeros((T, heads, 72))
    for h in range(heads):
        inverse = np.linalg.pinv(k.uk[h].astype(np.float64).T)
        q[:, h, :64] = (inverse @ (1.5 * c[aim[:, h]]).T).T
    want = c[aim]
    at, lengths = 0, [0, 0]
    for count in (129, 1, 1, 61, 1, 63, 2, 1, 141):   # ends at and around page borders, prompts and single rows
        p = Pass([count], [1], lengths)
        k.lengths.copy_(p.lengths)
        k.prepare(p, dev(rows[at:at + count]))
        _, out = k.attend(p, q[at:at + count], 420)
        # a key beyond the row's own position, had it been seen, would be missed here: the row's own key is its last one
        assert np.abs(out - want[at:at + count]).max() < 0.06 * np.abs(want).max(), (at, count)
        p.advance()
        torch.cuda.synchronize()
        lengths, at = p.lengths.cpu().tolist(), at + count
    assert at == T
    k.close()


def test_standing_out_inputs_discriminate():
    """The same inputs with the mistake planted in the plain statement: dropping the asked key changes the answer altogether."""
    rng = np.random.default_rng(2)
    c = O.rms(rng.normal(size=(50, 64)), 1e-5)
    score = 1.5 * c[7] @ c.T
    p = np.exp(score - score.max())
    masked = np.where(np.arange(50) == 7, 0.0, p)
    assert np.abs(p @ c / p.sum() - c[7]).max() < 0.05 and np.abs(masked @ c / masked.sum() - c[7]).max() > 0.5


# ---- whole models -----------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", H.CASES)
def test_prompt_matches_the_statement_layer_by_layer(name, dtype):
    model, w = model_of(name, dtype)
    c = H.CASES[name]
    ids = H.tokens(c, 71)
    trail = []
    want = O.forward(c, w, ids, trail)
    model.new_cache(2, 80)
    got_trail = model.trail(1, ids)
    for i, rows in enumerate(trail):
        assert ratio(got_trail[i], rows) < TOLERANCE[dtype], f"layer run {i}"
    assert ratio(model.run([(0, ids, all_places(71))]), want) < TOLERANCE[dtype]


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("name", H.CASES)
def test_decoding_and_portions_equal_the_whole_prompt(name, dtype):
    """Token by token, portions of two, unequal portions: the logits of every position equal those of one pass."""
    model, _ = model_of(name, dtype)
    c = H.CASES[name]
    ids = H.tokens(c, 70, seed=3)
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
@pytest.mark.parametrize("name", ["mixed", "large", "odd"])
def test_unequal_batches_equal_each_alone_and_slots_are_reused(name, dtype):
    model, _ = model_of(name, dtype)
    c = H.CASES[name]
    prompts = [H.tokens(c, n, seed=n) for n in (1, 67, 20, 3, 130)]
    tails = [4, 6, 1, 9, 5]
    full = [np.concatenate([p, H.tokens(c, t, seed=100 + t)]) for p, t in zip(prompts, tails)]
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
            if t % 2:
                parts = parts[::-1]   # the order of the rows in a batch does not matter either
            step(parts)
            for i, n in enumerate(tails):
                if t + 1 == n:
                    model.cache.release(slots[i])
        for i in range(len(full)):
            assert ratio(np.concatenate(got[i]), alone[i]) < tol, (slots, i)
        assert all(model.cache.length(s) == 0 for s in slots)


def test_long_pass_is_cut_and_joined():
    """More rows than one pass over the layers takes: the cut falls inside a sequence and between sequences."""
    model, _ = model_of("ones", "f32")
    c = H.CASES["ones"]
    ids = [H.tokens(c, n, seed=n) for n in (5000, 6000, 40)]
    model.new_cache(3, 6000)
    want_places = [[0, 4999], [3190, 3191, 3192, 5999], [39]]
    got = model.run([(i, t, p) for i, (t, p) in enumerate(zip(ids, want_places))])
    at = 0
    for i, (t, places) in enumerate(zip(ids, want_places)):
        model.cache.release(i)
        alone = []
        for a in range(0, len(t), 2500):
            part = t[a:a + 2500]
            alone.append(model.run([(i, part, [p - a for p in places if a <= p < a + len(part)])]))
        assert ratio(got[at:at + len(places)], np.concatenate(alone)) < 2e-5
        at += len(places)


@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_long_decoding_stays_with_the_statement(dtype):
    model, w = model_of("mixed", dtype)
    c = H.CASES["mixed"]
    ids = H.tokens(c, 300, seed=8)
    want = O.forward(c, w, ids)
    model.new_cache(1, 300)
    model.run([(0, ids[:5], [])])
    got = np.concatenate([model.run([(0, [t], [0])]) for t in ids[5:]])
    assert ratio(got, want[5:]) < TOLERANCE[dtype]


@pytest.mark.parametrize("name", ["mixed", "odd", "large"])
def test_greedy_generation_equals_the_statement(name):
    """The framework's own loop: prompts of unequal length in one batch, the token loop in a captured graph."""
    model, w = model_of(name, "f32")
    c = H.CASES[name]
    prompts, steps = [H.tokens(c, n, seed=n) for n in (9, 2, 31)], 12
    got = model.generate(prompts, steps)
    for row, prompt in zip(got, prompts):
        want, margin = O.greedy(c, w, prompt, steps)
        assert margin > 1e-4 and list(row) == want


@pytest.mark.parametrize("batch", [1, 20])
def test_bf16_generation_feeds_back_its_own_choice(batch):
    """bf16 loop (fused logits + choice; streaming and dense projections): replaying its tokens gives logits whose best is the
    token chosen next, and the logits asked for on demand are those."""
    model, _ = model_of("mixed", "bf16")
    c = H.CASES["mixed"]
    steps, prompts = 8, np.stack([H.tokens(c, 10, seed=b) for b in range(batch)])
    model.new_cache(batch, 10 + steps)
    gen = B.Generation(model, batch, steps)
    gen.prefill(prompts)
    gen.step(steps - 1)
    tokens, last = gen.tokens(), gen.logits()
    assert gen.launches_per_step() > 0 and tokens.shape == (batch, steps)
    model.new_cache(1, 10 + steps)
    for b in range(batch):
        ids = np.concatenate([prompts[b], tokens[b]])
        logits = model.run([(0, ids, all_places(len(ids)))])
        model.cache.release(0)
        for s in range(steps):
            row = logits[9 + s]
            assert row.max() - row[tokens[b, s]] < 1e-2 * np.abs(row).max()
        assert ratio(last[b], logits[9 + steps - 1]) < 1e-2


def test_sampling_and_host_steps():
    model, _ = model_of("mixed", "f32")
    c = H.CASES["mixed"]
    prompts = np.stack([H.tokens(c, 7, seed=b) for b in range(3)])
    greedy = model.generate(list(prompts), 6)
    assert np.array_equal(model.generate(list(prompts), 6, temperature=1e-4), greedy)   # cold sampling is the greedy choice
    model.new_cache(3, 13)
    gen = B.Generation(model, 3, 6)
    gen.prefill(prompts)
    first = gen.tokens()[:, 0].copy()
    assert np.array_equal(gen.run_host(first, 5).T, greedy[:, 1:])
    profile = None
    model.new_cache(3, 13)
    gen = B.Generation(model, 3, 6)
    gen.prefill(prompts)
    profile = gen.profile_step()
    assert profile["launches"] > 10 and profile["attention_ms"] > 0


def test_cache_errors_leave_the_model_usable():
    model, _ = model_of("mixed", "f32")
    c = H.CASES["mixed"]
    model.new_cache(2, 10)
    ids = H.tokens(c, 10)
    want = model.run([(1, ids, [9])])
    model.cache.release(1)
    for entries, message in (([(0, H.tokens(c, 11), [])], "capacity"), ([(2, ids, [])], "slot out of range"), ([(0, ids[:2], []), (0, ids[:2], [])], "twice"),
                             ([(0, [c["vocab"]], [])], "out of range"), ([(0, ids[:2], [2])], "wanted place"), ([(0, [], [])], "at least one token")):
        with pytest.raises(B.B200Error, match=message):
            model.run(entries)
    assert ratio(model.run([(1, ids, [9])]), want) < 1e-6
    with pytest.raises(B.B200Error, match="truncation to 0"):
        B.check(B.lib().dl_decoder_cache_truncate(model.cache.h, 3))
    B.check(B.lib().dl_decoder_cache_truncate(model.cache.h, 0))
    assert model.cache.length(1) == 0


def test_module_forward_equals_the_statement():
    model, w = model_of("mixed", "f32")
    c = H.CASES["mixed"]
    ids = np.stack([H.tokens(c, 12, seed=1), H.tokens(c, 12, seed=2)])
    got = model.module(B.Tensor.from_numpy(ids.astype(np.int64))).numpy()
    for b in range(2):
        assert ratio(got[b], O.forward(c, w, ids[b])) < TOLERANCE["f32"]


def test_single_plane_activations():
    """The bf16-activation option (one plane in passes over more than 16 rows) stays inside the bf16 tolerance."""
    weights = H.make_weights(H.CASES["mixed"], 0)
    model = B.LanguageModel(H.CASES["mixed"], weights)
    model.set_activation_dtype("bf16")
    ids = H.tokens(H.CASES["mixed"], 60)
    model.new_cache(1, 60)
    assert ratio(model.run([(0, ids, all_places(60))]), O.forward(H.CASES["mixed"], weights, ids)) < 4e-2


def test_ragged_prompts_of_the_grouped_query_decoder():
    """The same loop with the other design: unequal prompts in one batch equal each prompt alone."""
    c = {"architecture": "TransformerDecoder", "vocab": 90, "layers": 2, "width": 64, "heads": 4, "kv_heads": 2, "ff": 96, "context": 64}
    host = B.LanguageModel(c, None, dtype="f32", device=None)
    rng = np.random.default_rng(0)
    weights = {n: (np.ones(t.shape) if "norm" in n else rng.normal(0, 0.15, t.shape)).astype(np.float32)
               for n, t in host.module.state().items() if "rotary" not in n}
    for dtype in ("f32", "bf16"):
        model = B.LanguageModel(c, weights, dtype=dtype)
        prompts = [rng.integers(0, 90, n) for n in (5, 30, 1)]
        together = model.generate(prompts, 10)
        if dtype == "f32":
            for row, prompt in zip(together, prompts):
                assert np.array_equal(row, model.generate([prompt], 10)[0])


def test_command_lines(tmp_path):
    """The generation command and the trace runner as a user starts them."""
    c = H.CASES["mixed"]
    w = H.make_weights(c, 2)
    folder, out = tmp_path / "model", tmp_path / "out"
    folder.mkdir()
    out.mkdir()
    H.write_folder(folder, c, w)
    prompts = [H.tokens(c, 5, seed=1).tolist(), H.tokens(c, 3, seed=2).tolist()]
    run = subprocess.run([sys.executable, "-m", "ctorch_b200.generate", "--model", str(folder), "--dtype", "f32", "--steps", "4",
                          *[",".join(map(str, p)) for p in prompts]], cwd=ROOT, capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [[int(t) for t in line.split(",")] for line in run.stdout.split()] == [O.greedy(c, w, p, 4)[0] for p in prompts]
    a, b = H.tokens(c, 12, seed=5).tolist(), H.tokens(c, 4, seed=6).tolist()
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": b[:3], "want": []}, {"id": "y", "tokens": a[:9], "want": [0, 8]}], "end": []},
             {"step": 1, "entries": [{"id": "y", "tokens": a[9:10], "want": []}, {"id": "x", "tokens": b[3:], "want": []}], "end": ["x"]},
             {"step": 2, "entries": [{"id": "y", "tokens": a[10:11], "want": [0]}], "end": ["y"]},
             {"step": 3, "entries": [{"id": "z", "tokens": b, "want": [3]}], "end": ["z"]}]
    for dtype, tol in (("float32", 2e-5), ("bfloat16", 2e-2)):
        run = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens", "40"],
                             input="".join(json.dumps(s) + "\n" for s in steps), cwd=ROOT, capture_output=True, text=True, timeout=600)
        assert run.returncode == 0, run.stderr
        assert [line for line in run.stdout.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        full_a, full_b = O.forward(c, w, a), O.forward(c, w, b)
        for step, want in ((0, full_a[[0, 8]]), (2, full_a[[10]]), (3, full_b[[3]])):
            got = np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(-1, c["vocab"])
            assert ratio(got, want) < tol
        assert not (out / "1.f32").exists()
