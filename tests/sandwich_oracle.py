"""Plain, slow statement of the sandwich decoder ("Lozepel"): a norm before and after every sublayer; two kinds of grouped-query
attention, a pair of mixers side by side (softmax attention and lightning attention), a clamped gated feed-forward or a mixture of gated
experts with identity experts, an embedding of token pairs beside the embedding, and a soft cap on the logits.  numpy float64, one function
per mechanism, the recurrence one token at a time.  Shares no code with the library.

`weights` maps state names to float arrays (bf16 weights widened); `config` is the dictionary of config.json.
"""
from __future__ import annotations

import numpy as np

from hybrid_oracle import rms, rotate, sigmoid, silu

F = np.float64


def zero_centred_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (1.0 + w)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


def pair_row(previous, token, spec):
    """Row of the pair table; `previous` is None for a sequence's first token."""
    if previous is None:
        return spec["buckets"]
    return (int(previous) * spec["mul_prev"] + int(token) * spec["mul_cur"]) % spec["buckets"]


def embedding(w, tokens, config):
    spec = config["embedding"]["bigram"]
    rows = [pair_row(tokens[t - 1] if t else None, tokens[t], spec) for t in range(len(tokens))]
    return w["embed"][np.asarray(tokens)] + w["bigram"][rows]


def sink_softmax(score, sink):
    """Softmax over the last axis whose denominator also holds exp(sink); sink None: no such term."""
    top = score.max(axis=-1, keepdims=True)
    if sink is not None:
        top = np.maximum(top, sink)
    e = np.exp(score - top)
    return e / (e.sum(axis=-1, keepdims=True) + (np.exp(sink - top) if sink is not None else 0.0))


def attend(q, k, v, scale, cap, sinks):
    """q [H, T, d], k [G, T, d], v [G, T, e] -> [T, H, e]; every position sees itself and all before it."""
    H, T, _ = q.shape
    group = H // k.shape[0]
    seen = np.tril(np.ones((T, T), dtype=bool))
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        score = (q[h] @ k[h // group].T) * scale
        if cap is not None:
            score = soft_cap(score, cap)
        out[:, h] = sink_softmax(np.where(seen, score, -np.inf), None if sinks is None else sinks[h]) @ v[h // group]
    return out


def heads_of(x, heads):
    return x.reshape(x.shape[0], heads, -1).transpose(1, 0, 2)


def attention_keys_as_values(h, w, p, m):
    """Biased queries and keys, rotated; unrotated, the keys serve as values too; a sink of score 0; one gate per head."""
    H, G, pos = m["heads"], m["kv_heads"], np.arange(h.shape[0])
    q = heads_of(h @ w[p + "q"].T + w[p + "q.b"], H)
    k = heads_of(h @ w[p + "k"].T + w[p + "k.b"], G)
    turn = lambda x: rotate(x, pos, m["rot"]["dims"], m["rot"]["base"])
    o = attend(turn(q), turn(k), k, m["scale"], None, np.zeros(H))
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


def attention_head_norms(h, w, p, m, eps, shared):
    """Rotated queries and keys over their root mean square per head, capped scores, a learned sink per head.  `shared` keeps the keys and
    values that layers have made, for the layers that take them over; `shared["at"]` is the layer's own number."""
    H, G, pos = m["heads"], m["kv_heads"], np.arange(h.shape[0])
    turn = lambda x: rms(rotate(x, pos, m["rot"]["dims"], m["rot"]["base"]), eps)
    q = turn(heads_of(h @ w[p + "q"].T, H))
    if m.get("kv_from") is None:
        shared[shared["at"]] = turn(heads_of(h @ w[p + "k"].T, G)), heads_of(h @ w[p + "v"].T, G)
    k, v = shared[m["kv_from"] if m.get("kv_from") is not None else shared["at"]]
    o = attend(q, k, v, m["scale"], m.get("softcap"), w[p + "sink"])
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


def attention_projection_norms(h, w, p, m, eps):
    """No positions; RMS norms over all query heads and over all key heads at once; a learned sink and a gate per head."""
    H, G = m["heads"], m["kv_heads"]
    q = heads_of(rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"], H)
    k = heads_of(rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"], G)
    o = attend(q, k, heads_of(h @ w[p + "v"].T, G), m["scale"], None, w[p + "sink"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(h.shape[0], -1) @ w[p + "o"].T


def lightning_recurrence(q, k, v, decay):
    """q, k [T, H, d], v [T, H, e], decay [H]: S = decay S + k v^T, o = S^T q, token by token."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]))
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = np.asarray(decay)[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hde,hd->he", S, q[t])
    return out


def lightning(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    part = lambda name: silu(h @ w[p + name].T).reshape(T, H, -1)
    o = lightning_recurrence(part("q"), part("k"), part("v"), m["decay"]).reshape(T, -1)
    return (rms(o, eps) * w[p + "norm"] * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def side_by_side(h, w, p, m, eps):
    return (m["left_scale"] * attention_projection_norms(h, w, p + "left.", m["left"], eps)
            + m["right_scale"] * lightning(h, w, p + "right.", m["right"], eps))


def clamped_units(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, w, p, mlp):
    return clamped_units(h @ w[p + "gate"].T, h @ w[p + "up"].T, mlp["limit"]) @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def route(logits, correction, top):
    """Chosen outputs [T, top] by falling corrected score, and their scores without the correction."""
    s = softmax(logits)
    chosen = np.argsort(-(s + correction), axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def closest_call(logits, correction, top):
    """Smallest distance, over the tokens, between the choice scores of the last output chosen and the first one not chosen."""
    c = np.sort(softmax(logits) + correction, axis=1)[:, ::-1]
    return float((c[:, top - 1] - c[:, top]).min()) if c.shape[1] > top else np.inf


def mixture(h, w, p, mlp, calls=None):
    r = mlp["router"]
    logits = h @ w[p + "router"].T
    chosen, score = route(logits, w[p + "correction"], r["top"])
    if calls is not None:
        calls.append(closest_call(logits, w[p + "correction"], r["top"]))
    out = np.zeros_like(h)
    for e in np.unique(chosen):
        t, slot = np.nonzero(chosen == e)
        y = expert(h[t], w, f"{p}e{e}.") if e < r["experts"] else h[t]      # the last outputs hand the input through
        out[t] += score[t, slot][:, None] * y
    return out


def mixer(h, w, i, spec, eps, shared):
    p, m = f"l{i}.mix.", spec["mixer"]
    shared["at"] = i
    if spec["type"] == "attention":
        return attention_keys_as_values(h, w, p, m)
    if spec["type"] == "attention_2":
        return attention_head_norms(h, w, p, m, eps, shared)
    return side_by_side(h, w, p, m, eps)


def layer(x, w, i, spec, eps, shared, calls=None):
    p = f"l{i}."
    x = x + zero_centred_norm(mixer(zero_centred_norm(x, w[p + "norm1"], eps), w, i, spec, eps, shared), w[p + "norm1b"], eps)
    if spec.get("mlp"):
        h = zero_centred_norm(x, w[p + "norm2"], eps)
        y = dense_ff(h, w, p + "mlp.", spec["mlp"]) if spec["mlp"]["kind"] == "dense" else mixture(h, w, p + "mlp.", spec["mlp"], calls)
        x = x + zero_centred_norm(y, w[p + "norm2b"], eps)
    return x


def forward(config, weights, tokens, trail=None, calls=None):
    """Logits [T, vocab] of one sequence; `trail` collects the residual stream after every layer, `calls` the routers' closest calls."""
    w = {n: np.asarray(a, dtype=F) for n, a in weights.items()}
    eps = config["norm"]["eps"]
    x, shared = embedding(w, tokens, config), {}
    for i, spec in enumerate(config["layers"]):
        x = layer(x, w, i, spec, eps, shared, calls)
        if trail is not None:
            trail.append(x.copy())
    return soft_cap(zero_centred_norm(x, w["final.norm"], eps) @ w["head"].T, config["logit_softcap"])


def greedy(config, weights, prompt, steps):
    """Greedy continuation of one prompt and the smallest top-1 / top-2 margin met, by whole passes."""
    ids, margin = list(prompt), np.inf
    for _ in range(steps):
        last = forward(config, weights, ids)[-1]
        top = np.sort(last)[-2:]
        margin = min(margin, top[1] - top[0])
        ids.append(int(last.argmax()))
    return ids[len(prompt):], margin
