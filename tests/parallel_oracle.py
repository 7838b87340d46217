"""Plain, slow statement of the parallel decoder ("Sinezen"): chunked grouped-query attention with whole-projection query and key
norms and one gate per head, beside a dense feed-forward or a mixture of experts that reads the same norm, RMS norms, and a loop whose
passes are entered through a projection of the stream and the embedding.  numpy float64, one function per mechanism.  Shares no code
with the library.

`weights` maps state names to float arrays (bf16 weights widened); `config` is the dictionary of config.json.
"""
from __future__ import annotations

import math

import numpy as np

from hybrid_oracle import rms, run_order, sigmoid, silu

F = np.float64
_erf = np.vectorize(math.erf, otypes=[F])


def gelu_exact(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def rotate_half(x, positions, dims, base):
    """Entry i turns together with entry i + dims / 2, i < dims / 2; the entries from `dims` on stay.  x [..., T, d], positions [T]."""
    out = x.copy()
    half = dims // 2
    for i in range(half):
        angle = positions * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(angle), np.sin(angle)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def chunk_visible(i, j, size):
    """Whether position i sees position j: not later, and in the same chunk of `size` positions (None: no chunks)."""
    return j <= i and (size is None or i // size == j // size)


def chunked_attention(q, k, v, scale, size):
    """q [H, T, d], k [G, T, d], v [G, T, e] -> [T, H, e]."""
    H, T, _ = q.shape
    group = H // k.shape[0]
    seen = np.array([[chunk_visible(i, j, size) for j in range(T)] for i in range(T)])
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        score = np.where(seen, (q[h] @ k[h // group].T) * scale, -np.inf)
        p = np.exp(score - score.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[h // group]
    return out


def attention(h, w, prefix, m, eps):
    H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    T = h.shape[0]
    positions = np.arange(T)
    q = rms_norm(h @ w[prefix + "q"].T, w[prefix + "q.norm"], eps)      # over all heads at once
    k = rms_norm(h @ w[prefix + "k"].T, w[prefix + "k.norm"], eps)
    v = (h @ w[prefix + "v"].T).reshape(T, G, e).transpose(1, 0, 2)
    q = rotate_half(q.reshape(T, H, d).transpose(1, 0, 2), positions, m["rot"]["dims"], m["rot"]["base"])
    k = rotate_half(k.reshape(T, G, d).transpose(1, 0, 2), positions, m["rot"]["dims"], m["rot"]["base"])
    o = chunked_attention(q, k, v, m["scale"], m["mask"]["size"] if m.get("mask") else None)
    o = o * sigmoid(h @ w[prefix + "g"].T)[:, :, None]
    return o.reshape(T, H * e) @ w[prefix + "o"].T


def dense_ff(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def expert(h, w, prefix):
    return gelu_exact(h @ w[prefix + "up"].T) @ w[prefix + "down"].T


def route(h, w, prefix, top):
    """Chosen experts [T, top] by falling score, and their scores."""
    scores = sigmoid(h @ w[prefix + "router"].T)
    chosen = np.argsort(-scores, axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(scores, chosen, axis=1)


def closest_call(h, w, prefix, top):
    """Smallest distance, over the tokens, between the logits of the last expert chosen and the first one not chosen."""
    z = np.sort(h @ w[prefix + "router"].T, axis=1)[:, ::-1]
    return float((z[:, top - 1] - z[:, top]).min()) if z.shape[1] > top else np.inf


def mixture(h, w, prefix, spec, calls=None):
    chosen, score = route(h, w, prefix, spec["router"]["top"])
    if calls is not None:
        calls.append(closest_call(h, w, prefix, spec["router"]["top"]))
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(chosen[t], score[t]):
            out[t] += expert((s * h[t])[None], w, f"{prefix}e{e}.")[0]
    return out + expert(h, w, prefix + "shared.") if spec.get("shared") else out


def layer(x, w, i, spec, eps, calls=None):
    h = rms_norm(x, w[f"l{i}.norm1"], eps)
    total = attention(h, w, f"l{i}.mix.", spec["mixer"], eps)
    if spec.get("mlp"):
        total = total + (dense_ff(h, w, f"l{i}.mlp.") if spec["mlp"]["kind"] == "dense" else mixture(h, w, f"l{i}.mlp.", spec["mlp"], calls))
    return x + total


def enter_pass(x, first, w):
    return np.concatenate([x, first], axis=-1) @ w["loop.in"].T


def forward(config, weights, tokens, trail=None, calls=None):
    """Logits [T, vocab] of one sequence; `trail` collects the residual stream after every layer run, `calls` the routers' closest calls."""
    w = {n: np.asarray(a, dtype=F) for n, a in weights.items()}
    eps = config["norm"]["eps"]
    x = first = w["embed"][np.asarray(tokens)]
    for i, _, begins in run_order(config):
        if begins:
            x = enter_pass(x, first, w)
        x = layer(x, w, i, config["layers"][i], eps, calls)
        if trail is not None:
            trail.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(config, weights, prompt, steps):
    """Greedy continuation of one prompt and the smallest top-1 / top-2 margin met, by whole passes."""
    ids, margin = list(prompt), np.inf
    for _ in range(steps):
        last = forward(config, weights, ids)[-1]
        top = np.sort(last)[-2:]
        margin = min(margin, top[1] - top[0])
        ids.append(int(last.argmax()))
    return ids[len(prompt):], margin
