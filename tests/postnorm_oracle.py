"""Plain, slow statement of the post-norm decoder ("Rizovik"): sublayers that read the residual stream itself and whose results are normed
before they are added; attention over a window of tokens and pooled blocks before it, attention over a window and the first tokens with
mixed head weights, the gated delta rule, a mixture of gated experts under a router with biased logits, tied embeddings.  numpy float64,
one function per mechanism, the recurrence one token at a time.  Shares no code with the library.

`weights` maps state names to float arrays (bf16 weights widened); `config` is the dictionary of config.json.
"""
from __future__ import annotations

import numpy as np

from hybrid_oracle import rms, sigmoid, silu, softplus

F = np.float64


def rotate_halves(x, positions, dims, base, factor=1.0):
    """Entry i with entry i + dims / 2 of the last axis by the angle position * base^(-2i/dims) / factor; x [..., T, d]."""
    out = x.copy()
    for i in range(dims // 2):
        angle = positions * (float(base) ** (-2.0 * i / dims) / factor)
        c, s = np.cos(angle), np.sin(angle)
        u, v = x[..., i], x[..., i + dims // 2]
        out[..., i] = u * c - v * s
        out[..., i + dims // 2] = v * c + u * s
    return out


def heads_of(x, heads):
    return x.reshape(x.shape[0], heads, -1).transpose(1, 0, 2)


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def seen_tokens(T, size, keep):
    """[i, j]: whether position i sees token j - the last `size` up to itself, and the sequence's first `keep`."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep))


def seen_blocks(T, size, pool):
    """[i, b]: whether position i sees the pooled block b: its last token lies before the window."""
    i, b = np.arange(T)[:, None], np.arange(T // pool)[None, :]
    return b * pool + pool - 1 <= i - size


def block_means(x, pool):
    """[..., T, d] -> [..., T // pool, d]: the mean of every complete block."""
    n = x.shape[-2] // pool
    return x[..., :n * pool, :].reshape(*x.shape[:-2], n, pool, x.shape[-1]).mean(axis=-2)


def pooled_window_weights(q, k, scale, size, pool):
    """q [H, T, d], k [G, T, d] -> softmax weights [H, T, T + blocks] over tokens and blocks together."""
    H, T, _ = q.shape
    group = H // k.shape[0]
    keys = np.concatenate([k, block_means(k, pool)], axis=1)
    seen = np.concatenate([seen_tokens(T, size, 0), seen_blocks(T, size, pool)], axis=1)
    return softmax(np.where(seen, np.einsum("htd,hjd->htj", q, np.repeat(keys, group, axis=0)) * scale, -np.inf))


def attention_pooled(h, w, p, m, eps):
    """Norms over the whole projections, rotation, normed values, window and pooled blocks, a gate per value."""
    T, H, G, pos = h.shape[0], m["heads"], m["kv_heads"], np.arange(h.shape[0])
    turn = lambda x: rotate_halves(x, pos, m["rot"]["dims"], m["rot"]["base"])
    q = turn(heads_of(rms(h @ w[p + "q"].T, eps) * w[p + "q.norm"], H))
    k = turn(heads_of(rms(h @ w[p + "k"].T, eps) * w[p + "k.norm"], G))
    v = rms(heads_of(h @ w[p + "v"].T, G), eps)
    weights = pooled_window_weights(q, k, m["scale"], m["mask"]["size"], m["mask"]["pool"])
    values = np.concatenate([v, block_means(v, m["mask"]["pool"])], axis=1)
    o = np.einsum("htj,hje->the", weights, np.repeat(values, H // G, axis=0)).reshape(T, -1)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def mixed_heads(weights, talk):
    """weights [H, T, J] -> sum over g of talk[h, g] weights[g]."""
    return np.einsum("hg,gtj->htj", talk, weights)


def attention_mixed(h, w, p, m, eps):
    """Weighted norms per head, rotation with stretched positions, window and first tokens, softmax weights mixed over the heads."""
    T, H, G, pos = h.shape[0], m["heads"], m["kv_heads"], np.arange(h.shape[0])
    turn = lambda x: rotate_halves(x, pos, m["rot"]["dims"], m["rot"]["base"], m["rot"]["scaling"]["factor"])
    q = turn(rms(heads_of(h @ w[p + "q"].T, H), eps) * w[p + "q.norm"])
    k = turn(rms(heads_of(h @ w[p + "k"].T, G), eps) * w[p + "k.norm"])
    v = heads_of(h @ w[p + "v"].T, G)
    group = H // G
    score = np.einsum("htd,hjd->htj", q, np.repeat(k, group, axis=0)) * m["scale"]
    weights = softmax(np.where(seen_tokens(T, m["mask"]["size"], m["mask"]["keep_first"]), score, -np.inf))
    o = np.einsum("htj,hje->the", mixed_heads(weights, w[p + "talk"]), np.repeat(v, group, axis=0))
    return o.reshape(T, -1) @ w[p + "o"].T


def short_conv(x, weight):
    """Causal convolution per channel, x [T, C], weight [C, taps] (last column: the current token), then SiLU."""
    T, C = x.shape
    taps = weight.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, C)), x])
    return silu(sum(weight[:, j] * padded[j:j + T] for j in range(taps)))


def unit(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, beta, g):
    """q, k [T, H, d] (one per value head), v [T, H, e], beta and g [T, H]; token by token.  Returns the read-outs and the last state."""
    T, H, d = q.shape
    S = np.zeros((H, d, v.shape[2]))
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] = S[h] + np.outer(k[t, h], u)
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def delta(h, w, p, m, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    part = lambda name: short_conv(h @ w[p + name].T, w[p + name + ".conv"]).reshape(T, -1, e if name == "v" else d)
    q = np.repeat(unit(part("q")) * d ** -0.5, H // G, axis=1)
    k = np.repeat(unit(part("k")), H // G, axis=1)
    beta = sigmoid(h @ w[p + "b"].T)
    g = np.exp(-np.exp(w[p + "A_log"]) * softplus(h @ w[p + "a"].T + w[p + "dt_bias"]))
    o, _ = delta_rule(q, k, part("v"), beta, g)
    o = rms(o, eps) * w[p + "norm"] * silu(h @ w[p + "g"].T).reshape(T, H, e)
    return o.reshape(T, -1) @ w[p + "o"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(logits, top):
    """Chosen experts [T, top] by falling logit, and the softmax over the chosen ones' logits."""
    chosen = np.argsort(-logits, axis=1, kind="stable")[:, :top]
    return chosen, softmax(np.take_along_axis(logits, chosen, axis=1))


def closest_call(logits, top):
    """Smallest distance, over the tokens, between the logits of the last expert chosen and the first one not chosen."""
    z = np.sort(logits, axis=1)[:, ::-1]
    return float((z[:, top - 1] - z[:, top]).min()) if z.shape[1] > top else np.inf


def mixture(h, w, p, mlp, calls=None):
    logits = h @ w[p + "router"].T + w[p + "router.b"]
    top = mlp["router"]["top"]
    chosen, score = route(logits, top)
    if calls is not None:
        calls.append(closest_call(logits, top))
    out = np.zeros_like(h)
    for e in np.unique(chosen):
        t, slot = np.nonzero(chosen == e)
        out[t] += score[t, slot][:, None] * expert(h[t], w, f"{p}e{e}.")
    return out


def mixer(h, w, p, spec, eps):
    form = {"attention": attention_pooled, "attention_2": attention_mixed, "delta": delta}[spec["type"]]
    return form(h, w, p + "mix.", spec["mixer"], eps)


def layer(x, w, i, config, calls=None):
    spec, eps, m = config["layers"][i], config["norm"]["eps"], config["residual_mult"]
    while spec.get("weights_of") is not None:
        i = spec["weights_of"]
        spec = config["layers"][i]
    p = f"l{i}."
    x = x + m * rms(mixer(x, w, p, spec, eps), eps) * w[p + "norm1"]
    if spec.get("mlp"):
        x = x + m * rms(mixture(x, w, p + "mlp.", spec["mlp"], calls), eps) * w[p + "norm2"]
    return x


def forward(config, weights, tokens, trail=None, calls=None):
    """Logits [T, vocab] of one sequence; `trail` collects the residual stream after every layer, `calls` the routers' closest calls."""
    w = {n: np.asarray(a, dtype=F) for n, a in weights.items()}
    x = w["embed"][np.asarray(tokens)]
    for i in range(len(config["layers"])):
        x = layer(x, w, i, config, calls)
        if trail is not None:
            trail.append(x.copy())
    return (rms(x, config["norm"]["eps"]) * w["final.norm"]) @ w["embed"].T


def greedy(config, weights, prompt, steps):
    """Greedy continuation of one prompt and the smallest top-1 / top-2 margin met, by whole passes."""
    ids, margin = list(prompt), np.inf
    for _ in range(steps):
        last = forward(config, weights, ids)[-1]
        top = np.sort(last)[-2:]
        margin = min(margin, top[1] - top[0])
        ids.append(int(last.argmax()))
    return ids[len(prompt):], margin
