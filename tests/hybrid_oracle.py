"""Plain, slow statement of the hybrid decoder (Mamba-2 and latent-attention layers, Dynamic Tanh norms, looped layers,
"Ripitar") in numpy float64: one function per mechanism, one token at a time where the mechanism is a recurrence.  Shares
no code with the library.

`weights` maps state names to float arrays (bf16 weights widened); `config` is the dictionary of config.json.
"""
from __future__ import annotations

import numpy as np

F = np.float64


def silu(z):
    return z / (1.0 + np.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def rms(x, eps):
    """x over its root mean square along the last axis."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def dynamic_tanh(x, alpha, weight, bias):
    return np.tanh(alpha * x) * weight + bias


def rotate(x, positions, dims, base):
    """Interleaved rotary positions on the first `dims` entries of the last axis; x [..., T, d], positions [T]."""
    out = x.copy()
    for i in range(dims // 2):
        angle = positions * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(angle), np.sin(angle)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def short_conv(x, weight, bias):
    """Causal convolution per channel, x [T, C], weight [C, taps] (last column = current token)."""
    T, C = x.shape
    taps = weight.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, C)), x])
    out = np.zeros((T, C))
    for t in range(T):
        for j in range(taps):
            out[t] += weight[:, j] * padded[t + j]
    return out + bias


def ssm_recurrence(x, B, C, dt, A_log, D, return_state=False):
    """x [T, H, P], B and C [T, G, N], dt [T, H] (after softplus): the state-space recurrence token by token."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, P))
    y = np.zeros((T, H, P))
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.exp(-np.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return (y, S) if return_state else y


def gated_norm(y, z, weight, parts, eps):
    """Gate first, then the RMS norm of each of `parts` equal parts."""
    v = y * silu(z)
    T, inner = v.shape
    return rms(v.reshape(T, parts, inner // parts), eps).reshape(T, inner) * weight


def mamba2(h, w, prefix, m, eps):
    heads, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = heads * P
    T = h.shape[0]
    rows = h @ w[prefix + "in"].T
    z, xbc, dt = rows[:, :inner], rows[:, inner:2 * inner + 2 * G * N], rows[:, 2 * inner + 2 * G * N:]
    xbc = silu(short_conv(xbc, w[prefix + "conv"], w[prefix + "conv.b"]))
    x = xbc[:, :inner].reshape(T, heads, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    dt = softplus(dt + w[prefix + "dt_bias"])
    y = ssm_recurrence(x, B, C, dt, w[prefix + "A_log"], w[prefix + "D"]).reshape(T, inner)
    return gated_norm(y, z, w[prefix + "norm"], m["norm_groups"], eps) @ w[prefix + "o"].T


def causal_softmax_attention(q, k, v, scale):
    """q, k [H, T, d], v [H, T, e] -> [T, H, e]."""
    H, T, _ = q.shape
    out = np.zeros((T, H, v.shape[2]))
    for h in range(H):
        score = (q[h] @ k[h].T) * scale
        score[np.triu_indices(T, 1)] = -np.inf
        p = np.exp(score - score.max(axis=1, keepdims=True))
        out[:, h] = (p / p.sum(axis=1, keepdims=True)) @ v[h]
    return out


def latent_attention(h, w, prefix, m, eps):
    H, d, r, e, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    T = h.shape[0]
    positions = np.arange(T)
    cq = rms(h @ w[prefix + "dq"].T, eps) * w[prefix + "dq.norm"]
    q = (cq @ w[prefix + "uq"].T).reshape(T, H, d + r).transpose(1, 0, 2)
    down = h @ w[prefix + "dkv"].T
    c = rms(down[:, :K], eps) * w[prefix + "dkv.norm"]
    shared = rotate(down[:, K:], positions, m["rot"]["dims"], m["rot"]["base"])
    q = np.concatenate([q[..., :d], rotate(q[..., d:], positions, m["rot"]["dims"], m["rot"]["base"])], axis=-1)
    k = (c @ w[prefix + "uk"].T).reshape(T, H, d).transpose(1, 0, 2)
    k = np.concatenate([k, np.broadcast_to(shared, (H, T, r))], axis=-1)
    v = (c @ w[prefix + "uv"].T).reshape(T, H, e).transpose(1, 0, 2)
    o = causal_softmax_attention(q, k, v, m["scale"]).reshape(T, H * e)
    return (o * sigmoid(h @ w[prefix + "g"].T)) @ w[prefix + "o"].T


def dense_mlp(h, w, prefix):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def layer(x, w, i, spec, eps):
    def norm(name, value):
        return dynamic_tanh(value, w[name + ".alpha"], w[name], w[name + ".b"])
    mixer = {"mamba2": mamba2, "latent_attention": latent_attention}[spec["type"]]
    x = x + mixer(norm(f"l{i}.norm1", x), w, f"l{i}.mix.", spec["mixer"], eps)
    if spec.get("mlp") is not None:
        x = x + dense_mlp(norm(f"l{i}.norm2", x), w, f"l{i}.mlp.")
    return x


def run_order(config):
    """(layer, pass or None, first layer of a pass) in the order the layers run."""
    loop = config.get("loop") or {"start": 0, "stop": 0, "times": 0}
    order = [(i, None, False) for i in range(loop["start"])]
    for t in range(loop["times"]):
        order += [(i, t, i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return order + [(i, None, False) for i in range(loop["stop"], len(config["layers"]))]


def forward(config, weights, tokens, trail=None):
    """Logits [T, vocab] of one sequence; `trail` collects the residual stream after every layer run."""
    w = {n: np.asarray(a, dtype=F) for n, a in weights.items()}
    eps = config["norm"]["eps"]
    x = first = w["embed"][np.asarray(tokens)] * config["embedding"]["scale"]
    for i, t, begins in run_order(config):
        if begins:
            if t > 0:
                x = x + first
            x = x + w["loop.step"][t]
        x = layer(x, w, i, config["layers"][i], eps)
        if trail is not None:
            trail.append(x.copy())
    x = dynamic_tanh(x, w["final.norm.alpha"], w["final.norm"], w["final.norm.b"])
    return (x @ w["head"].T) * config["logit_scale"]


def greedy(config, weights, prompt, steps):
    """Greedy continuation of one prompt and the smallest top-1 / top-2 margin met, by whole passes."""
    ids, margin = list(prompt), np.inf
    for _ in range(steps):
        last = forward(config, weights, ids)[-1]
        top = np.sort(last)[-2:]
        margin = min(margin, top[1] - top[0])
        ids.append(int(last.argmax()))
    return ids[len(prompt):], margin
