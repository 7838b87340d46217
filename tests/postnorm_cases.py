"""Small post-norm-decoder configurations and seeded weights for the tests."""
from __future__ import annotations

import numpy as np

from ctorch_b200.workloads import bf16_bits, bf16_to_f32
import postnorm_oracle
from hybrid_cases import tokens, write_folder  # noqa: F401


def moe(experts, top, ff):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def pooled(heads, kv_heads, dim, vdim, size, pool, mlp, dims=None, base=10000.0, scale=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "pool": pool},
                                                       "rot": {"base": base, "dims": dims or dim}, "scale": scale if scale is not None else dim ** -0.5}}


def mixing(heads, kv_heads, dim, vdim, size, keep, mlp, dims=None, base=10000.0, factor=1.0, scale=None):
    return {"type": "attention_2", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size, "keep_first": keep},
                                                         "rot": {"base": base, "dims": dims or dim, "scaling": {"factor": factor}},
                                                         "scale": scale if scale is not None else dim ** -0.5}}


def delta(heads, kv_heads, dim, vdim, conv, mlp):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def config(width, layers, vocab=96, eps=1e-5, factor=0.8, weights_of=()):
    """`weights_of`: (layer, source) pairs of layers that are put in front of the given ones' places, as copies of their source."""
    layers = list(layers)
    for at, source in weights_of:
        layers.insert(at, None)
    for at, source in weights_of:
        layers[at] = {**layers[source], "weights_of": source}
    return {"architecture": "Rizovik", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "residual_mult": factor}


CASES = {
    # every mixer, keys and values of different widths, partial rotation, layers that run other layers' weights (one of them an earlier copy)
    "mixed": config(80, [delta(4, 2, 24, 16, 3, moe(6, 2, 40)), pooled(4, 2, 16, 24, 20, 4, moe(5, 3, 24), dims=8, base=500.0),
                         mixing(6, 2, 24, 16, 18, 3, moe(6, 1, 32), dims=8, base=100.0, factor=2.5), mixing(3, 3, 16, 32, 33, 10, moe(7, 2, 24), factor=1.5)],
                    vocab=104, weights_of=((3, 0), (5, 1), (6, 5))),
    # sizes equal or one
    "ones": config(16, [delta(1, 1, 16, 16, 1, moe(1, 1, 16)), pooled(1, 1, 16, 16, 1, 1, moe(1, 1, 16)), mixing(1, 1, 16, 16, 1, 1, moe(1, 1, 16))], vocab=16, factor=1.0),
    # nothing a multiple of 8: the kernels without vector loads; blocks longer than the window
    "odd": config(36, [pooled(3, 1, 10, 14, 7, 11, moe(5, 2, 21), dims=6), delta(6, 3, 9, 7, 5, moe(3, 3, 13)), mixing(3, 3, 14, 6, 5, 9, moe(4, 4, 9), dims=2, factor=3.0),
                       delta(5, 5, 7, 9, 2, None)], vocab=53, eps=0.03, factor=0.9),
    # layers without a feed-forward, every expert chosen, windows longer than most sequences, no kept tokens
    "plain": config(72, [mixing(5, 5, 40, 72, 200, 0, None), pooled(10, 5, 40, 72, 128, 64, moe(4, 4, 56)), delta(2, 1, 40, 8, 4, None), mixing(10, 5, 40, 24, 64, 70, moe(3, 3, 40), factor=8.0)],
                    vocab=200, weights_of=((4, 1),)),
    # heads past a step's tile and past the registers of the mixing kernel, many experts, larger states
    "wide": config(128, [pooled(40, 2, 16, 16, 65, 16, moe(40, 1, 64)), mixing(72, 2, 8, 8, 40, 5, moe(9, 9, 32)), delta(2, 2, 130, 64, 4, moe(12, 2, 32)), mixing(20, 1, 128, 64, 48, 2, None)],
                   vocab=304),
    # the larger head sizes of the tensor-core attention, a state beyond the narrow scan
    "deep": config(96, [mixing(2, 1, 192, 128, 30, 4, moe(8, 1, 48), dims=32), pooled(2, 2, 256, 256, 24, 5, None), delta(3, 1, 264, 128, 4, moe(6, 2, 40)), pooled(3, 1, 72, 96, 63, 2, None, dims=10)],
                   vocab=131),
    # the recurrence alone, with mixtures; then attention alone, without
    "recurrent": config(40, [delta(4, 4, 96, 16, 3, moe(2, 2, 64)), delta(9, 3, 40, 32, 4, moe(2, 1, 16))], vocab=64, weights_of=((2, 0),)),
    "attending": config(48, [pooled(2, 2, 32, 32, 12, 6, None), mixing(4, 1, 16, 16, 9, 2, None)], vocab=70),
    # planes between the kernels, but head sizes and experts without vector loads; an odd vocabulary
    "uneven": config(64, [mixing(4, 2, 20, 12, 25, 6, moe(5, 2, 21), dims=6), delta(4, 4, 10, 6, 3, moe(3, 1, 9)), pooled(4, 1, 12, 18, 31, 6, moe(6, 2, 24), dims=6)], vocab=97, factor=0.5),
}


def weight_shapes(c):
    D, V = c["width"], c["vocab"]
    shapes = {"embed": (V, D), "final.norm": (D,)}
    for i, spec in enumerate(c["layers"]):
        if spec.get("weights_of") is not None:
            continue
        p, m, mlp = f"l{i}.", spec["mixer"], spec["mlp"]
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        shapes[p + "norm1"] = (D,)
        x = p + "mix."
        if spec["type"] == "delta":
            for name, rows in (("q", G * d), ("k", G * d), ("v", H * e)):
                shapes.update({x + name: (rows, D), x + name + ".conv": (rows, m["conv"])})
            shapes.update({x + "b": (H, D), x + "A_log": (H,), x + "norm": (e,), x + "a": (H, D), x + "dt_bias": (H,), x + "g": (H * e, D), x + "o": (D, H * e)})
        else:
            whole = spec["type"] == "attention"
            shapes.update({x + "q": (H * d, D), x + "k": (G * d, D), x + "v": (G * e, D), x + "q.norm": (H * d if whole else d,), x + "k.norm": (G * d if whole else d,)})
            shapes.update({x + "g": (H * e, D)} if whole else {x + "talk": (H, H)})
            shapes[x + "o"] = (D, H * e)
        if not mlp:
            continue
        shapes[p + "norm2"] = (D,)
        E, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
        for k in range(E):
            shapes.update({f"{p}mlp.e{k}.gate": (ff, D), f"{p}mlp.e{k}.up": (ff, D), f"{p}mlp.e{k}.down": (D, ff)})
        shapes.update({p + "mlp.router": (E, D), p + "mlp.router.b": (E,)})
    return shapes


def make_weights(c, seed=0):
    """bf16-representable f32 weights by name: rows of about unit gain, norm weights away from one, routers with clear choices, decays
    that remember."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in weight_shapes(c).items():
        leaf = name.split(".")[-1]
        if leaf == "A_log":
            w = rng.uniform(-3.0, 0.5, shape)
        elif leaf == "dt_bias":
            w = rng.uniform(-3.0, 0.5, shape)
        elif leaf == "b" and len(shape) == 1:
            w = rng.normal(0, 0.8, shape)
        elif leaf == "talk":
            w = np.eye(shape[0]) * rng.uniform(0.5, 1.0, shape[0]) + rng.normal(0, 0.5 / np.sqrt(shape[0]), shape)
        elif leaf == "conv":
            w = rng.normal(0, 0.7, shape)
        elif len(shape) == 1:
            w = rng.uniform(0.6, 1.4, shape)
        elif name == "embed":
            w = rng.normal(0, 1.0, shape)
        else:
            w = rng.normal(0, {"router": 1.5, "g": 1.5, "gate": 1.5, "up": 1.5}.get(leaf, 1.0) / np.sqrt(shape[-1]), shape)
        out[name] = bf16_to_f32(bf16_bits(np.asarray(w, dtype=np.float32))).reshape(shape)
    return out


def decided_tokens(c, weights, count, seed=1, margin=0.06):
    """Random tokens on which no router's choice is a close call, which rounding could turn either way: the first of a few draws."""
    best, at = None, -1.0
    for draw in range(40):
        ids = tokens(c, count, seed=seed + 1000 * draw)
        calls = [np.inf]
        postnorm_oracle.forward(c, weights, ids, calls=calls)
        if min(calls) > at:
            best, at = ids, min(calls)
        if at > margin:
            break
    return best
