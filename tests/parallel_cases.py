"""Small parallel-decoder configurations and seeded weights for the tests."""
from __future__ import annotations

import numpy as np

from ctorch_b200.workloads import bf16_bits, bf16_to_f32
import parallel_oracle
from hybrid_cases import tokens, write_folder  # noqa: F401


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}, "shared": {"ff": shared} if shared else None}


def layer(heads, kv_heads, dim, vdim, size, mlp, dims=None, base=10000.0, scale=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
                      "rot": {"base": base, "dims": dims or dim}, "scale": scale if scale is not None else dim ** -0.5}}


def config(width, layers, loop=None, vocab=96, eps=1e-5):
    c = {"architecture": "Sinezen", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CASES = {
    # both feed-forwards, grouped heads, partial rotation, chunks of different sizes in one model, a loop in the middle
    "mixed": config(64, [layer(4, 2, 16, 24, 16, dense(48), dims=8), layer(6, 3, 24, 16, 7, moe(6, 2, 40, 24), base=100.0),
                         layer(4, 1, 32, 8, 33, dense(80), scale=0.3)], loop=(1, 2, 3), vocab=104),
    # sizes equal or one, a loop over everything, one expert, chunks of one position
    "ones": config(16, [layer(1, 1, 16, 16, 1, moe(1, 1, 16, 16)), layer(1, 1, 16, 16, 2, dense(16))], loop=(0, 2, 1), vocab=16),
    # nothing a multiple of 8: the kernels without vector loads
    "odd": config(36, [layer(3, 3, 10, 14, 5, moe(5, 3, 21, 13), dims=6), layer(6, 2, 14, 10, 20, dense(30), dims=2)], loop=(0, 1, 2), vocab=53),
    # every expert chosen, no shared expert, a layer without a feed-forward, no loop
    "plain": config(72, [layer(5, 5, 40, 72, 11, moe(4, 4, 56, 0)), layer(2, 1, 8, 8, 64, None, dims=4)], vocab=200, eps=1e-3),
    # heads larger than a step's tile, many experts, a chunk longer than every test's sequence
    "wide": config(128, [layer(40, 2, 16, 16, 4096, moe(64, 2, 64, 72)), layer(4, 2, 64, 128, 65, dense(136), base=500.0),
                         layer(2, 2, 128, 64, 130, moe(24, 6, 32, 8))], loop=(2, 3, 2), vocab=304),
    # the larger head sizes of the tensor-core attention
    "deep": config(96, [layer(2, 1, 192, 128, 48, dense(64), dims=32), layer(2, 2, 256, 200, 100, moe(8, 1, 48, 16)), layer(3, 1, 72, 96, 31, dense(40))],
                   vocab=131),
    # planes between the kernels, but head sizes and experts without vector loads; an odd vocabulary
    "uneven": config(64, [layer(3, 1, 12, 8, 9, moe(5, 2, 21, 16), dims=6), layer(4, 2, 20, 18, 14, dense(24)), layer(2, 2, 16, 12, 6, moe(3, 1, 9, 8))],
                     loop=(0, 1, 2), vocab=97),
}


def weight_shapes(c):
    D, V = c["width"], c["vocab"]
    shapes = {"embed": (V, D), "head": (V, D), "final.norm": (D,)}
    for i, spec in enumerate(c["layers"]):
        p, m, mlp = f"l{i}.", spec["mixer"], spec["mlp"]
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        shapes.update({p + "norm1": (D,), p + "mix.q": (H * d, D), p + "mix.k": (G * d, D), p + "mix.v": (G * e, D), p + "mix.q.norm": (H * d,),
                       p + "mix.k.norm": (G * d,), p + "mix.g": (H, D), p + "mix.o": (D, H * e)})
        if mlp and mlp["kind"] == "dense":
            shapes.update({p + "mlp.gate": (mlp["ff"], D), p + "mlp.up": (mlp["ff"], D), p + "mlp.down": (D, mlp["ff"])})
        elif mlp:
            for x in range(mlp["router"]["experts"]):
                shapes.update({f"{p}mlp.e{x}.up": (mlp["expert"]["ff"], D), f"{p}mlp.e{x}.down": (D, mlp["expert"]["ff"])})
            shapes[p + "mlp.router"] = (mlp["router"]["experts"], D)
            if mlp["shared"]:
                shapes.update({p + "mlp.shared.up": (mlp["shared"]["ff"], D), p + "mlp.shared.down": (D, mlp["shared"]["ff"])})
    if c.get("loop"):
        shapes["loop.in"] = (D, 2 * D)
    return shapes


def make_weights(c, seed=0):
    """bf16-representable f32 weights by name: rows of about unit gain, norm weights away from one, routers with clear choices, queries
    that tell keys apart."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in weight_shapes(c).items():
        leaf = name.split(".")[-1]
        if len(shape) == 1:
            w = rng.uniform(0.6, 1.4, shape) * (2.0 if name.endswith("q.norm") else 1.0)
        elif name == "embed":
            w = rng.normal(0, 1.0, shape)
        else:
            w = rng.normal(0, {"router": 2.5, "g": 1.5, "down": 1.5, "up": 1.5}.get(leaf, 1.0) / np.sqrt(shape[-1]), shape)
        out[name] = bf16_to_f32(bf16_bits(np.asarray(w, dtype=np.float32))).reshape(shape)
    return out


def decided_tokens(c, weights, count, seed=1, margin=0.008):
    """Random tokens on which no router's choice is a close call, which rounding could turn either way: the first of a few draws."""
    best, at = None, -1.0
    for draw in range(30):
        ids = tokens(c, count, seed=seed + 1000 * draw)
        calls = [np.inf]
        parallel_oracle.forward(c, weights, ids, calls=calls)
        if min(calls) > at:
            best, at = ids, min(calls)
        if at > margin:
            break
    return best
