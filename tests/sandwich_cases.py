"""Small sandwich-decoder configurations and seeded weights for the tests."""
from __future__ import annotations

import numpy as np

from ctorch_b200.workloads import bf16_bits, bf16_to_f32
import sandwich_oracle
from hybrid_cases import tokens, write_folder  # noqa: F401


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, identity):
    return {"kind": "moe", "router": {"experts": experts, "top": top, "identity": identity}, "expert": {"ff": ff}}


def rotating(type_, heads, kv_heads, dim, vdim, mlp, dims=None, base=10000.0, scale=None, **more):
    return {"type": type_, "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": {"base": base, "dims": dims or dim},
                                                 "scale": scale if scale is not None else dim ** -0.5, **more}}


def first(heads, kv_heads, dim, mlp, **more):
    return rotating("attention", heads, kv_heads, dim, dim, mlp, **more)


def second(heads, kv_heads, dim, vdim, mlp, softcap=20.0, **more):
    return rotating("attention_2", heads, kv_heads, dim, vdim, mlp, softcap=softcap, **more)


def pair(left, right, mlp, scales=(0.75, 1.3), scale=None):
    (heads, kv_heads, dim, vdim), (rheads, rdim, rvdim, decay) = left, right
    assert len(decay) == rheads
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale if scale is not None else dim ** -0.5},
                      "right": {"heads": rheads, "dim": rdim, "vdim": rvdim, "decay": list(decay)}, "left_scale": scales[0], "right_scale": scales[1]}}


def config(width, layers, vocab=96, eps=1e-5, buckets=61, mul_prev=31, mul_cur=7, cap=25.0):
    return {"architecture": "Lozepel", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "logit_softcap": cap,
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}}


CASES = {
    # every mixer and both feed-forwards, keys and values of different widths, partial rotation, a layer that reads another's keys
    "mixed": config(64, [first(4, 2, 16, moe(6, 2, 40, 2), dims=8), second(4, 2, 24, 16, dense(48, 1.5), base=500.0), pair((4, 1, 32, 8), (3, 24, 16, (0.5, 0.9, 0.999)), moe(5, 3, 24, 1)),
                         second(8, 2, 24, 16, moe(6, 3, 16, 3), dims=24, base=500.0, kv_from=1, softcap=4.0), first(2, 2, 32, dense(80, 0.7))], vocab=104, cap=3.0),
    # sizes equal or one
    "ones": config(16, [first(1, 1, 16, moe(1, 1, 16, 0)), second(1, 1, 16, 16, dense(16, 1.0), dims=2), pair((1, 1, 16, 16), (1, 16, 16, (1.0,)), moe(1, 2, 16, 1), scales=(1.0, 1.0))],
                   vocab=16, buckets=1, mul_prev=1, mul_cur=1, cap=1.0),
    # nothing a multiple of 8: the kernels without vector loads
    "odd": config(36, [pair((3, 3, 10, 14), (5, 9, 7, (0.1, 0.5, 0.7, 0.95, 1.0)), dense(30, 2.5)), first(6, 2, 14, moe(5, 2, 21, 2), dims=6), second(3, 1, 10, 6, dense(21, 0.9), dims=2),
                       second(6, 1, 10, 6, moe(3, 4, 13, 4), dims=2, kv_from=2, scale=0.4)], vocab=53, buckets=200, mul_prev=1009, mul_cur=3, cap=6.0),
    # layers without a feed-forward, every output of a router chosen, more identity experts than others, the same keys read twice
    "plain": config(72, [second(5, 5, 40, 72, None), second(10, 5, 40, 72, moe(2, 6, 56, 4), kv_from=0), first(2, 1, 8, None, dims=4), second(5, 5, 40, 72, dense(40, 3.0), kv_from=0, softcap=2.0)],
                    vocab=200, eps=1e-3),
    # heads past a step's tile, many experts, larger recurrent states
    "wide": config(128, [first(40, 2, 16, moe(64, 3, 64, 16)), pair((24, 1, 64, 128), (2, 130, 64, (0.8, 0.99)), moe(24, 6, 32, 8), scales=(-0.4, 2.0)), second(4, 2, 128, 64, dense(136, 2.0), base=500.0)],
                   vocab=304),
    # the larger head sizes of the tensor-core attention
    "deep": config(96, [second(2, 1, 192, 128, dense(64, 1.2), dims=32), first(2, 2, 256, moe(8, 1, 48, 1)), pair((3, 1, 72, 96), (4, 64, 128, (0.3, 0.6, 0.9, 0.97)), dense(40, 4.0))], vocab=131),
    # planes between the kernels, but head sizes and experts without vector loads; an odd vocabulary
    "uneven": config(64, [first(4, 2, 20, moe(5, 2, 21, 1), dims=6), second(4, 1, 12, 18, dense(24, 1.0), dims=6), pair((2, 1, 12, 12), (4, 10, 6, (0.2, 0.9, 0.99, 0.4)), moe(3, 1, 9, 2))], vocab=97),
}


def weight_shapes(c):
    D, V = c["width"], c["vocab"]
    shapes = {"embed": (V, D), "bigram": (c["embedding"]["bigram"]["buckets"] + 1, D), "head": (V, D), "final.norm": (D,)}

    def attention(p, m, bias, values, norms, sink, gate):
        H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        own = m.get("kv_from") is None
        shapes.update({p + "q": (H * d, D), p + "o": (D, H * e)})
        for wanted, name, shape in ((own, "k", (G * d, D)), (own and values, "v", (G * e, D)), (bias, "q.b", (H * d,)), (bias, "k.b", (G * d,)), (norms, "q.norm", (H * d,)),
                                    (norms, "k.norm", (G * d,)), (sink, "sink", (H,)), (gate, "g", (H, D))):
            if wanted:
                shapes[p + name] = shape

    for i, spec in enumerate(c["layers"]):
        p, m, mlp = f"l{i}.", spec["mixer"], spec["mlp"]
        shapes.update({p + "norm1": (D,), p + "norm1b": (D,)})
        if spec["type"] == "attention":
            attention(p + "mix.", m, True, False, False, False, True)
        elif spec["type"] == "attention_2":
            attention(p + "mix.", m, False, True, False, True, False)
        else:
            attention(p + "mix.left.", m["left"], False, True, True, True, True)
            r = m["right"]
            n, inner = r["heads"] * r["dim"], r["heads"] * r["vdim"]
            shapes.update({p + "mix.right.q": (n, D), p + "mix.right.k": (n, D), p + "mix.right.v": (inner, D), p + "mix.right.g": (inner, D), p + "mix.right.o": (D, inner),
                           p + "mix.right.norm": (inner,)})
        if not mlp:
            continue
        shapes.update({p + "norm2": (D,), p + "norm2b": (D,)})
        if mlp["kind"] == "dense":
            shapes.update({p + "mlp.gate": (mlp["ff"], D), p + "mlp.up": (mlp["ff"], D), p + "mlp.down": (D, mlp["ff"])})
        else:
            outputs = mlp["router"]["experts"] + mlp["router"]["identity"]
            for x in range(mlp["router"]["experts"]):
                shapes.update({f"{p}mlp.e{x}.gate": (mlp["expert"]["ff"], D), f"{p}mlp.e{x}.up": (mlp["expert"]["ff"], D), f"{p}mlp.e{x}.down": (D, mlp["expert"]["ff"])})
            shapes.update({p + "mlp.router": (outputs, D), p + "mlp.correction": (outputs,)})
    return shapes


def make_weights(c, seed=0):
    """bf16-representable f32 weights by name: rows of about unit gain, norm weights away from one, routers with clear choices, queries
    that tell keys apart."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in weight_shapes(c).items():
        leaf = name.split(".")[-1]
        if leaf == "sink":
            w = rng.uniform(-1.0, 2.5, shape)
        elif leaf == "correction":
            w = rng.normal(0, 0.3, shape)
        elif leaf == "b":
            w = rng.normal(0, 0.4, shape)
        elif len(shape) == 1 and (name.endswith(("q.norm", "k.norm", "right.norm"))):
            w = rng.uniform(0.6, 1.4, shape) * (2.0 if name.endswith("q.norm") else 1.0)
        elif len(shape) == 1:
            w = rng.uniform(-0.4, 0.4, shape)      # around zero: the weight is one plus it
        elif name in ("embed", "bigram"):
            w = rng.normal(0, 1.0, shape)
        else:
            w = rng.normal(0, {"router": 1.5, "g": 1.5, "gate": 1.5, "up": 1.5}.get(leaf, 1.0) / np.sqrt(shape[-1]), shape)
        out[name] = bf16_to_f32(bf16_bits(np.asarray(w, dtype=np.float32))).reshape(shape)
    return out


def decided_tokens(c, weights, count, seed=1, margin=0.004):
    """Random tokens on which no router's choice is a close call, which rounding could turn either way: the first of a few draws."""
    best, at = None, -1.0
    for draw in range(30):
        ids = tokens(c, count, seed=seed + 1000 * draw)
        calls = [np.inf]
        sandwich_oracle.forward(c, weights, ids, calls=calls)
        if min(calls) > at:
            best, at = ids, min(calls)
        if at > margin:
            break
    return best
