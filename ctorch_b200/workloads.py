"""Seeded synthetic decoder workloads: shapes, weights and prompts.

The five shapes are the benchmark configurations of the decoder token loop.  No dataset or checkpoint is
involved: weights are N(0, 0.02) from a fixed numpy seed (RMSNorm weights 1 + small noise so that the norm
weight product is exercised), prompts are uniform random token ids.  bf16 tensors travel as uint16 bit
patterns (round-to-nearest-even of the f32 draw), which is how every consumer here takes them.
"""
from __future__ import annotations

import numpy as np

CONFIGS = {
    # byte-level decoder the reference can run on a CPU in seconds
    "c1": dict(vocab=256, d_model=256, layers=4, heads=8, kv_heads=2, hidden=688, dtype="f32",
               batch=1, prompt=64, steps=128),
    # small GQA decoder, the single-GPU benchmark workload
    "c2": dict(vocab=32000, d_model=768, layers=12, heads=12, kv_heads=4, hidden=2048, dtype="bf16",
               batch=16, prompt=512, steps=256),
    # decode-attention microbenchmark (attention only)
    "c3": dict(batch=64, heads=32, kv_heads=8, head_dim=128, min_context=1024, max_context=32768, dtype="bf16"),
    # 1B-shape decoder, batch sharded over GPUs by sequence
    "c4": dict(vocab=32000, d_model=2048, layers=16, heads=32, kv_heads=8, hidden=8192, dtype="bf16",
               batch=256, prompt=1024, steps=512),
    # 8B-shape decoder with rank-16 adapters on q and v, KV-head tensor parallel
    "c5": dict(vocab=128256, d_model=4096, layers=32, heads=32, kv_heads=8, hidden=14336, dtype="bf16",
               batch=32, prompt=4096, steps=256, lora_rank=16, lora_alpha=32.0),
}
for _c in CONFIGS.values():
    if "prompt" in _c:
        _c.setdefault("context", _c["prompt"] + _c["steps"])
        _c.setdefault("tied", True)
        _c.setdefault("eps", 1e-5)
        _c.setdefault("rope_base", 10000.0)


def tiny(dtype: str = "f32", **overrides) -> dict:
    """A decoder small enough for exhaustive CPU comparison (the shape of the reference's own state test)."""
    spec = dict(vocab=97, d_model=64, layers=2, heads=4, kv_heads=2, hidden=96, dtype=dtype, batch=2,
                prompt=6, steps=5, context=24, tied=True, eps=1e-5, rope_base=10000.0)
    spec.update(overrides)
    return spec


def bf16_bits(values: np.ndarray) -> np.ndarray:
    """float32 -> bf16 bit patterns, round to nearest even."""
    u = np.ascontiguousarray(values, dtype=np.float32).view(np.uint32)
    return ((u + np.uint32(0x7FFF) + ((u >> np.uint32(16)) & np.uint32(1))) >> np.uint32(16)).astype(np.uint16)


def bf16_to_f32(bits: np.ndarray) -> np.ndarray:
    return (np.ascontiguousarray(bits, dtype=np.uint16).astype(np.uint32) << np.uint32(16)).view(np.float32)


def tensor_shapes(spec: dict) -> list[tuple[str, tuple[int, ...]]]:
    """(state name, shape) in the canonical order every implementation here consumes."""
    D, F = spec["d_model"], spec["hidden"]
    kv = spec["kv_heads"] * (D // spec["heads"])
    out = [("tokens.weight", (spec["vocab"], D))]
    for i in range(spec["layers"]):
        p = f"decoder.layer{i}."
        out += [(p + "attention.query.weight", (D, D)), (p + "attention.key.weight", (kv, D)),
                (p + "attention.value.weight", (kv, D)), (p + "attention.output.weight", (D, D)),
                (p + "feedforward.gate.weight", (F, D)), (p + "feedforward.up.weight", (F, D)),
                (p + "feedforward.down.weight", (D, F)), (p + "attention_norm.weight", (D,)),
                (p + "feedforward_norm.weight", (D,))]
    out.append(("decoder.normalization.weight", (D,)))
    if not spec.get("tied", True):
        out.append(("output.weight", (spec["vocab"], D)))
    return out


def make_weights(spec: dict, seed: int = 1234, scale: float = 0.02, threads: int | None = None) -> list[np.ndarray]:
    """Ordered tensors in the model dtype (float32 arrays, or uint16 bf16 bit patterns).  Every tensor has its own
    generator seeded by (seed, index), so the draws do not depend on how many worker threads make them."""
    def one(item):
        index, (name, shape) = item
        rng = np.random.default_rng([seed, index])
        if name.endswith("norm.weight") or name.endswith("normalization.weight"):
            w = (1.0 + 0.1 * rng.standard_normal(shape)).astype(np.float32)
        else:
            w = rng.standard_normal(shape, dtype=np.float32)
            w *= np.float32(scale)
        return bf16_bits(w) if spec["dtype"] == "bf16" else w

    items = list(enumerate(tensor_shapes(spec)))
    if threads is None:
        import os
        threads = min(16, len(os.sched_getaffinity(0)) if hasattr(os, "sched_getaffinity") else (os.cpu_count() or 1))
    if threads <= 1 or len(items) < 4:
        return [one(item) for item in items]
    from concurrent.futures import ThreadPoolExecutor
    with ThreadPoolExecutor(max_workers=threads) as pool:   # numpy releases the GIL inside the generators
        return list(pool.map(one, items))


def make_lora(spec: dict, seed: int = 4321) -> list[np.ndarray] | None:
    """Per layer: q.down [r,D], q.up [D,r], v.down [r,D], v.up [kv,r].  `up` is non-zero on purpose (the
    reference initialises it to zero, which would make the adapter a no-op)."""
    r = spec.get("lora_rank", 0)
    if not r:
        return None
    D = spec["d_model"]
    kv = spec["kv_heads"] * (D // spec["heads"])
    out = []
    for i in range(spec["layers"]):
        for j, shape in enumerate([(r, D), (D, r), (r, D), (kv, r)]):
            rng = np.random.default_rng([seed, i, j])
            w = (0.05 * rng.standard_normal(shape, dtype=np.float32)).astype(np.float32)
            out.append(bf16_bits(w) if spec["dtype"] == "bf16" else w)
    return out


def make_prompts(spec: dict, batch: int | None = None, length: int | None = None, seed: int = 99) -> np.ndarray:
    batch = spec["batch"] if batch is None else batch
    length = spec["prompt"] if length is None else length
    rng = np.random.default_rng([seed, batch, length])
    return rng.integers(0, spec["vocab"], size=(batch, length), dtype=np.int64)


def weight_bytes(spec: dict) -> int:
    """Bytes of weights one decode step must read (tied table counted once)."""
    size = 2 if spec["dtype"] == "bf16" else 4
    return sum(int(np.prod(shape)) for _, shape in tensor_shapes(spec)) * size


def kv_bytes_per_token(spec: dict, kv_dtype: str) -> int:
    """Bytes of K and V one cached position holds across all layers, per sequence."""
    hd = spec["d_model"] // spec["heads"]
    return 2 * spec["layers"] * spec["kv_heads"] * hd * (2 if kv_dtype == "bf16" else 4)


def hybrid_config(width: int, layers: int, ff: int, heads: int, ssm_heads: int, loop: tuple[int, int, int] | None = None,
                  vocab: int = 32000) -> dict:
    """Hybrid decoder of a real model's layer sizes: state-space and latent-attention layers in turn, each with a feed-forward."""
    ssm = {"type": "mamba2", "mixer": {"heads": ssm_heads, "vdim": 64, "state": 128, "groups": 8, "conv": 4, "norm_groups": 8},
           "mlp": {"kind": "dense", "ff": ff}}
    latent = {"type": "latent_attention",
              "mixer": {"heads": heads, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "q_rank": 768, "scale": 192 ** -0.5,
                        "rot": {"dims": 64, "base": 10000.0}},
              "mlp": {"kind": "dense", "ff": ff}}
    config = {"architecture": "Ripitar", "vocab": vocab, "width": width, "layers": [(ssm, latent)[i % 2] for i in range(layers)],
              "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0}, "logit_scale": 1.0}
    if loop:
        config["loop"] = dict(zip(("start", "stop", "times"), loop))
    return config


def parallel_config(width: int, layers: int, ff: int, heads: int, kv_heads: int, experts: int, top: int = 2, chunk: int = 2048,
                    loop: tuple[int, int, int] | None = None, vocab: int = 32000) -> dict:
    """Parallel decoder of a real model's layer sizes: dense and mixture layers in turn; `top` experts and the shared one have the dense
    feed-forward's active weights (two matrices of width * ff_expert each against three of width * ff)."""
    expert = 3 * ff // (2 * (top + 1))
    dim = width // heads
    mixer = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": chunk}, "rot": {"dims": dim, "base": 500000.0},
             "scale": dim ** -0.5}
    mlps = ({"kind": "dense", "ff": ff},
            {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": expert}, "shared": {"ff": expert}})
    config = {"architecture": "Sinezen", "vocab": vocab, "width": width,
              "layers": [{"type": "attention", "mixer": mixer, "mlp": mlps[i % 2]} for i in range(layers)], "norm": {"eps": 1e-5}}
    if loop:
        config["loop"] = dict(zip(("start", "stop", "times"), loop))
    return config


def sandwich_config(width: int, layers: int, ff: int, heads: int, kv_heads: int, experts: int, lightning_heads: int, top: int = 2, identity: int = 2,
                    vocab: int = 32000) -> dict:
    """Sandwich decoder of a real model's layer sizes: its three mixers in turn, the second kind of attention twice (the second time with the
    first's keys); dense and mixture layers in turn, `top` experts with the dense feed-forward's weights."""
    dim = width // heads
    rot = {"dims": dim, "base": 100000.0}
    sizes = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5}
    mlps = ({"kind": "dense", "ff": ff, "limit": 7.0},
            {"kind": "moe", "router": {"experts": experts, "top": top, "identity": identity}, "expert": {"ff": ff // top}})
    decay = [float(1.0 - 2.0 ** -(1 + 8.0 * h / lightning_heads)) for h in range(lightning_heads)]
    mixers = (("attention", {**sizes, "rot": rot}), ("attention_2", {**sizes, "rot": rot, "softcap": 40.0}),
              ("parallel", {"left": sizes, "right": {"heads": lightning_heads, "dim": 128, "vdim": 128, "decay": decay}, "left_scale": 0.8, "right_scale": 0.4}),
              ("attention_2", {**sizes, "rot": rot, "softcap": 40.0}))
    config = {"architecture": "Lozepel", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "logit_softcap": 20.0, "layers": [],
              "embedding": {"bigram": {"buckets": vocab - 1, "mul_prev": 1021, "mul_cur": 31}}}
    for i in range(layers):
        kind, mixer = mixers[i % 4]
        config["layers"].append({"type": kind, "mixer": {**mixer, "kv_from": i - 2} if i % 4 == 3 else mixer, "mlp": mlps[i % 2]})
    return config


def postnorm_config(width: int, layers: int, ff: int, heads: int, kv_heads: int, experts: int, delta_heads: int, top: int = 2, window: int = 512, pool: int = 16,
                    keep: int = 8, vocab: int = 32000) -> dict:
    """Post-norm decoder of a real model's layer sizes: the delta rule, the window with pooled blocks and the window with mixed heads in turn, a
    mixture behind each of them, `top` experts with a dense feed-forward's weights."""
    dim = width // heads
    sizes = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": dim ** -0.5}
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff // top}}
    mixers = (("delta", {"heads": delta_heads, "kv_heads": delta_heads // 2, "dim": 128, "vdim": 128, "conv": 4}),
              ("attention", {**sizes, "mask": {"size": window, "pool": pool}, "rot": {"base": 500000.0, "dims": dim // 2}}),
              ("attention_2", {**sizes, "mask": {"size": window, "keep_first": keep}, "rot": {"base": 10000.0, "dims": dim // 2, "scaling": {"factor": 8.0}}}))
    return {"architecture": "Rizovik", "vocab": vocab, "width": width, "norm": {"eps": 1e-5}, "residual_mult": 0.8,
            "layers": [{"type": mixers[i % 3][0], "mixer": mixers[i % 3][1], "mlp": mlp} for i in range(layers)]}


def transformer_config(width: int, layers: int, ff: int, heads: int, kv_heads: int, context: int, vocab: int = 32000) -> dict:
    return {"architecture": "TransformerDecoder", "vocab": vocab, "layers": layers, "width": width, "heads": heads, "kv_heads": kv_heads,
            "ff": ff, "context": context, "tied": 1}


# (hybrid, grouped-query) arguments of equal width, feed-forward width and number of layer runs
HYBRID_SIZES = {
    "1k": (dict(width=1024, layers=12, ff=4096, heads=8, ssm_heads=32), dict(width=1024, layers=12, ff=4096, heads=16, kv_heads=4)),
    "2k": (dict(width=2048, layers=12, ff=8192, heads=16, ssm_heads=64, loop=(4, 8, 2)), dict(width=2048, layers=16, ff=8192, heads=32, kv_heads=8)),
    "4k": (dict(width=4096, layers=8, ff=14336, heads=32, ssm_heads=128), dict(width=4096, layers=8, ff=14336, heads=32, kv_heads=8)),
}

# (parallel, grouped-query) arguments, likewise
PARALLEL_SIZES = {
    "1k": (dict(width=1024, layers=12, ff=4096, heads=16, kv_heads=4, experts=16), HYBRID_SIZES["1k"][1]),
    "2k": (dict(width=2048, layers=12, ff=8192, heads=32, kv_heads=8, experts=16, loop=(4, 8, 2)), HYBRID_SIZES["2k"][1]),
    "4k": (dict(width=4096, layers=8, ff=14336, heads=32, kv_heads=8, experts=8), HYBRID_SIZES["4k"][1]),
}

# (sandwich, grouped-query) arguments, likewise
SANDWICH_SIZES = {
    "1k": (dict(width=1024, layers=12, ff=4096, heads=16, kv_heads=4, experts=16, lightning_heads=8), HYBRID_SIZES["1k"][1]),
    "2k": (dict(width=2048, layers=16, ff=8192, heads=32, kv_heads=8, experts=16, lightning_heads=16), HYBRID_SIZES["2k"][1]),
    "4k": (dict(width=4096, layers=8, ff=14336, heads=32, kv_heads=8, experts=8, lightning_heads=32), HYBRID_SIZES["4k"][1]),
}

# (post-norm, sandwich) arguments: the closest design, of equal width, heads, layers and experts
POSTNORM_SIZES = {
    "1k": (dict(width=1024, layers=12, ff=4096, heads=16, kv_heads=4, experts=16, delta_heads=8), SANDWICH_SIZES["1k"][0]),
    "2k": (dict(width=2048, layers=16, ff=8192, heads=32, kv_heads=8, experts=16, delta_heads=16), SANDWICH_SIZES["2k"][0]),
    "4k": (dict(width=4096, layers=8, ff=14336, heads=32, kv_heads=8, experts=8, delta_heads=32), SANDWICH_SIZES["4k"][0]),
}


def random_state(shapes: dict[str, tuple[int, ...]], seed: int = 7) -> dict[str, np.ndarray]:
    """bf16 bit patterns for every named shape, cut from one seeded block (norm-like vectors around 1)."""
    block = np.random.default_rng(seed).standard_normal(1 << 22, dtype=np.float32)
    out = {}
    for i, (name, shape) in enumerate(shapes.items()):
        count = int(np.prod(shape)) if shape else 1
        values = np.resize(block[i * 9973 % 65536:], count).reshape(shape)
        if len(shape) == 2:
            values = values * np.float32(shape[1] ** -0.5)
        elif name.endswith("correction"):   # the scores decide, so that the experts share the rows
            values = 0.002 * values
        elif not name.endswith((".b", "A_log", "dt_bias")):
            values = 1.0 + 0.05 * values
        else:
            values = 0.2 * values
        out[name] = bf16_bits(values).reshape(shape)
    return out
