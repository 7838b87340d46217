"""Small hybrid-decoder configurations and seeded weights for the tests; files in the layout the loader reads."""
from __future__ import annotations

import json
import os
import struct

import numpy as np

from ctorch_b200.workloads import bf16_bits, bf16_to_f32


def mamba(heads, vdim, state, groups, conv, norm_groups, ff=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, ff=None, base=10000.0, dims=None, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "scale": scale if scale is not None else (dim + rot_dim) ** -0.5, "rot": {"dims": dims or rot_dim, "base": base}},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, layers, loop=None, vocab=96, eps=1e-5, embed=3.0, logit=1.5):
    c = {"architecture": "Ripitar", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "embedding": {"scale": embed},
         "logit_scale": logit}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


CASES = {
    # every kind of layer with and without a feed-forward, a loop in the middle
    "mixed": config(64, [latent(4, 16, 8, 24, 32, 40), mamba(4, 16, 24, 2, 4, 4, ff=48), latent(4, 16, 8, 24, 32, 40, ff=56), mamba(6, 8, 16, 3, 3, 2)],
                    loop=(1, 3, 2), vocab=101),
    # sizes equal or one, no loop
    "ones": config(16, [mamba(1, 16, 16, 1, 1, 1), latent(1, 16, 16, 16, 16, 16, ff=16)], vocab=16, embed=1.0, logit=1.0),
    # nothing a multiple of 8: the kernels without vector loads
    "odd": config(36, [mamba(3, 10, 7, 1, 5, 3, ff=30), latent(3, 10, 6, 14, 22, 13, ff=21, dims=4)], loop=(0, 1, 3), vocab=53),
    # more heads than a 16-row tile, groups = heads, loop over everything with one pass
    "wide": config(72, [latent(20, 24, 16, 16, 144, 48), mamba(8, 12, 100, 8, 2, 1, ff=80)], loop=(0, 2, 1), vocab=200, eps=1e-3),
    # the largest latent the tensor-core attention takes, a state of 200, loop at the end
    "large": config(128, [mamba(2, 64, 128, 1, 4, 2), mamba(2, 36, 200, 2, 4, 1), latent(16, 32, 64, 40, 512, 96, ff=136, base=500.0)],
                    loop=(1, 3, 2), vocab=300),
    # heads beyond a 32-row tile, a latent between the kernel's sizes
    "heads": config(80, [latent(40, 8, 24, 8, 200, 24, scale=0.3), latent(33, 16, 32, 8, 264, 32, ff=64)], loop=(1, 2, 2), vocab=128),
}


def weight_shapes(c):
    D, V = c["width"], c["vocab"]
    shapes = {"embed": (V, D), "head": (V, D)}

    def norm(name):
        shapes.update({name: (D,), name + ".b": (D,), name + ".alpha": ()})
    for i, layer in enumerate(c["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        norm(p + "norm1")
        if layer["type"] == "mamba2":
            inner, gn = m["heads"] * m["vdim"], m["groups"] * m["state"]
            shapes.update({p + "mix.in": (2 * inner + 2 * gn + m["heads"], D), p + "mix.conv": (inner + 2 * gn, m["conv"]),
                           p + "mix.conv.b": (inner + 2 * gn,), p + "mix.dt_bias": (m["heads"],), p + "mix.A_log": (m["heads"],),
                           p + "mix.D": (m["heads"],), p + "mix.norm": (inner,), p + "mix.o": (D, inner)})
        else:
            H = m["heads"]
            shapes.update({p + "mix.dq": (m["q_rank"], D), p + "mix.dq.norm": (m["q_rank"],),
                           p + "mix.uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]), p + "mix.dkv": (m["kv_rank"] + m["rot_dim"], D),
                           p + "mix.dkv.norm": (m["kv_rank"],), p + "mix.uk": (H * m["dim"], m["kv_rank"]),
                           p + "mix.uv": (H * m["vdim"], m["kv_rank"]), p + "mix.g": (H * m["vdim"], D), p + "mix.o": (D, H * m["vdim"])})
        if layer["mlp"]:
            norm(p + "norm2")
            ff = layer["mlp"]["ff"]
            shapes.update({p + "mlp.gate": (ff, D), p + "mlp.up": (ff, D), p + "mlp.down": (D, ff)})
    norm("final.norm")
    if c.get("loop"):
        shapes["loop.step"] = (c["loop"]["times"], D)
    return shapes


def make_weights(c, seed=0):
    """bf16-representable f32 weights by name: rows of about unit gain, parameters away from their neutral values."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in weight_shapes(c).items():
        leaf = name.split(".")[-1]
        if leaf == "alpha":
            w = np.asarray(rng.uniform(0.3, 0.7))
        elif leaf == "A_log":
            w = rng.uniform(-1.5, 1.5, shape)
        elif leaf == "dt_bias":
            w = rng.uniform(-3.0, 1.0, shape)
        elif leaf == "D" or (leaf == "norm" and len(shape) == 1) or leaf in ("norm1", "norm2"):
            w = rng.uniform(0.6, 1.4, shape)
        elif leaf == "b":
            w = rng.normal(0, 0.2, shape)
        elif name == "embed" or name == "loop.step":
            w = rng.normal(0, 0.5, shape)
        elif leaf == "conv":
            w = rng.normal(0, 0.6, shape)
        else:
            gain = 2.0 if leaf in ("uq", "uk", "in") else 1.0
            w = rng.normal(0, gain / np.sqrt(shape[-1]), shape)
        out[name] = bf16_to_f32(bf16_bits(np.asarray(w, dtype=np.float32))).reshape(shape)
    return out


def tokens(c, count, seed=1):
    return np.random.default_rng(seed).integers(0, c["vocab"], count)


def write_safetensors(path, tensors):
    """bf16 tensors from f32 arrays (int32 arrays stay)."""
    header, blobs, at = {"__metadata__": {"made": "by \"tests\""}}, [], 0
    for name, array in tensors.items():
        if np.issubdtype(np.asarray(array).dtype, np.integer):
            data, kind = np.ascontiguousarray(array, dtype="<i4").tobytes(), "I32"
        else:
            data, kind = bf16_bits(np.asarray(array, dtype=np.float32)).tobytes(), "BF16"
        header[name] = {"dtype": kind, "shape": list(np.shape(array)), "data_offsets": [at, at + len(data)]}
        blobs.append(data)
        at += len(data)
    text = json.dumps(header).encode()
    with open(path, "wb") as f:
        f.write(struct.pack("<Q", len(text)) + text + b"".join(blobs))


def write_folder(folder, c, weights):
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(c, f)
    write_safetensors(os.path.join(folder, "model.safetensors"), weights)
