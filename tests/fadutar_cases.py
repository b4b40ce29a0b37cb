"""Small Fadutar configurations and weights for the tests.  Tensor names and shapes are written down here from the
design, not taken from the package, so that a wrong name or shape in the package shows.

The cases differ from one another in every size and option: the order of the layers; layers with and without a
feed-forward; limits that clip much and little; blocks of channels that are a multiple of 8 (the kernels with tensor
cores) and that are not (the 32-bit ones), larger than one stretch of the step kernel, one block and as many blocks as
channels; 1 to 5 taps; key and value sizes that differ, that are no multiple of 16, that reach 128; as many kv heads as
heads, one kv head for all; chunks of one position, shorter and longer than a cache block, longer than the prompt, and no
chunks; a reader right behind its owner and far behind it, with a wider chunk, a narrower one and none; latent rows that
are no multiple of 16, wider than 256, and more than 16 latent heads; widths that are no multiple of 8.
"""
from __future__ import annotations

import json
import os

import numpy as np


def attn(heads, kv, dim, vdim, chunk, scale, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def latent(heads, dim, rot_dim, vdim, rank, base, scale):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank,
            "rot": {"dims": rot_dim, "base": base}, "scale": scale}


def rglru(width, blocks, conv):
    return {"width": width, "blocks": blocks, "conv": conv}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


CASE_MIXED = {
    "architecture": "Fadutar", "vocab": 101, "width": 64, "norm": {"eps": 1e-5},
    "layers": [
        layer("rglru", rglru(96, 4, 4), dense(40, 1.5)),
        layer("attention", attn(4, 2, 16, 16, 40, 0.5), dense(88, 7.0)),
        layer("latent_attention", latent(3, 8, 8, 16, 24, 5000.0, 0.4), None),
        layer("attention", attn(6, 2, 16, 16, 90, 0.3, kv_from=1), dense(48, 0.7)),
        layer("rglru", rglru(48, 6, 2), None),
    ],
}

CASE_ODD = {
    "architecture": "Fadutar", "vocab": 50, "width": 36, "norm": {"eps": 1e-6},
    "layers": [
        layer("latent_attention", latent(20, 12, 6, 20, 13, 300.0, 0.5), dense(20, 3.0)),
        layer("rglru", rglru(60, 5, 1), dense(28, 1.0)),
        layer("attention", attn(3, 3, 24, 40, 70, 0.25), None),
        layer("attention", attn(2, 1, 8, 24, 1, 1.0), dense(12, 0.5)),
        layer("attention", attn(3, 3, 24, 40, 20, 0.4, kv_from=2), None),
        layer("rglru", rglru(33, 33, 5), dense(36, 2.0)),
        layer("attention", attn(9, 3, 24, 40, None, 0.3, kv_from=2), dense(8, 4.0)),
    ],
}

# heads of 64 and 128 and a width of 384: with prompts of more than 128 tokens the tiled tensor-core products run too,
# and the attention kernels that only take such heads
CASE_WIDE = {
    "architecture": "Fadutar", "vocab": 300, "width": 384, "norm": {"eps": 1e-5},
    "layers": [
        layer("attention", attn(4, 2, 128, 128, 100, 0.09), dense(512, 2.5)),
        layer("latent_attention", latent(6, 64, 64, 48, 248, 10000.0, 0.09), None),
        layer("rglru", rglru(576, 2, 3), dense(256, 5.0)),
        layer("attention", attn(8, 2, 128, 128, 230, 0.1, kv_from=0), dense(136, 1.2)),
        layer("attention", attn(5, 5, 64, 64, 64, 0.125), dense(128, 1.0)),
        layer("attention", attn(6, 3, 128, 80, 400, 0.08), None),
    ],
}

CASES = {"mixed": (CASE_MIXED, 41), "odd": (CASE_ODD, 42), "wide": (CASE_WIDE, 43)}


def tensor_shapes(config: dict) -> dict:
    """{name: shape} of every tensor of a model of this configuration."""
    d = config["width"]
    shapes = {"embed": (config["vocab"], d), "final.norm": (d,), "head": (config["vocab"], d)}
    for i, entry in enumerate(config["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        shapes.update({p + "norm1": (d,), p + "norm1b": (d,)})
        q = p + "mix."
        if entry["type"] == "attention":
            H, G, kd, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            shapes.update({q + "q": (H * kd, d), q + "sink": (H,), q + "o": (d, H * vd)})
            if m.get("kv_from") is None:
                shapes.update({q + "k": (G * kd, d), q + "v": (G * vd, d)})
        elif entry["type"] == "latent_attention":
            H, kd, rd, vd, r = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            shapes.update({q + "q": (H * (kd + rd), d), q + "dkv": (r + rd, d), q + "dkv.norm": (r,),
                           q + "uk": (H * kd, r), q + "uv": (H * vd, r), q + "sink": (H,), q + "o": (d, H * vd)})
        else:
            n, b = m["width"], m["blocks"]
            for name in ("y", "x"):
                shapes.update({q + name: (n, d), f"{q}{name}.b": (n,)})
            shapes.update({q + "conv": (n, m["conv"]), q + "conv.b": (n,), q + "lam": (n,), q + "o": (d, n)})
            for name in ("ra", "ri"):
                shapes.update({q + name: (b, n // b, n // b), f"{q}{name}.b": (b, n // b)})
        mlp = entry.get("mlp")
        if mlp:
            shapes.update({p + "norm2": (d,), p + "norm2b": (d,)})
            for name, shape in (("gate", (mlp["ff"], d)), ("up", (mlp["ff"], d)), ("down", (d, mlp["ff"]))):
                shapes.update({f"{p}mlp.{name}": shape, f"{p}mlp.{name}.b": (shape[0],)})
    return shapes


def _bf16(x: np.ndarray) -> np.ndarray:
    """Rounded to bfloat16 (to nearest even) and back, so that file and oracle hold the same numbers."""
    bits = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    rounded = ((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16).astype(np.uint32) << 16
    return rounded.view(np.float32).reshape(np.shape(x))


def random_weights(config: dict, seed: int) -> dict:
    """Decays that remember from a few to some hundreds of tokens, sinks that weigh about as much as the keys, norms
    around zero."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        if name.endswith("dkv.norm"):
            w = 1.0 + rng.normal(0.0, 0.15, shape)
        elif leaf.startswith("norm"):
            w = rng.normal(0.0, 0.15, shape)
        elif leaf == "sink":
            w = rng.normal(1.0, 1.5, shape)
        elif leaf == "lam":
            w = rng.normal(-4.0, 1.5, shape)
        elif leaf == "b":
            w = rng.normal(0.0, 0.3, shape)
        elif leaf == "conv":
            w = rng.normal(0.0, 0.7, shape)
        elif leaf in ("ra", "ri"):
            w = rng.normal(0.0, 1.5 / np.sqrt(shape[-1]), shape)
        elif leaf == "embed":
            w = rng.normal(0.0, 1.0, shape)
        else:
            w = rng.normal(0.0, (1.5 if leaf in ("q", "k") else 1.0) / np.sqrt(shape[1]), shape)
        out[name] = _bf16(np.asarray(w, dtype=np.float32))
    return out


def write_folder(path: str, config: dict, weights: dict) -> str:
    """config.json and model.safetensors (bfloat16) in ``path``."""
    import torch
    from xeno_rt_b200.weights import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(config, fh)
    write_safetensors(os.path.join(path, "model.safetensors"),
                      {k: torch.from_numpy(np.array(v, dtype=np.float32)).reshape(np.shape(v)).to(torch.bfloat16)
                       for k, v in weights.items()})
    return path


def make_case(tmp_path, name: str):
    """(folder, config, weights) of a named case."""
    config, seed = CASES[name]
    weights = random_weights(config, seed)
    return write_folder(os.path.join(str(tmp_path), name), config, weights), config, weights


def random_config(rng) -> dict:
    """A configuration drawn at random: any order of layers, any of the sizes and options the cases above use and more."""
    pick = lambda *values: values[int(rng.integers(len(values)))]
    chunk = lambda: pick(1, 5, 33, 64, 70, 128, 130, 400, None)
    layers, owners = [], []
    for i in range(int(rng.integers(2, 8))):
        kind = rng.random()
        if kind < 0.3:
            blocks, size = pick(1, 2, 3, 4, 8), pick(1, 4, 8, 12, 16, 24, 40, 72)
            entry = ("rglru", rglru(blocks * size, blocks, pick(1, 2, 3, 4, 5, 9)))
        elif kind < 0.55:
            rot = pick(2, 4, 8, 16, 32, 64)
            m = latent(pick(1, 2, 3, 4, 8, 17), pick(4, 8, 12, 16, 32, 64), rot, pick(4, 8, 16, 20, 32, 64),
                       pick(5, 12, 16, 24, 40, 64, 128, 200, 300), pick(100.0, 10000.0, 1e6),
                       float(pick(0.5, 1.0, 2.0)) / np.sqrt(16))
            entry = ("latent_attention", m)
        elif owners and kind < 0.75:
            j = pick(*owners)
            o = layers[j]["mixer"]
            m = attn(o["kv_heads"] * pick(1, 2, 3, 4), o["kv_heads"], o["dim"], o["vdim"], chunk(),
                     float(pick(0.5, 1.0, 2.0)) / np.sqrt(o["dim"]), kv_from=j)
            entry = ("attention", m)
        else:
            kv, dim = pick(1, 2, 3), pick(8, 16, 24, 32, 48, 64, 128, 256)
            m = attn(kv * pick(1, 2, 3, 4, 8, 17), kv, dim, pick(8, 16, 24, 40, 64, 128), chunk(),
                     float(pick(0.5, 1.0, 2.0)) / np.sqrt(dim))
            entry = ("attention", m)
            owners.append(i)
        layers.append(layer(*entry, dense(pick(8, 12, 33, 64, 136), float(pick(0.5, 1.0, 2.0, 7.0))) if rng.random() < 0.75 else None))
    return {"architecture": "Fadutar", "vocab": pick(50, 101, 256), "width": pick(32, 36, 64, 96, 128, 200),
            "norm": {"eps": pick(1e-5, 1e-6)}, "layers": layers}
