"""Small Zivovik configurations and weights for the tests.  Tensor names and shapes are written down here from the
design, not taken from the package, so that a wrong name or shape in the package shows.

The cases differ from one another in every size and option: the order of the layers; layers with and without a
feed-forward; stretches that run twice, three times, once, from the first layer or to the last, and no loop; residual
multipliers and embedding scales that are 1 and that are not; temperatures of several steps and none; key and value sizes
that differ, that are no multiple of 16, that reach 128; as many kv heads as heads, one kv head for all, groups of more
than 16; recurrences with 1 to 5 taps and as many q/k heads as heads or fewer; decays near and far from one; 1 to all
experts a token; widths that are no multiple of 8.
"""
from __future__ import annotations

import json
import os

import numpy as np


def temp(coef, every):
    return {"coef": coef, "every": every}


def attn(heads, kv, dim, scale, q_temp=None, vdim=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": dim if vdim is None else vdim, "scale": scale}
    if q_temp is not None:
        m["q_temp"] = q_temp
    return m


def delta(heads, kv, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}


def light(dim, vdim, decay):
    return {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": list(decay)}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


def model(vocab, width, layers, loop=None, scale=1.0, mult=1.0, eps=1e-5, positions=420):
    out = {"architecture": "Zivovik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers,
           "embedding": {"scale": scale}, "residual_mult": mult, "max_positions": positions}
    if loop is not None:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


CASE_MIXED = model(101, 64, [
    layer("lightning", light(16, 24, [0.5, 0.9, 0.99]), moe(24, 6, 2)),
    layer("attention", attn(4, 2, 16, 0.3, temp(0.4, 40)), moe(40, 5, 3)),
    layer("parallel", {"left": attn(6, 2, 32, 0.2, temp(0.7, 30), vdim=16), "right": delta(4, 2, 16, 32, 4)}, moe(16, 8, 2)),
    layer("attention", attn(2, 1, 48, 0.2, temp(0.3, 7)), None),
    layer("lightning", light(32, 8, [0.97, 0.3]), None),
], loop=(1, 3, 2), scale=2.5, mult=0.4)

CASE_ODD = model(50, 36, [
    layer("parallel", {"left": attn(6, 3, 20, 0.25, None, vdim=12), "right": delta(3, 3, 12, 20, 1)}, moe(20, 5, 5)),
    layer("attention", attn(17, 1, 24, 0.4, temp(1.0, 1)), None),
    layer("lightning", light(12, 20, [1.0, 0.8, 0.25, 0.999, 0.6]), moe(12, 3, 1)),
    layer("attention", attn(3, 3, 40, 0.2), moe(33, 4, 2)),
    layer("parallel", {"left": attn(2, 2, 12, 0.5, temp(-0.3, 60), vdim=28), "right": delta(6, 2, 40, 9, 5)}, None),
], loop=(0, 2, 3), mult=0.7, eps=1e-6)

# heads of 64 and 128 and a width of 384: with prompts of more than 128 tokens the tiled tensor-core products run too,
# the attention kernels that only take such heads, the single-token attention that takes the product's rows itself, and
# the experts' products over sorted rows
CASE_WIDE = model(300, 384, [
    layer("attention", attn(4, 2, 128, 0.12, temp(0.5, 70)), moe(136, 8, 2)),
    layer("parallel", {"left": attn(8, 2, 64, 0.1, temp(0.6, 50)), "right": delta(4, 4, 128, 128, 4)}, moe(64, 16, 4)),
    layer("lightning", light(128, 64, [0.95, 0.999]), None),
    layer("attention", attn(6, 2, 64, 0.15, temp(0.25, 200)), moe(72, 4, 2)),
    layer("parallel", {"left": attn(4, 4, 128, 0.08, None), "right": delta(4, 2, 64, 72, 2)}, None),
], loop=(2, 5, 2), scale=0.7, mult=0.5)

CASES = {"mixed": (CASE_MIXED, 51), "odd": (CASE_ODD, 52), "wide": (CASE_WIDE, 53)}


def tensor_shapes(config: dict) -> dict:
    """{name: shape} of every tensor of a model of this configuration."""
    d = config["width"]
    shapes = {"embed": (config["vocab"], d), "pos": (config["max_positions"], d), "final.norm": (d,),
              "head": (config["vocab"], d)}

    def attention(p, m, tied):
        H, G, kd, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        shapes.update({p + "q": (H * kd, d), p + "k": (G * kd, d), p + "g": (H * vd if tied else H, d), p + "o": (d, H * vd)})
        if not tied:
            shapes[p + "v"] = (G * vd, d)

    for i, entry in enumerate(config["layers"]):
        p, m = f"l{i}.", entry["mixer"]
        q = p + "mix."
        shapes[p + "norm1"] = (d,)
        if entry["type"] == "attention":
            attention(q, m, True)
        elif entry["type"] == "lightning":
            H, kd, vd = m["heads"], m["dim"], m["vdim"]
            shapes.update({q + "q": (H * kd, d), q + "k": (H * kd, d), q + "v": (H * vd, d), q + "g": (H * vd, d),
                           q + "norm": (H * vd,), q + "o": (d, H * vd)})
        else:
            attention(q + "left.", m["left"], False)
            r, b = q + "right.", m["right"]
            H, G, kd, vd, taps = b["heads"], b["kv_heads"], b["dim"], b["vdim"], b["conv"]
            for name, rows in (("q", G * kd), ("k", G * kd), ("v", H * vd)):
                shapes.update({r + name: (rows, d), f"{r}{name}.conv": (rows, taps)})
            shapes.update({r + "b": (H, d), r + "a": (H, d), r + "A_log": (H,), r + "dt_bias": (H,), r + "g": (H * vd, d),
                           r + "norm": (vd,), r + "o": (d, H * vd), q + "left.out": (d,), q + "right.out": (d,)})
        mlp = entry.get("mlp")
        if mlp:
            shapes.update({p + "norm2": (d,), p + "mlp.router": (mlp["router"]["experts"], d)})
            for e in range(mlp["router"]["experts"]):
                ff = mlp["expert"]["ff"]
                shapes.update({f"{p}mlp.e{e}.gate": (ff, d), f"{p}mlp.e{e}.up": (ff, d), f"{p}mlp.e{e}.down": (d, ff)})
    return shapes


def _bf16(x: np.ndarray) -> np.ndarray:
    """Rounded to bfloat16 (to nearest even) and back, so that file and oracle hold the same numbers."""
    bits = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    rounded = ((bits + 0x7FFF + ((bits >> 16) & 1)) >> 16).astype(np.uint32) << 16
    return rounded.view(np.float32).reshape(np.shape(x))


def random_weights(config: dict, seed: int) -> dict:
    """Scores that single out keys, states that remember from a few to hundreds of tokens, routers whose last chosen
    expert weighs little (a choice that rounding turns then moves the result little), norms around zero (the weights
    of the state mixers' norms and of a parallel mixer's results around one)."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(config).items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2") or name == "final.norm":
            w = rng.normal(0.0, 0.15, shape)
        elif leaf in ("norm", "out"):
            w = rng.normal(1.0, 0.15, shape)
        elif leaf == "A_log":
            w = rng.normal(0.0, 0.7, shape)
        elif leaf == "dt_bias":
            w = rng.normal(-3.5, 1.5, shape)
        elif leaf == "conv":
            w = rng.normal(0.0, 0.7, shape)
        elif leaf in ("embed", "pos"):
            w = rng.normal(0.0, 1.0 if leaf == "embed" else 0.7, shape)
        else:
            w = rng.normal(0.0, {"q": 1.5, "k": 1.5, "router": 3.0}.get(leaf, 1.0) / np.sqrt(shape[1]), shape)
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
    some_temp = lambda: pick(None, temp(float(pick(0.2, 0.5, 1.0, -0.2)), pick(1, 3, 16, 50, 64, 100, 300)))

    def some_attention(tied):
        kv, dim = pick(1, 2, 3), pick(8, 12, 16, 24, 32, 48, 64, 96, 128, 256)
        vdim = dim if tied else pick(8, 16, 24, 40, 64, 96, 128)
        return attn(kv * pick(1, 2, 3, 4, 8, 17), kv, dim, float(pick(0.5, 1.0, 2.0)) / np.sqrt(dim), some_temp(), vdim)

    layers = []
    for _ in range(int(rng.integers(1, 7))):
        kind = pick("attention", "parallel", "lightning")
        if kind == "attention":
            mixer = some_attention(True)
        elif kind == "parallel":
            kv = pick(1, 2, 3)
            mixer = {"left": some_attention(False),
                     "right": delta(kv * pick(1, 2, 4), kv, pick(4, 8, 15, 16, 24, 32, 64, 100, 128),
                                    pick(5, 8, 16, 32, 40, 64, 130), pick(1, 2, 3, 4, 5, 9))}
        else:
            mixer = light(pick(4, 8, 12, 16, 32, 50, 64, 128), pick(3, 8, 16, 32, 48, 64, 200),
                          [float(pick(0.1, 0.5, 0.9, 0.99, 0.999, 1.0)) for _ in range(pick(1, 2, 3, 4, 8))])
        experts = pick(1, 2, 5, 8, 12, 33)
        layers.append(layer(kind, mixer, moe(pick(4, 8, 12, 33, 64), experts, min(experts, pick(1, 2, 3, 4)))
                            if rng.random() < 0.75 else None))
    loop = None
    if rng.random() < 0.7:
        start = int(rng.integers(len(layers)))
        loop = (start, int(rng.integers(start + 1, len(layers) + 1)), pick(1, 2, 3))
    return model(pick(50, 101, 256), pick(32, 36, 64, 96, 128, 200), layers, loop, float(pick(1.0, 0.5, 3.0)),
                 float(pick(1.0, 0.3, 0.8)), pick(1e-5, 1e-6))
