"""Fadutar: a decoder whose layers norm every sublayer before and after it, x <- x + N(mixer(N(x))), then, where the
layer has a feed-forward, x <- x + N(ff(N(x))), with norms whose stored weight is a difference from one.  A layer's mixer
is a gated linear recurrence a channel ("rglru", ``parts/linear_recurrence.py``), grouped-query attention without a
rotation whose queries see only their own chunk of positions ("attention"; a layer may read the keys and values that an
earlier layer cached instead of making its own), or latent attention over all earlier tokens ("latent_attention": the
keys and values of all heads are read out of one small normed vector a token, one rotated key part of split-half pairs is
shared by all heads).  Both attentions have a learned sink a head.  A feed-forward is dense with a limited gate and
biases on all three products.  The logits are the final norm times the head matrix.

config.json keys: ``architecture`` "Fadutar", ``vocab``, ``width``, ``norm.eps``, ``layers`` (a list of ``{"type",
"mixer", "mlp"}``), ``max_positions`` (optional).  An rglru mixer: ``width``, ``blocks``, ``conv`` (taps).  An attention
mixer: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``, ``mask.size`` (of a chunk; optional), ``kv_from`` (optional: the
layer whose keys and values it reads).  A latent mixer: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``,
``rot`` (``dims``, ``base``).  ``mlp``: null or ``{"kind": "dense", "ff", "limit"}``.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass

from ..config import ModelConfig, register_architecture
from ..core import ConfigError
from ..parts import LayerSpec, ModelSpec, PartSpec, SchedulePlace
from .givopel import DEFAULT_MAX_POSITIONS, _positive, _positive_int
from .zogevik import _check_attention, _check_latent, _rotation

# constants that the design fixes
DECAY_SCALE = 8.0    # log a = -DECAY_SCALE * r * softplus(lam)
GATE_ALPHA = 1.702   # of the feed-forward's gate g * sigmoid(GATE_ALPHA g)
NORM_OFFSET = 1.0    # a norm multiplies by NORM_OFFSET + its stored weight


def _check_recurrence(problems, where, m):
    width, blocks = _positive_int(problems, where, m, "width"), _positive_int(problems, where, m, "blocks")
    _positive_int(problems, where, m, "conv")
    if width % blocks:
        problems.append(f"{where}: width {width} does not form {blocks} equal blocks")


def _check_mlp(problems, where, mlp):
    if not isinstance(mlp, dict) or mlp.get("kind") != "dense":
        problems.append(f"{where}.kind {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} is not dense")
        return
    _positive_int(problems, where, mlp, "ff")
    _positive(problems, where, mlp, "limit")


@dataclass(frozen=True)
class FadutarConfig(ModelConfig):
    architecture: str
    vocab: int
    width: int
    layers: tuple          # of dicts as config.json writes them (checked)
    norm_eps: float
    max_positions: int
    eos_token_ids: tuple = ()

    @classmethod
    def from_dict(cls, raw: dict) -> "FadutarConfig":
        problems: list[str] = []
        vocab = _positive_int(problems, "config", raw, "vocab")
        width = _positive_int(problems, "config", raw, "width")
        eps = _positive(problems, "norm", raw.get("norm"), "eps")
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            problems.append("'layers' must be a non-empty list")
            layers = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or not isinstance(layer.get("mixer"), dict):
                problems.append(f"{where} must be an object with a 'mixer'")
                continue
            kind, m = layer.get("type"), layer["mixer"]
            if kind == "rglru":
                _check_recurrence(problems, where + ".mixer", m)
            elif kind == "attention":
                _check_attention(problems, where + ".mixer", m, i, layers)
                if m.get("rot") is not None:
                    problems.append(f"{where}.mixer.rot: attention layers of this design have no rotation")
            elif kind == "latent_attention":
                _check_latent(problems, where + ".mixer", m)
                if m.get("mask") is not None:
                    problems.append(f"{where}.mixer.mask: latent attention of this design sees every earlier key")
            else:
                problems.append(f"{where}.type {kind!r} is not one of rglru, attention, latent_attention")
            if layer.get("mlp") is not None:
                _check_mlp(problems, where + ".mlp", layer["mlp"])
        max_positions = raw.get("max_positions", DEFAULT_MAX_POSITIONS)
        if isinstance(max_positions, bool) or not isinstance(max_positions, int) or max_positions <= 0:
            problems.append(f"max_positions must be a positive integer, got {max_positions!r}")
        if problems:
            raise ConfigError("config.json: " + "; ".join(problems))
        eos = raw.get("eos_token_id")
        eos = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(architecture="Fadutar", vocab=vocab, width=width, layers=tuple(copy.deepcopy(layers)), norm_eps=eps,
                   max_positions=max_positions, eos_token_ids=eos)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps}}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            out["max_positions"] = self.max_positions
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out


def _norm(width, eps, name):
    return PartSpec("rmsnorm", {"width": width, "eps": eps, "offset": NORM_OFFSET}, {"weight": name})


def _recurrence_spec(width, eps, m, prefix):
    params = {"width": width, "inner": m["width"], "blocks": m["blocks"], "taps": m["conv"], "decay_scale": DECAY_SCALE}
    names = {"y": "y", "y_bias": "y.b", "x": "x", "x_bias": "x.b", "conv": "conv", "conv_bias": "conv.b", "r": "ra",
             "r_bias": "ra.b", "i": "ri", "i_bias": "ri.b", "lam": "lam", "o": "o"}
    return PartSpec("gated_linear_recurrence", params, {role: prefix + name for role, name in names.items()})


def _attention_spec(width, eps, m, prefix):
    own = m.get("kv_from") is None
    params = {"width": width, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"],
              "v_head_dim": m["vdim"], "qk_norm": False, "eps": eps, "scale": m["scale"], "sink": "learned",
              "chunk": (m.get("mask") or {}).get("size"), "own_kv": own, "position": {"kind": "none", "params": {}}}
    return PartSpec("attention", params, {r: prefix + r for r in ("q", "o", "sink") + (("k", "v") if own else ())})


def _latent_spec(width, eps, m, prefix):
    params = {"width": width, "n_heads": m["heads"], "head_dim": m["dim"], "rot_dim": m["rot_dim"],
              "v_head_dim": m["vdim"], "kv_rank": m["kv_rank"], "eps": eps, "window": None, "scale": m["scale"],
              "sink": "learned", "position": _rotation(m, "split_half")}
    names = {"q": prefix + "q", "down": prefix + "dkv", "down_norm": prefix + "dkv.norm", "up_k": prefix + "uk",
             "up_v": prefix + "uv", "o": prefix + "o", "sink": prefix + "sink"}
    return PartSpec("latent_attention", params, names)


_MIXERS = {"rglru": _recurrence_spec, "attention": _attention_spec, "latent_attention": _latent_spec}


def _feed_forward(width, mlp, prefix):
    names = {role: prefix + role for role in ("gate", "up", "down")}
    names.update({role + "_bias": f"{prefix}{role}.b" for role in ("gate", "up", "down")})
    return PartSpec("swiglu", {"width": width, "inner": mlp["ff"], "activation": "gated_sigmoid", "limit": mlp["limit"],
                               "alpha": GATE_ALPHA, "bias": True}, names)


def build_spec(cfg: FadutarConfig) -> ModelSpec:
    d, eps = cfg.width, cfg.norm_eps
    layers, schedule = [], []
    for i, layer in enumerate(cfg.layers):
        p, m = f"l{i}.", layer["mixer"]
        parts = {"mixer_norm": ("norm", _norm(d, eps, p + "norm1")),
                 "mixer": ("mixer", _MIXERS[layer["type"]](d, eps, m, p + "mix.")),
                 "mixer_post": ("norm", _norm(d, eps, p + "norm1b"))}
        if layer.get("mlp"):
            parts.update({"ffn_norm": ("norm", _norm(d, eps, p + "norm2")),
                          "ffn": ("feed_forward", _feed_forward(d, layer["mlp"], p + "mlp.")),
                          "ffn_post": ("norm", _norm(d, eps, p + "norm2b"))})
        layers.append(LayerSpec(parts, "sandwich_residual"))
        # a layer that reads another's keys and values is a place that reads that place's cache (places = layers here)
        schedule.append(SchedulePlace(i, cache_from=m.get("kv_from") if layer["type"] == "attention" else None))
    ignorable = tuple(f"l{i}.{n}" for i, layer in enumerate(cfg.layers) if not layer.get("mlp") for n in ("norm2", "norm2b"))
    return ModelSpec(
        vocab_size=cfg.vocab, hidden_size=d, max_positions=cfg.max_positions,
        embedding=PartSpec("token", {"vocab_size": cfg.vocab, "width": d}, {"weight": "embed"}),
        layers=layers, schedule=schedule, final_norm=_norm(d, eps, "final.norm"),
        lm_head=PartSpec("linear", {"vocab_size": cfg.vocab, "width": d}, {"weight": "head"}),
        stop_ids=tuple(cfg.eos_token_ids), ignorable_tensors=ignorable)


register_architecture("Fadutar", FadutarConfig, build_spec)
