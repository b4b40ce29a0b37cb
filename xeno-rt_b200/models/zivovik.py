"""Zivovik: a decoder whose input is a scaled token embedding plus a learned row a position, and whose layers add their
sublayers times a number m, x <- x + m * mixer(N(x)), then, where the layer has a feed-forward, x <- x + m * ff(N(x)),
with norms N whose stored weight is a difference from one.  A layer's mixer is grouped-query attention whose values are
the projected keys ("attention": unit-RMS q and k, one sigmoid gate a column), or two mixers side by side whose results
are RMS-normed and averaged ("parallel": grouped-query attention with one sigmoid gate a head, and a gated delta rule
with short convolutions and one decay a head), or linear attention with a constant decay a head ("lightning").  The
attentions have no rotation: their queries are multiplied by a temperature that grows with the logarithm of the position.
A feed-forward is a mixture of gated silu experts routed by softmax scores that are normalized over the chosen.  A stretch
of layers (``loop``) runs several times in a row with the same weights and a cache of its own each time; every pass but
the first begins by adding the embedding's output to the stream.  The logits are the final norm times the head matrix.

config.json keys: ``architecture`` "Zivovik", ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``residual_mult``,
``layers`` (a list of ``{"type", "mixer", "mlp"}``), ``loop`` (``start``, ``stop``, ``times``; optional),
``max_positions`` (rows of the position table; read from the table's shape where the key is missing).  An attention
mixer: ``heads``, ``kv_heads``, ``dim``, ``vdim`` (= dim), ``scale``, ``q_temp`` (``coef``, ``every``; optional).  A
parallel mixer: ``left`` (the same keys, any vdim) and ``right`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``conv``).
A lightning mixer: ``heads``, ``dim``, ``vdim``, ``decay`` (a number a head).  ``mlp``: null or ``{"kind": "moe",
"expert": {"ff"}, "router": {"experts", "top"}}``.
"""
from __future__ import annotations

import copy
import dataclasses
import math
from dataclasses import dataclass

from ..config import ModelConfig, register_architecture
from ..core import ConfigError
from ..parts import LayerSpec, ModelSpec, PartSpec, SchedulePlace
from .givopel import _check_delta, _positive, _positive_int

# constants that the design fixes
NORM_OFFSET = 1.0       # a norm multiplies by NORM_OFFSET + its stored weight
WEIGHT_SUM_EPS = 1e-20  # added to the sum of the chosen experts' scores


def _number(problems, where, d, key, default=None, nonzero=False):
    v = d.get(key, default) if isinstance(d, dict) else default
    if isinstance(v, bool) or not isinstance(v, (int, float)) or not math.isfinite(v) or (nonzero and v == 0):
        problems.append(f"{where}.{key} must be a number{' other than 0' if nonzero else ''}, got {v!r}")
        return 1.0
    return float(v)


def _check_attention(problems, where, m):
    heads, kv = _positive_int(problems, where, m, "heads"), _positive_int(problems, where, m, "kv_heads")
    for key in ("dim", "vdim"):
        _positive_int(problems, where, m, key)
    _positive(problems, where, m, "scale")
    if heads % kv:
        problems.append(f"{where}: {heads} heads are not a multiple of {kv} kv_heads")
    temp = m.get("q_temp")
    if temp is not None:
        _number(problems, where + ".q_temp", temp, "coef")
        _positive_int(problems, where + ".q_temp", temp, "every")


def _check_tied_attention(problems, where, m):
    _check_attention(problems, where, m)
    if m.get("dim") != m.get("vdim"):
        problems.append(f"{where}: values that are the projected keys have their size, vdim {m.get('vdim')!r} is not "
                        f"dim {m.get('dim')!r}")


def _check_parallel(problems, where, m):
    for side, check in (("left", _check_attention), ("right", _check_delta)):
        if not isinstance(m.get(side), dict):
            problems.append(f"{where}.{side} is missing")
        else:
            check(problems, f"{where}.{side}", m[side])


def _check_lightning(problems, where, m):
    heads = _positive_int(problems, where, m, "heads")
    for key in ("dim", "vdim"):
        _positive_int(problems, where, m, key)
    decay = m.get("decay")
    if not isinstance(decay, list) or any(isinstance(v, bool) or not isinstance(v, (int, float)) for v in decay):
        problems.append(f"{where}.decay must be a list of numbers, got {decay!r}")
    elif len(decay) != heads:
        problems.append(f"{where}.decay: {len(decay)} numbers for {heads} heads")


_CHECKS = {"attention": _check_tied_attention, "parallel": _check_parallel, "lightning": _check_lightning}


def _check_mlp(problems, where, mlp):
    if not isinstance(mlp, dict) or mlp.get("kind") != "moe":
        problems.append(f"{where}.kind {mlp.get('kind') if isinstance(mlp, dict) else mlp!r} is not moe")
        return
    _positive_int(problems, where + ".expert", mlp.get("expert"), "ff")
    experts = _positive_int(problems, where + ".router", mlp.get("router"), "experts")
    top = _positive_int(problems, where + ".router", mlp.get("router"), "top")
    if top > experts:
        problems.append(f"{where}.router: top {top} exceeds the {experts} experts")


@dataclass(frozen=True)
class ZivovikConfig(ModelConfig):
    architecture: str
    vocab: int
    width: int
    layers: tuple          # of dicts as config.json writes them (checked)
    loop: tuple | None     # (start, stop, times)
    norm_eps: float
    embedding_scale: float
    residual_mult: float
    max_positions: int | None  # None: not known before the position table's shape is seen
    eos_token_ids: tuple = ()

    @classmethod
    def from_dict(cls, raw: dict) -> "ZivovikConfig":
        problems: list[str] = []
        vocab = _positive_int(problems, "config", raw, "vocab")
        width = _positive_int(problems, "config", raw, "width")
        eps = _positive(problems, "norm", raw.get("norm"), "eps")
        scale = _number(problems, "embedding", raw.get("embedding"), "scale", 1.0, nonzero=True)
        mult = _number(problems, "config", raw, "residual_mult", 1.0)
        layers = raw.get("layers")
        if not isinstance(layers, list) or not layers:
            problems.append("'layers' must be a non-empty list")
            layers = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or not isinstance(layer.get("mixer"), dict):
                problems.append(f"{where} must be an object with a 'mixer'")
                continue
            check = _CHECKS.get(layer.get("type"))
            if check is None:
                problems.append(f"{where}.type {layer.get('type')!r} is not one of {', '.join(_CHECKS)}")
            else:
                check(problems, where + ".mixer", layer["mixer"])
            if layer.get("mlp") is not None:
                _check_mlp(problems, where + ".mlp", layer["mlp"])
        loop = raw.get("loop")
        if loop is not None:
            start, stop, times = (loop.get(k) if isinstance(loop, dict) else None for k in ("start", "stop", "times"))
            ok = all(isinstance(v, int) and not isinstance(v, bool) for v in (start, stop, times))
            if not ok or not (0 <= start < stop <= len(layers)) or times < 1:
                problems.append(f"loop {loop!r} must give 0 <= start < stop <= {len(layers)} layers and times >= 1")
                loop = None
            else:
                loop = (start, stop, times)
        max_positions = raw.get("max_positions")
        if max_positions is not None and (isinstance(max_positions, bool) or not isinstance(max_positions, int)
                                          or max_positions <= 0):
            problems.append(f"max_positions must be a positive integer, got {max_positions!r}")
        if problems:
            raise ConfigError("config.json: " + "; ".join(problems))
        eos = raw.get("eos_token_id")
        eos = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(eos))
        return cls(architecture="Zivovik", vocab=vocab, width=width, layers=tuple(copy.deepcopy(layers)), loop=loop,
                   norm_eps=eps, embedding_scale=scale, residual_mult=mult, max_positions=max_positions, eos_token_ids=eos)

    def to_dict(self) -> dict:
        out = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
               "layers": copy.deepcopy(list(self.layers)), "norm": {"eps": self.norm_eps},
               "embedding": {"scale": self.embedding_scale}, "residual_mult": self.residual_mult}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.max_positions is not None:
            out["max_positions"] = self.max_positions
        if self.eos_token_ids:
            out["eos_token_id"] = list(self.eos_token_ids)
        return out

    def with_tensor_shapes(self, shapes: dict) -> "ZivovikConfig":
        """The same configuration with ``max_positions`` taken from the position table's shape in ``shapes`` ({tensor
        name: shape}) where the configuration does not name it."""
        shape = shapes.get("pos")
        if self.max_positions is not None or shape is None or len(shape) != 2:
            return self
        return dataclasses.replace(self, max_positions=int(shape[0]))

    def order(self) -> list:
        """[(layer, whether the embedding's output is added to the stream first)] in the order the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        start, stop, times = self.loop
        order = [(i, False) for i in range(start)]
        for t in range(times):
            order += [(i, t > 0 and i == start) for i in range(start, stop)]
        return order + [(i, False) for i in range(stop, n)]


def _norm(width, eps, name):
    return PartSpec("rmsnorm", {"width": width, "eps": eps, "offset": NORM_OFFSET}, {"weight": name})


def _attention(width, eps, m, prefix, tied: bool):
    params = {"width": width, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"],
              "v_head_dim": m["vdim"], "qk_norm": "unit" if tied else False, "eps": eps, "scale": m["scale"],
              "gate": "sigmoid" if tied else "sigmoid_head", "tied_values": tied, "q_temp": m.get("q_temp"),
              "position": {"kind": "none", "params": {}}}
    return "attention", params, {r: prefix + r for r in ("q", "k", "g", "o") + (() if tied else ("v",))}


def _delta(width, eps, m, prefix):
    params = {"width": width, "n_heads": m["heads"], "n_qk_heads": m["kv_heads"], "key_dim": m["dim"],
              "value_dim": m["vdim"], "taps": m["conv"], "gate_act": "silu", "eps": eps}
    names = {r: prefix + r for r in ("q", "k", "v", "g", "b", "a", "A_log", "dt_bias", "norm", "o")}
    names.update({r + "_conv": f"{prefix}{r}.conv" for r in ("q", "k", "v")})
    return "gated_delta_rule", params, names


def _mixer(width, eps, kind, m, prefix) -> PartSpec:
    if kind == "attention":
        return PartSpec(*_attention(width, eps, m, prefix, tied=True))
    if kind == "lightning":
        params = {"width": width, "n_heads": m["heads"], "key_dim": m["dim"], "value_dim": m["vdim"],
                  "decay": list(m["decay"]), "eps": eps}
        return PartSpec("constant_decay_linear_attention", params, {r: prefix + r for r in ("q", "k", "v", "g", "norm", "o")})
    branches, names = [], {}
    for side, (part, params, own) in (("left", _attention(width, eps, m["left"], prefix + "left.", tied=False)),
                                      ("right", _delta(width, eps, m["right"], prefix + "right."))):
        branches.append({"name": side, "kind": part, "params": params})
        names.update({f"{side}.{role}": tensor for role, tensor in own.items()})
        names[f"{side}.out"] = f"{prefix}{side}.out"
    return PartSpec("side_by_side", {"width": width, "eps": eps, "branches": branches}, names)


def _experts(width, mlp, prefix) -> PartSpec:
    n = mlp["router"]["experts"]
    names = {"router": prefix + "router"}
    for i in range(n):
        names.update({f"{role}{i}": f"{prefix}e{i}.{role}" for role in ("gate", "up", "down")})
    return PartSpec("routed_experts", {"width": width, "inner": mlp["expert"]["ff"], "experts": n,
                                       "top": mlp["router"]["top"], "activation": "gated_silu", "routing": "scores",
                                       "scores": "softmax", "normalize": True, "sum_eps": WEIGHT_SUM_EPS,
                                       "router_bias": False}, names)


def build_spec(cfg: ZivovikConfig) -> ModelSpec:
    if cfg.max_positions is None:
        raise ConfigError("max_positions is not known: it is neither in the configuration nor in a model file's shapes")
    d, eps = cfg.width, cfg.norm_eps
    add = ("add", PartSpec("scaled", {"width": d, "factor": cfg.residual_mult}))
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        parts = {"mixer_norm": ("norm", _norm(d, eps, p + "norm1")),
                 "mixer": ("mixer", _mixer(d, eps, layer["type"], layer["mixer"], p + "mix.")), "mixer_add": add}
        if layer.get("mlp"):
            parts.update({"ffn_norm": ("norm", _norm(d, eps, p + "norm2")),
                          "ffn": ("feed_forward", _experts(d, layer["mlp"], p + "mlp.")), "ffn_add": add})
        layers.append(LayerSpec(parts, "added_residual"))
    schedule = [SchedulePlace(i, before="pass_in" if again else None) for i, again in cfg.order()]
    stream_parts = {"pass_in": PartSpec("add_embedding", {"width": d})} if any(p.before for p in schedule) else {}
    return ModelSpec(
        vocab_size=cfg.vocab, hidden_size=d, max_positions=cfg.max_positions,
        embedding=PartSpec("token", {"vocab_size": cfg.vocab, "width": d, "scale": cfg.embedding_scale,
                                     "positions": cfg.max_positions}, {"weight": "embed", "positions": "pos"}),
        layers=layers, schedule=schedule, final_norm=_norm(d, eps, "final.norm"),
        lm_head=PartSpec("linear", {"vocab_size": cfg.vocab, "width": d}, {"weight": "head"}),
        stop_ids=tuple(cfg.eos_token_ids),
        ignorable_tensors=tuple(f"l{i}.norm2" for i, layer in enumerate(cfg.layers) if not layer.get("mlp")),
        stream_parts=stream_parts)


register_architecture("Zivovik", ZivovikConfig, build_spec)
