"""Plain, slow restatement of the Zivovik decoder, one function per mechanism.

The oracle of the Zivovik tests.  It shares no code with the product package: whole sequences, no cache, numpy
float64 throughout, every head by itself, every recurrence token by token.

The design in short.  x = scale * E[token] + P[position].  A layer adds its sublayers behind a norm and times a number m,
x <- x + m mixer(N_1(x)), then, if it has a feed-forward, x <- x + m ff(N_2(x)); N is an RMSNorm whose stored weight is a
difference from one.  A stretch of layers may run several times in a row; every pass but the first begins by adding what
the embedding gave.  A mixer is one of
  * "attention": grouped-query attention over every earlier key whose values are the projected keys themselves; q and k
    heads are then divided by their root mean square, q is multiplied by a temperature that grows with the logarithm of
    the position, and the heads side by side are multiplied by a sigmoid gate a column;
  * "parallel": two mixers that read the same input, each result RMS-normed with its own plain weight, their mean being
    the result.  Left: grouped-query attention with the same temperature, without norms, one sigmoid gate a head.  Right:
    a gated delta rule with short convolutions, unit q and k, and one decay a head;
  * "lightning": a linear recurrence of silu'd q, k, v with one constant decay a head, one norm over all heads and a
    sigmoid gate.
A feed-forward is a mixture of gated silu experts; a token's weights are its largest softmax scores divided by their sum.
"""
from __future__ import annotations

import math

import numpy as np

F64 = np.float64

UNIT_EPS = 1e-6    # inside the root of the delta rule's unit q and k
SUM_EPS = 1e-20    # added to the sum of the chosen experts' scores


# ----------------------------------------------------------------------------- small functions
def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    x = np.asarray(x, F64)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps)


def rms_norm(x, weight, eps):
    return unit_rms(x, eps) * np.asarray(weight, F64)


def offset_norm(x, weight, eps):
    """An RMSNorm whose weight is stored as its difference from one."""
    return rms_norm(x, 1.0 + np.asarray(weight, F64), eps)


def sigmoid(z):
    z = np.asarray(z, F64)
    e = np.exp(-np.abs(z))
    return np.where(z >= 0, 1.0 / (1.0 + e), e / (1.0 + e))


def silu(z):
    return np.asarray(z, F64) * sigmoid(z)


def softplus(z):
    z = np.asarray(z, F64)
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def softmax(z):
    e = np.exp(z - np.max(z, axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


# ----------------------------------------------------------------------------- embedding
def embed(tokens, table, positions, scale, start=0):
    rows = np.asarray(table, F64)[list(tokens)] * scale
    return rows + np.asarray(positions, F64)[start:start + len(rows)]


# ----------------------------------------------------------------------------- attention
def temperature(position: int, temp) -> float:
    """What a query at ``position`` is multiplied by; ``temp`` is {"coef", "every"} or None."""
    if not temp:
        return 1.0
    return 1.0 + temp["coef"] * math.log((position + 1) // temp["every"] + 1)


def attend(q, k, v, scale, temp):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim] -> [T, H, vdim]: every query over the keys up to its own."""
    n, heads = q.shape[:2]
    group = heads // k.shape[1]
    out = np.zeros((n, heads, v.shape[2]), F64)
    for t in range(n):
        for a in range(heads):
            s = k[:t + 1, a // group] @ (q[t, a] * temperature(t, temp)) * scale
            out[t, a] = softmax(s) @ v[:t + 1, a // group]
    return out


def tied_attention(h, w, m, eps):
    """Mixer "attention": values are the keys as projected, before their norm."""
    n = h.shape[0]
    q = (h @ w["q"].T).reshape(n, m["heads"], m["dim"])
    k = (h @ w["k"].T).reshape(n, m["kv_heads"], m["dim"])
    out = attend(unit_rms(q, eps), unit_rms(k, eps), k, m["scale"], m.get("q_temp"))
    return (out.reshape(n, -1) * sigmoid(h @ w["g"].T)) @ w["o"].T


def head_gated_attention(h, w, m):
    """The left half of mixer "parallel"."""
    n = h.shape[0]
    q = (h @ w["q"].T).reshape(n, m["heads"], m["dim"])
    k = (h @ w["k"].T).reshape(n, m["kv_heads"], m["dim"])
    v = (h @ w["v"].T).reshape(n, m["kv_heads"], m["vdim"])
    out = attend(q, k, v, m["scale"], m.get("q_temp")) * sigmoid(h @ w["g"].T)[:, :, None]
    return out.reshape(n, -1) @ w["o"].T


# ----------------------------------------------------------------------------- recurrences
def short_convolution(u, taps_weight):
    """silu of sum_j w[c, j] u_(t - taps + 1 + j)[c], zeros before the start.  u [T, C], w [C, taps]."""
    u, w = np.asarray(u, F64), np.asarray(taps_weight, F64)
    taps = w.shape[1]
    out = np.zeros_like(u)
    for t in range(u.shape[0]):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] += w[:, j] * u[src]
    return silu(out)


def unit_vectors(x):
    return x / np.sqrt((x * x).sum(axis=-1, keepdims=True) + UNIT_EPS)


def head_decay(raw, a_log, dt_bias):
    """g = exp(-exp(A_log) softplus(raw + dt_bias)), one a head.  raw [T, H]."""
    return np.exp(-np.exp(np.asarray(a_log, F64)) * softplus(raw + np.asarray(dt_bias, F64)))


def delta_scan(q, k, v, decay, beta):
    """S <- g S; S <- S + k (beta (v - S^T k))^T; o = S^T q for one head.  q, k [T, d], v [T, e], decay, beta [T]."""
    state = np.zeros((k.shape[1], v.shape[1]), F64)
    out = np.zeros(v.shape, F64)
    for t in range(len(q)):
        state = decay[t] * state
        state = state + np.outer(k[t], beta[t] * (v[t] - state.T @ k[t]))
        out[t] = state.T @ q[t]
    return out


def delta_rule(h, w, m, eps):
    """The right half of mixer "parallel"."""
    n, heads, kv = h.shape[0], m["heads"], m["kv_heads"]
    through = lambda name: short_convolution(h @ w[name].T, w[name + ".conv"])
    q = unit_vectors(through("q").reshape(n, kv, m["dim"])) * m["dim"] ** -0.5
    k = unit_vectors(through("k").reshape(n, kv, m["dim"]))
    v = through("v").reshape(n, heads, m["vdim"])
    beta = sigmoid(h @ w["b"].T)
    decay = head_decay(h @ w["a"].T, w["A_log"], w["dt_bias"])
    out = np.stack([delta_scan(q[:, a // (heads // kv)], k[:, a // (heads // kv)], v[:, a], decay[:, a], beta[:, a])
                    for a in range(heads)], axis=1)
    out = rms_norm(out, w["norm"], eps).reshape(n, -1) * silu(h @ w["g"].T)
    return out @ w["o"].T


def parallel(h, w, m, eps):
    left = head_gated_attention(h, _sub(w, "left."), m["left"])
    right = delta_rule(h, _sub(w, "right."), m["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


def constant_decay_scan(q, k, v, decay):
    """S <- decay S + k v^T; o = S^T q for one head."""
    state = np.zeros((k.shape[1], v.shape[1]), F64)
    out = np.zeros(v.shape, F64)
    for t in range(len(q)):
        state = decay * state + np.outer(k[t], v[t])
        out[t] = state.T @ q[t]
    return out


def lightning(h, w, m, eps):
    n, heads = h.shape[0], m["heads"]
    q, k, v = (silu(h @ w[name].T).reshape(n, heads, -1) for name in ("q", "k", "v"))
    out = np.stack([constant_decay_scan(q[:, a], k[:, a], v[:, a], m["decay"][a]) for a in range(heads)], axis=1)
    return (rms_norm(out.reshape(n, -1), w["norm"], eps) * sigmoid(h @ w["g"].T)) @ w["o"].T


# ----------------------------------------------------------------------------- experts
def route(logits, top: int):
    """(chosen experts, their weights) of one token."""
    s = softmax(np.asarray(logits, F64))
    chosen = np.argsort(-s, kind="stable")[:top]
    return chosen, s[chosen] / (s[chosen].sum() + SUM_EPS)


def experts_ff(h, w, mlp):
    logits = h @ w["router"].T
    out = np.zeros(h.shape, F64)
    for t in range(h.shape[0]):
        for e, weight in zip(*route(logits[t], mlp["router"]["top"])):
            act = silu(w[f"e{e}.gate"] @ h[t]) * (w[f"e{e}.up"] @ h[t])
            out[t] += weight * (w[f"e{e}.down"] @ act)
    return out


# ----------------------------------------------------------------------------- the model
def _sub(tensors, prefix):
    return {k[len(prefix):]: np.asarray(v, F64) for k, v in tensors.items() if k.startswith(prefix)}


def order(config):
    """[(layer, whether the embedding output is added first)] as the layers run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    start, stop = loop["start"], loop["stop"]
    out = [(i, False) for i in range(start)]
    for t in range(loop["times"]):
        out += [(i, t > 0 and i == start) for i in range(start, stop)]
    return out + [(i, False) for i in range(stop, n)]


def forward(config, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the stream after every layer run."""
    eps, mult = config["norm"]["eps"], config.get("residual_mult", 1.0)
    x0 = embed(tokens, tensors["embed"], tensors["pos"], config.get("embedding", {}).get("scale", 1.0))
    x = x0
    for i, again in order(config):
        layer = config["layers"][i]
        p, m = f"l{i}.", layer["mixer"]
        w = _sub(tensors, p + "mix.")
        if again:
            x = x + x0
        h = offset_norm(x, tensors[p + "norm1"], eps)
        if layer["type"] == "attention":
            y = tied_attention(h, w, m, eps)
        elif layer["type"] == "parallel":
            y = parallel(h, w, m, eps)
        elif layer["type"] == "lightning":
            y = lightning(h, w, m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + mult * y
        if layer.get("mlp"):
            x = x + mult * experts_ff(offset_norm(x, tensors[p + "norm2"], eps), _sub(tensors, p + "mlp."), layer["mlp"])
        if layers_out is not None:
            layers_out.append(x.copy())
    return offset_norm(x, tensors["final.norm"], eps) @ np.asarray(tensors["head"], F64).T
