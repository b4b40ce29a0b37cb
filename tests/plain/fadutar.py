"""Plain, slow restatement of the Fadutar decoder, one function per mechanism.

The oracle of the Fadutar tests.  It shares no code with the product package: whole sequences, no cache, numpy
float64 throughout, every head by itself, the recurrence token by token.

The design in short.  x = E[token].  A layer norms every sublayer before and after it, x <- x + N_1b(mixer(N_1(x))), then,
if it has a feed-forward, x <- x + N_2b(ff(N_2(x))), where N is an RMSNorm whose stored weight is a difference from
one.  A mixer is one of
  * a gated linear recurrence a channel: two branches of one size, one through the tanh gelu, the other through a short
    causal convolution over time and then S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with the decay and the input gate
    computed from the convolved branch by square matrices a block of channels;
  * grouped-query attention without a rotation whose queries see only the keys of their own chunk of positions, with a
    learned sink a head in the softmax's denominator; a layer may take keys and values from an earlier layer;
  * latent attention: keys and values of all heads are read out of one small normed vector a token, one rotated key
    part (split-half pairs) is shared by all heads; every earlier key is seen; a learned sink a head.
A feed-forward is dense with a limited gate and biases on all three products.  The logits are the final norm times the
head matrix.
"""
from __future__ import annotations

import math

import numpy as np

F64 = np.float64

DECAY_SCALE = 8.0   # log a = -DECAY_SCALE * r * softplus(lam)
GATE_ALPHA = 1.702  # of the feed-forward's gate


# ----------------------------------------------------------------------------- small functions
def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    x = np.asarray(x, F64)
    return x / np.sqrt((x * x).mean(axis=-1, keepdims=True) + eps) * np.asarray(weight, F64)


def offset_norm(x, weight, eps):
    """The same with a weight stored as its difference from one."""
    return rms_norm(x, 1.0 + np.asarray(weight, F64), eps)


def sigmoid(z):
    z = np.asarray(z, F64)
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def softplus(z):
    z = np.asarray(z, F64)
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    z = np.asarray(z, F64)
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def short_convolution(u, taps_weight, bias):
    """y_t[c] = b[c] + sum_j w[c, j] * u_(t - taps + 1 + j)[c], zeros before the start.  u [T, C], w [C, taps]."""
    u, w = np.asarray(u, F64), np.asarray(taps_weight, F64)
    taps = w.shape[1]
    out = np.zeros_like(u) + np.asarray(bias, F64)
    for t in range(u.shape[0]):
        for j in range(taps):
            src = t - taps + 1 + j
            if src >= 0:
                out[t] += w[:, j] * u[src]
    return out


def rotate_split_half(vec, position: int, dims: int, base: float):
    """The first ``dims`` entries of ``vec``: entry i pairs with entry i + dims / 2; the rest stays."""
    out = np.array(vec, F64)
    half = dims // 2
    a = position * np.power(F64(base), -2.0 * np.arange(half, dtype=F64) / dims)
    u, v = out[:half].copy(), out[half:dims].copy()
    out[:half] = u * np.cos(a) - v * np.sin(a)
    out[half:dims] = v * np.cos(a) + u * np.sin(a)
    return out


def sink_weights(scores, sink: float):
    """exp(s_j) / (sum exp(s) + exp(sink))."""
    s = np.asarray(scores, F64)
    m = max(s.max(), sink)
    e = np.exp(s - m)
    return e / (e.sum() + math.exp(sink - m))


# ----------------------------------------------------------------------------- the recurrence
def block_product(u, matrices, bias):
    """Part b of every row of ``u`` times the square matrix b, plus its bias.  u [T, width], matrices [blocks, n, n]."""
    blocks, n, _ = matrices.shape
    parts = np.asarray(u, F64).reshape(u.shape[0], blocks, n)
    return np.stack([parts[:, b] @ np.asarray(matrices[b], F64).T + np.asarray(bias[b], F64) for b in range(blocks)],
                    axis=1).reshape(u.shape[0], blocks * n)


def linear_recurrence(u, decay_gate, input_gate, lam):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t for every channel, from zero.  All [T, width], lam [width]."""
    log_a = -DECAY_SCALE * np.asarray(decay_gate, F64) * softplus(lam)
    state = np.zeros(u.shape[1], F64)
    out = np.zeros(u.shape, F64)
    for t in range(u.shape[0]):
        a = np.exp(log_a[t])
        state = a * state + np.sqrt(-np.expm1(2.0 * log_a[t])) * input_gate[t] * u[t]
        out[t] = state
    return out


def recurrent(h, w):
    y = gelu_tanh(h @ w["y"].T + w["y.b"])
    u = short_convolution(h @ w["x"].T + w["x.b"], w["conv"], w["conv.b"])
    r = sigmoid(block_product(u, w["ra"], w["ra.b"]))
    i = sigmoid(block_product(u, w["ri"], w["ri.b"]))
    return (linear_recurrence(u, r, i, w["lam"]) * y) @ w["o"].T


# ----------------------------------------------------------------------------- attention within chunks
def visible(i: int, chunk):
    """Keys that query i sees: those of its chunk of positions up to its own (every earlier key without chunks)."""
    return range(i // chunk * chunk if chunk else 0, i + 1)


def attention_keys_values(h, w, m):
    n = h.shape[0]
    return ((h @ w["k"].T).reshape(n, m["kv_heads"], m["dim"]), (h @ w["v"].T).reshape(n, m["kv_heads"], m["vdim"]))


def attention(h, w, m, keys_values):
    """The mixer's result [T, width]; ``keys_values`` from this layer or from the one it shares with."""
    n, heads = h.shape[0], m["heads"]
    k, v = keys_values
    q = (h @ w["q"].T).reshape(n, heads, m["dim"])
    chunk = (m.get("mask") or {}).get("size")
    out = np.zeros((n, heads, m["vdim"]), F64)
    for t in range(n):
        js = visible(t, chunk)
        for a in range(heads):
            kv = a // (heads // m["kv_heads"])
            p = sink_weights(k[js.start:js.stop, kv] @ q[t, a] * m["scale"], float(w["sink"][a]))
            out[t, a] = p @ v[js.start:js.stop, kv]
    return out.reshape(n, heads * m["vdim"]) @ w["o"].T


# ----------------------------------------------------------------------------- latent attention
def latent_attention(h, w, m, eps):
    n = h.shape[0]
    heads, dim, rot, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    base = m["rot"]["base"]
    q = (h @ w["q"].T).reshape(n, heads, dim + rot)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :rank], w["dkv.norm"], eps)
    shared = np.stack([rotate_split_half(down[t, rank:], t, rot, base) for t in range(n)])
    k_plain = (c @ w["uk"].T).reshape(n, heads, dim)
    v = (c @ w["uv"].T).reshape(n, heads, vdim)
    out = np.zeros((n, heads, vdim), F64)
    for t in range(n):
        for a in range(heads):
            q_rot = rotate_split_half(q[t, a, dim:], t, rot, base)
            s = (k_plain[:t + 1, a] @ q[t, a, :dim] + shared[:t + 1] @ q_rot) * m["scale"]
            out[t, a] = sink_weights(s, float(w["sink"][a])) @ v[:t + 1, a]
    return out.reshape(n, heads * vdim) @ w["o"].T


# ----------------------------------------------------------------------------- feed-forward
def limited_gate(gate, up, limit: float):
    g = np.minimum(np.asarray(gate, F64), limit)
    u = np.clip(np.asarray(up, F64), -limit, limit)
    return g * sigmoid(GATE_ALPHA * g) * (u + 1.0)


def dense_ff(h, w, limit: float):
    act = limited_gate(h @ w["gate"].T + w["gate.b"], h @ w["up"].T + w["up.b"], limit)
    return act @ w["down"].T + w["down.b"]


# ----------------------------------------------------------------------------- the model
def _sub(tensors, prefix):
    return {k[len(prefix):]: np.asarray(v, F64) for k, v in tensors.items() if k.startswith(prefix)}


def forward(config, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence.  ``layers_out``: a list that receives the stream after every layer."""
    eps = config["norm"]["eps"]
    x = np.asarray(tensors["embed"], F64)[list(tokens)]
    kept = {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        w = _sub(tensors, p + "mix.")
        h = offset_norm(x, tensors[p + "norm1"], eps)
        if layer["type"] == "rglru":
            y = recurrent(h, w)
        elif layer["type"] == "attention":
            if m.get("kv_from") is None:
                kept[i] = attention_keys_values(h, w, m)
            y = attention(h, w, m, kept[i if m.get("kv_from") is None else m["kv_from"]])
        elif layer["type"] == "latent_attention":
            y = latent_attention(h, w, m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + offset_norm(y, tensors[p + "norm1b"], eps)
        if layer.get("mlp"):
            h = offset_norm(x, tensors[p + "norm2"], eps)
            x = x + offset_norm(dense_ff(h, _sub(tensors, p + "mlp."), layer["mlp"]["limit"]), tensors[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return offset_norm(x, tensors["final.norm"], eps) @ np.asarray(tensors["head"], F64).T
