"""Mixers that keep a matrix state per head instead of keys and values: gated linear attention, linear attention
with a constant decay a head, the gated delta
rule, and a delta rule with a decay and a removal rate per key channel (``DecayRemovalRule``, whose recurrence is in
its own text).  All run a scan over the tokens of a step (csrc/state_mixers.cu; where the decay is one number a head
csrc/head_scan.cu),

    S_t = diag(a_t) S_(t-1) + k_t u_t^T,        o_t = S_t^T q_t,

with S [key size, value size] per head, a_t a decay per key channel, and u_t = v_t (gated linear
attention) or u_t = b_t (v_t - (diag(a_t) S_(t-1))^T k_t) (delta rule: the state is corrected by what it
already answers for k_t; the read-out sees the write).  The state, the decays, the unit norms and the
head norms are 32-bit in both compute dtypes; products take their inputs in the compute dtype.

The state lives in the cache as a ``StateNeed``: zero when a slot opens, carried from step to step,
laid out [heads, value size, key size] (a column of S is contiguous, which is how the kernel holds it).
"""
from __future__ import annotations

import torch

from ..cache import StateNeed
from ..core import ConfigError, DType, torch_dtype
from ..csrc import ops
from .linear import linear
from .registry import register_part


def _vector(t):
    """Small tensors of the recurrence are kept in 32-bit whatever the compute dtype."""
    return t.to(torch.float32).contiguous()


class _StateMixer:
    graph_safe = True

    def forward(self, h, residual, ctx, store, owns_cache=True):
        ctx.then_norm = None
        linear(self.heads_out(h, ctx, store, owns_cache), self.w_o, accumulate_into=residual)

    def mix(self, h, ctx, store, owns_cache=True, out=None):
        ctx.then_norm = None
        return linear(self.heads_out(h, ctx, store, owns_cache), self.w_o, out_dtype=torch.float32, out=out)

    @staticmethod
    def _rows(ctx):
        """How to make a buffer that the per-sequence kernels fill: they skip rows of no sequence (the padding rows
        of a captured step), which must then hold zeros and not whatever the memory held."""
        padded = getattr(ctx, "captured", False) or sum(ctx.new_lens) < ctx.n_tokens  # a captured step is replayed with padding rows
        return torch.zeros if padded else torch.empty

    @staticmethod
    def _owning(owns_cache):
        if not owns_cache:
            raise ConfigError("a mixer with a state cannot read another place's: the state is what the tokens left there")


class GatedLinearAttention(_StateMixer):
    """q = W_q h / sqrt(key size), k = W_k h, v = W_v h; decay a = sigmoid(W_a2 (W_a1 h) + bias)^(1 / tau) per
    head and key channel; scan; every head's o RMS-normed over the value size with one shared weight, times
    silu(W_g h), then W_o.
    params: ``width``, ``n_heads``, ``key_dim``, ``value_dim``, ``decay_rank`` (rows of a1), ``tau``, ``eps``.
    weights: ``q``, ``k`` [heads * key_dim, width], ``v``, ``g`` [heads * value_dim, width], ``a1`` [rank, width],
    ``a2`` [heads * key_dim, rank], ``a2_bias`` [heads * key_dim], ``norm`` [value_dim], ``o`` [width, heads * value_dim]."""

    @classmethod
    def fused_weights(cls, params):
        return {"qkvg": ("q", "k", "v", "g")}

    @classmethod
    def weight_shapes(cls, params):
        d, nh, kd, vd, r = (params[k] for k in ("width", "n_heads", "key_dim", "value_dim", "decay_rank"))
        return {"q": ((nh * kd, d), "matrix"), "k": ((nh * kd, d), "matrix"), "v": ((nh * vd, d), "matrix"),
                "g": ((nh * vd, d), "matrix"), "a1": ((r, d), "matrix"), "a2": ((nh * kd, r), "matrix"),
                "a2_bias": ((nh * kd,), "vector"), "norm": ((vd,), "vector"), "o": ((d, nh * vd), "matrix")}

    def __init__(self, params, weights, dtype: DType, device):
        self.n_heads, self.key_dim, self.value_dim = (int(params[k]) for k in ("n_heads", "key_dim", "value_dim"))
        self.tau, self.eps = float(params["tau"]), float(params["eps"])
        if not self.tau > 0:
            raise ConfigError(f"tau {self.tau} must be positive")
        self.w_in = weights.get("qkvg")
        if self.w_in is None:
            self.w_in = torch.cat([weights[r] for r in ("q", "k", "v", "g")], dim=0).contiguous()
        self.w_a1, self.w_a2, self.w_o = weights["a1"], weights["a2"], weights["o"]
        self.a2_bias, self.norm = _vector(weights["a2_bias"]), _vector(weights["norm"])
        self.act_dtype = torch_dtype(dtype)

    def cache_need(self):
        return StateNeed((self.n_heads, self.value_dim, self.key_dim), "float32")

    def heads_out(self, h, ctx, store, owns_cache=True):
        self._owning(owns_cache)
        nh, kd, vd = self.n_heads, self.key_dim, self.value_dim
        n = h.shape[0]
        p = linear(h, self.w_in, out_dtype=torch.float32)
        decay = linear(linear(h, self.w_a1, out_dtype=self.act_dtype), self.w_a2, out_dtype=torch.float32)
        ops.decay_from_gate(decay, self.a2_bias, nh, kd, self.tau)
        o = self._rows(ctx)((n, nh * vd), dtype=torch.float32, device=h.device)
        ops.state_scan(o, p, p[:, nh * kd:], p[:, 2 * nh * kd:], decay, None, store.state, ctx.cu_seqlens, ctx.seq_slot,
                       nh, nh, kd, vd, q_scale=kd ** -0.5, max_new=ctx.max_new)
        y = torch.empty((n, nh * vd), dtype=self.act_dtype, device=h.device)
        ops.head_norm_gate(y, o, self.norm, p[:, 2 * nh * kd + nh * vd:], nh, vd, self.eps, "silu")
        return y


class GatedDeltaRule(_StateMixer):
    """q = W_q h, k = W_k h (``n_qk_heads`` heads of key_dim), v = W_v h (``n_heads`` heads of value_dim; head i
    uses q/k head i // (n_heads / n_qk_heads)); each passes a short causal convolution per channel and silu; q and
    k become unit vectors per head (x / sqrt(sum x^2 + 1e-6)), q times key_dim^(-1/2); b = sigmoid(W_b h) per
    head; decay a = exp(-exp(A_log[head]) * softplus(W_a2 (W_a1 h) + dt_bias)) per head and key channel; scan with
    the delta rule; every head's o divided by its root mean square (eps), times the shared weight ``norm``, times
    sigmoid(W_g2 (W_g1 h)); then W_o.  The last taps - 1 inputs of the convolutions are state as well.
    Without ``decay_rank`` and ``gate_rank`` (both or neither): ONE decay a head from a product ``a`` [heads, width]
    with ``dt_bias`` [heads], and the gate is a product ``g`` [heads * value_dim, width].  ``gate_act``: "sigmoid"
    (default) or "silu".
    params: ``width``, ``n_heads``, ``n_qk_heads``, ``key_dim``, ``value_dim``, ``taps``, ``decay_rank``,
    ``gate_rank``, ``eps``.
    weights: ``q``, ``k`` [qk heads * key_dim, width], ``v`` [heads * value_dim, width], ``q_conv``, ``k_conv``,
    ``v_conv`` [channels, taps], ``b`` [heads, width], ``A_log`` [heads], ``a1`` [decay_rank, width], ``a2``
    [heads * key_dim, decay_rank], ``dt_bias`` [heads * key_dim], ``g1`` [gate_rank, width], ``g2``
    [heads * value_dim, gate_rank], ``norm`` [value_dim], ``o`` [width, heads * value_dim]."""

    UNIT_EPS = 1e-6  # inside the root of the unit norms of q and k; a constant of the mixer

    @classmethod
    def _inputs(cls, params):
        """The matrices that one product of the mixer's input serves, in the order of its columns."""
        return ("q", "k", "v", "g", "b", "a") if cls._head_decay(params) else ("q", "k", "v", "b")

    @staticmethod
    def _head_decay(params) -> bool:
        if (params.get("decay_rank") is None) != (params.get("gate_rank") is None):
            raise ConfigError("a gated delta rule has low-rank products for both its decay and its gate, or for neither")
        return params.get("decay_rank") is None

    @classmethod
    def fused_weights(cls, params):
        if cls._head_decay(params):
            return {"qkvgba": cls._inputs(params)}
        return {"qkvb": cls._inputs(params), "a1g1": ("a1", "g1")}

    @classmethod
    def weight_shapes(cls, params):
        d, nh, nq, kd, vd, taps = (params[k] for k in ("width", "n_heads", "n_qk_heads", "key_dim", "value_dim", "taps"))
        shapes = {"q": ((nq * kd, d), "matrix"), "k": ((nq * kd, d), "matrix"), "v": ((nh * vd, d), "matrix"),
                  "b": ((nh, d), "matrix"), "q_conv": ((nq * kd, taps), "vector"), "k_conv": ((nq * kd, taps), "vector"),
                  "v_conv": ((nh * vd, taps), "vector"), "A_log": ((nh,), "vector"), "norm": ((vd,), "vector"),
                  "o": ((d, nh * vd), "matrix")}
        if cls._head_decay(params):
            shapes.update({"a": ((nh, d), "matrix"), "dt_bias": ((nh,), "vector"), "g": ((nh * vd, d), "matrix")})
        else:
            ra, rg = params["decay_rank"], params["gate_rank"]
            shapes.update({"a1": ((ra, d), "matrix"), "a2": ((nh * kd, ra), "matrix"), "dt_bias": ((nh * kd,), "vector"),
                           "g1": ((rg, d), "matrix"), "g2": ((nh * vd, rg), "matrix")})
        return shapes

    def __init__(self, params, weights, dtype: DType, device):
        self.n_heads, self.n_qk_heads, self.key_dim, self.value_dim, self.taps = (
            int(params[k]) for k in ("n_heads", "n_qk_heads", "key_dim", "value_dim", "taps"))
        self.head_decay = self._head_decay(params)
        self.decay_rank = int(params.get("decay_rank") or 0)
        self.gate_act = params.get("gate_act", "sigmoid")
        if self.gate_act not in ("sigmoid", "silu"):
            raise ConfigError(f"a delta rule's gate {self.gate_act!r} is not sigmoid or silu")
        self.eps = float(params["eps"])
        if self.n_heads % self.n_qk_heads:
            raise ConfigError(f"{self.n_heads} heads are not a multiple of {self.n_qk_heads} q/k heads")
        if not (1 <= self.taps <= 9):
            raise ConfigError(f"a short convolution of {self.taps} taps is outside 1 to 9")
        self.w_in = weights.get("qkvgba" if self.head_decay else "qkvb")
        if self.w_in is None:
            self.w_in = torch.cat([weights[r] for r in self._inputs(params)], dim=0).contiguous()
        self.w_o = weights["o"]
        if not self.head_decay:
            self.w_low = weights.get("a1g1")
            if self.w_low is None:
                self.w_low = torch.cat([weights["a1"], weights["g1"]], dim=0).contiguous()
            self.w_a2, self.w_g2 = weights["a2"], weights["g2"]
        self.conv = torch.cat([_vector(weights[r]) for r in ("q_conv", "k_conv", "v_conv")], dim=0).contiguous()
        self.a_log, self.dt_bias, self.norm = _vector(weights["A_log"]), _vector(weights["dt_bias"]), _vector(weights["norm"])
        self.channels = 2 * self.n_qk_heads * self.key_dim + self.n_heads * self.value_dim
        self.act_dtype = torch_dtype(dtype)

    def cache_need(self):
        needs = [StateNeed((self.n_heads, self.value_dim, self.key_dim), "float32")]
        if self.taps > 1:
            needs.append(StateNeed((self.taps - 1, self.channels), "float32"))
        return needs

    def heads_out(self, h, ctx, store, owns_cache=True):
        self._owning(owns_cache)
        nh, nq, kd, vd = self.n_heads, self.n_qk_heads, self.key_dim, self.value_dim
        n = h.shape[0]
        p = linear(h, self.w_in, out_dtype=torch.float32)          # q | k | v | b, or q | k | v | g | b | a
        if self.head_decay:
            return self._heads_out_one_decay(p, ctx, store)
        low = linear(h, self.w_low, out_dtype=self.act_dtype)      # a1 h | g1 h
        decay = linear(low[:, :self.decay_rank], self.w_a2, out_dtype=torch.float32)
        gate = linear(low[:, self.decay_rank:], self.w_g2, out_dtype=torch.float32)
        ops.decay_from_step(decay, self.dt_bias, self.a_log, nh, kd)
        qkv = self._rows(ctx)((n, self.channels), dtype=torch.float32, device=h.device)
        conv_state = store[1].state if self.taps > 1 else None
        ops.short_conv(qkv, p, self.conv, conv_state, ctx.cu_seqlens, ctx.seq_slot, ctx.max_new, "silu")
        ops.unit_heads(qkv, 2 * nq, kd, self.UNIT_EPS, scaled_heads=nq, scale=kd ** -0.5)
        o = self._rows(ctx)((n, nh * vd), dtype=torch.float32, device=h.device)
        ops.state_scan(o, qkv, qkv[:, nq * kd:], qkv[:, 2 * nq * kd:], decay, p[:, self.channels:], store[0].state,
                       ctx.cu_seqlens, ctx.seq_slot, nh, nq, kd, vd, delta=True, max_new=ctx.max_new)
        y = torch.empty((n, nh * vd), dtype=self.act_dtype, device=h.device)
        ops.head_norm_gate(y, o, self.norm, gate, nh, vd, self.eps, self.gate_act)
        return y

    def _heads_out_one_decay(self, p, ctx, store):
        nh, nq, kd, vd = self.n_heads, self.n_qk_heads, self.key_dim, self.value_dim
        n = p.shape[0]
        qkv = self._rows(ctx)((n, self.channels), dtype=torch.float32, device=p.device)
        conv_state = store[1].state if self.taps > 1 else None
        ops.short_conv(qkv, p, self.conv, conv_state, ctx.cu_seqlens, ctx.seq_slot, ctx.max_new, "silu")
        o = self._rows(ctx)((n, nh * vd), dtype=torch.float32, device=p.device)
        gate, beta = p[:, self.channels:], p[:, self.channels + nh * vd:]
        ops.head_scan(o, qkv, qkv[:, nq * kd:], qkv[:, 2 * nq * kd:], store[0].state, ctx.cu_seqlens, ctx.seq_slot, nh, nq,
                      kd, vd, decay_raw=beta[:, nh:], a_log=self.a_log, dt_bias=self.dt_bias, beta=beta,
                      q_scale=kd ** -0.5, unit_eps=self.UNIT_EPS, max_new=ctx.max_new)
        y = torch.empty((n, nh * vd), dtype=self.act_dtype, device=p.device)
        ops.head_norm_gate(y, o, self.norm, gate, nh, vd, self.eps, self.gate_act)
        return y


class ConstantDecayLinearAttention(_StateMixer):
    """q = silu(W_q h), k = silu(W_k h), v = silu(W_v h), head by head; S_t = decay_h S_(t-1) + k_t v_t^T,
    o_t = S_t^T q_t with one constant decay a head and no other scale; the heads side by side are RMS-normed together,
    times the weight ``norm``, times sigmoid(W_g h); then W_o.
    params: ``width``, ``n_heads``, ``key_dim``, ``value_dim``, ``decay`` (a number a head), ``eps``.
    weights: ``q``, ``k`` [heads * key_dim, width], ``v``, ``g`` [heads * value_dim, width], ``norm``
    [heads * value_dim], ``o`` [width, heads * value_dim]."""

    @classmethod
    def fused_weights(cls, params):
        return {"qkvg": ("q", "k", "v", "g")}

    @classmethod
    def weight_shapes(cls, params):
        d, nh, kd, vd = (params[k] for k in ("width", "n_heads", "key_dim", "value_dim"))
        return {"q": ((nh * kd, d), "matrix"), "k": ((nh * kd, d), "matrix"), "v": ((nh * vd, d), "matrix"),
                "g": ((nh * vd, d), "matrix"), "norm": ((nh * vd,), "vector"), "o": ((d, nh * vd), "matrix")}

    def __init__(self, params, weights, dtype: DType, device):
        self.n_heads, self.key_dim, self.value_dim = (int(params[k]) for k in ("n_heads", "key_dim", "value_dim"))
        self.eps = float(params["eps"])
        decay = [float(d) for d in params["decay"]]
        if len(decay) != self.n_heads:
            raise ConfigError(f"{len(decay)} decays for {self.n_heads} heads")
        self.decay = torch.tensor(decay, dtype=torch.float32, device=device)
        self.w_in = weights.get("qkvg")
        if self.w_in is None:
            self.w_in = torch.cat([weights[r] for r in ("q", "k", "v", "g")], dim=0).contiguous()
        self.w_o, self.norm = weights["o"], _vector(weights["norm"])
        self.act_dtype = torch_dtype(dtype)

    def cache_need(self):
        return StateNeed((self.n_heads, self.value_dim, self.key_dim), "float32")

    def heads_out(self, h, ctx, store, owns_cache=True):
        self._owning(owns_cache)
        nh, kd, vd = self.n_heads, self.key_dim, self.value_dim
        n = h.shape[0]
        p = linear(h, self.w_in, out_dtype=torch.float32)   # q | k | v | g
        o = self._rows(ctx)((n, nh * vd), dtype=torch.float32, device=h.device)
        qkv, single = p, ctx.max_new == 1  # (the scan of single tokens takes silu along; in portions it would do so many times)
        if not single:
            qkv = torch.empty((n, 2 * nh * kd + nh * vd), dtype=torch.float32, device=h.device)
            ops.act_cast(qkv, p[:, :2 * nh * kd + nh * vd], "silu")
        ops.head_scan(o, qkv, qkv[:, nh * kd:], qkv[:, 2 * nh * kd:], store.state, ctx.cu_seqlens, ctx.seq_slot, nh, nh, kd, vd,
                      decay=self.decay, silu=single, max_new=ctx.max_new)
        y = torch.empty((n, nh * vd), dtype=self.act_dtype, device=h.device)
        ops.head_norm_gate(y, o, self.norm, p[:, 2 * nh * kd + nh * vd:], 1, nh * vd, self.eps, "sigmoid")
        return y


class DecayRemovalRule(_StateMixer):
    """r = W_r h, k = W_k h, v = W_v h, all heads of ``dim``.  Per head and key channel a decay
    w = exp(-decay_rate * sigmoid(W_w2 tanh(W_w1 h) + w0)) and a removal rate a = sigmoid(W_a h + a_bias).  With the
    unit key n = k / sqrt(sum(k^2) + unit_eps) of a head, its state S [key, value] becomes
    S <- diag(w) S - (a * n) (n^T S) + k v^T, the decay and the removal both reading the state as the token found it,
    and o = S^T r.  Every head's o is divided by its root mean square (``eps``), times the weight ``norm`` (one a column
    of all heads), times sigmoid(W_g h); then W_o.  State, decays, rates, unit keys and head norms are 32-bit.
    params: ``width``, ``n_heads``, ``dim``, ``decay_rank`` (rows of w1), ``eps``, ``decay_rate``, ``unit_eps``.
    weights: ``r``, ``k``, ``v``, ``g``, ``a`` [heads * dim, width], ``a_bias``, ``w0``, ``norm`` [heads * dim],
    ``w1`` [decay_rank, width], ``w2`` [heads * dim, decay_rank], ``o`` [width, heads * dim]."""

    @classmethod
    def fused_weights(cls, params):
        return {"rkvgaw": ("r", "k", "v", "g", "a", "w1")}

    @classmethod
    def weight_shapes(cls, params):
        d, nh, hd, rank = (params[k] for k in ("width", "n_heads", "dim", "decay_rank"))
        shapes = {r: ((nh * hd, d), "matrix") for r in ("r", "k", "v", "g", "a")}
        shapes.update({"w1": ((rank, d), "matrix"), "w2": ((nh * hd, rank), "matrix"), "o": ((d, nh * hd), "matrix"),
                       "a_bias": ((nh * hd,), "vector"), "w0": ((nh * hd,), "vector"), "norm": ((nh * hd,), "vector")})
        return shapes

    def __init__(self, params, weights, dtype: DType, device):
        self.n_heads, self.dim, self.decay_rank = (int(params[k]) for k in ("n_heads", "dim", "decay_rank"))
        self.eps, self.decay_rate, self.unit_eps = (float(params[k]) for k in ("eps", "decay_rate", "unit_eps"))
        if not self.decay_rate > 0:
            raise ConfigError(f"decay_rate {self.decay_rate} must be positive")
        self.w_in = weights.get("rkvgaw")
        if self.w_in is None:
            self.w_in = torch.cat([weights[r] for r in ("r", "k", "v", "g", "a", "w1")], dim=0).contiguous()
        self.w_w2, self.w_o = weights["w2"], weights["o"]
        self.a_bias, self.w0, self.norm = _vector(weights["a_bias"]), _vector(weights["w0"]), _vector(weights["norm"])
        self.act_dtype = torch_dtype(dtype)

    def cache_need(self):
        return StateNeed((self.n_heads, self.dim, self.dim), "float32")

    def heads_out(self, h, ctx, store, owns_cache=True):
        self._owning(owns_cache)
        nh, hd = self.n_heads, self.dim
        n, w = h.shape[0], self.n_heads * self.dim
        p = linear(h, self.w_in, out_dtype=torch.float32)                   # r | k | v | g | a | w1 h
        low = torch.empty((n, self.decay_rank), dtype=self.act_dtype, device=h.device)
        ops.act_cast(low, p[:, 5 * w:], "tanh")
        decay = linear(low, self.w_w2, out_dtype=torch.float32)
        unit = torch.empty((n, w), dtype=torch.float32, device=h.device)
        removal = p[:, 4 * w:5 * w]
        ops.removal_gates(decay, self.w0, removal, self.a_bias, unit, p[:, w:2 * w], nh, hd, self.decay_rate, self.unit_eps)
        o = self._rows(ctx)((n, w), dtype=torch.float32, device=h.device)
        ops.state_scan(o, p, p[:, w:], p[:, 2 * w:], decay, None, store.state, ctx.cu_seqlens, ctx.seq_slot, nh, nh, hd, hd,
                       max_new=ctx.max_new, unit=unit, removal=removal)
        y = torch.empty((n, w), dtype=self.act_dtype, device=h.device)
        ops.head_norm_gate(y, o, self.norm, p[:, 3 * w:], nh, hd, self.eps, "sigmoid")
        return y


register_part("mixer", "decay_removal_rule", DecayRemovalRule)
register_part("mixer", "gated_linear_attention", GatedLinearAttention)
register_part("mixer", "gated_delta_rule", GatedDeltaRule)
register_part("mixer", "constant_decay_linear_attention", ConstantDecayLinearAttention)
