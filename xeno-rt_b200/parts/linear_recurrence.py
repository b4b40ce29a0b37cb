"""A mixer whose state is ONE number a channel: the recurrent block with a real-gated linear recurrent unit (De et al.,
"Griffin: Mixing Gated Linear Recurrences with Local Attention for Efficient Language Models").

    y = gelu_tanh(W_y h + b_y),   u = conv(W_x h + b_x)        (a short causal convolution a channel with a bias)
    r = sigmoid(R u + b_r),   i = sigmoid(I u + b_i)           (one square matrix a block of neighbouring channels)
    log a = -decay_scale * r * softplus(lam)
    S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t,   out = W_o (S * y)

The state S (float32, zero when a slot opens) and the convolution's inputs of the last ``taps`` positions (a ring, position
p at entry p % taps) are the sequence's state.  From the branches' products on everything is 32-bit in both compute
dtypes, the gates' products too: in bfloat16 their matrices meet u as a sum of three bfloat16 numbers on the tensor
cores (csrc/linear_recurrence.cu)."""
from __future__ import annotations

import torch

from ..cache import StateNeed
from ..core import ConfigError, DType, torch_dtype
from ..csrc import ops
from .linear import linear
from .registry import register_part
from .state_mixers import _StateMixer, _vector


class GatedLinearRecurrence(_StateMixer):
    """params: ``width`` (model width), ``inner`` (channels), ``blocks``, ``taps``, ``decay_scale``.
    weights: ``y``, ``x`` [inner, width] with ``y_bias``, ``x_bias`` [inner]; ``conv`` [inner, taps], ``conv_bias`` [inner];
    ``r``, ``i`` [blocks, inner / blocks, inner / blocks] ([out, in] each) with ``r_bias``, ``i_bias`` [blocks, inner /
    blocks]; ``lam`` [inner]; ``o`` [width, inner]."""

    @classmethod
    def fused_weights(cls, params):
        return {"yx": ("y", "x")}

    @classmethod
    def weight_shapes(cls, params):
        d, n, blocks, taps = (params[k] for k in ("width", "inner", "blocks", "taps"))
        size = n // blocks
        return {"y": ((n, d), "matrix"), "x": ((n, d), "matrix"), "y_bias": ((n,), "vector"), "x_bias": ((n,), "vector"),
                "conv": ((n, taps), "vector"), "conv_bias": ((n,), "vector"), "r": ((blocks, size, size), "matrix"),
                "i": ((blocks, size, size), "matrix"), "r_bias": ((blocks, size), "vector"),
                "i_bias": ((blocks, size), "vector"), "lam": ((n,), "vector"), "o": ((d, n), "matrix")}

    def __init__(self, params, weights, dtype: DType, device):
        self.inner, self.blocks, self.taps = (int(params[k]) for k in ("inner", "blocks", "taps"))
        if self.inner % self.blocks:
            raise ConfigError(f"{self.inner} channels do not form {self.blocks} equal blocks")
        if not 1 <= self.taps <= 9:
            raise ConfigError(f"a short convolution of {self.taps} taps is outside 1 to 9")
        self.w_in = weights.get("yx")
        if self.w_in is None:
            self.w_in = torch.cat([weights["y"], weights["x"]], dim=0).contiguous()
        self.w_o = weights["o"]
        lam = weights["lam"].to(torch.float64)
        rate = (-float(params["decay_scale"]) * torch.nn.functional.softplus(lam, threshold=1e9)).to(torch.float32)
        r, i = weights["r"].contiguous(), weights["i"].contiguous()
        self.one_launch = dtype is DType.BF16 and r.shape[1] % 8 == 0  # a step of single tokens, with bfloat16 matrices
        if not self.one_launch:  # matrices whose rows the vector loads do not take are kept in 32-bit
            r, i = _vector(r), _vector(i)
        flat = lambda role: _vector(weights[role]).reshape(-1)
        self.weights = ops.RecurrenceWeights(
            y_bias=flat("y_bias"), x_bias=flat("x_bias"), conv=_vector(weights["conv"]), conv_bias=flat("conv_bias"),
            r_bias=flat("r_bias"), i_bias=flat("i_bias"), rate=rate.contiguous(), r=r, i=i)
        self.act_dtype = torch_dtype(dtype)

    def cache_need(self):
        needs = [StateNeed((self.inner,), "float32")]
        if self.taps > 1:
            needs.append(StateNeed((self.taps, self.inner), "float32"))
        return needs

    def heads_out(self, h, ctx, store, owns_cache=True):
        self._owning(owns_cache)
        n = h.shape[0]
        p = linear(h, self.w_in, out_dtype=torch.float32)   # y | x
        state, ring = store[0].state, store[1].state if self.taps > 1 else None
        if self.one_launch and ctx.all_single:
            out = torch.empty((n, self.inner), dtype=self.act_dtype, device=h.device)
            ops.linear_recurrence_step(out, p, self.weights, state, ring, ctx.tok_slot, ctx.tok_pos, ctx.cu_seqlens,
                                       ctx.seq_slot, ctx.seq_start)
            return out
        out = self._rows(ctx)((n, self.inner), dtype=self.act_dtype, device=h.device)
        ops.linear_recurrence(out, p, self.weights, state, ring, ctx.cu_seqlens, ctx.seq_slot, ctx.seq_start, ctx.max_new)
        return out


register_part("mixer", "gated_linear_recurrence", GatedLinearRecurrence)
