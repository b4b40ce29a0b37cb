"""How a sublayer's result enters the residual stream (role ``add``), for layers that norm only what a sublayer reads."""
from __future__ import annotations

import torch

from ..core import ConfigError
from ..csrc import ops
from .norm import RMSNorm, WeightedParts
from .registry import register_part


class ScaledAdd:
    """x <- x + factor * y in 32-bit.  params: ``width``, ``factor``.  No weights.
    ``add_into(x, y, then)``: ``y`` float32 [T, width] or [parts, T, width] (added in index order), or a ``WeightedParts``
    of any form but one with a bias.  ``then``: the RMSNorm that the next sublayer begins with; its result over the new
    stream is returned, computed in the same pass (None where it is another kind of norm, or not given)."""

    graph_safe = True

    @classmethod
    def weight_shapes(cls, params):
        return {}

    def __init__(self, params, weights, dtype, device):
        self.width, self.factor = int(params["width"]), float(params["factor"])

    def add_into(self, x, y, then=None):
        options = {}
        if isinstance(y, WeightedParts):
            if y.bias is not None:
                raise ConfigError("a result that leaves a bias to be added cannot be scaled into the stream")
            options = {"rows": y.rows, "row_scales": y.row_scales, "scales": y.scales, "part_norms": y.norms,
                       "part_eps": y.eps}
            y = y.parts
        out = None
        if isinstance(then, RMSNorm) and then.width == self.width:
            out = torch.empty(x.shape, dtype=then.out_dtype, device=x.device)
            options["then"] = (then.weight, then.eps, out)
        ops.stream_add(x, y, self.factor, **options)
        return out


register_part("add", "scaled", ScaledAdd)
