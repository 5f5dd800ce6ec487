"""What a layer adds to the stream from the token itself: a small row per token and layer, read from a table."""

from __future__ import annotations

import torch

from ..kernels import ops
from .base import Runtime, register_token_side
from .util import matrix, vector


@register_token_side("gated_rows")
class GatedTokenRows:
    """x + rms_norm(W_proj (gelu(W_gate x) * e)), e the token's row of a table (gelu in its tanh form; the norm with a plain gain per
    coordinate). The table may hold the rows of several layers side by side; this part takes the `dim` columns from `column` on.

    params: column, dim, eps. weights (matrices stored [out, in]): table [V, >= column + dim], gate [dim, D], proj [D, dim], norm [D]."""

    gathered = ("table",)   # read by rows, not as a whole

    def __init__(self, params: dict, weights: dict, rt: Runtime):
        at, dim, self.eps = int(params["column"]), int(params["dim"]), float(params["eps"])
        table, gate, proj = weights["table"], weights["gate"], weights["proj"]
        if at < 0 or table.shape[1] < at + dim or gate.shape[0] != dim or tuple(proj.shape) != (gate.shape[1], dim) or weights["norm"].shape[0] != gate.shape[1]:
            raise ValueError(f"token rows: table {tuple(table.shape)}, gate {tuple(gate.shape)}, proj {tuple(proj.shape)} do not fit {dim} columns from {at} on")
        self.table = matrix(table[:, at: at + dim], rt)
        self.gate, self.proj = matrix(gate, rt), matrix(proj, rt)
        self.norm = vector(weights["norm"], rt)

    def join(self, x, h, ctx, rounded_dtype=None):
        """x: the stream's rows in float32, h: the same rows in the compute dtype -> (new x, its rows in `rounded_dtype` or None)."""
        y = ops.gated_token_rows(ops.linear(h, self.gate, None, w_is_nk=True, out_dtype=torch.float32), ctx.input_ids, self.table)
        y = ops.linear(y, self.proj, None, w_is_nk=True, out_dtype=torch.float32)
        if rounded_dtype is None:
            return ops.norm_add(x, y, self.norm, self.eps), None
        return ops.norm_add(x, y, self.norm, self.eps, rounded_dtype=rounded_dtype)
