"""What stands before a pass of a stretch of layers that runs several times (``ModelSpec.loop``).

    x <- A x + B x0 + S[t]          one stored matrix W = [A | B] [H, 2 H];  x0 the rows that entered the first layer;  t the pass

B x0 is the same in every pass of a step, so it is made once, from the embedded rows, before any layer runs (``begin``), and
the stored matrix is kept as its two halves; a pass (``enter``) is then one element-wise kernel, which leaves the rows rounded for the
product and starts the sum with B x0 + S[t], and one product with A that adds into the residual stream.  Both sums are
float32.  Nothing outlasts its step.
"""
from __future__ import annotations

from typing import List

import torch

from .. import kernels as K
from ..weights.loader import WeightSpec
from . import linear
from .base import Part


class LoopEntry(Part):
    def __init__(self, spec, width: int):
        self.spec, self.W = spec, width
        self.w_x = self.w_x0 = self.step = None

    def weight_specs(self, prefix: str = "") -> List[WeightSpec]:
        s, out = self.spec, []
        if s.mix is not None:
            out.append(WeightSpec(prefix + s.mix, (self.W, 2 * self.W)))
        if s.step is not None:
            out.append(WeightSpec(prefix + s.step, (s.times, self.W), "vector", ("normal", 0.1)))
        return out

    def bind(self, get) -> None:
        s = self.spec
        if s.mix is not None:
            w = get(s.mix)
            self.w_x, self.w_x0 = w[:, :self.W].contiguous(), w[:, self.W:].contiguous()
        if s.step is not None:
            self.step = get(s.step).contiguous()

    def begin(self, x: torch.Tensor, ctx) -> None:
        """Before the first layer of a step: x are the rows that every pass is given again."""
        if self.w_x0 is None:
            return
        rows = x
        if ctx.dtype != torch.float32:
            rows = ctx.empty(tuple(x.shape))
            K.round_rows(x, rows, ctx.stream)
        base = ctx.carried["loop_base"] = ctx.empty(tuple(x.shape), torch.float32)
        linear.matmul(rows, self.w_x0, base, linear.EPI_F32, ctx)

    def enter(self, x: torch.Tensor, ctx, t: int) -> None:
        """Before the first layer of pass ``t``; x in place."""
        for made_ahead in ("normed_rows", "rounded_rows"):     # what a block prepared from the rows as they were
            ctx.carried.pop(made_ahead, None)
        step = None if self.step is None else self.step[t]
        if self.w_x is None:
            if step is not None:
                K.pass_entry(x, None, step, None, ctx.stream)
            return
        rows = ctx.empty(tuple(x.shape))
        K.pass_entry(x, ctx.carried["loop_base"], step, rows, ctx.stream)
        linear.matmul(rows, self.w_x, x, linear.EPI_ADD, ctx)
