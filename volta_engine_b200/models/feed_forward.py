"""Feed-forwards of decoders whose ``config.json`` lists its layers. ``rows`` takes the rows a layer reads and returns the result's rows;
``step`` is the same on a few decode rows, reading the residual through the layer's norm and putting the result into it.
"""
from __future__ import annotations

import copy

import torch

from ..ops.routed import FEW_ROWS, ExpertWeights, Router, routed_few, routed_many, routed_reference
from ..ops.rowops import ClampedGlu, gemv_rows
from .mixers import apply_linear, make_linear


class DenseFF:
    """Linear, row operator, linear. In decode steps the operator is the epilogue of the first linear (``act.epilogue()``) or the
    prologue of the second."""

    def __init__(self, up, act, down):
        self.up, self.act, self.down = up, act, down

    @classmethod
    def gated(cls, src, p: str, unit: ClampedGlu, device, dtype) -> "DenseFF":
        """Tensors ``gate``, ``up`` and ``down`` under the prefix ``p``; gate and up rows in blocks where the widths allow it."""
        down = make_linear(src, p + "down", device, dtype)
        act = copy.copy(unit)
        act.blocks = down.in_features % 8 == 0
        return cls(make_linear(src, [p + "gate", p + "up"], device, dtype, join=ClampedGlu.interleave if act.blocks else None), act, down)

    def linears(self):
        return [self.up, self.down]

    def nbytes(self, step: bool = False) -> int:
        return self.up.nbytes() + self.down.nbytes()

    def rows(self, x, b):
        z = apply_linear(self.up, x, out_f32=b.row_path)
        return apply_linear(self.down, self.act.rows(z, x.dtype))

    def step(self, res, norm, write, b) -> None:
        epi = self.act.epilogue()
        z = gemv_rows(self.up, b.n, out_f32=epi is None, **res.read(norm), **(epi or {}))
        res.put(write)(self.down, **(self.act.prologue(z) if epi is None else {"x": z}))


class RoutedFF:
    """Mixture of experts: an fp32 router over all experts, gated units as experts (tensors ``router`` and ``e0.gate``, ``e0.up``,
    ``e0.down``, ... under the prefix). Prompt rows return their results unsummed where the norm behind can sum them."""

    def __init__(self, src, p: str, router: Router, unit: ClampedGlu, device, dtype):
        self.choice = router
        self.router = make_linear(src, p + "router", device, dtype)
        if self.router.out_features != router.experts:
            raise ValueError(f"{p}: a router over {self.router.out_features} of {router.experts} experts")
        gu = down = None
        for e in range(router.experts):                  # filled in place: no second copy of all experts
            g, u, d = (src.tensor(f"{p}e{e}.{n}", device, dtype) for n in ("gate", "up", "down"))
            if gu is None:
                (ff, W) = g.shape
                gu = torch.zeros(router.experts, 2 * ff, W + -W % 8, dtype=dtype, device=device)
                down = torch.zeros(router.experts, W, ff + -ff % 8, dtype=dtype, device=device)
            gu[e, :ff, :W], gu[e, ff:, :W], down[e, :, :ff] = g, u, d
        self.experts = ExpertWeights(gu, down, unit, ff)

    def linears(self):
        return [self.router]

    def nbytes(self, step: bool = False) -> int:
        n = self.experts.nbytes()
        return self.router.nbytes() + (n * self.choice.top // self.choice.experts if step else n)

    def rows(self, x, b):
        z = apply_linear(self.router, x, out_f32=True)
        if not x.is_cuda:
            return routed_reference(self.choice, self.experts, z, x, x.dtype)
        if x.dtype == torch.float32 or x.shape[0] <= FEW_ROWS:
            return routed_few(self.choice, self.experts, z, x, x.dtype)
        return routed_many(self.choice, self.experts, z, x)

    def step(self, res, norm, write, b) -> None:
        pro, x = res.read(norm), res.h
        if pro.get("b") is not None:                     # the experts read the normed row, which the router's linear stores
            x = pro["x_out"] = torch.empty(x.shape, dtype=torch.bfloat16, device=x.device)
        z = gemv_rows(self.router, b.n, out_f32=True, **pro)
        if getattr(write, "deferred", False):
            res.later(routed_few(self.choice, self.experts, z, x, torch.float32), write)
        elif write is None:
            routed_few(self.choice, self.experts, z, x, residual=res.h)
        else:
            raise NotImplementedError(f"routed results through {type(write).__name__}")
