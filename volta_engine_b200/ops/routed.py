"""Routed feed-forwards (mixture of experts) with bf16 or fp32 weights for decoders with an fp32 residual (csrc/cuda/routed.cu; prompt
rows: csrc/cuda/moe.cu sorts the routes, gemm_tcgen05.cu multiplies them expert by expert). CPU tensors run the same formulas in
PyTorch.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .._lib import call, ptr
from . import kernels as K
from .rowops import ClampedGlu, RoutedRows

MAX_EXPERTS, MAX_TOP = 1024, 32           # of the kernels
FEW_ROWS = 16                             # rows that run route by route


@dataclass
class Router:
    """Scores are the softmax over all experts, or (``sigmoid``) the sigmoid of every logit, in fp32. With ``groups`` > ``keep`` the experts form equal groups of neighbours, of which
    the ``keep`` best stay open; a group's score is its best member's (``best2``: the sum of its two best). The ``top`` best open experts
    are taken, their scores are the weights (``renorm``: over their sum), times ``factor``. Ties go to the lower index. A weight multiplies
    its expert's output, or (``weigh_input``) what the expert reads."""
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    best2: bool = False
    renorm: bool = False
    factor: float = 1.0
    sigmoid: bool = False
    weigh_input: bool = False

    def __post_init__(self):
        if self.experts > MAX_EXPERTS or self.top > MAX_TOP:
            raise NotImplementedError(f"{self.top} of {self.experts} experts (at most {MAX_TOP} of {MAX_EXPERTS})")
        if self.groups < 1 or self.experts % self.groups or not 1 <= self.keep <= self.groups or not 1 <= self.top <= self.keep * (self.experts // self.groups):
            raise ValueError(f"{self.top} of {self.experts} experts out of {self.keep} of {self.groups} groups")

    def choose(self, z):
        """CPU statement: logits [rows, experts] -> (experts int32 [rows, top], weights fp32 [rows, top])."""
        s = torch.sigmoid(z.float()) if self.sigmoid else torch.softmax(z.float(), -1)
        rows = s.shape[0]
        rank = open_ = z.float() if self.sigmoid else s                  # (sigmoids near one cannot be told apart)
        if self.keep < self.groups:
            g = rank.reshape(rows, self.groups, -1)
            gs = s.reshape(g.shape).topk(min(2, g.shape[2]), -1).values.sum(-1) if self.best2 else g.amax(-1)
            best = torch.sort(gs, dim=-1, descending=True, stable=True).indices[:, : self.keep]
            kept = torch.zeros_like(gs, dtype=torch.bool).scatter_(1, best, True)
            open_ = torch.where(kept[:, :, None], g, torch.full_like(g, -torch.inf)).reshape(rows, -1)
        ids = torch.sort(open_, dim=-1, descending=True, stable=True).indices[:, : self.top]
        w = s.gather(1, ids)
        if self.renorm:
            w = w / w.sum(-1, keepdim=True)
        return ids.int(), w * self.factor

    @property
    def args(self):
        return self.experts, self.top, self.groups, self.keep, int(self.best2), int(self.renorm), float(self.factor), int(self.sigmoid)


_R = "iiiiiifi"


class ExpertWeights:
    """gate_up [experts, 2 ff, width] (gate rows, then up rows) and down [experts, width, ff], rows padded with zeros to 16 bytes."""

    def __init__(self, gate_up, down, unit: ClampedGlu, ff: int):
        self.experts, self.width = down.shape[:2]
        self.ff, self.gate_up, self.down, self.unit = ff, gate_up, down, unit

    def nbytes(self) -> int:
        return (self.gate_up.numel() + self.down.numel()) * self.down.element_size()


def route(router: Router, z):
    """Router logits fp32 [rows, experts] -> (experts int32 [rows, top], weights fp32 [rows, top])."""
    if not z.is_cuda:
        return router.choose(z)
    ids = torch.empty(z.shape[0], router.top, dtype=torch.int32, device=z.device)
    w = torch.empty(z.shape[0], router.top, dtype=torch.float32, device=z.device)
    call("route_rows", _R + "plppi", *router.args, ptr(z), z.stride(0), ptr(ids), ptr(w), z.shape[0])
    return ids, w


def routed_reference(router: Router, ex: ExpertWeights, z, x, out_dtype):
    """CPU statement: every chosen expert on its rows; what a matrix product gives or takes is rounded to the weights' type."""
    dt = ex.down.dtype
    ids, w = router.choose(z)
    x = x.to(dt).float()
    y = torch.zeros(x.shape[0], ex.width)
    for e in ids.unique().tolist():
        r, k = (ids == e).nonzero(as_tuple=True)
        gu = x[r] @ ex.gate_up[e, :, : ex.width].float().t()
        f = w[r, k, None]
        if router.weigh_input:
            gu, f = gu * f, 1.0
        a = ex.unit.of(gu[:, : ex.ff], gu[:, ex.ff:]).to(dt).float()
        y.index_add_(0, r, f * (a @ ex.down[e, :, : ex.ff].float().t()))
    return y.to(out_dtype)


def routed_few(router: Router, ex: ExpertWeights, z, x, out_dtype=None, residual=None):
    """Rows one by one: two launches, the first routes too. ``x``: rows of the weights' type, or fp32 (rounded to it). ``residual``: fp32 rows
    that the results are added to (nothing is returned)."""
    n, dev, dt = x.shape[0], x.device, ex.down.dtype
    f32 = int(dt == torch.float32)
    ids = torch.empty(n, router.top, dtype=torch.int32, device=dev)
    w = torch.empty(n, router.top, dtype=torch.float32, device=dev)
    a = torch.empty(n * router.top, ex.ff, dtype=dt, device=dev)
    call("routed_up", _R + "plplipl" + "plpp" + "iiifffii", *router.args, ptr(z), z.stride(0), ptr(x), x.stride(0), int(x.dtype == torch.float32), ptr(ex.gate_up),
         ex.gate_up.stride(1), ptr(a), a.stride(0), ptr(ids), ptr(w), n, ex.width, ex.ff, *ex.unit.constants, int(router.weigh_input), f32)
    out = torch.empty(n, ex.width, dtype=out_dtype, device=dev) if residual is None else residual
    call("routed_down", "plplppiplii" + "iiii", ptr(a), a.stride(0), ptr(ex.down), ex.down.stride(1), ptr(ids), 0 if router.weigh_input else ptr(w), router.top, ptr(out),
         out.stride(0), int(out.dtype == torch.float32), n, ex.width, ex.ff, int(residual is not None), f32)
    return out if residual is None else None


def routed_many(router: Router, ex: ExpertWeights, z, x) -> RoutedRows:
    """bf16 rows of a prompt: routes sorted by expert, gate and up, unit and down over all of them."""
    n, dev, top = x.shape[0], x.device, router.top
    ids, w = route(router, z)
    routes = n * top
    per = routes / ex.experts
    bn = 16 if per <= 8 else 32 if per <= 24 else 64 if per <= 96 else 128 if per <= 512 else 256
    tiles = routes // bn + ex.experts + 1
    inv, order = torch.empty(n, top, dtype=torch.int32, device=dev), torch.empty(routes, dtype=torch.int32, device=dev)
    tab, totals = torch.empty(tiles, 4, dtype=torch.int32, device=dev), torch.empty(2, dtype=torch.int32, device=dev)
    call("moe_sort", "piiiipppip", ptr(ids), routes, 0, ex.experts, bn, ptr(inv), ptr(order), ptr(tab), tiles, ptr(totals))
    st = K.status_word(dev)
    if x.shape[1] % 8 or x.stride(0) % 8:                    # rows of whole 16-byte pieces for the copies
        x = torch.nn.functional.pad(x, (0, -x.shape[1] % 8)).contiguous()
    xs = torch.empty(routes, x.shape[1], dtype=x.dtype, device=dev)
    call("moe_gather", "plppiplii", ptr(x), x.stride(0), ptr(order), ptr(totals), top, ptr(xs), xs.stride(0), x.shape[1], routes)

    def grouped(W, a, cols, k):
        out = torch.empty(routes, cols, dtype=a.dtype, device=dev)
        call("gemm_grouped_bf16", "plplpliiiiipip", ptr(W), W.stride(1), ptr(a), a.stride(0), ptr(out), out.stride(0), routes, ex.experts, cols, k, bn, ptr(tab),
             tiles, ptr(st))
        return out
    by = (w.reshape(-1), order) if router.weigh_input else None
    a = ex.unit.rows(grouped(ex.gate_up, xs, 2 * ex.ff, ex.width), x.dtype, by)
    if ex.ff % 8:
        a = torch.nn.functional.pad(a, (0, -ex.ff % 8))
    return RoutedRows(grouped(ex.down, a, ex.width, ex.ff), inv, None if router.weigh_input else w)
