"""Row operators of decoders with an fp32 residual stream, and the linears of their decode steps that take the operator in
front as a prologue (csrc/cuda/rowops.cu, gemv_rows.cu). CPU tensors run the same formulas in fp32 PyTorch.

Activations are bf16, or fp32 for the all-32-bit form of a model; the residual is always fp32 and every operator computes
in fp32.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .._lib import call, ptr

FUSED_ROWS = 8            # decode rows that take the prologue forms
FUSED_SMEM = 100 << 10


def _f32(t) -> int:
    return 1 if t.dtype == torch.float32 else 0


@dataclass
class DynamicTanh:
    """y = tanh(alpha x) * w + b: an element-wise stand-in for a norm layer (no statistics)."""
    w: torch.Tensor           # fp32
    b: torch.Tensor           # fp32
    alpha: float

    @classmethod
    def load(cls, src, name: str, device):
        return cls(src.tensor(name, device, torch.float32).contiguous(), src.tensor(name + ".b", device, torch.float32).contiguous(),
                   float(src.tensor(name + ".alpha").float()))

    def rows(self, h, out_dtype, part=None, scale=None):
        """h += scale * part (in place, optional), then the norm of h."""
        rows, H = h.shape
        if not h.is_cuda:
            if part is not None:
                h += part.float() * (scale if scale is not None else 1.0)
            return (torch.tanh(self.alpha * h) * self.w + self.b).to(out_dtype)
        out = torch.empty(rows, H, dtype=out_dtype, device=h.device)
        call("dyt_rows", "pplpppfpliii", ptr(h), ptr(part), part.stride(0) if part is not None else 0, ptr(scale), ptr(self.w), ptr(self.b),
             self.alpha, ptr(out), out.stride(0), rows, H, _f32(out))
        return out

    def prologue(self, h):
        return {"pro": 1, "x": h, "w": self.w, "b": self.b, "alpha": self.alpha}


@dataclass
class GroupRMS:
    """RMS norm over groups of ``group`` columns (0: the whole row) with a plain weight that repeats with its own length,
    optionally times sigmoid(gate) (``silu``: times silu(gate))."""
    w: torch.Tensor           # fp32
    eps: float
    group: int = 0
    silu: bool = False

    def rows(self, x, out_dtype, gate=None, out=None):
        rows, cols = x.shape
        G = self.group or cols
        if not x.is_cuda:
            v = x.float().reshape(rows, cols // G, G)
            v = (v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + self.eps)).reshape(rows, cols)
            v = v * self.w.repeat(cols // self.w.numel())
            if gate is not None:
                v = v * (torch.nn.functional.silu(gate.float()) if self.silu else torch.sigmoid(gate.float()))
            if out is None:
                return v.to(out_dtype)
            return out.copy_(v)
        if out is None:
            out = torch.empty(rows, cols, dtype=out_dtype, device=x.device)
        assert gate is None or gate.dtype == x.dtype
        call("group_rms", "plipipli" + "pliiifi", ptr(x), x.stride(0), _f32(x), ptr(self.w), self.w.numel(), ptr(gate),
             gate.stride(0) if gate is not None else 0, int(self.silu), ptr(out), out.stride(0), rows, cols, G, float(self.eps), _f32(out))
        return out

    def prologue(self, x, gate=None, head=None):
        """``head``: fp32 columns in front of the normed ones, taken as they are."""
        return {"pro": 2, "x": x, "w": self.w, "G": self.group or x.shape[1], "wlen": self.w.numel(), "gate": gate, "eps": self.eps,
                "head": head, "silu": self.silu}


@dataclass
class PolyNorm:
    """c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3 with N = division by the row's root mean square."""
    coef: torch.Tensor        # fp32 [4]
    eps: float

    def rows(self, z, out_dtype):
        rows, F = z.shape
        if not z.is_cuda:
            v = z.float()
            n = [p / torch.sqrt(p.pow(2).mean(-1, keepdim=True) + self.eps) for p in (v, v * v, v * v * v)]
            return (self.coef[0] * n[0] + self.coef[1] * n[1] + self.coef[2] * n[2] + self.coef[3]).to(out_dtype)
        out = torch.empty(rows, F, dtype=out_dtype, device=z.device)
        call("polynorm", "plipplii" + "fi", ptr(z), z.stride(0), _f32(z), ptr(self.coef), ptr(out), out.stride(0), rows, F, float(self.eps), _f32(out))
        return out

    def epilogue(self):
        return None             # statistics over the whole row

    def prologue(self, z):
        return {"pro": 3, "x": z, "coef": self.coef, "eps": self.eps}


@dataclass
class ClampedGlu:
    """Rows [gate | up]: g sigmoid(alpha g) (u + shift) with g = min(gate, limit), u = up clamped to +-limit. ``blocks``: the columns come
    as blocks of [4 gate | 4 up] (``interleave`` reorders a weight for it), which a decode linear can finish in its epilogue."""
    limit: float
    alpha: float
    blocks: bool = False
    shift: float = 1.0

    @classmethod
    def silu(cls, blocks: bool = False):
        """silu(gate) * up."""
        return cls(math.inf, 1.0, blocks, 0.0)

    @property
    def constants(self) -> tuple:
        return float(self.alpha), float(self.limit), float(self.shift)

    def of(self, g, u):
        """CPU statement on fp32 halves."""
        g = g.clamp(max=self.limit)
        return g * torch.sigmoid(self.alpha * g) * (u.clamp(-self.limit, self.limit) + self.shift)

    @staticmethod
    def interleave(gate, up):
        """Weights of the two halves [F, K] (F a multiple of 4) -> one weight whose outputs are in blocks."""
        F, K = gate.shape
        return torch.stack([gate.reshape(F // 4, 4, K), up.reshape(F // 4, 4, K)], 1).reshape(2 * F, K)

    def rows(self, z, out_dtype, by=None):
        """``by`` = (weights fp32, index int32 [rows]): row r of z is first multiplied with weights[index[r]]."""
        rows, F = z.shape[0], z.shape[1] // 2
        if not z.is_cuda:
            if by is not None:
                z = z.float() * by[0][by[1].long()][:, None]
            v = z.float().reshape(rows, F // 4, 2, 4).transpose(1, 2).reshape(rows, 2 * F) if self.blocks else z.float()
            return self.of(v[:, :F], v[:, F:]).to(out_dtype)
        out = torch.empty(rows, F, dtype=out_dtype, device=z.device)
        w, index = by if by is not None else (None, None)
        call("clamped_glu", "plipliiifffppi", ptr(z), z.stride(0), _f32(z), ptr(out), out.stride(0), rows, F, int(self.blocks), *self.constants, ptr(w), ptr(index), _f32(out))
        return out

    def epilogue(self):
        """Operands of a decode linear that ends with this operator; None: it goes into the prologue of the next one."""
        return {"glu": self.constants} if self.blocks else None

    def prologue(self, z):
        assert not self.blocks
        return {"pro": 5, "x": z, "kx": z.shape[1] // 2, "unit": self.constants}


@dataclass
class StreamWrite:
    """How a sublayer's result y enters residual streams [rows, streams, H]: x_t <- sum_s mix[s, t] x_s + out[t] y."""
    mix: torch.Tensor         # fp32 [streams, streams], [from, to]
    out: torch.Tensor         # fp32 [streams]

    def add(self, h, part):
        h.copy_(torch.einsum("rsd,st->rtd", h, self.mix) + self.out[:, None] * part.float()[:, None, :])


@dataclass
class StreamNorm:
    """Layer norm (weight, no shift) of the weighted sum of the residual streams [rows, streams, H]."""
    w: torch.Tensor           # fp32 [H]
    eps: float
    read: torch.Tensor        # fp32 [streams]

    def rows(self, h, out_dtype, part=None, write: StreamWrite | None = None):
        """The streams rewritten with ``part`` (in place, optional), then the norm of what is read from them."""
        rows, S, H = h.shape
        if not h.is_cuda:
            if part is not None:
                write.add(h, part)
            u = torch.einsum("rsd,s->rd", h, self.read)
            u = u - u.mean(-1, keepdim=True)
            return (u / torch.sqrt(u.pow(2).mean(-1, keepdim=True) + self.eps) * self.w).to(out_dtype)
        out = torch.empty(rows, H, dtype=out_dtype, device=h.device)
        call("stream_norm", "pplpppppliiifi", ptr(h), ptr(part), part.stride(0) if part is not None else 0, ptr(write.mix) if part is not None else 0,
             ptr(write.out) if part is not None else 0, ptr(self.read), ptr(self.w), ptr(out), out.stride(0), rows, H, S, float(self.eps), _f32(out))
        return out

    def prologue(self, h):
        S, H = h.shape[1:]
        return {"pro": 4, "x": h.view(h.shape[0], S * H), "kx": H, "w": self.w, "G": S, "coef": self.read, "eps": self.eps}


@dataclass
class RoutedRows:
    """Results of a routed feed-forward that are not summed yet: a row's result is sum_k w[row, k] d[inv[row, k]]."""
    d: torch.Tensor           # [routes, H]
    inv: torch.Tensor         # int32 [rows, top]
    w: torch.Tensor | None = None         # fp32 [rows, top] (None: all one)

    def tensor(self):
        rows, top = self.inv.shape
        d = self.d[self.inv.long().reshape(-1)].reshape(rows, top, -1).float()
        return (d.sum(1) if self.w is None else torch.einsum("rk,rkh->rh", self.w, d)).to(self.d.dtype)


@dataclass
class NormedWrite:
    """How a sublayer's result enters the residual behind a norm of its own: h += RMS norm(y) * w (a factor on it is part of w).
    Needs the whole row of y, so the linear that makes y cannot add it; the reader behind does (``ResidualNorm``)."""
    w: torch.Tensor           # fp32 [H]
    eps: float
    deferred = True

    def add(self, h, part):
        p = (part.tensor() if isinstance(part, RoutedRows) else part).float()
        h += p / torch.sqrt(p.pow(2).mean(-1, keepdim=True) + self.eps) * self.w


@dataclass
class ResidualNorm:
    """What is read of an fp32 residual: the residual itself (``w`` None) or its RMS norm. A sublayer's result enters it behind a norm of its
    own (``write``: NormedWrite) or as it is (None)."""
    w: torch.Tensor | None
    eps: float
    takes_routed = True

    @staticmethod
    def add(h, part, write: NormedWrite | None = None):
        """CPU statement: a result enters the residual."""
        if write is not None:
            write.add(h, part)
        else:
            h += (part.tensor() if isinstance(part, RoutedRows) else part).float()

    def rows(self, h, out_dtype, part=None, write: NormedWrite | None = None):
        """The result in front enters the residual (in place, optional), then what is read of it."""
        rows, H = h.shape
        if not h.is_cuda:
            if part is not None:
                self.add(h, part, write)
            v = h if self.w is None else h / torch.sqrt(h.pow(2).mean(-1, keepdim=True) + self.eps) * self.w
            return v.to(out_dtype)
        assert part is None or write is None or write.eps == self.eps
        out = torch.empty(rows, H, dtype=out_dtype, device=h.device)
        d, inv, w, top = (part.d, part.inv, part.w, part.inv.shape[1]) if isinstance(part, RoutedRows) else (part, None, None, 0)
        call("residual_norm", "pplppippplii" + "fi", ptr(h), ptr(d), d.stride(0) if d is not None else 0, ptr(inv), ptr(w), top,
             ptr(write.w) if part is not None and write is not None else 0, ptr(self.w), ptr(out), out.stride(0), rows, H, float(self.eps), _f32(out))
        return out

    def prologue(self, h, part=None, write: NormedWrite | None = None):
        """``h_out``: the residual with ``part`` (fp32) in it, stored by the linear."""
        assert part is None or write.eps == self.eps
        return {"pro": 6, "x": h, "part": part, "w": write.w if part is not None else None, "b": self.w, "eps": self.eps,
                "h_out": torch.empty(h.shape, dtype=torch.float32, device=h.device) if part is not None else None}


def soft_cap_(x, cap: float):
    """x <- cap tanh(x / cap), in place (fp32)."""
    if not x.is_cuda:
        return x.copy_(cap * torch.tanh(x / cap))
    call("soft_cap", "plf", ptr(x), x.numel(), float(cap))
    return x


class SinusoidalPositions:
    """Position vectors: sine in column 2i, cosine in 2i + 1 of position * base^(-2i / width). Half circles per position are kept
    in double, so that angles are exact at any position."""

    def __init__(self, width: int, base: float, device):
        i = torch.arange((width + 1) // 2, dtype=torch.float64)
        self.width = width
        self.freq = torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / width)
        self.half_turns = (self.freq / torch.pi).to(device)

    def vectors(self, pos):
        ang = pos.double()[:, None] * self.freq[None, :]
        return torch.stack([ang.sin(), ang.cos()], -1).flatten(1)[:, : self.width].float()


def embed_rows(ids, table, pos=None, positions: SinusoidalPositions | None = None, streams: int = 0, scale: float = 1.0):
    """-> fp32 [rows, H], times ``scale``; with ``positions`` their vectors of ``pos`` are added; with ``streams`` the rows come that many times
    ([rows, streams, H])."""
    S = max(1, streams)
    if not table.is_cuda:
        x = table[ids.long()].float() * scale
        if positions is not None:
            x = x + positions.vectors(pos)
        return x[:, None, :].repeat(1, S, 1) if streams else x
    V, H = table.shape
    n = ids.numel()
    out = torch.empty((n, S, H) if streams else (n, H), dtype=torch.float32, device=table.device)
    call("embed_rows", "pppppiiiifi", ptr(ids), ptr(table), ptr(pos) if positions is not None else 0, ptr(positions.half_turns) if positions is not None else 0,
         ptr(out), n, H, V, S, float(scale), _f32(table))
    return out


def fused_fits(lin, rows: int) -> bool:
    """The prologue form of ``lin`` takes this many rows."""
    return rows <= FUSED_ROWS and rows * (lin.weight.shape[1] + 64) * 2 <= FUSED_SMEM


def gemv_rows(lin, M: int, *, x, pro=0, kx=0, w=None, b=None, alpha=0.0, G=0, wlen=0, gate=None, coef=None, eps=0.0, head=None, silu=False,
              glu=None, unit=None, part=None, h_out=None, x_out=None, cap=0.0, out_f32=False, residual=None):
    """A bf16 linear (with its bias, if it has one) on ``M`` <= 16 rows. ``pro`` and its operands: the ``prologue`` dictionaries above (0: ``x`` is bf16).
    ``glu`` = (alpha, limit, shift): the clamped gated unit of its outputs, which come in blocks, in bf16. ``cap``: soft cap of fp32 outputs.
    ``residual`` = (h fp32, scale | None): h += scale * y in place, (streams, StreamWrite): the streams rewritten in place; otherwise
    the product is returned."""
    W = lin.weight
    N, K = W.shape
    dev = W.device
    if pro == 0 and x.shape[1] != K:              # weight rows padded to 16 bytes
        x = torch.nn.functional.pad(x, (0, K - x.shape[1]))
    k0 = head.shape[1] if head is not None else 0
    out = None
    if residual is None:
        N_out = N // 2 if glu else N
        out = torch.empty(M, N_out, dtype=torch.float32 if out_f32 else torch.bfloat16, device=dev)
    h, scale = residual if residual is not None else (None, None)
    streams, mix = 0, None
    if isinstance(scale, StreamWrite):
        streams, mix, scale = h.shape[1], scale.mix, scale.out
    call("gemv_rows", "pliiiii" + "plppfiiplpf" + "pplplp" + "pliiifffip" + "fplppp", ptr(W), W.stride(0), N, K, M, pro, kx or k0 + x.shape[1], ptr(x), x.stride(0), ptr(w), ptr(b),
         float(alpha), G, wlen, ptr(gate), gate.stride(0) if gate is not None else 0, ptr(coef), float(eps),
         ptr(out) if out_f32 else 0, ptr(out) if out is not None and not out_f32 else 0, out.stride(0) if out is not None else 0, ptr(h), h.stride(0) if h is not None else 0, ptr(scale),
         ptr(head), head.stride(0) if head is not None else 0, k0, int(silu), int(glu is not None), *(glu or unit or (0.0, 0.0, 0.0)), streams, ptr(mix),
         float(cap), ptr(part), part.stride(0) if part is not None else 0, ptr(h_out), ptr(x_out), ptr(getattr(lin, "bias", None)))
    return out
