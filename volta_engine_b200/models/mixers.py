"""Token mixers of decoders whose ``config.json`` lists its layers one by one, each with its own mixer type and sizes. A mixer
reads normed rows and returns the rows of its output projection; ``step`` is the same on a few decode rows with the norm in
front, the layer scale and the residual add inside the linears' launches.

``MIXERS`` maps the type names to classes; a class takes (mixer sizes, eps, tensor source, name prefix, device, dtype).
"""
from __future__ import annotations

import torch

from ..ops.latent import LatentSpec, latent_rows
from ..ops.linear import LinearBF16, LinearF32
from ..ops.linear_attn import LinAttnSpec, LinAttnState, linattn_rows
from ..ops.rowops import GroupRMS, gemv_rows


def make_linear(src, names, device, dtype):
    """One linear computing the stacked outputs of the tensors ``names``."""
    names = [names] if isinstance(names, str) else names
    w = torch.cat([src.tensor(n, device, dtype) for n in names], 0) if len(names) > 1 else src.tensor(names[0], device, dtype)
    return LinearF32(w) if dtype == torch.float32 else LinearBF16(w)


def apply_linear(lin, x, out_f32: bool = False):
    """``lin`` on rows of its activation type: the decode kernel up to 16 rows, the tensor-core GEMM above."""
    if x.is_cuda and isinstance(lin, LinearBF16) and x.shape[0] <= 16:
        return gemv_rows(lin, x.shape[0], x=x, out_f32=out_f32)
    return lin.forward(x, out_f32=out_f32)


class LinearRecurrence:
    """HGRN2 and lightning attention: one fused input projection [q | forget gate or k | v | gate], the decayed outer-product
    recurrence, an RMS norm of its output (per head, or over all heads and gated), the output projection."""
    cached = False

    def __init__(self, kind: str, m: dict, eps: float, src, p: str, device, dtype):
        H, dk, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        f32 = lambda name: src.tensor(p + name, device, torch.float32).reshape(-1).contiguous()
        self.gated = kind == "lightning"
        if kind == "lightning":
            decay = m["decay"] if isinstance(m["decay"], (list, tuple)) else [m["decay"]] * H
            self.spec = LinAttnSpec(H, dk, dv, decay=torch.tensor([float(d) for d in decay], dtype=torch.float32, device=device))
            if self.spec.decay.numel() != H:
                raise ValueError(f"{p}: {self.spec.decay.numel()} decays for {H} heads")
        else:
            self.spec = LinAttnSpec(H, dk, dv, lower=f32("lower"), bias=f32("f.b"))
        self.in_proj = make_linear(src, [p + n for n in (("q", "k", "v", "g") if self.gated else ("q", "f", "v"))], device, dtype)
        self.out = make_linear(src, p + "o", device, dtype)
        self.norm = GroupRMS(f32("norm"), eps, 0 if self.gated else dv)
        self.dtype = dtype
        self.state: LinAttnState | None = None

    def bind(self, kv):
        if self.state is None:
            self.state = LinAttnState(self.spec, kv.max_slots, kv.page_table.device)
        return self.state

    def linears(self):
        return [self.in_proj, self.out]

    def _gate(self, proj):
        return proj[:, self.spec.cols:] if self.gated else None

    def rows(self, x, b, kv, journal=(None, None)):
        proj = apply_linear(self.in_proj, x, out_f32=True)         # gates and keys enter the recurrence unrounded
        o = linattn_rows(proj, b, self.bind(kv), self.spec, *journal, chunked=self.dtype != torch.float32)
        y = self.norm.rows(o, self.dtype, gate=self._gate(proj))
        return apply_linear(self.out, y)

    def step(self, pro, residual, b, kv, journal=(None, None)):
        proj = gemv_rows(self.in_proj, b.n, out_f32=True, **pro)
        o = linattn_rows(proj, b, self.bind(kv), self.spec, *journal)
        gemv_rows(self.out, b.n, residual=residual, **self.norm.prologue(o, self._gate(proj)) if self.gated else self.norm.prologue(o))


class LatentAttention:
    """Multi-head attention over a low-rank latent per token, with a low-rank query and a rotated key part shared by the heads."""
    cached = True                   # owns one layer of the paged cache (``cache_index``)
    state = None

    def __init__(self, kind: str, m: dict, eps: float, src, p: str, device, dtype):
        rot = m["rot"]
        if int(rot["dims"]) != int(m["rot_dim"]):
            raise ValueError(f"{p}: the rotated part is turned as a whole")
        self.spec = LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]),
                               float(rot["base"]), eps).bind(device)
        self.q_rank = int(m["q_rank"])
        f32 = lambda name: src.tensor(p + name, device, torch.float32).reshape(-1).contiguous()
        self.down = make_linear(src, [p + "dq", p + "dkv"], device, dtype)
        self.uq = make_linear(src, p + "uq", device, dtype)
        self.w_uk = src.tensor(p + "uk", device, dtype).contiguous()
        self.w_uv = src.tensor(p + "uv", device, dtype).contiguous()
        self.ukv = LinearBF16(torch.cat([self.w_uk, self.w_uv], 0)) if dtype != torch.float32 else None
        if self.ukv is not None and self.ukv.weight.shape[1] == self.spec.kv_rank:      # one copy: the absorbed form reads slices of the stacked weight
            self.w_uk, self.w_uv = self.ukv.weight[: self.w_uk.shape[0]], self.ukv.weight[self.w_uk.shape[0]:]
        self.out = make_linear(src, p + "o", device, dtype)
        self.q_norm = GroupRMS(f32("dq.norm"), eps)
        self.kv_norm = f32("dkv.norm")
        self.dtype = dtype
        self.cache_index = -1

    def linears(self):
        return [self.down, self.uq, self.out]

    def extra_bytes(self) -> int:
        return (self.w_uk.numel() + self.w_uv.numel()) * self.w_uk.element_size()

    def _attend(self, q, a, b, kv):
        return latent_rows(self.spec, q, a[:, self.q_rank:], self.kv_norm, self.w_uk, self.w_uv, self.ukv, b, kv, kv.k[self.cache_index])

    def rows(self, x, b, kv, journal=None):
        a = apply_linear(self.down, x, out_f32=True)
        q = apply_linear(self.uq, self.q_norm.rows(a[:, : self.q_rank], self.dtype), out_f32=x.shape[0] <= 16)
        return apply_linear(self.out, self._attend(q, a, b, kv))

    def step(self, pro, residual, b, kv, journal=None):
        a = gemv_rows(self.down, b.n, out_f32=True, **pro)
        q = gemv_rows(self.uq, b.n, out_f32=True, **self.q_norm.prologue(a[:, : self.q_rank]))
        att = self._attend(q, a, b, kv)
        gemv_rows(self.out, b.n, residual=residual, x=att)


MIXERS = {"hgrn2": LinearRecurrence, "lightning": LinearRecurrence, "latent_attention": LatentAttention}
