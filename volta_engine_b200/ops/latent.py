"""Latent attention with its sizes as parameters (csrc/cuda/latent.cu, the decode kernel in mla.cu): queries of ``dim`` plain and
``rot`` rotated columns per head, one cached row per token [ latent c (kv_rank) | rotated key part (rot) ] shared by all heads,
keys W_uk c and values W_uv c per head. Rotation pairs are neighbouring columns; frequencies may be scaled (ops/rotary.py). A sliding
window hides the keys in front of it.

Decode rows run the absorbed form over the paged rows; prompt portions expand keys and values of their sequence and run a
flash kernel; the all-32-bit form, and sizes outside the tensor-core kernels' range, run the absorbed form on the CUDA cores.
"""
from __future__ import annotations

import os
from dataclasses import dataclass

import torch

from .._lib import call, ptr
from . import kernels as K
from .rotary import Rotation

PAGE = K.PAGE
# prompt rows on the tcgen05 kernel where it applies; "mma" keeps the mma.sync kernel
TC_PREFILL = os.environ.get("VOLTA_LATENT_PREFILL", "tc") != "mma"


def _up(n: int, m: int) -> int:
    return (n + m - 1) // m * m


@dataclass
class LatentSpec:
    heads: int
    dim: int
    rot: int
    vdim: int
    kv_rank: int
    scale: float
    theta: float
    eps: float
    scaling: dict | None = None               # of the rotation's frequencies
    window: int = 0                           # a key is seen at distances below it (0: all in front)

    def __post_init__(self):
        self.turn = Rotation(self.rot, self.theta, True, self.scaling)
        self.rot0 = _up(self.kv_rank, 16)                 # column of the rotated part in the cache row
        nb = 1 if self.kv_rank <= 64 else 2 if self.kv_rank <= 128 else 4 if self.kv_rank <= 256 else 8
        self.lat_cols = nb * 64                           # columns of the decode kernel's partial outputs
        self.width = max(_up(self.rot0 + self.rot, 64), self.lat_cols if self.kv_rank <= 512 else 0)

    def bind(self, device):
        self.turn.bind(device)
        return self

    @property
    def tc_decode(self) -> bool:
        return self.kv_rank <= 512 and self.width <= 704

    @property
    def tc_prefill(self) -> bool:
        return (self.dim % 8 == 0 and self.rot % 8 == 0 and self.vdim % 8 == 0 and self.kv_rank % 8 == 0 and self.dim + self.rot <= 256
                and self.vdim <= 256)

    @property
    def tcgen05(self) -> bool:
        return self.tc_prefill and -(-self.dim // 64) - (-self.rot // 64) <= 3 and self.vdim <= 128 and self.scale > 0

    def dims(self, pool):
        return (self.heads, self.dim, self.rot, self.vdim, self.kv_rank, self.rot0, self.width, pool.shape[-1])


_D = "iiiiiiii"


def latent_reference(spec: LatentSpec, q, kv, w_norm, w_uk, w_uv, b, cache, pool) -> torch.Tensor:
    """CPU statement: cache rows written, then every row's softmax over its sequence (fp32) -> [rows, heads * vdim]."""
    n, H, d, r, dv, kr = q.shape[0], spec.heads, spec.dim, spec.rot, spec.vdim, spec.kv_rank
    dt = pool.dtype
    qh = q.float().reshape(n, H, d + r).clone()
    qh[..., d:] = spec.turn.turn(qh[..., d:], b.pos)
    qh = qh.to(dt).float()
    kv = kv.float()
    c = kv[:, :kr]
    c = c / torch.sqrt(c.pow(2).mean(-1, keepdim=True) + spec.eps) * w_norm
    kr_rot = spec.turn.turn(kv[:, kr: kr + r], b.pos)
    out = torch.zeros(n, H, dv)
    for i in range(n):
        s, p = int(b.slot[i]), int(b.pos[i])
        if s < 0:
            continue
        row = pool[int(cache.page_table[s, p // PAGE]), 0, p % PAGE]
        row[:kr], row[spec.rot0: spec.rot0 + r] = c[i].to(dt), kr_rot[i].to(dt)
    uk, uv = w_uk.float().reshape(H, d, kr), w_uv.float().reshape(H, dv, kr)
    for i in range(n):
        s, p = int(b.slot[i]), int(b.pos[i])
        if s < 0:
            continue
        a = max(0, p - spec.window + 1) if spec.window else 0          # first key it sees
        rows = pool[cache.page_table[s, a // PAGE: p // PAGE + 1].long(), 0].reshape(-1, pool.shape[-1])[a % PAGE: p + 1 - a // PAGE * PAGE].float()
        lat, rot = rows[:, :kr], rows[:, spec.rot0: spec.rot0 + r]
        sc = torch.einsum("hd,hdc->hc", qh[i, :, :d], uk) @ lat.t() + qh[i, :, d:] @ rot.t()
        pr = torch.softmax(sc * spec.scale, -1)
        out[i] = torch.einsum("hc,hvc->hv", pr @ lat, uv)
    return out.reshape(n, H * dv).to(dt)


def _absorbed(spec, q, kv, w_norm, w_uk, w_uv, pos, slot, cache, pool):
    """Absorbed attention of the rows of ``q``; writes their cache rows first (rows of one sequence may follow each other: all
    cache rows are written before the attention launch)."""
    n, dev, dt = q.shape[0], q.device, pool.dtype
    f32, x32 = int(dt == torch.float32), int(q.dtype == torch.float32)
    D = spec.dims(pool)
    qw = spec.width
    q_abs = torch.empty(n, spec.heads, qw, dtype=dt, device=dev)
    table = cache.page_table
    call("latent_absorb", _D + "plplii" + "pppf" + "pppip" + "piifi", *D, ptr(q), q.stride(0), ptr(kv), kv.stride(0), x32, int(kv.dtype == torch.float32), ptr(w_norm),
         ptr(w_uk), ptr(spec.turn.half_turns), spec.turn.mul, ptr(pos), ptr(slot), ptr(table), table.shape[1], ptr(pool), ptr(q_abs), qw, n, float(spec.eps), f32)
    out = torch.empty(n, spec.heads * spec.vdim, dtype=dt, device=dev)
    if spec.tc_decode and not f32:
        nsplit = max(1, min(64, 296 // (n * ((spec.heads + 15) // 16))))        # two CTAs per SM, whatever the position
        if spec.window:
            nsplit = min(nsplit, (spec.window + PAGE - 2) // PAGE + 1)          # pages a window lies in at most
        part = torch.empty(n, spec.heads, nsplit, spec.lat_cols, dtype=torch.float32, device=dev)
        lse = torch.empty(n, spec.heads, nsplit, dtype=torch.float32, device=dev)
        call("latent_decode", "ppppppiplii" + "iiiifip", ptr(q_abs), ptr(part), ptr(lse), ptr(pos), ptr(slot), ptr(table), table.shape[1], ptr(pool),
             pool.shape[0], pool.shape[-1], spec.width, spec.kv_rank, n, spec.heads, nsplit, float(spec.scale), spec.window, ptr(K.status_word(dev)))
        ld = spec.lat_cols
    else:
        nsplit, lse, ld = 1, None, spec.kv_rank
        part = torch.empty(n, spec.heads, spec.kv_rank, dtype=torch.float32, device=dev)
        call("latent_attn", _D + "pipppipfipii", *D, ptr(q_abs), qw, ptr(pos), ptr(slot), ptr(table), table.shape[1], ptr(pool), float(spec.scale), spec.window,
             ptr(part), n, f32)
    call("latent_expand", _D + "ppiipp" + "plii", *D, ptr(part), ptr(lse), nsplit, ld, ptr(w_uv), ptr(slot), ptr(out), out.stride(0), n, f32)
    return out


def _expanded(spec, q, kv, w_norm, ukv, b, cache, pool, out, r0):
    """Prompt rows [r0, n) of the batch: the keys and values that their sequences see, expanded from the cached latents."""
    t = b.segments().context(spec.window)
    D = spec.dims(pool)
    table = cache.page_table
    n = q.shape[0]
    dev = q.device
    x32 = int(q.dtype == torch.float32)
    qr = q[r0:]
    same = not x32
    qo = qr if same else torch.empty(qr.shape, dtype=pool.dtype, device=dev)
    kvr = kv[r0:]
    call("latent_rope_store", _D + "plplplii" + "ppf" + "pppip" + "ifi", *D, ptr(qr), qr.stride(0), ptr(qo), qo.stride(0), ptr(kvr), kvr.stride(0), x32,
         int(kv.dtype == torch.float32), ptr(w_norm), ptr(spec.turn.half_turns), spec.turn.mul, ptr(b.pos[r0:]), ptr(b.slot[r0:]), ptr(table), table.shape[1], ptr(pool), n - r0, float(spec.eps), 0)
    lat = torch.empty(t.total, spec.width, dtype=pool.dtype, device=dev)
    call("latent_gather", "pipipppi" + "pii", ptr(pool), pool.shape[-1], ptr(table), table.shape[1], ptr(t.slot), ptr(t.base), ptr(t.start), t.slot.numel(),
         ptr(lat), spec.width, t.total)
    up = ukv.forward(lat[:, : spec.kv_rank])
    if spec.tcgen05 and TC_PREFILL and qo.stride(0) % 8 == 0 and qo.data_ptr() % 16 == 0:
        tf, tc, tb, tk = t.tiles[128]
        call("latent_prefill_tc", _D + "plplpil" + "pppppii" + "plfp", *D, ptr(qo), qo.stride(0), ptr(up), up.stride(0), ptr(lat), spec.width, t.total,
             ptr(b.pos[r0:]), ptr(tf), ptr(tc), ptr(tb), ptr(tk), tf.numel(), spec.window, ptr(out[r0:]), out.stride(0), float(spec.scale), ptr(K.status_word(dev)))
        return
    tf, tc, tb, tk = t.tiles[64]
    call("latent_prefill", _D + "plplpip" + "ppppii" + "plf", *D, ptr(qo), qo.stride(0), ptr(up), up.stride(0), ptr(lat), spec.width, ptr(b.pos[r0:]),
         ptr(tf), ptr(tc), ptr(tb), ptr(tk), tf.numel(), spec.window, ptr(out[r0:]), out.stride(0), float(spec.scale))


def latent_rows(spec: LatentSpec, q, kv, w_norm, w_uk, w_uv, ukv, b, cache, pool) -> torch.Tensor:
    """All rows of batch ``b``: q [rows, heads (dim + rot)] not yet rotated (overwritten when it is bf16), kv [rows, kv_rank + rot]
    as projected (views of any row pitch; kv fp32, or of q's type). ``ukv``: the stacked linear [W_uk; W_uv]. -> [rows, heads * vdim] in the cache's type."""
    if not q.is_cuda:
        return latent_reference(spec, q, kv, w_norm, w_uk, w_uv, b, cache, pool)
    n = q.shape[0]
    if b.row_path or pool.dtype == torch.float32 or not spec.tc_prefill:
        return _absorbed(spec, q, kv, w_norm, w_uk, w_uv, b.pos, b.slot, cache, pool)
    t = b.segments()
    out = torch.empty(n, spec.heads * spec.vdim, dtype=pool.dtype, device=q.device)
    r0 = t.short_rows
    if r0:
        out[:r0] = _absorbed(spec, q[:r0], kv[:r0], w_norm, w_uk, w_uv, b.pos[:r0], b.slot[:r0], cache, pool)
    _expanded(spec, q, kv, w_norm, ukv, b, cache, pool, out, r0)
    return out
