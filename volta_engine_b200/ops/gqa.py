"""Grouped-query softmax attention with its sizes and score terms as parameters (csrc/cuda/gqa.cu): rotary positions, RMS norm of
queries and keys behind them or in front (with or without a weight), query temperature by position, factor per head, soft cap of the
scores, sliding window (the first tokens in sight or not), bias by distance, sink, values rotated by their position (the result is turned
back by the query's), output gate, unlike query / key and value widths.

The paged cache's rows are as wide as the widest layer needs (``row_widths``); a layer sees a page as [kv heads, 64, width].

Decode rows run a split-key tensor-core kernel, prompt portions a tcgen05 kernel; the all-32-bit form, and sizes outside the
tensor-core kernels' range, run on the CUDA cores.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .._lib import call, ptr
from . import kernels as K
from .rotary import Rotation

PAGE = K.PAGE
MAX_TICKETS = 1 << 16


def _up8(n: int) -> int:
    return (n + 7) // 8 * 8


def log_bucket(n: int, rows: int, far: int) -> int:
    """Row of a bias table of ``rows`` rows for a key ``n`` tokens back: one row per distance in the first half, then rows over
    logarithmically growing ranges that end at distance ``far``."""
    half = rows / 2
    if n < half:
        return n
    return int(min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half))))


def distance_bias(table, far: int):
    """table [rows, heads] -> fp32 [heads, L]: the bias by distance; its last entry holds for all larger distances."""
    rows = table.shape[0]
    if rows % 2 or rows < 2 or far <= rows // 2:
        raise ValueError(f"bias table of {rows} rows for distances up to {far}")
    idx = []
    while not idx or idx[-1] < rows - 1:
        idx.append(log_bucket(len(idx), rows, far))
    return table.float().t()[:, torch.tensor(idx, device=table.device)].contiguous()


@dataclass
class GqaSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    eps: float = 1e-6
    q_norm: torch.Tensor | None = None        # fp32 [dim]
    k_norm: torch.Tensor | None = None
    temp_coef: float = 0.0                    # queries times 1 + coef * ln(floor((position + 1) / every) + 1); every 0: off
    temp_every: int = 0
    bias: torch.Tensor | None = None          # fp32 [heads, L] (distance_bias)
    sink: torch.Tensor | None = None          # fp32 [heads]: log of one more term of the denominator
    out_scale: float = 1.0                    # factor on the result
    rot: Rotation | None = None               # of queries and keys, in front of their norm
    unit: bool = False                        # queries and keys are normed without a weight
    window: int = 0                           # a key is seen at distances below it (0: all in front)
    gated: bool = False                       # columns behind the values: the result is multiplied with their sigmoid
    norm_first: bool = False                  # the norm of queries and keys stands in front of their rotation
    head_mul: torch.Tensor | None = None      # fp32 [heads]: factor on a head's queries
    softcap: float = 0.0                      # scores are softcap * tanh(score / softcap), in front of the bias (0: as they are)
    keep_first: int = 0                       # the first tokens of a sequence that a window never leaves
    v_rot: Rotation | None = None             # of the values over their whole width, pairs as in ``rot``

    def __post_init__(self):
        if self.heads % self.kv_heads:
            raise ValueError(f"{self.heads} query heads over {self.kv_heads} key / value heads")
        self.kw, self.vw = _up8(self.dim), _up8(self.vdim)
        self.group = self.heads // self.kv_heads
        if self.v_rot is not None and (self.v_rot.dims != self.vdim or self.v_rot.mul != 1.0 or (self.rot is not None and self.rot.neighbours != self.v_rot.neighbours)):
            raise ValueError("values are turned as a whole, in pairs laid out as those of the keys")

    @property
    def cols(self) -> int:
        """Columns of a projection row [q | k | v | gate]."""
        return self.gate_col + (self.heads * self.vdim if self.gated else 0)

    @property
    def gate_col(self) -> int:
        return self.heads * self.dim + self.kv_heads * (self.dim + self.vdim)

    def gate(self, proj):
        """The gate's columns of projection rows."""
        return proj[:, self.gate_col: self.cols] if self.gated else None

    @property
    def row_widths(self) -> tuple[int, int]:
        """Elements of a token's row in the key and in the value pool."""
        return self.kv_heads * self.kw, self.kv_heads * self.vw

    @property
    def tc_decode(self) -> bool:
        return self.kw <= 256 and self.vw <= 256

    @property
    def tc_prefill(self) -> bool:
        return self.kw <= 256 and self.vw <= 128 and self.group <= 128 and self.scale > 0 and (self.v_rot is None or self.v_rot.neighbours)

    def temperature(self, pos):
        return 1.0 + self.temp_coef * torch.log(((pos + 1) // self.temp_every + 1).float()) if self.temp_every > 0 else torch.ones(pos.shape)


def _norm(v, w, unit, eps):
    if w is None and not unit:
        return v
    v = v / torch.sqrt(v.pow(2).mean(-1, keepdim=True) + eps)
    return v if w is None else v * w


def gqa_reference(spec: GqaSpec, proj, b, cache, kpool, vpool, out):
    """CPU statement: cache rows written, then every row's softmax over its sequence (fp32)."""
    n, H, G, d, dv = proj.shape[0], spec.heads, spec.kv_heads, spec.dim, spec.vdim
    dt = kpool.dtype
    pf = proj.float()
    turn = (lambda x: spec.rot.turn(x, b.pos)) if spec.rot is not None else (lambda x: x)
    place = (lambda x, w: turn(_norm(x, w, spec.unit, spec.eps))) if spec.norm_first else (lambda x, w: _norm(turn(x), w, spec.unit, spec.eps))
    q = place(pf[:, : H * d].reshape(n, H, d), spec.q_norm) * spec.temperature(b.pos)[:, None, None]
    if spec.head_mul is not None:
        q = q * spec.head_mul[:, None]
    q = q.to(dt).float()
    k = place(pf[:, H * d: (H + G) * d].reshape(n, G, d), spec.k_norm)
    v = pf[:, (H + G) * d: spec.gate_col].reshape(n, G, dv)
    if spec.v_rot is not None:
        v = spec.v_rot.turn(v, b.pos)
    gate = torch.sigmoid(spec.gate(pf)) if spec.gated else None
    kp = kpool.reshape(kpool.shape[0], -1)[:, : G * PAGE * spec.kw].view(-1, G, PAGE, spec.kw)
    vp = vpool.reshape(vpool.shape[0], -1)[:, : G * PAGE * spec.vw].view(-1, G, PAGE, spec.vw)
    rows = [(i, int(b.slot[i]), int(b.pos[i])) for i in range(n)]
    for i, s, p in rows:
        if s >= 0:
            pg = int(cache.page_table[s, p // PAGE])
            kp[pg, :, p % PAGE] = torch.nn.functional.pad(k[i], (0, spec.kw - d)).to(dt)
            vp[pg, :, p % PAGE] = torch.nn.functional.pad(v[i], (0, spec.vw - dv)).to(dt)
    for i, s, p in rows:
        if s < 0:
            out[i] = 0
            continue
        a = max(0, p - spec.window + 1) if spec.window else 0          # first key it sees
        seen = torch.cat([torch.arange(min(a, spec.keep_first)), torch.arange(a, p + 1)])
        pgs = cache.page_table[s, : p // PAGE + 1].long()
        ks = kp[pgs].transpose(1, 2).reshape(-1, G, spec.kw)[seen, :, :d].float()
        vs = vp[pgs].transpose(1, 2).reshape(-1, G, spec.vw)[seen, :, :dv].float()
        sc = torch.einsum("gud,jgd->guj", q[i].reshape(G, spec.group, d), ks).reshape(H, -1) * spec.scale
        if spec.softcap:
            sc = spec.softcap * torch.tanh(sc / spec.softcap)
        if spec.bias is not None:
            sc = sc + spec.bias[:, (p - seen).clamp(max=spec.bias.shape[1] - 1)]
        if spec.sink is not None:
            sc = torch.cat([sc, spec.sink[:, None]], 1)
        pr = torch.softmax(sc, -1)[:, : len(seen)].reshape(G, spec.group, -1)
        r = torch.einsum("guj,jgv->guv", pr, vs) * spec.out_scale
        if spec.v_rot is not None:
            r = spec.v_rot.turn(r[None], -b.pos[i: i + 1])
        r = r.reshape(-1)
        out[i] = (r if gate is None else r * gate[i]).to(out.dtype)
    return out


_tickets: dict = {}


def _ticket_words(dev):
    t = _tickets.get(str(dev))
    if t is None:
        t = _tickets[str(dev)] = torch.zeros(MAX_TICKETS, dtype=torch.int32, device=dev)
    return t


_D, _R, _S = "iiiiiill", "pppi", "fpipfipli" + "ifpii"


def _dims(spec, kpool, vpool):
    return (spec.heads, spec.kv_heads, spec.dim, spec.vdim, spec.kw, spec.vw, kpool[0].numel(), vpool[0].numel())


def _rows(pos, slot, cache):
    return (ptr(pos), ptr(slot), ptr(cache.page_table), cache.page_table.shape[1])


def _score(spec, gate, back):
    return (float(spec.scale), ptr(spec.bias), spec.bias.shape[1] if spec.bias is not None else 0, ptr(spec.sink), float(spec.out_scale), spec.window,
            ptr(gate), gate.stride(0) if gate is not None else 0, int(gate is not None and gate.dtype == torch.float32), spec.keep_first, float(spec.softcap),
            ptr(back), spec.v_rot.pairs if back is not None else 0, int(back is not None and spec.v_rot.neighbours))


def gqa_store(spec: GqaSpec, proj, pos, slot, cache, kpool, vpool):
    """Rotation, norms, temperature, cache rows -> (queries [rows, heads, kw] of the cache's type, fp32 [rows, pairs, 2] cosines and sines that
    results are turned back by, or None)."""
    n, f32 = proj.shape[0], kpool.dtype == torch.float32
    q = torch.empty(n, spec.heads, spec.kw, dtype=kpool.dtype, device=proj.device)
    rot, vr = spec.rot, spec.v_rot
    back = torch.empty(n, vr.pairs, 2, dtype=torch.float32, device=proj.device) if vr is not None else None
    norm = int(spec.unit or spec.q_norm is not None or spec.k_norm is not None) * (2 if spec.norm_first else 1)
    call("gqa_store", _D + _R + "pli" + "pifi" + "ippffi" + "ppip" + "pppii", *_dims(spec, kpool, vpool), *_rows(pos, slot, cache), ptr(proj), proj.stride(0),
         int(proj.dtype == torch.float32), ptr(rot.half_turns) if rot is not None else 0, rot.pairs if rot is not None else 0, rot.mul if rot is not None else 1.0,
         int((rot or vr).neighbours) if rot is not None or vr is not None else 0, norm, ptr(spec.q_norm), ptr(spec.k_norm), float(spec.eps), float(spec.temp_coef),
         int(spec.temp_every), ptr(spec.head_mul), ptr(vr.half_turns) if vr is not None else 0, vr.pairs if vr is not None else 0, ptr(back), ptr(q), ptr(kpool), ptr(vpool),
         n, int(f32))
    return q, back


def _each_row(spec, q, back, gate, pos, slot, cache, kpool, vpool, out):
    """Every row by itself: the split-key kernel, or the CUDA-core one."""
    n, dev, f32 = q.shape[0], q.device, kpool.dtype == torch.float32
    o32 = int(out.dtype == torch.float32)
    if f32 or not spec.tc_decode:
        call("gqa_rows", _D + _R + _S + "ppp" + "pliii", *_dims(spec, kpool, vpool), *_rows(pos, slot, cache), *_score(spec, gate, back), ptr(q), ptr(kpool), ptr(vpool),
             ptr(out), out.stride(0), o32, n, int(f32))
        return
    units = n * spec.kv_heads * ((spec.group + 15) // 16)
    nsplit = max(16, min(64, 148 // units)) if units <= MAX_TICKETS else 1          # a row takes as many of them as its position asks for,
    if spec.window:                                                                 # each at least two pages
        nsplit = max(1, min(nsplit, ((spec.window + PAGE - 2) // PAGE + 2 + (spec.keep_first + PAGE - 1) // PAGE) // 2))
    part = lse = None
    if nsplit > 1:
        part = torch.empty(n, spec.heads, nsplit, spec.vdim, dtype=torch.float32, device=dev)
        lse = torch.empty(n, spec.heads, nsplit, dtype=torch.float32, device=dev)
    call("gqa_decode", _D + _R + _S + "pppl" + "pppi" + "pliip", *_dims(spec, kpool, vpool), *_rows(pos, slot, cache), *_score(spec, gate, back), ptr(q), ptr(kpool), ptr(vpool),
         kpool.shape[0], ptr(part), ptr(lse), ptr(_ticket_words(dev)), nsplit, ptr(out), out.stride(0), o32, n, ptr(K.status_word(dev)))


def gqa_attend(spec: GqaSpec, proj, b, cache, kpool, vpool, out):
    """All rows of batch ``b``: ``proj`` rows start with [q | k | v | gate] as projected; the result goes to ``out`` [rows, heads * vdim] (a
    view of any row pitch; fp32, or bf16 as the cache). ``kpool`` / ``vpool``: this layer's pages."""
    if not proj.is_cuda:
        return gqa_reference(spec, proj, b, cache, kpool, vpool, out)
    q, back = gqa_store(spec, proj, b.pos, b.slot, cache, kpool, vpool)
    return gqa_scores(spec, q, b, cache, kpool, vpool, out, spec.gate(proj), back)


def gqa_scores(spec: GqaSpec, q, b, cache, kpool, vpool, out, gate=None, back=None):
    """Attention of the queries of ``gqa_store`` over the cached rows. ``gate``: the gate's columns as projected; ``back``: its second result."""
    n = q.shape[0]
    if b.row_path or kpool.dtype == torch.float32 or not spec.tc_prefill or out.dtype != torch.bfloat16:
        _each_row(spec, q, back, gate, b.pos, b.slot, cache, kpool, vpool, out)
        return out
    t = b.segments()
    r0 = t.short_rows
    if r0:
        _each_row(spec, q[:r0], back, None if gate is None else gate[:r0], b.pos[:r0], b.slot[:r0], cache, kpool, vpool, out[:r0])
    if r0 < n:
        tf, tc = t.tiles(128 // spec.group)
        call("gqa_prefill", _D + _R + _S + "pppl" + "ppi" + "plp", *_dims(spec, kpool, vpool), *_rows(b.pos, b.slot, cache), *_score(spec, gate, back), ptr(q), ptr(kpool),
             ptr(vpool), kpool.shape[0], ptr(tf), ptr(tc), tf.numel(), ptr(out), out.stride(0), ptr(K.status_word(q.device)))
    return out
