"""Linear attention with a decayed outer-product state (csrc/cuda/linattn.cu): per slot and head an fp32 state S [dk, dv] with

    S_t = diag(d_t) S_(t-1) + k_t v_t^T,     o_t = S_t^T q_t

over projection rows [ q (heads dk) | x (heads dk) | v (heads dv) | ... ] and one of

  * ``decay`` given (lightning attention): d = decay[head], k = silu(x), v = silu(v), q = silu(q); with ``plain`` (retention) k = x and v as
    projected, q times ``q_scale``;
  * ``lower`` / ``bias`` given (HGRN2): the forget gate f = lower + (1 - lower) sigmoid(x + bias) per channel is the decay and
    its complement 1 - f the key; v as projected, q = silu(q);
  * ``w2`` / ``bias`` given (gated linear attention): d = sigmoid(w2 a + bias)^(1 / tau) per channel from a low-rank part a of the
    row (columns from ``a_col``); k = x and v as projected, q times ``q_scale``.

A row at position 0 starts its slot from a zero state; rows of one slot inside a batch are consecutive positions in order.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from .._lib import call, ptr
from .gdn import GDNJournal

@dataclass
class LinAttnSpec:
    heads: int
    dk: int
    dv: int
    decay: torch.Tensor | None = None       # fp32 [heads]
    lower: torch.Tensor | None = None       # fp32 [heads * dk]
    bias: torch.Tensor | None = None        # fp32 [heads * dk]
    w2: torch.Tensor | None = None          # fp32 [heads * dk, rank]
    a_col: int = 0
    tau: float = 1.0
    q_scale: float = 1.0
    plain: bool = False

    @property
    def mode(self) -> int:
        return 0 if self.decay is not None else 2 if self.w2 is not None else 1

    @property
    def rank(self) -> int:
        return self.w2.shape[1] if self.w2 is not None else 0

    @property
    def chunks(self) -> bool:
        """The chunked kernels take these sizes."""
        return self.dk <= 128 and self.dv <= 128 and self.rank <= 320

    @property
    def cols(self) -> int:
        return self.heads * (2 * self.dk + self.dv)


class LinAttnState:
    """rec [slots, heads, dk, dv] fp32 of one layer."""
    conv = None

    def __init__(self, spec: LinAttnSpec, max_slots: int, device):
        self.rec = torch.zeros(max_slots, spec.heads, spec.dk, spec.dv, dtype=torch.float32, device=device)

    def nbytes(self):
        return self.rec.numel() * 4

    def snapshot(self, slot: int) -> dict:
        return {"rec": self.rec[slot].cpu().clone()}

    def restore(self, slot: int, snap: dict):
        self.rec[slot].copy_(snap["rec"])


def gates(pf, spec: LinAttnSpec):
    """fp32 projection rows -> (decay, key), each [rows, heads, dk]."""
    n, D = pf.shape[0], spec.heads * spec.dk
    x = pf[:, D: 2 * D]
    if spec.mode == 2:
        z = pf[:, spec.a_col: spec.a_col + spec.rank] @ spec.w2.t() + spec.bias
        return torch.exp(torch.nn.functional.logsigmoid(z) / spec.tau).reshape(n, spec.heads, spec.dk), x.reshape(n, spec.heads, spec.dk)
    if spec.mode == 0:
        k = (x if spec.plain else torch.nn.functional.silu(x)).reshape(n, spec.heads, spec.dk)
        return spec.decay.reshape(1, spec.heads, 1).expand_as(k), k
    z = x + spec.bias
    f = spec.lower + (1.0 - spec.lower) * torch.sigmoid(z)
    k = (1.0 - spec.lower) * torch.sigmoid(-z)
    return f.reshape(n, spec.heads, spec.dk), k.reshape(n, spec.heads, spec.dk)


def linattn_reference(proj, pos, slot, st: LinAttnState, spec: LinAttnSpec) -> torch.Tensor:
    """CPU statement over the rows of a batch; updates ``st`` in place -> fp32 [rows, heads * dv]."""
    n, H, dk, dv = proj.shape[0], spec.heads, spec.dk, spec.dv
    pf = proj.float()
    q = (pf[:, : H * dk] * spec.q_scale if spec.mode == 2 or spec.plain else torch.nn.functional.silu(pf[:, : H * dk])).reshape(n, H, dk)
    d, k = gates(pf, spec)
    v = pf[:, 2 * H * dk: spec.cols].reshape(n, H, dv)
    if spec.mode == 0 and not spec.plain:
        v = torch.nn.functional.silu(v)
    o = torch.zeros(n, H, dv)
    for i in range(n):
        s = int(slot[i])
        if s < 0:
            continue
        S = st.rec[s]
        if int(pos[i]) == 0:
            S.zero_()
        S.mul_(d[i][:, :, None]).add_(k[i][:, :, None] * v[i][:, None, :])
        o[i] = torch.einsum("hkv,hk->hv", S, q[i])
    return o.reshape(n, H * dv)


def _step(proj, pos, slot, st, spec, o, rows, segs=None):
    x32 = 1 if proj.dtype == torch.float32 else 0
    first, count, n = segs if segs is not None else (None, None, 0)
    call("linattn_step", "plipp" + "ppi" + "pppp" + "pliiiii" + "piiffi", ptr(proj), proj.stride(0), x32, ptr(pos), ptr(slot), ptr(first), ptr(count), n,
         ptr(st.rec), ptr(spec.bias), ptr(spec.lower), ptr(spec.decay), ptr(o), o.stride(0), rows, spec.heads, spec.dk, spec.dv, spec.mode,
         ptr(spec.w2), spec.rank, spec.a_col, 1.0 / spec.tau, float(spec.q_scale), int(spec.plain))


def linattn_rows(proj, b, st: LinAttnState, spec: LinAttnSpec, journal: GDNJournal | None = None, rows=None,
                 chunked: bool = True) -> torch.Tensor:
    """Rows of batch ``b`` through the recurrence -> fp32 [rows, heads * dv]. ``chunked``: long portions may take the
    tensor-core form, which rounds the values v to bf16 (off in the all-32-bit form of a model). ``rows`` = (pos, slot) that outlive the step
    when ``journal`` keeps the block's operands for a replay."""
    pos, slot = rows if rows is not None else (b.pos, b.slot)
    if journal is not None:
        journal.begin(st, slot)
    if not proj.is_cuda:
        if journal is not None:
            journal.fn = lambda keep: linattn_reference(proj[:keep], pos[:keep], slot[:keep], st, spec)
        return linattn_reference(proj, pos, slot, st, spec)
    n = proj.shape[0]
    o = torch.empty(n, spec.heads * spec.dv, dtype=torch.float32, device=proj.device)
    if b.row_path:
        _step(proj, pos, slot, st, spec, o, n)
        if journal is not None:
            o2 = torch.empty_like(o)
            journal.fn = lambda keep: _step(proj, pos, slot, st, spec, o2, keep)
        return o
    t = b.segments()
    if not chunked or not spec.chunks or proj.dtype != torch.float32:
        _step(proj, pos, slot, st, spec, o, n, (t.first, t.count, t.n))
        return o
    if t.n_short:
        _step(proj, pos, slot, st, spec, o, n, (t.first, t.count, t.n_short))
    if t.chunks:
        multi = t.longest > 1
        start = torch.empty((t.chunks, spec.heads, spec.dk, spec.dv) if multi else (1,), dtype=torch.float32, device=proj.device)
        total = torch.empty((t.chunks, spec.heads, spec.dk) if multi else (1,), dtype=torch.float32, device=proj.device)
        dec = None
        if spec.mode == 2:
            dec = torch.empty(n, spec.heads * spec.dk, dtype=torch.float32, device=proj.device)
            a = proj[:, spec.a_col:]
            call("linattn_decay", "plippp" + "iiif", ptr(a), a.stride(0), 1, ptr(spec.w2), ptr(spec.bias), ptr(dec), n, spec.heads * spec.dk, spec.rank, 1.0 / spec.tau)
        call("linattn_chunk", "plpppppp" + "iii" + "ppp" + "pppp" + "liiii" + "pfi", ptr(proj), proj.stride(0), ptr(pos), ptr(slot), ptr(t.chunk_seg), ptr(t.chunk_first),
             ptr(t.chunk_count), ptr(t.seg_chunk0), t.chunks, t.seg_chunk0.numel() - 1, t.longest, ptr(st.rec), ptr(start), ptr(total), ptr(spec.bias),
             ptr(spec.lower), ptr(spec.decay), ptr(o), o.stride(0), spec.heads, spec.dk, spec.dv, spec.mode, ptr(dec), float(spec.q_scale), int(spec.plain))
    return o
