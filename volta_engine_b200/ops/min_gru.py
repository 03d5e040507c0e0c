"""Gated recurrence per channel whose gate and candidate read the current row alone (minGRU: L. Feng et al.,
"Were RNNs All We Needed?"; csrc/cuda/mingru.cu): per slot an fp32 state S [width] with

    S_t = (1 - z_t) S_(t-1) + z_t c_t,     y_t = S_t silu(g_t)

over fp32 projection rows [ z | u | g ]; z behind a sigmoid, c = u + 1/2 for u >= 0 and sigmoid(u) below. A row at position 0 starts its slot
from a zero state; rows of one slot inside a batch are consecutive positions in order.
"""
from __future__ import annotations

import torch

from .._lib import call, ptr
from .gdn import GDNJournal


class MinGruState:
    """rec [slots, width] fp32 of one layer."""
    conv = None

    def __init__(self, width: int, max_slots: int, device):
        self.rec = torch.zeros(max_slots, width, dtype=torch.float32, device=device)

    def nbytes(self):
        return self.rec.numel() * 4

    def snapshot(self, slot: int) -> dict:
        return {"rec": self.rec[slot].cpu().clone()}

    def restore(self, slot: int, snap: dict):
        self.rec[slot].copy_(snap["rec"])


def min_gru_reference(proj, pos, slot, st: MinGruState) -> torch.Tensor:
    """CPU statement over the rows of a batch; updates ``st`` in place -> fp32 [rows, width]."""
    W = st.rec.shape[1]
    z, u, g = proj[:, : 3 * W].float().split(W, 1)
    take, keep = torch.sigmoid(z), torch.sigmoid(-z)
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    S = torch.zeros(proj.shape[0], W)
    for i in range(proj.shape[0]):
        s = int(slot[i])
        if s < 0:
            continue
        if int(pos[i]) == 0:
            st.rec[s].zero_()
        S[i] = st.rec[s].mul_(keep[i]).add_(take[i] * c[i])
    return S * torch.nn.functional.silu(g)


def _step(proj, pos, slot, st, y, rows, segs=(None, None, 0)):
    first, count, n = segs
    call("mingru_step", "plppppip" + "pliiii", ptr(proj), proj.stride(0), ptr(pos), ptr(slot), ptr(first), ptr(count), n, ptr(st.rec), ptr(y), y.stride(0), rows,
         st.rec.shape[1], y.shape[1], int(y.dtype == torch.float32))


def min_gru_rows(proj, b, st: MinGruState, dtype, cols: int = 0, journal: GDNJournal | None = None, rows=None) -> torch.Tensor:
    """Rows of batch ``b`` through the recurrence -> [rows, cols or width] of ``dtype`` (columns behind the width are zero). ``rows`` = (pos, slot)
    that outlive the step when ``journal`` keeps the block's operands for a replay."""
    pos, slot = rows if rows is not None else (b.pos, b.slot)
    n, W = proj.shape[0], st.rec.shape[1]
    if journal is not None:
        journal.begin(st, slot)
    if not proj.is_cuda:
        if journal is not None:
            journal.fn = lambda keep: min_gru_reference(proj[:keep], pos[:keep], slot[:keep], st)
        y = min_gru_reference(proj, pos, slot, st).to(dtype)
        return torch.nn.functional.pad(y, (0, cols - W)) if cols > W else y
    assert proj.dtype == torch.float32
    y = torch.empty(n, max(cols, W), dtype=dtype, device=proj.device)
    if b.row_path:
        _step(proj, pos, slot, st, y, n)
        if journal is not None:
            y2 = torch.empty_like(y)
            journal.fn = lambda keep: _step(proj, pos, slot, st, y2, keep)
        return y
    t = b.segments()
    if t.n_short:
        _step(proj, pos, slot, st, y, n, (t.first, t.count, t.n_short))
    if t.chunks:
        new = lambda *s: torch.empty(*s, dtype=torch.float32, device=proj.device)
        total, start = new(t.chunks, 2, W), new(t.seg_chunk0.numel() - 1, W)
        call("mingru_chunk", "plpp" + "ppppi" + "ppp" + "pliii", ptr(proj), proj.stride(0), ptr(pos), ptr(slot), ptr(t.chunk_seg), ptr(t.chunk_first),
             ptr(t.chunk_count), ptr(t.seg_chunk0), t.chunks, ptr(st.rec), ptr(total), ptr(start), ptr(y), y.stride(0), W, y.shape[1],
             int(dtype == torch.float32))
    return y
