"""Per-forward row descriptor, resident on the device so one CUDA graph per row count serves every step.

Equivalent of the reference's ``BatchRows`` / ``SlotRef`` (inc/engine/core/batch.h:11-105): each row
names its sequence slot and position; prefill chunks carry the tile grouping for the attention kernel;
the logits mode says which rows reach the LM head.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

MAX_GRAPH_ROWS = 16    # decode / verify row counts that get a captured graph
MAX_CHUNK_ROWS = 4096  # prefill chunk upper bound

LOGITS_ALL = "all"
LOGITS_LAST = "last"
LOGITS_NONE = "none"
LOGITS_ROWS = "rows"   # the rows listed in BatchRows.want

CHUNK_ROWS = 128       # rows of one chunk of the chunked recurrences (half of it in small batches, for more parallel work)
LONG_SEGMENT = 16      # portions of at least this many rows take the prompt kernels, shorter ones the decode kernels


@dataclass
class Contexts:
    """Contexts of segments, one after the other: per segment its slot, the first row of its context and that row's position; ``tiles``
    of at most 64 or 128 rows of one segment: (first row, counted from the table's ``short_rows``; rows; first row of the segment's
    context; that row's position)."""
    slot: torch.Tensor
    base: torch.Tensor
    start: torch.Tensor
    total: int
    tiles: dict


@dataclass
class SegmentTable:
    """Runs of consecutive rows of one slot inside a batch that is known on the host. Device tables are int32."""
    n: int                          # segments
    first: torch.Tensor             # [n] first row
    count: torch.Tensor             # [n] rows
    host: list                      # [(slot, first row, rows, first position)]
    short_rows: int                 # leading rows that belong to segments shorter than LONG_SEGMENT
    chunk_seg: torch.Tensor | None   # chunks of at most CHUNK_ROWS rows of these segments: segment (0 = the first behind short_rows),
    chunk_first: torch.Tensor | None  # first row (in the batch) and rows
    chunk_count: torch.Tensor | None
    seg_chunk0: torch.Tensor | None   # [segments + 1] first chunk of every such segment
    n_short: int = 0                  # leading segments that make up short_rows
    chunks: int = 0
    longest: int = 0                  # most chunks of any segment
    made: dict = field(default_factory=dict)

    def _dev(self, v):
        return torch.tensor(list(v), dtype=torch.int32).to(self.first.device, non_blocking=True)

    def context(self, window: int = 0) -> "Contexts":
        """What the segments behind ``short_rows`` see (a sliding window: none of their rows sees further back), laid out one after
        the other."""
        t = self.made.get(("context", window))
        if t is None:
            rest = self.host[self.n_short:]
            start = [max(0, p0 - window + 1) if window else 0 for _, _, _, p0 in rest]
            base, total = [], 0
            for a, (_, _, c, p0) in zip(start, rest):
                base.append(total)
                total += p0 + c - a
            tiles = {}
            for per in (64, 128):
                rows = [(f + o - self.short_rows, min(per, c - o), z, a) for a, z, (_, f, c, _) in zip(start, base, rest) for o in range(0, c, per)]
                tiles[per] = tuple(self._dev(v) for v in zip(*rows))
            t = self.made["context", window] = Contexts(self._dev([h[0] for h in rest]), self._dev(base), self._dev(start), total, tiles)
        return t

    def tiles(self, per: int):
        """(first row in the batch, rows) of tiles of at most ``per`` rows over the segments behind ``short_rows``."""
        t = self.made.get(per)
        if t is None:
            rows = [(f + o, min(per, c - o)) for _, f, c, _ in self.host[self.n_short:] for o in range(0, c, per)]
            t = self.made[per] = tuple(self._dev(v) for v in zip(*rows))
        return t

    @classmethod
    def build(cls, slots, pos, device):
        host, i, n = [], 0, len(slots)
        while i < n:
            j = i
            while j < n and slots[j] == slots[i] and pos[j] == pos[i] + (j - i):
                j += 1
            host.append((slots[i], i, j - i, pos[i]))
            i = j

        def dev(v):
            return torch.tensor(v, dtype=torch.int32).to(device, non_blocking=True)
        k = 0
        while k < len(host) and host[k][2] < LONG_SEGMENT:
            k += 1
        rest = host[k:]
        short = rest[0][1] if rest else n
        t = cls(len(host), dev([h[1] for h in host]), dev([h[2] for h in host]), host, short, *([None] * 4), n_short=k)
        if rest:
            cs, cf, cc, c0 = [], [], [], [0]
            per = CHUNK_ROWS if n >= 1024 else CHUNK_ROWS // 2
            for g, (s, f, c, p0) in enumerate(rest):
                for o in range(0, c, per):
                    cs.append(g)
                    cf.append(f + o)
                    cc.append(min(per, c - o))
                c0.append(len(cs))
            t.chunks, t.longest = len(cs), max(b - a for a, b in zip(c0, c0[1:]))
            t.chunk_seg, t.chunk_first, t.chunk_count, t.seg_chunk0 = dev(cs), dev(cf), dev(cc), dev(c0)
        return t


@dataclass
class BatchRows:
    ids: torch.Tensor      # [n] int32
    pos: torch.Tensor      # [n] int32
    slot: torch.Tensor     # [n] int32 (-1 = padding row)
    n: int
    logits: str = LOGITS_ALL
    tiles: tuple | None = None      # (tile_first, tile_count, ntiles) for prefill attention
    nsplit: int = 1                 # split-KV factor for decode attention
    key_end: torch.Tensor | None = None
    host_slots: list = field(default_factory=list)
    host_pos: list = field(default_factory=list)
    pos3: torch.Tensor | None = None        # [3, n] int32 rotary positions (time, height, width) of multimodal prompts
    embeds: torch.Tensor | None = None      # [n, H] rows that replace the token embedding where embed_mask is set
    embed_mask: torch.Tensor | None = None  # [n] bool
    tree: tuple | None = None               # (base int32 [n], mask int64 [n]): rows of a verification tree (ops.kernels.attention)

    want: torch.Tensor | None = None        # LOGITS_ROWS: int64 row indices
    seg_table: SegmentTable | None = None

    @property
    def row_path(self) -> bool:
        """Few rows: kernels that handle every row by itself (and find rows of one slot on the device)."""
        return self.n <= MAX_GRAPH_ROWS

    def segments(self) -> SegmentTable:
        if self.seg_table is None:
            assert len(self.host_slots) == self.n, "the batch's rows are not known on the host"
            self.seg_table = SegmentTable.build(self.host_slots, self.host_pos, self.ids.device)
        return self.seg_table

    def select_logits(self, x):
        """Rows of ``x`` whose logits are asked for (None: no rows)."""
        if self.logits == LOGITS_NONE:
            return None
        if self.logits == LOGITS_LAST:
            return x[self.n - 1: self.n]
        return x.index_select(0, self.want) if self.logits == LOGITS_ROWS else x

    @classmethod
    def make(cls, ids, pos, slots, device, logits=LOGITS_ALL, G=1, prefill=False, nsplit=1):
        from ..ops.kernels import make_prefill_tiles
        n = len(ids)
        t_ids = torch.tensor(ids, dtype=torch.int32).to(device, non_blocking=True)
        t_pos = torch.tensor(pos, dtype=torch.int32).to(device, non_blocking=True)
        t_slot = torch.tensor(slots, dtype=torch.int32).to(device, non_blocking=True)
        tiles = make_prefill_tiles(list(slots), G, device) if prefill else None
        return cls(t_ids, t_pos, t_slot, n, logits, tiles, nsplit, None, list(slots), list(pos))
