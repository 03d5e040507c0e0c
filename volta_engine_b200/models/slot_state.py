"""Recurrent state that a model keeps per slot beside the paged cache: journalled verify blocks and their rollback, and the
state as part of sequence snapshots. Models list their layers' states (:class:`~..ops.gdn.GDNState`,
:class:`~..ops.linear_attn.LinAttnState`; None for layers without one) through ``layer_states``.
"""
from __future__ import annotations

import torch

from ..ops.gdn import GDNJournal


class SlotStates:
    journal_on = False            # set by the engine for a verify step (rows of one slot that may be rejected)

    def layer_states(self) -> list:
        """The states of all layers, once they exist (an empty list before the first forward)."""
        raise NotImplementedError

    def begin_journal(self, on: bool, tag=0) -> None:
        """Called before a forward. ``tag`` names the set of operands this forward records into (the engine passes the
        row count: a CUDA graph of that row count keeps writing the tensors its capture pass recorded)."""
        self.journal_on = bool(on)
        if not hasattr(self, "_jsets"):
            self._jsets, self._shadows = {}, {}
        if on:
            self._jcur = self._jsets.setdefault(tag, {"rows": None, "layers": {}})
            self._jcur["rows"] = None
            self._jlast = tag

    def journal_of(self, li: int, st, b):
        """-> (journal of layer ``li`` or None, (pos, slot) of the rows) for this forward."""
        if not (self.journal_on and b.tiles is None):
            return None, (b.pos, b.slot)
        # rows of a speculative verify block (one slot): keep what is needed to take rejected rows back
        js = self._jcur
        jn = js["layers"].get(li)
        if jn is None:
            sh = self._shadows.get(li)
            if sh is None:
                sh = self._shadows[li] = GDNJournal.make_shadow(st)
            jn = js["layers"][li] = GDNJournal(st, sh)
        if js["rows"] is None:
            js["rows"] = (b.pos.clone(), b.slot.clone())      # the engine advances its row descriptor after the step
        return jn, js["rows"]

    def rollback_state(self, slot: int, keep: int) -> None:
        """After a journalled block: leave the slot's recurrent and convolution state as if only the block's first
        ``keep`` rows had run (the KV pool needs nothing: rejected rows are overwritten by the next step)."""
        js = getattr(self, "_jsets", {}).get(getattr(self, "_jlast", None))
        if js is None:
            raise RuntimeError("rollback without a journalled step")
        states = self.layer_states()
        for li, jn in js["layers"].items():
            jn.replay(states[li], slot, keep)

    # recurrent state travels with sequence snapshots
    def snapshot_state(self, slot: int) -> list:
        return [s.snapshot(slot) if s is not None else None for s in self.layer_states()]

    def restore_state(self, slot: int, snaps: list):
        for s, snap in zip(self.layer_states(), snaps):
            if s is not None and snap is not None:
                s.restore(slot, snap)

    def pack_state(self, slot: int) -> dict:
        """The slot's state of every layer as one or two flat host tensors (what a prefix snapshot stores)."""
        sts = [s for s in self.layer_states() if s is not None]
        out = {}
        if sts:
            out["gdn_rec"] = torch.cat([s.rec[slot].reshape(-1) for s in sts]).cpu()
        conv = [s.conv[slot].reshape(-1) for s in sts if s.conv is not None]
        if conv:
            out["gdn_conv"] = torch.cat(conv).cpu()
        return out

    def unpack_state(self, slot: int, snap: dict, kv) -> None:
        at = {"gdn_rec": 0, "gdn_conv": 0}

        def take(key, dst):
            n = dst.numel()
            dst.copy_(snap[key].reshape(-1)[at[key]: at[key] + n].reshape(dst.shape))
            at[key] += n
        for s in self._states(kv):
            if s is not None:
                take("gdn_rec", s.rec[slot])
                if s.conv is not None:
                    take("gdn_conv", s.conv[slot])
