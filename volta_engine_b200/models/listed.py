"""Decoders whose configuration lists its layers one by one: every layer has a token mixer of its own type and sizes
(:mod:`.mixers`) and an optional feed-forward, with a norm in front of each (or behind it, on its result) and an fp32 residual. A range
of layers may run several times in a row with the same weights; every pass has its own cache layer and state.

A design supplies the parts (:meth:`ListedModel.load_layer`, ``load_ends``, ``embed_batch``); loading order, cache layers, state
slots, batches and the forward pass are here. A layer's parts are row operators of :mod:`..ops.rowops`:

  norm1, norm2     ``rows(h, dtype, part, write)``: the sublayer result in front enters the residual, then the norm of it;
                   ``prologue(h)``: the norm as the prologue of a decode linear
  write1, write2   how a sublayer's result enters the residual (an element-wise scale, a StreamWrite, or a NormedWrite: that one needs
                   whole rows, so the reader behind adds the result)
  ff               the feed-forward (:mod:`.feed_forward`)
"""
from __future__ import annotations

import copy
import json
from dataclasses import dataclass, field
from pathlib import Path
from typing import ClassVar

import torch

from ..ops.rowops import RoutedRows, fused_fits, gemv_rows, soft_cap_
from ..runtime.batch import LOGITS_ALL, BatchRows
from .dense import DenseConfig, DenseModel
from .mixers import MIXERS, apply_linear
from .slot_state import SlotStates

DTYPES = {"bf16": torch.bfloat16, "bfloat16": torch.bfloat16, "fp32": torch.float32, "float32": torch.float32}


@dataclass
class ListedConfig(DenseConfig):
    mixers: ClassVar[dict] = MIXERS                 # the design's mixer types
    layers: list = field(default_factory=list)      # [{"type", "mixer": {sizes}, "mlp": {"kind", ...} | None}]
    loop: tuple = (0, 0, 1)                         # layers [start, stop) run this many times in a row
    v_width: int = 8                                # elements of a token's row in the value pool
    residual: str = "fp32"

    @classmethod
    def listed(cls, c: dict, feed_forwards=("dense",), **kw):
        """The fields every design of this form has. ``feed_forwards``: the kinds the design has."""
        layers = [dict(L) for L in c["layers"]]
        for i, L in enumerate(layers):
            if L["type"] not in cls.mixers:
                raise NotImplementedError(f"layer {i}: no mixer {L['type']!r} in this build")
            if L.get("mlp") is not None and L["mlp"].get("kind", "dense") not in feed_forwards:
                raise NotImplementedError(f"layer {i}: no feed-forward {L['mlp']['kind']!r} in this build")
        lp = c.get("loop")
        loop = (int(lp["start"]), int(lp["stop"]), int(lp["times"])) if lp else (0, 0, 1)
        if not 0 <= loop[0] <= loop[1] <= len(layers) or loop[2] < 1:
            raise ValueError(f"loop over layers {loop[0]} .. {loop[1]} of {len(layers)}, {loop[2]} times")
        widths = [cls.mixers[L["type"]].row_widths(L["mixer"]) for L in layers]
        return cls(n_layers=len(layers), hidden=int(c["width"]), vocab=int(c["vocab"]), rms_eps=float(c["norm"]["eps"]), layers=layers, loop=loop,
                   n_q=1, n_kv=1, ffn=max([int((L["mlp"].get("expert") or L["mlp"])["ff"]) for L in layers if L.get("mlp") is not None] or [1]), quant="bf16",
                   head_dim=max([k for k, _ in widths] + [0]) or 64, v_width=max([v for _, v in widths] + [8]), **kw)

    def runs(self) -> list:
        """Layer indices in the order they run."""
        a, b, times = self.loop
        return list(range(a)) + list(range(a, b)) * times + list(range(b, len(self.layers)))


class ListedLayer:
    __slots__ = ("mixer", "norm1", "write1", "norm2", "write2", "ff")

    def __init__(self, mixer, norm1, write1):
        self.mixer, self.norm1, self.write1 = mixer, norm1, write1
        self.norm2 = self.write2 = self.ff = None

    def again(self) -> "ListedLayer":
        """Another pass of this layer: the same weights, a cache layer and a state of its own."""
        L = copy.copy(self)
        L.mixer = copy.copy(self.mixer)
        return L


def read_rows(norm, h, dtype, part, write):
    """``norm.rows``; results of a routed feed-forward are summed in front of norms that do not sum them."""
    if isinstance(part, RoutedRows) and not getattr(norm, "takes_routed", False):
        part = part.tensor()
    return norm.rows(h, dtype, part, write)


class StepResidual:
    """The residual of a decode step whose linears carry norms and updates, with a result that the next reader adds to it."""

    def __init__(self, h):
        self.h, self.part, self.write = h, None, None

    def read(self, norm) -> dict:
        """Operands of a linear that reads the residual through ``norm``."""
        if self.part is None:
            return norm.prologue(self.h)
        pro = norm.prologue(self.h, self.part, self.write)
        self.h, self.part = pro["h_out"], None
        return pro

    def put(self, write):
        """-> ``finish(linear, **operands)``: the linear whose result enters the residual through ``write``."""
        def finish(lin, **pro):
            if getattr(write, "deferred", False):
                self.later(gemv_rows(lin, self.h.shape[0], out_f32=True, **pro), write)
            else:
                gemv_rows(lin, self.h.shape[0], residual=(self.h, write), **pro)
        return finish

    def later(self, part, write):
        self.part, self.write = part, write


class ListedModel(SlotStates, DenseModel):
    supports_mixed = True           # prompt portions and decode rows of several sequences run in one forward
    kv_layers = 0
    kv_v_dim = 8

    def __init__(self, cfg: ListedConfig, device, comm=None, dtype="bf16"):
        super().__init__(cfg, device, comm)
        if self.comm.size != 1:
            raise NotImplementedError("this model runs on one GPU (its norms over all heads and over the feed-forward width are not split)")
        self.dtype = DTYPES[dtype] if isinstance(dtype, str) else dtype
        self.vocab_pad = self.vocab_local = cfg.vocab
        self.kv_v_dim = cfg.v_width
        self.layer_tap = None       # a list that receives the residual after every layer run (tests, inspection)

    @property
    def prefix_resume(self) -> str:
        """What a prefix snapshot holds: the paged cache, and the slot's state where a layer has one."""
        return "kv+state" if any(L.mixer.recurrent for L in self.layers) else "kv"

    # ------------------------------------------------------------------------------------------ what a design supplies
    def load_ends(self, src) -> None:
        """Sets ``embed``, ``final_norm`` and ``lm_head``."""
        raise NotImplementedError

    def load_layer(self, i: int, spec: dict, src) -> ListedLayer:
        raise NotImplementedError

    def embed_batch(self, b: BatchRows):
        """-> the fp32 residual the first layer reads."""
        raise NotImplementedError

    def residual_rows(self, h, part=None, write=None):
        """The residual as rows [tokens, hidden] for ``layer_tap``, with a result that is still on its way into it."""
        raise NotImplementedError

    # ------------------------------------------------------------------------------------------ weights
    def load(self, src):
        """``src``: has ``tensor(name, device, dtype)`` (a checkpoint's tensor source, or a random one)."""
        self.load_ends(src)
        once = [self.load_layer(i, spec, src) for i, spec in enumerate(self.cfg.layers)]
        self.layers, n_cached, seen = [], 0, set()
        for i in self.cfg.runs():
            L = once[i].again() if i in seen else once[i]
            seen.add(i)
            if L.mixer.cached:
                L.mixer.cache_index = n_cached
                n_cached += 1
            self.layers.append(L)
        self.own_layers = once                                   # every layer's weights once
        self.kv_layers = n_cached
        return self

    def link_prefetch(self) -> None:
        pass

    def ensure_workspace(self, max_rows: int, max_splits: int):
        pass

    @staticmethod
    def _layer_bytes(layers, step: bool) -> int:
        n = 0
        for L in layers:
            n += sum(lin.nbytes() for lin in L.mixer.linears()) + L.mixer.extra_bytes()
            if L.ff is not None:
                n += L.ff.nbytes(step)
        return n

    def decode_bytes_per_token(self) -> int:
        """Weight bytes a decode step of one row reads (a looped layer's once per pass)."""
        return self.lm_head.nbytes() + self._layer_bytes(self.layers, True)

    def weight_bytes(self) -> int:
        tied = self.lm_head.weight.data_ptr() == self.embed.data_ptr()
        return self.lm_head.nbytes() + self._layer_bytes(self.own_layers, False) + (0 if tied else self.embed.numel() * self.embed.element_size())

    # ------------------------------------------------------------------------------------------ state slots
    def _states(self, kv) -> list:
        return [L.mixer.bind(kv) if L.mixer.recurrent else None for L in self.layers]

    def layer_states(self) -> list:
        return [L.mixer.state for L in self.layers]

    def reset_states(self) -> None:
        """Forget the slots' states (an engine with another slot count is about to be built on this model)."""
        self.journal_on = False
        for L in self.layers:
            L.mixer.state = None
        for name in ("_jsets", "_shadows"):
            if hasattr(self, name):
                delattr(self, name)

    def state_bytes_per_slot(self) -> int:
        return sum(4 * L.mixer.state_elements() for L in self.layers)

    def _journal(self, li, L, b, kv):
        return self.journal_of(li, L.mixer.bind(kv), b) if L.mixer.recurrent else (None, None)

    # ------------------------------------------------------------------------------------------ forward
    def forward(self, b: BatchRows, kv) -> torch.Tensor | None:
        if self.kv_layers and kv.k.dtype != self.dtype:
            raise ValueError(f"cache of {kv.k.dtype} under a model of {self.dtype}")
        h = self.embed_batch(b)
        if h.is_cuda and self.dtype == torch.bfloat16 and fused_fits(self._widest(), b.n):
            return self._forward_fused(b, kv, h)
        dt, part, write = self.dtype, None, None
        for li, L in enumerate(self.layers):
            x = read_rows(L.norm1, h, dt, part, write)
            part, write = L.mixer.rows(x, b, kv, self._journal(li, L, b, kv)), L.write1
            if L.ff is not None:
                x = read_rows(L.norm2, h, dt, part, write)
                part, write = L.ff.rows(x, b), L.write2
            if self.layer_tap is not None:
                self.layer_tap.append(self.residual_rows(h, part, write))
        x = read_rows(self.final_norm, h, dt, part, write)
        self.last_hidden, self.last_residual = x, h
        x = b.select_logits(x)
        return None if x is None else self.capped(apply_linear(self.lm_head, x, out_f32=True))

    def capped(self, logits):
        return soft_cap_(logits, self.cfg.logit_softcap) if self.cfg.logit_softcap > 0 else logits

    def _forward_fused(self, b: BatchRows, kv, h):
        """A few decode rows: norms, activations and residual updates ride in the linears' launches."""
        res = StepResidual(h)
        for li, L in enumerate(self.layers):
            L.mixer.step(res.read(L.norm1), res.put(L.write1), b, kv, self._journal(li, L, b, kv))
            if L.ff is not None:
                L.ff.step(res, L.norm2, L.write2, b)
            if self.layer_tap is not None:
                self.layer_tap.append(self.residual_rows(res.h, res.part, res.write))
        if res.part is not None and b.logits != LOGITS_ALL:          # the head reads some of the rows
            self.final_norm.rows(res.h, torch.float32, res.part, res.write)
            res.part = None
        pro = res.read(self.final_norm)
        self.last_residual = res.h
        if b.logits != LOGITS_ALL:
            h = b.select_logits(res.h)
            if h is None:
                return None
            pro = self.final_norm.prologue(h)
        return gemv_rows(self.lm_head, pro["x"].shape[0], out_f32=True, cap=self.cfg.logit_softcap, **pro)

    def _widest(self):
        """The linear with the longest input rows of those that take a prologue."""
        w = getattr(self, "_widest_lin", None)
        if w is None:
            lins = [self.lm_head] + [x for L in self.own_layers for x in (*L.mixer.linears(), *(L.ff.linears() if L.ff is not None else ()))]
            w = self._widest_lin = max(lins, key=lambda x: x.weight.shape[1])
        return w


# ---------------------------------------------------------------------------------------------- random weights
class RandomTensors:
    """Random weights under checkpoint names: every tensor has a generator of its own, so any subset can be drawn in any order.
    ``draw(name, shape, rnd, uni)`` gives a tensor from functions that return normal / uniform numbers of the tensor's shape."""

    def __init__(self, shapes: dict, seed: int, device="cpu"):
        self.shapes, self.seed, self.device = shapes, seed, torch.device(device)
        self.order = {n: i for i, n in enumerate(sorted(shapes))}

    def draw(self, name, shape, rnd, uni):
        raise NotImplementedError

    def has(self, name: str) -> bool:
        return name in self.shapes

    def tensor(self, name: str, device=None, dtype=None):
        shape = self.shapes[name]
        g = torch.Generator(device=self.device).manual_seed(self.seed * 1000003 + self.order[name])
        t = self.draw(name, shape, lambda: torch.randn(shape, generator=g, device=self.device), lambda: torch.rand(shape, generator=g, device=self.device))
        t = t.to(torch.bfloat16)                 # what a checkpoint would hold
        return t.to(device=device or self.device, dtype=dtype or t.dtype)


def save_listed(model_dir, config: dict, src: RandomTensors, tensors: dict | None = None):
    """Write a model directory (config.json + model.safetensors) with random weights; ``tensors`` replaces some of them."""
    from ..loader.safetensors import write_safetensors
    d = Path(model_dir)
    d.mkdir(parents=True, exist_ok=True)
    (d / "config.json").write_text(json.dumps(config, indent=1))
    out = {n: src.tensor(n) for n in src.shapes}
    out.update({n: t.to(torch.bfloat16) for n, t in (tensors or {}).items()})
    write_safetensors(d / "model.safetensors", out)
