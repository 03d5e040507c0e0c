"""Token mixers of decoders whose ``config.json`` lists its layers one by one, each with its own mixer type and sizes. A mixer
reads normed rows and returns the rows of its output projection; ``step`` is the same on a few decode rows with the norm in
front, the layer scale and the residual add inside the linears' launches (``finish(linear, **operands)`` runs the last one).

``MIXERS`` maps type names to classes (a design may give its own names, ``ListedConfig.mixers``); a class takes (mixer sizes, eps, tensor source, name prefix, device, dtype).
"""
from __future__ import annotations

import copy

import torch

from ..ops.gqa import GqaSpec, distance_bias, gqa_attend
from ..ops.latent import LatentSpec, latent_rows
from ..ops.linear import LinearBF16, LinearF32
from ..ops.linear_attn import LinAttnSpec, LinAttnState, linattn_rows
from ..ops.min_gru import MinGruState, min_gru_rows
from ..ops.rotary import Rotation
from ..ops.rowops import GroupRMS, gemv_rows


def make_linear(src, names, device, dtype, dim: int = 0, join=None, bias=None):
    """One linear computing the stacked outputs of the tensors ``names`` (``dim`` 1: the sum of their outputs on stacked inputs;
    ``join``: a function that makes one weight of them; ``bias``: fp32, of its outputs)."""
    names = [names] if isinstance(names, str) else names
    parts = [src.tensor(n, device, dtype) for n in names]
    w = join(*parts) if join is not None else torch.cat(parts, dim) if len(parts) > 1 else parts[0]
    return LinearF32(w, bias) if dtype == torch.float32 else LinearBF16(w, bias)


def apply_linear(lin, x, out_f32: bool = False):
    """``lin`` on rows of its activation type: the decode kernel up to 16 rows, the tensor-core GEMM above."""
    if x.is_cuda and isinstance(lin, LinearBF16) and x.shape[0] <= 16:
        return gemv_rows(lin, x.shape[0], x=x, out_f32=out_f32)
    return lin.forward(x, out_f32=out_f32)


def window_of(m: dict) -> int:
    """Size of a mixer's sliding window (0: none)."""
    mask = m.get("mask")
    if not mask:
        return 0
    if int(mask["size"]) < 1:
        raise ValueError(f"a window of {mask['size']} keys")
    return int(mask["size"])


class Mixer:
    """What the decoder asks of a mixer beside ``rows`` and ``step``."""
    cached = False                  # owns one layer of the paged cache (``cache_index``)
    recurrent = False               # has a state per slot (``bind``, ``state``)
    cache_index = -1
    state = None

    @staticmethod
    def row_widths(m: dict) -> tuple[int, int]:
        """Elements of a token's row in the key and in the value pool, from the mixer's sizes."""
        return 0, 0

    def linears(self):
        return [self.in_proj, self.out]

    def extra_bytes(self) -> int:
        """Bytes of further matrices a decode step reads."""
        return 0

    def state_elements(self) -> int:
        return 0


class MinGru(Mixer):
    """A gated recurrence per channel whose gate and candidate read the current token alone: one fused input projection [gate | candidate |
    output gate] with biases on the first two, the recurrence with the output gate, the output projection."""
    recurrent = True

    def __init__(self, kind: str, m: dict, eps: float, src, p: str, device, dtype):
        self.width = int(m["width"])
        b = torch.cat([src.tensor(p + n, device, torch.float32).reshape(-1) for n in ("z.b", "x.b")])
        self.in_proj = make_linear(src, [p + "z", p + "x", p + "g"], device, dtype, bias=torch.nn.functional.pad(b, (0, self.width)))
        self.out = make_linear(src, p + "o", device, dtype)
        if self.in_proj.out_features != 3 * self.width:
            raise ValueError(f"{p}: projections of {self.in_proj.out_features} rows for three times {self.width} channels")
        self.dtype = dtype
        self.state: MinGruState | None = None

    def bind(self, kv):
        if self.state is None:
            self.state = MinGruState(self.width, kv.max_slots, kv.page_table.device)
        return self.state

    def state_elements(self) -> int:
        return self.width

    def recur(self, proj, b, kv, journal):
        return min_gru_rows(proj, b, self.bind(kv), self.dtype, self.out.weight.shape[1], *journal)

    def rows(self, x, b, kv, journal=(None, None)):
        return apply_linear(self.out, self.recur(apply_linear(self.in_proj, x, out_f32=True), b, kv, journal))

    def step(self, pro, finish, b, kv, journal=(None, None)):
        finish(self.out, x=self.recur(gemv_rows(self.in_proj, b.n, out_f32=True, **pro), b, kv, journal))


class LinearRecurrence(Mixer):
    """HGRN2, lightning attention, retention and gated linear attention: one fused input projection [q | forget gate or k | v | gate | low-rank
    decay], the decayed outer-product recurrence, an RMS norm of its output (per head, or over all heads; gated), the output
    projection. ``out_scale``: a factor on what enters the output projection."""
    recurrent = True
    PARTS = {"hgrn2": ("q", "f", "v"), "lightning": ("q", "k", "v", "g"), "retention": ("q", "k", "v", "g"),
             "gated_linear_attention": ("q", "k", "v", "g", "a1")}

    def __init__(self, kind: str, m: dict, eps: float, src, p: str, device, dtype, linears: bool = True, out_scale: float = 1.0):
        H, dk, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        f32 = lambda name: src.tensor(p + name, device, torch.float32).reshape(-1).contiguous()
        self.parts = [p + n for n in self.PARTS[kind]]
        self.gated = "g" in self.PARTS[kind]
        if kind in ("lightning", "retention"):
            decay = m["decay"] if isinstance(m["decay"], (list, tuple)) else [m["decay"]] * H
            self.spec = LinAttnSpec(H, dk, dv, decay=torch.tensor([float(d) for d in decay], dtype=torch.float32, device=device),
                                    **({"plain": True, "q_scale": dk ** -0.5} if kind == "retention" else {}))
            if self.spec.decay.numel() != H:
                raise ValueError(f"{p}: {self.spec.decay.numel()} decays for {H} heads")
        elif kind == "hgrn2":
            self.spec = LinAttnSpec(H, dk, dv, lower=f32("lower"), bias=f32("f.b"))
        else:
            self.spec = LinAttnSpec(H, dk, dv, bias=f32("a2.b"), w2=src.tensor(p + "a2", device, torch.float32).contiguous(), a_col=H * (2 * dk + 2 * dv),
                                    tau=float(m["tau"]), q_scale=dk ** -0.5)
        if linears:
            self.in_proj = make_linear(src, self.parts, device, dtype)
            self.out = make_linear(src, p + "o", device, dtype)
        w = torch.ones(dv, device=device) if kind == "retention" else f32("norm")
        self.norm = GroupRMS(w * out_scale, eps, 0 if kind == "lightning" else dv, silu=kind in ("retention", "gated_linear_attention"))
        self.dtype = dtype
        self.state: LinAttnState | None = None

    def bind(self, kv):
        if self.state is None:
            self.state = LinAttnState(self.spec, kv.max_slots, kv.page_table.device)
        return self.state

    def state_elements(self) -> int:
        return self.spec.heads * self.spec.dk * self.spec.dv

    def extra_bytes(self) -> int:
        return self.spec.w2.numel() * 4 if self.spec.w2 is not None else 0

    def gate(self, proj):
        return proj[:, self.spec.cols: self.spec.cols + self.spec.heads * self.spec.dv] if self.gated else None

    def recur(self, proj, b, kv, journal, chunked: bool):
        return linattn_rows(proj, b, self.bind(kv), self.spec, *journal, chunked=chunked)

    def rows(self, x, b, kv, journal=(None, None)):
        proj = apply_linear(self.in_proj, x, out_f32=True)         # gates and keys enter the recurrence unrounded
        o = self.recur(proj, b, kv, journal, self.dtype != torch.float32)
        return apply_linear(self.out, self.norm.rows(o, self.dtype, gate=self.gate(proj)))

    def step(self, pro, finish, b, kv, journal=(None, None)):
        proj = gemv_rows(self.in_proj, b.n, out_f32=True, **pro)
        o = self.recur(proj, b, kv, journal, True)
        finish(self.out, **self.norm.prologue(o, self.gate(proj)))


class GroupedAttention(Mixer):
    """Grouped-query softmax attention without rotation: normed queries and keys, a query temperature, a bias by distance and a sink;
    one fused input projection [q | k | v]. ``out_scale`` as above."""
    cached = True
    PARTS = ("q", "k", "v")

    @staticmethod
    def row_widths(m: dict) -> tuple[int, int]:
        return GqaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), 1.0).row_widths

    def __init__(self, kind: str, m: dict, eps: float, src, p: str, device, dtype, linears: bool = True, out_scale: float = 1.0):
        f32 = lambda name: src.tensor(p + name, device, torch.float32).contiguous()
        temp = m.get("q_temp") or {"coef": 0.0, "every": 0}
        self.spec = GqaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), eps, q_norm=f32("q.norm"),
                            k_norm=f32("k.norm"), temp_coef=float(temp["coef"]), temp_every=int(temp["every"]),
                            bias=distance_bias(f32("rel"), int(m["bias_max"])), sink=f32("sink"), out_scale=out_scale)
        self.parts = [p + n for n in self.PARTS]
        if linears:
            self.in_proj = make_linear(src, self.parts, device, dtype)
            self.out = make_linear(src, p + "o", device, dtype)
        self.dtype = dtype

    def in_bias(self, src):
        """Biases of the input projection's outputs, or None."""
        return None

    def out_bias(self, src):
        return None

    def attend(self, proj, b, kv, out):
        return gqa_attend(self.spec, proj, b, kv, kv.k[self.cache_index], kv.v[self.cache_index], out)

    def _out(self, proj):
        return torch.empty(proj.shape[0], self.spec.heads * self.spec.vdim, dtype=self.dtype, device=proj.device)

    def rows(self, x, b, kv, journal=None):
        proj = apply_linear(self.in_proj, x, out_f32=True)
        return apply_linear(self.out, self.attend(proj, b, kv, self._out(proj)))

    def step(self, pro, finish, b, kv, journal=None):
        proj = gemv_rows(self.in_proj, b.n, out_f32=True, **pro)
        finish(self.out, x=self.attend(proj, b, kv, self._out(proj)))


class WindowedAttention(GroupedAttention):
    """Grouped-query softmax attention with rotary positions, queries and keys brought to unit root mean square behind them, a sliding
    window, a sink, and a sigmoid gate on the result; one fused input projection [q | k | v | gate]."""
    PARTS = ("q", "k", "v", "g")

    def __init__(self, kind: str, m: dict, eps: float, src, p: str, device, dtype):
        rot = m.get("rot")
        self.spec = GqaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), float(m["scale"]), eps, unit=True, gated=True,
                            sink=src.tensor(p + "sink", device, torch.float32).reshape(-1).contiguous(), window=window_of(m),
                            rot=Rotation.from_config(rot, False).bind(device) if rot else None)
        if rot and self.spec.rot.dims > self.spec.dim:
            raise ValueError(f"{p}: {self.spec.rot.dims} rotated columns of {self.spec.dim}")
        self.parts = [p + n for n in self.PARTS]
        self.in_proj = make_linear(src, self.parts, device, dtype)
        self.out = make_linear(src, p + "o", device, dtype)
        self.dtype = dtype

    def rows(self, x, b, kv, journal=None):
        proj = apply_linear(self.in_proj, x, out_f32=b.row_path)
        return apply_linear(self.out, self.attend(proj, b, kv, self._out(proj)))


class RotatedValueAttention(GroupedAttention):
    """Grouped-query softmax attention with rotary positions on queries and keys (behind their norm) and on values (taken back from the
    result), a number per head on the scores, a soft cap, a sliding window that keeps the first tokens in sight, and biases on all
    projections. ``out_scale`` as above."""

    def __init__(self, kind: str, m: dict, eps: float, src, p: str, device, dtype, linears: bool = True, out_scale: float = 1.0):
        f32 = lambda name: src.tensor(p + name, device, torch.float32).reshape(-1).contiguous()
        rot, vdim, window = m["rot"], int(m["vdim"]), window_of(m)
        self.spec = GqaSpec(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), vdim, float(m["scale"]), eps, q_norm=f32("q.norm"), k_norm=f32("k.norm"),
                            norm_first=True, head_mul=f32("temp"), softcap=float(m.get("softcap") or 0.0), out_scale=out_scale, window=window,
                            keep_first=int(m["mask"].get("keep_first") or 0) if window else 0, rot=Rotation.from_config(rot, True).bind(device),
                            v_rot=Rotation(vdim, float(rot["base"]), True).bind(device))
        if self.spec.rot.dims > self.spec.dim:
            raise ValueError(f"{p}: {self.spec.rot.dims} rotated columns of {self.spec.dim}")
        self.p, self.out_scale, self.device = p, out_scale, device
        self.parts = [p + n for n in self.PARTS]
        if linears:
            self.in_proj = make_linear(src, self.parts, device, dtype, bias=self.in_bias(src))
            self.out = make_linear(src, p + "o", device, dtype, bias=self.out_bias(src))
        self.dtype = dtype

    def in_bias(self, src):
        return torch.cat([src.tensor(self.p + n + ".b", self.device, torch.float32).reshape(-1) for n in self.PARTS])

    def out_bias(self, src):
        return (src.tensor(self.p + "o.b", self.device, torch.float32).reshape(-1) * self.out_scale).contiguous()


class Parallel(Mixer):
    """Attention and a linear recurrence side by side on the same rows: one input projection for both, and one output projection over the
    two results put next to each other (each times its scale)."""
    LEFT, RIGHT = (GroupedAttention, "grouped_attention"), (LinearRecurrence, "gated_linear_attention")
    cached = recurrent = True

    @staticmethod
    def row_widths(m: dict) -> tuple[int, int]:
        return GroupedAttention.row_widths(m["left"])

    def __init__(self, kind: str, m: dict, eps: float, src, p: str, device, dtype):
        side = lambda which, name: which[0](which[1], m[name], eps, src, f"{p}{name}.", device, dtype, False, float(m[name + "_scale"]))
        self.left, self.right = side(self.LEFT, "left"), side(self.RIGHT, "right")
        self.in_proj = make_linear(src, self.left.parts + self.right.parts, device, dtype)
        self.out = make_linear(src, [p + "left.o", p + "right.o"], device, dtype, dim=1, bias=self.left.out_bias(src))
        b = self.left.in_bias(src)
        if b is not None:
            self.in_proj.bias = torch.nn.functional.pad(b, (0, self.in_proj.out_features - b.numel())).contiguous()
        self.k0 = self.left.spec.heads * self.left.spec.vdim         # columns of the left result
        self.k1 = self.right.spec.heads * self.right.spec.dv
        self.dtype = dtype

    def __copy__(self):
        new = object.__new__(type(self))
        new.__dict__.update(self.__dict__)
        new.left, new.right = copy.copy(self.left), copy.copy(self.right)
        return new

    cache_index = property(lambda self: self.left.cache_index, lambda self, i: setattr(self.left, "cache_index", i))
    state = property(lambda self: self.right.state, lambda self, s: setattr(self.right, "state", s))

    def bind(self, kv):
        return self.right.bind(kv)

    def state_elements(self) -> int:
        return self.right.state_elements()

    def extra_bytes(self) -> int:
        return self.right.extra_bytes()

    def rows(self, x, b, kv, journal=(None, None)):
        proj = apply_linear(self.in_proj, x, out_f32=True)
        y = torch.empty(x.shape[0], self.k0 + self.k1, dtype=self.dtype, device=x.device)
        self.left.attend(proj, b, kv, y[:, : self.k0])
        pr = proj[:, self.left.spec.cols:]
        o = self.right.recur(pr, b, kv, journal, self.dtype != torch.float32)
        self.right.norm.rows(o, self.dtype, gate=self.right.gate(pr), out=y[:, self.k0:])
        return apply_linear(self.out, y)

    def step(self, pro, finish, b, kv, journal=(None, None)):
        proj = gemv_rows(self.in_proj, b.n, out_f32=True, **pro)
        att = self.left.attend(proj, b, kv, torch.empty(b.n, self.k0, dtype=torch.float32, device=proj.device))
        pr = proj[:, self.left.spec.cols:]
        o = self.right.recur(pr, b, kv, journal, True)
        finish(self.out, **self.right.norm.prologue(o, self.right.gate(pr), head=att))


class RotatedRetention(Parallel):
    """Attention with rotated values beside retention."""
    LEFT, RIGHT = (RotatedValueAttention, "rotated_value_attention"), (LinearRecurrence, "retention")


class LatentAttention(Mixer):
    """Multi-head attention over a low-rank latent per token and a rotated key part shared by the heads, with a sliding window or
    without. Queries come from a normed low-rank projection, or (no ``q_rank``) straight from the input: then one fused input
    projection [q | latent and rotated part]."""
    cached = True

    @staticmethod
    def row_widths(m: dict) -> tuple[int, int]:
        return LatentSpec(1, 1, int(m["rot_dim"]), 1, int(m["kv_rank"]), 1.0, 2.0, 1e-5).width, 0

    def __init__(self, kind: str, m: dict, eps: float, src, p: str, device, dtype):
        rot = m["rot"]
        if int(rot["dims"]) != int(m["rot_dim"]):
            raise ValueError(f"{p}: the rotated part is turned as a whole")
        self.spec = LatentSpec(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]),
                               float(rot["base"]), eps, rot.get("scaling"), window_of(m)).bind(device)
        f32 = lambda name: src.tensor(p + name, device, torch.float32).reshape(-1).contiguous()
        self.q_rank = int(m.get("q_rank") or 0)
        self.split = self.q_rank or self.spec.heads * (self.spec.dim + self.spec.rot)        # columns in front of the latent
        self.down = make_linear(src, [p + ("dq" if self.q_rank else "q"), p + "dkv"], device, dtype)
        self.uq = make_linear(src, p + "uq", device, dtype) if self.q_rank else None
        self.w_uk = src.tensor(p + "uk", device, dtype).contiguous()
        self.w_uv = src.tensor(p + "uv", device, dtype).contiguous()
        self.ukv = LinearBF16(torch.cat([self.w_uk, self.w_uv], 0)) if dtype != torch.float32 else None
        if self.ukv is not None and self.ukv.weight.shape[1] == self.spec.kv_rank:      # one copy: the absorbed form reads slices of the stacked weight
            self.w_uk, self.w_uv = self.ukv.weight[: self.w_uk.shape[0]], self.ukv.weight[self.w_uk.shape[0]:]
        self.out = make_linear(src, p + "o", device, dtype)
        self.q_norm = GroupRMS(f32("dq.norm"), eps) if self.q_rank else None
        self.kv_norm = f32("dkv.norm")
        self.dtype = dtype

    def linears(self):
        return [x for x in (self.down, self.uq, self.out) if x is not None]

    def extra_bytes(self) -> int:
        return (self.w_uk.numel() + self.w_uv.numel()) * self.w_uk.element_size()

    def _attend(self, q, a, b, kv):
        return latent_rows(self.spec, q, a[:, self.split:], self.kv_norm, self.w_uk, self.w_uv, self.ukv, b, kv, kv.k[self.cache_index])

    def rows(self, x, b, kv, journal=None):
        few = x.shape[0] <= 16
        if self.uq is None:
            a = apply_linear(self.down, x, out_f32=few)
            q = a[:, : self.split]
        else:
            a = apply_linear(self.down, x, out_f32=True)
            q = apply_linear(self.uq, self.q_norm.rows(a[:, : self.q_rank], self.dtype), out_f32=few)
        return apply_linear(self.out, self._attend(q, a, b, kv))

    def step(self, pro, finish, b, kv, journal=None):
        a = gemv_rows(self.down, b.n, out_f32=True, **pro)
        q = a[:, : self.split] if self.uq is None else gemv_rows(self.uq, b.n, out_f32=True, **self.q_norm.prologue(a[:, : self.q_rank]))
        finish(self.out, x=self._attend(q, a, b, kv))


MIXERS = {"hgrn2": LinearRecurrence, "lightning": LinearRecurrence, "latent_attention": LatentAttention,
          "gated_linear_attention": LinearRecurrence, "grouped_attention": GroupedAttention, "parallel": Parallel, "attention": WindowedAttention,
          "mingru": MinGru, "rotated_retention": RotatedRetention}
