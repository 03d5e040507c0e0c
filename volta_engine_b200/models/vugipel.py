"""Vugipel: a decoder whose configuration lists its layers one by one. Every layer mixes tokens by a gated recurrence per channel (minGRU) or
by windowed attention with rotated values beside retention, and has a mixture of gated SiLU experts (sigmoid router, weights on the
experts' inputs) or no feed-forward. RMS norms whose weights are stored as offsets from one stand in front of the sublayers, whose results are
added to an fp32 residual.

The decoder is the one of :mod:`.listed`, mixers and feed-forwards those of :mod:`.mixers` and :mod:`.feed_forward`, norms and
activations the row operators of :mod:`..ops.rowops`; cache, state slots, scheduling and sampling are the engine's. A model runs in bf16
(matrix products and activations; angles, scores, gates, states, router, norms and the residual in fp32) or, with ``dtype="fp32"``, in
fp32 throughout.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import ClassVar

import torch

from ..ops.routed import Router
from ..ops.rowops import ClampedGlu, ResidualNorm, embed_rows
from .feed_forward import RoutedFF
from .listed import ListedConfig, ListedLayer, ListedModel, RandomTensors, save_listed
from .mixers import MIXERS, make_linear

# CUDA sources whose kernels this model and its sampling launch
KERNEL_SOURCES = ("gemm_bf16_wide.cu", "gemm_tcgen05.cu", "gemv_rows.cu", "gqa.cu", "linattn.cu", "mingru.cu", "moe.cu", "routed.cu", "rowops.cu", "sampling.cu")


@dataclass
class VugipelConfig(ListedConfig):
    mixers: ClassVar[dict] = {"mingru": MIXERS["mingru"], "parallel": MIXERS["rotated_retention"]}
    model_type: str = "vugipel"

    @classmethod
    def from_dict(cls, c: dict) -> "VugipelConfig":
        return cls.listed(c, ("moe",))


def router_of(m: dict) -> Router:
    return Router(int(m["experts"]), int(m["top"]), sigmoid=True, weigh_input=True)


class VugipelModel(ListedModel):
    def _norm(self, src, name: str) -> ResidualNorm:
        return ResidualNorm((1.0 + src.tensor(name, self.device, torch.float32)).contiguous(), self.cfg.rms_eps)

    def load_ends(self, src) -> None:
        dev, dt = self.device, self.dtype
        self.embed = src.tensor("embed", dev, dt).contiguous()
        self.final_norm = self._norm(src, "final.norm")
        self.lm_head = make_linear(src, "head", dev, dt)

    def load_layer(self, i: int, spec: dict, src) -> ListedLayer:
        dev, dt, p = self.device, self.dtype, f"l{i}."
        mixer = self.cfg.mixers[spec["type"]]
        L = ListedLayer(mixer(spec["type"], spec["mixer"], self.cfg.rms_eps, src, p + "mix.", dev, dt), self._norm(src, p + "norm1"), None)
        if spec.get("mlp") is not None:
            L.norm2 = self._norm(src, p + "norm2")
            L.ff = RoutedFF(src, p + "mlp.", router_of(spec["mlp"]["router"]), ClampedGlu.silu(), dev, dt)
        return L

    def embed_batch(self, b):
        return embed_rows(b.ids, self.embed)

    def residual_rows(self, h, part=None, write=None):
        h = h.clone()
        if part is not None:
            ResidualNorm.add(h, part)
        return h

    def init_random(self, seed: int = 1, std: float = 0.02, search: bool = False):
        return self.load(RandomSource(self.cfg, seed, self.device, std))


# ---------------------------------------------------------------------------------------------- random weights
def tensor_shapes(cfg: VugipelConfig) -> dict:
    """Checkpoint tensor names -> shapes."""
    W = cfg.hidden
    out = {"embed": (cfg.vocab, W), "head": (cfg.vocab, W), "final.norm": (W,)}
    for i, spec in enumerate(cfg.layers):
        p, m = f"l{i}.", spec["mixer"]
        x = p + "mix."
        out[p + "norm1"] = (W,)
        if spec["type"] == "mingru":
            S = int(m["width"])
            out.update({x + "z": (S, W), x + "z.b": (S,), x + "x": (S, W), x + "x.b": (S,), x + "g": (S, W), x + "o": (W, S)})
        else:
            a, x = m["left"], p + "mix.left."
            H, G, d, dv = int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"])
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * dv)):
                out.update({x + n: (rows, W), x + n + ".b": (rows,)})
            out.update({x + "q.norm": (d,), x + "k.norm": (d,), x + "temp": (H,), x + "o": (W, H * dv), x + "o.b": (W,)})
            a, x = m["right"], p + "mix.right."
            H, d, dv = int(a["heads"]), int(a["dim"]), int(a["vdim"])
            out.update({x + "q": (H * d, W), x + "k": (H * d, W), x + "v": (H * dv, W), x + "g": (H * dv, W), x + "o": (W, H * dv)})
        f = spec.get("mlp")
        if f is not None:
            y, ff = p + "mlp.", int(f["expert"]["ff"])
            out.update({p + "norm2": (W,), y + "router": (int(f["router"]["experts"]), W)})
            for e in range(int(f["router"]["experts"])):
                out.update({f"{y}e{e}.gate": (ff, W), f"{y}e{e}.up": (ff, W), f"{y}e{e}.down": (W, ff)})
    return out


class RandomSource(RandomTensors):
    """N(0, std) matrices, norms near the identity, small biases, gates that remember, heads of unlike sharpness."""

    def __init__(self, cfg: VugipelConfig, seed: int, device="cpu", std: float | None = None):
        super().__init__(tensor_shapes(cfg), seed, device)
        self.std = std

    def draw(self, name, shape, rnd, uni):
        if len(shape) == 2:
            return rnd() * (self.std if self.std is not None else shape[1] ** -0.5 if name != "embed" else 1.0)
        if name.endswith(".z.b"):
            return rnd() - 2.0
        if name.endswith(".b"):
            return 0.2 * rnd()
        if name.endswith((".temp", "q.norm", "k.norm")):
            return 0.8 + 0.6 * uni()
        return 0.1 * rnd()


def save_checkpoint(model_dir, config: dict, seed: int = 0, tensors: dict | None = None):
    """Write a model directory with random weights; ``tensors`` replaces some of them."""
    save_listed(model_dir, config, RandomSource(VugipelConfig.from_dict(config), seed), tensors)


def load_vugipel(hf: dict, src, device, comm=None, dtype="bf16", **_):
    return VugipelModel(VugipelConfig.from_dict(hf), device, comm, dtype).load(src)
