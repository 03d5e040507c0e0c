"""Fofosun: a decoder whose configuration lists its layers one by one. Every layer has a token mixer of its own type and sizes
(HGRN2, lightning attention, latent attention) and an optional feed-forward; Dynamic-Tanh norms in front of the sublayers,
an element-wise layer scale on their results, an fp32 residual stream, a PolyNorm feed-forward.

The decoder is the one of :mod:`.listed`, the mixers those of :mod:`.mixers`, norms and activations the row operators of
:mod:`..ops.rowops`; cache, state slots, scheduling and sampling are the engine's. A model runs in bf16 (matrix products and activations; scores, gates, states,
norms and the residual in fp32) or, with ``dtype="fp32"``, in fp32 throughout.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..ops.rowops import DynamicTanh, PolyNorm, embed_rows
from .feed_forward import DenseFF
from .listed import ListedConfig, ListedLayer, ListedModel, RandomTensors, save_listed
from .mixers import MIXERS, make_linear

# CUDA sources whose kernels this model and its sampling launch
KERNEL_SOURCES = ("gemm_bf16_wide.cu", "gemm_tcgen05.cu", "gemv_rows.cu", "latent.cu", "linattn.cu", "mla.cu", "rowops.cu", "sampling.cu")


@dataclass
class FofosunConfig(ListedConfig):
    model_type: str = "fofosun"

    @classmethod
    def from_dict(cls, c: dict) -> "FofosunConfig":
        return cls.listed(c)


class FofosunModel(ListedModel):
    def load_ends(self, src) -> None:
        dev, dt = self.device, self.dtype
        self.embed = src.tensor("embed", dev, dt).contiguous()
        self.final_norm = DynamicTanh.load(src, "final.norm", dev)
        self.lm_head = make_linear(src, "head", dev, dt)

    def load_layer(self, i: int, spec: dict, src) -> ListedLayer:
        dev, dt, eps, p = self.device, self.dtype, self.cfg.rms_eps, f"l{i}."
        f32 = lambda name: src.tensor(name, dev, torch.float32).contiguous()
        L = ListedLayer(MIXERS[spec["type"]](spec["type"], spec["mixer"], eps, src, p + "mix.", dev, dt), DynamicTanh.load(src, p + "norm1", dev), f32(p + "ls1"))
        if spec.get("mlp") is not None:
            L.norm2, L.write2 = DynamicTanh.load(src, p + "norm2", dev), f32(p + "ls2")
            L.ff = DenseFF(make_linear(src, p + "mlp.up", dev, dt), PolyNorm(f32(p + "mlp.act"), eps), make_linear(src, p + "mlp.down", dev, dt))
        return L

    def embed_batch(self, b):
        return embed_rows(b.ids, self.embed)

    def residual_rows(self, h, part=None, write=None):
        return h.clone() if part is None else h + part.float() * write

    def init_random(self, seed: int = 1, std: float = 0.02, search: bool = False):
        return self.load(RandomSource(self.cfg, seed, self.device, std))


# ---------------------------------------------------------------------------------------------- random weights
def tensor_shapes(cfg: FofosunConfig) -> dict:
    """Checkpoint tensor names -> shapes."""
    W = cfg.hidden
    out = {"embed": (cfg.vocab, W), "head": (cfg.vocab, W)}

    def norm(name):
        out[name], out[name + ".b"], out[name + ".alpha"] = (W,), (W,), ()
    for i, spec in enumerate(cfg.layers):
        p, m = f"l{i}.", spec["mixer"]
        H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        x = p + "mix."
        norm(p + "norm1")
        out[p + "ls1"] = (W,)
        if spec["type"] == "latent_attention":
            qr, kr, rd = int(m["q_rank"]), int(m["kv_rank"]), int(m["rot_dim"])
            out.update({x + "dq": (qr, W), x + "dq.norm": (qr,), x + "uq": (H * (d + rd), qr), x + "dkv": (kr + rd, W), x + "dkv.norm": (kr,),
                        x + "uk": (H * d, kr), x + "uv": (H * dv, kr)})
        elif spec["type"] == "lightning":
            out.update({x + "q": (H * d, W), x + "k": (H * d, W), x + "v": (H * dv, W), x + "g": (H * dv, W), x + "norm": (H * dv,)})
        else:
            out.update({x + "q": (H * d, W), x + "f": (H * d, W), x + "f.b": (H * d,), x + "lower": (H * d,), x + "v": (H * dv, W), x + "norm": (dv,)})
        out[x + "o"] = (W, H * dv)
        if spec.get("mlp") is not None:
            norm(p + "norm2")
            ff = int(spec["mlp"]["ff"])
            out.update({p + "mlp.up": (ff, W), p + "mlp.down": (W, ff), p + "mlp.act": (4,), p + "ls2": (W,)})
    norm("final.norm")
    return out


class RandomSource(RandomTensors):
    """N(0, std) matrices, norms near the identity, forget gates spread over (lower, 1)."""

    def __init__(self, cfg: FofosunConfig, seed: int, device="cpu", std: float | None = None):
        super().__init__(tensor_shapes(cfg), seed, device)
        self.std = std

    def draw(self, name, shape, rnd, uni):
        leaf = name.rsplit(".", 1)[-1]
        if len(shape) == 2:
            return rnd() * (self.std if self.std is not None else shape[1] ** -0.5 if name != "embed" else 1.0)
        if leaf == "alpha":
            return torch.full(shape, 0.5, device=self.device)
        if leaf == "lower":
            return 0.9 * uni()
        if name.endswith("f.b"):
            return 2.0 + rnd()
        if leaf == "b":
            return 0.05 * rnd()
        if leaf == "act":
            return torch.tensor([0.6, 0.3, 0.2, 0.05], device=self.device)
        return 0.7 + 0.1 * rnd() if leaf in ("ls1", "ls2") else 1.0 + 0.1 * rnd()


def save_checkpoint(model_dir, config: dict, seed: int = 0, tensors: dict | None = None):
    """Write a model directory with random weights; ``tensors`` replaces some of them."""
    save_listed(model_dir, config, RandomSource(FofosunConfig.from_dict(config), seed), tensors)


def load_fofosun(hf: dict, src, device, comm=None, dtype="bf16", **_):
    return FofosunModel(FofosunConfig.from_dict(hf), device, comm, dtype).load(src)
