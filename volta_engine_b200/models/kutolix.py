"""Kutolix: a decoder whose configuration lists its layers one by one. Every layer mixes tokens by grouped-query attention (rotary
positions, normed queries and keys, a sliding window, a sink, an output gate) or by latent attention (direct queries, scaled rotary
positions, a sliding window), and has a gated SiLU feed-forward, a mixture of clamped gated experts, or none. Sublayers read the fp32
residual as it is; their results enter it through an RMS norm and a common factor. Scaled embeddings, tied head, soft-capped logits.

The decoder is the one of :mod:`.listed`, mixers and feed-forwards those of :mod:`.mixers` and :mod:`.feed_forward`, norms and
activations the row operators of :mod:`..ops.rowops`; cache, scheduling and sampling are the engine's. A model runs in bf16 (matrix
products and activations; angles, scores, router, norms and the residual in fp32) or, with ``dtype="fp32"``, in fp32 throughout.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..ops.linear import LinearBF16, LinearF32
from ..ops.routed import Router
from ..ops.rowops import ClampedGlu, NormedWrite, ResidualNorm, embed_rows
from .feed_forward import DenseFF, RoutedFF
from .listed import ListedConfig, ListedLayer, ListedModel, RandomTensors, save_listed
from .mixers import MIXERS

# CUDA sources whose kernels this model and its sampling launch
KERNEL_SOURCES = ("gemm_bf16_wide.cu", "gemm_tcgen05.cu", "gemv_rows.cu", "gqa.cu", "latent.cu", "mla.cu", "moe.cu", "routed.cu", "rowops.cu", "sampling.cu")
EXPERT_ALPHA = 1.702


@dataclass
class KutolixConfig(ListedConfig):
    residual_mult: float = 1.0
    model_type: str = "kutolix"

    @classmethod
    def from_dict(cls, c: dict) -> "KutolixConfig":
        return cls.listed(c, ("dense", "moe"), embed_scale=float(c["embedding"]["scale"]), residual_mult=float(c["residual_mult"]),
                          logit_softcap=float(c.get("logit_softcap") or 0.0), tie_embeddings=True)


def router_of(m: dict) -> Router:
    g = m.get("groups") or {"count": 1, "keep": 1}
    return Router(int(m["experts"]), int(m["top"]), int(g["count"]), int(g["keep"]))


class KutolixModel(ListedModel):
    def load_ends(self, src) -> None:
        dev, dt, cfg = self.device, self.dtype, self.cfg
        self.embed = src.tensor("embed", dev, dt).contiguous()
        self.final_norm = ResidualNorm(src.tensor("final.norm", dev, torch.float32).contiguous(), cfg.rms_eps)
        self.lm_head = LinearF32(self.embed) if dt == torch.float32 else LinearBF16(self.embed)

    def load_layer(self, i: int, spec: dict, src) -> ListedLayer:
        dev, dt, eps, p = self.device, self.dtype, self.cfg.rms_eps, f"l{i}."
        read = ResidualNorm(None, eps)
        write = lambda q: NormedWrite((src.tensor(f"{p}norm{q}", dev, torch.float32) * self.cfg.residual_mult).contiguous(), eps)
        L = ListedLayer(MIXERS[spec["type"]](spec["type"], spec["mixer"], eps, src, p + "mix.", dev, dt), read, write(1))
        m = spec.get("mlp")
        if m is not None:
            L.norm2, L.write2 = read, write(2)
            if m["kind"] == "moe":
                L.ff = RoutedFF(src, p + "mlp.", router_of(m["router"]), ClampedGlu(float(m["expert"]["limit"]), EXPERT_ALPHA), dev, dt)
            else:
                L.ff = DenseFF.gated(src, p + "mlp.", ClampedGlu.silu(), dev, dt)
        return L

    def embed_batch(self, b):
        return embed_rows(b.ids, self.embed, scale=self.cfg.embed_scale)

    def residual_rows(self, h, part=None, write=None):
        h = h.clone()
        if part is not None:
            write.add(h, part)
        return h

    def init_random(self, seed: int = 1, std: float = 0.02, search: bool = False):
        return self.load(RandomSource(self.cfg, seed, self.device, std))


# ---------------------------------------------------------------------------------------------- random weights
def tensor_shapes(cfg: KutolixConfig) -> dict:
    """Checkpoint tensor names -> shapes."""
    W = cfg.hidden
    out = {"embed": (cfg.vocab, W), "final.norm": (W,)}
    for i, spec in enumerate(cfg.layers):
        p, m = f"l{i}.", spec["mixer"]
        H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
        x = p + "mix."
        out[p + "norm1"] = (W,)
        if spec["type"] == "latent_attention":
            r, kr = int(m["rot_dim"]), int(m["kv_rank"])
            out.update({x + "q": (H * (d + r), W), x + "dkv": (kr + r, W), x + "dkv.norm": (kr,), x + "uk": (H * d, kr), x + "uv": (H * dv, kr)})
        else:
            G = int(m["kv_heads"])
            out.update({x + "q": (H * d, W), x + "k": (G * d, W), x + "v": (G * dv, W), x + "sink": (H,), x + "g": (H * dv, W)})
        out[x + "o"] = (W, H * dv)
        f = spec.get("mlp")
        if f is None:
            continue
        out[p + "norm2"] = (W,)
        y = p + "mlp."
        if f["kind"] == "moe":
            ff = int(f["expert"]["ff"])
            out[y + "router"] = (int(f["router"]["experts"]), W)
            for e in range(int(f["router"]["experts"])):
                out.update({f"{y}e{e}.gate": (ff, W), f"{y}e{e}.up": (ff, W), f"{y}e{e}.down": (W, ff)})
        else:
            ff = int(f["ff"])
            out.update({y + "gate": (ff, W), y + "up": (ff, W), y + "down": (W, ff)})
    return out


class RandomSource(RandomTensors):
    """N(0, std) matrices, norms near the identity."""

    def __init__(self, cfg: KutolixConfig, seed: int, device="cpu", std: float | None = None):
        super().__init__(tensor_shapes(cfg), seed, device)
        self.std = std

    def draw(self, name, shape, rnd, uni):
        if name.endswith(".sink"):
            return rnd()
        if len(shape) == 2:
            return rnd() * (self.std if self.std is not None else shape[1] ** -0.5 if name != "embed" else 1.0)
        return 1.0 + 0.1 * rnd()


def save_checkpoint(model_dir, config: dict, seed: int = 0, tensors: dict | None = None):
    """Write a model directory with random weights; ``tensors`` replaces some of them."""
    save_listed(model_dir, config, RandomSource(KutolixConfig.from_dict(config), seed), tensors)


def load_kutolix(hf: dict, src, device, comm=None, dtype="bf16", **_):
    return KutolixModel(KutolixConfig.from_dict(hf), device, comm, dtype).load(src)
