"""Siditar: a decoder whose configuration lists its layers one by one. Every layer mixes tokens by grouped-query attention (bias by
distance, sink, query temperature, normed queries and keys) and gated linear attention side by side; layer norms without shift
stand in front of the sublayers, several fp32 residual streams are read and rewritten with static weights (hyper-connections), the
feed-forward is a clamped gated unit, and positions enter the embedding as sinusoids. A range of layers runs several times.

The decoder is the one of :mod:`.listed`, the mixers those of :mod:`.mixers`, norms and activations the row operators of
:mod:`..ops.rowops`; cache, state slots, scheduling and sampling are the engine's. A model runs in bf16 (matrix products and
activations; scores, decays, states, norms and the residual streams in fp32) or, with ``dtype="fp32"``, in fp32 throughout.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

from ..ops.rowops import ClampedGlu, SinusoidalPositions, StreamNorm, StreamWrite, embed_rows
from .feed_forward import DenseFF
from .listed import ListedConfig, ListedLayer, ListedModel, RandomTensors, save_listed
from .mixers import MIXERS, make_linear

# CUDA sources whose kernels this model and its sampling launch
KERNEL_SOURCES = ("gemm_bf16_wide.cu", "gemm_tcgen05.cu", "gemv_rows.cu", "gqa.cu", "linattn.cu", "rowops.cu", "sampling.cu")
POSITION_BASE = 10000.0
GLU_ALPHA = 1.702
MAX_STREAMS = 8                 # of the stream kernels (csrc/cuda/rowmath.cuh)


@dataclass
class SiditarConfig(ListedConfig):
    streams: int = 1
    model_type: str = "siditar"

    @classmethod
    def from_dict(cls, c: dict) -> "SiditarConfig":
        S = int(c["streams"])
        if not 1 <= S <= MAX_STREAMS:
            raise NotImplementedError(f"{S} residual streams (1 to {MAX_STREAMS} in this build)")
        return cls.listed(c, streams=S)


class SiditarModel(ListedModel):
    def load_ends(self, src) -> None:
        dev, dt, cfg = self.device, self.dtype, self.cfg
        self.embed = src.tensor("embed", dev, dt).contiguous()
        self.positions = SinusoidalPositions(cfg.hidden, POSITION_BASE, dev)
        self.final_norm = StreamNorm(src.tensor("final.norm", dev, torch.float32).contiguous(), cfg.rms_eps, torch.ones(cfg.streams, device=dev))
        self.lm_head = make_linear(src, "head", dev, dt)

    def load_layer(self, i: int, spec: dict, src) -> ListedLayer:
        dev, dt, eps, p = self.device, self.dtype, self.cfg.rms_eps, f"l{i}."
        f32 = lambda name: src.tensor(name, dev, torch.float32).contiguous()
        norm = lambda q: StreamNorm(f32(f"{p}norm{q}"), eps, f32(f"{p}hc{q}.in"))
        write = lambda q: StreamWrite(f32(f"{p}hc{q}.mix"), f32(f"{p}hc{q}.out"))
        L = ListedLayer(MIXERS[spec["type"]](spec["type"], spec["mixer"], eps, src, p + "mix.", dev, dt), norm(1), write(1))
        if spec.get("mlp") is not None:
            L.norm2, L.write2 = norm(2), write(2)
            L.ff = DenseFF.gated(src, p + "mlp.", ClampedGlu(float(spec["mlp"]["limit"]), GLU_ALPHA), dev, dt)
        return L

    def embed_batch(self, b):
        return embed_rows(b.ids, self.embed, b.pos, self.positions, self.cfg.streams)

    def residual_rows(self, h, part=None, write=None):
        h = h.clone()
        if part is not None:
            write.add(h, part)
        return h.sum(1)

    def init_random(self, seed: int = 1, std: float = 0.02, search: bool = False):
        return self.load(RandomSource(self.cfg, seed, self.device, std))


# ---------------------------------------------------------------------------------------------- random weights
def tensor_shapes(cfg: SiditarConfig, bias_rows: int = 32, rank: int = 16) -> dict:
    """Checkpoint tensor names -> shapes. ``bias_rows``, ``rank``: rows of the distance tables and width of the low-rank decays, which
    only the tensors say."""
    W, S = cfg.hidden, cfg.streams
    out = {"embed": (cfg.vocab, W), "head": (cfg.vocab, W), "final.norm": (W,)}
    for i, spec in enumerate(cfg.layers):
        p, m = f"l{i}.", spec["mixer"]
        a, r = m["left"], m["right"]
        H, G, d, dv = int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"])
        x = p + "mix.left."
        out.update({p + "norm1": (W,), x + "q": (H * d, W), x + "k": (G * d, W), x + "v": (G * dv, W), x + "q.norm": (d,), x + "k.norm": (d,),
                    x + "rel": (bias_rows, H), x + "sink": (H,), x + "o": (W, H * dv)})
        H, d, dv = int(r["heads"]), int(r["dim"]), int(r["vdim"])
        x = p + "mix.right."
        out.update({x + "q": (H * d, W), x + "k": (H * d, W), x + "v": (H * dv, W), x + "g": (H * dv, W), x + "o": (W, H * dv), x + "norm": (dv,),
                    x + "a1": (rank, W), x + "a2": (H * d, rank), x + "a2.b": (H * d,)})
        subs = [1]
        if spec.get("mlp") is not None:
            ff = int(spec["mlp"]["ff"])
            out.update({p + "norm2": (W,), p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
            subs.append(2)
        for q in subs:
            out.update({f"{p}hc{q}.in": (S,), f"{p}hc{q}.out": (S,), f"{p}hc{q}.mix": (S, S)})
    return out


class RandomSource(RandomTensors):
    """N(0, std) matrices, norms near the identity, decays spread over long and short memories, streams that mix."""

    def __init__(self, cfg: SiditarConfig, seed: int, device="cpu", std: float | None = None, bias_rows: int = 32, rank: int = 16):
        super().__init__(tensor_shapes(cfg, bias_rows, rank), seed, device)
        self.std = std

    def draw(self, name, shape, rnd, uni):
        leaf = name.rsplit(".", 1)[-1]
        if leaf == "mix" and "hc" in name:
            return 0.7 * torch.eye(shape[0], device=self.device) + 0.3 * uni()
        if leaf in ("in", "out") and "hc" in name:
            return 0.3 + 0.7 * uni()
        if leaf in ("rel", "sink"):
            return rnd()
        if len(shape) == 2:
            return rnd() * (self.std if self.std is not None else shape[1] ** -0.5 if name != "embed" else 1.0)
        return 1.0 + 2.0 * rnd() if name.endswith("a2.b") else 1.0 + 0.1 * rnd()


def save_checkpoint(model_dir, config: dict, seed: int = 0, tensors: dict | None = None, **shapes):
    """Write a model directory with random weights; ``tensors`` replaces some of them."""
    save_listed(model_dir, config, RandomSource(SiditarConfig.from_dict(config), seed, **shapes), tensors)


def load_siditar(hf: dict, src, device, comm=None, dtype="bf16", **_):
    return SiditarModel(SiditarConfig.from_dict(hf), device, comm, dtype).load(src)
