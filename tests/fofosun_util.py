"""Small Fofosun configurations for the tests."""
import json

import torch

import fofosun_plain as plain
from listed_util import DEVICES, DTYPES, TOL, engine, off, one_thread, tokens  # noqa: F401
from volta_engine_b200.models.fofosun import FofosunConfig, FofosunModel, RandomSource


def hgrn2(heads, dim, vdim, ff=None):
    return {"type": "hgrn2", "mixer": {"heads": heads, "dim": dim, "vdim": vdim}, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def lightning(decay, dim, vdim, ff=None):
    return {"type": "lightning", "mixer": {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": decay},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads, dim, rot, vdim, kv_rank, q_rank, base=1000.0, scale=None, ff=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                      "rot": {"base": base, "dims": rot}, "scale": scale or (dim + rot) ** -0.5},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Fofosun", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}}


CONFIGS = {
    # widths that are multiples of 8 but of little else; mlp on every kind of layer
    "eights": config(104, 328, [latent(3, 40, 8, 24, 72, 56, ff=200), hgrn2(3, 24, 40, ff=88), lightning([0.5, 0.97, 0.999, 1.0], 16, 48),
                                hgrn2(1, 56, 16), latent(1, 16, 24, 72, 136, 24)]),
    # odd widths: no 16-byte rows anywhere
    "odd": config(75, 131, [lightning([0.9], 9, 21, ff=53), hgrn2(2, 13, 10), latent(3, 21, 6, 18, 50, 33, base=77.0, ff=101)], eps=3e-4),
    # widths of a larger model, two heads
    "wide": config(192, 512, [hgrn2(2, 128, 64), lightning([0.8, 0.995], 96, 128, ff=320), latent(2, 128, 64, 128, 320, 160)]),
    # no attention layer at all, one head everywhere
    "recurrent": config(64, 96, [hgrn2(1, 32, 32), lightning([0.99], 64, 32, ff=64)]),
    # attention only, latent wider than the tensor-core decode kernel takes
    "attention": config(128, 200, [latent(2, 24, 16, 40, 544, 48, ff=96)]),
}


class Weights:
    """Random weights with long memories: the forget gates of half the channels stay close to one."""

    def __init__(self, cfg, seed):
        self.src = RandomSource(FofosunConfig.from_dict(cfg), seed)
        self.t = {}
        for n in self.src.shapes:
            t = self.src.tensor(n)
            if n.endswith(".lower"):
                t = torch.where(torch.arange(t.numel()) % 2 == 0, 1.0 - (1.0 - t.float()) * 0.03, t.float()).to(torch.bfloat16)
            self.t[n] = t

    def has(self, name):
        return name in self.t

    def tensor(self, name, device=None, dtype=None):
        return self.t[name].to(device=device or "cpu", dtype=dtype or torch.bfloat16)


_made = {}


def make(name, device, dtype, seed=3):
    """-> (config, plain weights, model)."""
    key = (name, device, dtype, seed)
    if key not in _made:
        cfg = CONFIGS[name]
        w = Weights(cfg, seed)
        _made[key] = (cfg, w.t, FofosunModel(FofosunConfig.from_dict(cfg), device, None, dtype).load(w))
    return _made[key]


_want = {}


def reference(name, tokens, seed=3):
    """Plain logits of every position (cached: several tests share prompts)."""
    key = (name, tuple(tokens), seed)
    if key not in _want:
        _want[key] = plain.forward(CONFIGS[name], Weights(CONFIGS[name], seed).t, tokens)[0]
    return _want[key]


def write_model(path, name, seed=3):
    from volta_engine_b200.models.fofosun import save_checkpoint
    save_checkpoint(path, CONFIGS[name], seed, tensors=Weights(CONFIGS[name], seed).t)
    return json.loads((path / "config.json").read_text())
