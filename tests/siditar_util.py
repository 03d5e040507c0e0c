"""Small Siditar configurations for the tests."""
import json

import torch

import siditar_plain as plain
from listed_util import DEVICES, DTYPES, TOL, engine, off, one_thread, tokens  # noqa: F401
from volta_engine_b200.models.siditar import RandomSource, SiditarConfig, SiditarModel


def layer(left, right, ff=None, limit=1.5, scales=(0.9, 0.7)):
    """left = (heads, kv heads, dim, vdim, scale, farthest distance, temperature coefficient, every), right = (heads, dim, vdim, tau)."""
    H, G, d, dv, sc, far, coef, every = left
    return {"type": "parallel",
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": sc, "bias_max": far, "q_temp": {"coef": coef, "every": every}},
                      "right": dict(zip(("heads", "dim", "vdim", "tau"), right)), "left_scale": scales[0], "right_scale": scales[1]},
            "mlp": {"kind": "dense", "ff": ff, "limit": limit} if ff else None}


def config(width, vocab, layers, streams, loop=None, eps=1e-5):
    return {"architecture": "Siditar", "width": width, "vocab": vocab, "layers": layers, "streams": streams, "norm": {"eps": eps},
            "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None}


CONFIGS = {
    # widths that are multiples of 8 but of little else; unlike layers share one pool; a loop in the middle; a layer without feed-forward
    "eights": config(104, 328, [layer((4, 2, 24, 40, 0.31, 40, 0.4, 50), (3, 16, 24, 8.0), 88), layer((3, 1, 40, 16, 0.2, 90, 0.3, 16), (1, 32, 40, 1.0)),
                                layer((2, 2, 16, 72, 0.25, 17, -0.2, 7), (2, 56, 16, 3.5), 200, 0.4, (1.0, 1.3))], 3, (1, 3, 2)),
    # odd widths: no 16-byte rows anywhere; one stream
    "odd": config(75, 131, [layer((3, 3, 21, 13, 0.2, 30, 0.5, 11), (2, 9, 21, 16.0), 53), layer((2, 1, 9, 18, 0.4, 9, 0.1, 100), (3, 13, 10, 2.0), 101)], 1,
                  (0, 1, 1), 3e-4),
    # widths of a larger model; the whole stack runs twice
    "wide": config(192, 512, [layer((8, 2, 128, 128, 0.09, 128, 0.2, 64), (2, 128, 128, 16.0), 320, 7.0), layer((4, 4, 64, 128, 0.12, 64, 0.2, 64), (2, 96, 64, 4.0), 96)],
                   2, (0, 2, 2)),
    # one head, one kv head for many heads, widths outside the tensor-core kernels' range
    "edges": config(64, 96, [layer((18, 1, 16, 8, 0.3, 24, 0.2, 9), (1, 40, 136, 5.0), 64), layer((1, 1, 264, 24, 0.06, 50, 0.2, 20), (1, 200, 8, 9.0)),
                             layer((2, 2, 200, 160, 0.07, 33, 0.0, 1), (1, 8, 8, 1.0), 40)], 5),
}
SHAPES = {"eights": {"bias_rows": 16, "rank": 12}, "odd": {"bias_rows": 6, "rank": 5}, "wide": {"bias_rows": 32, "rank": 16}, "edges": {"bias_rows": 8, "rank": 40}}


class Weights:
    """Random weights with long memories: the decays of half the channels stay close to one."""

    def __init__(self, name, seed):
        self.src = RandomSource(SiditarConfig.from_dict(CONFIGS[name]), seed, **SHAPES[name])
        self.t = {}
        for n in self.src.shapes:
            t = self.src.tensor(n)
            if n.endswith("a2.b"):
                t = torch.where(torch.arange(t.numel()) % 2 == 0, t.float() + 5.0, t.float()).to(torch.bfloat16)
            self.t[n] = t

    def has(self, name):
        return name in self.t

    def tensor(self, name, device=None, dtype=None):
        return self.t[name].to(device=device or "cpu", dtype=dtype or torch.bfloat16)


_made, _want = {}, {}


def make(name, device, dtype, seed=3):
    """-> (config, plain weights, model)."""
    key = (name, device, dtype, seed)
    if key not in _made:
        w = Weights(name, seed)
        _made[key] = (CONFIGS[name], w.t, SiditarModel(SiditarConfig.from_dict(CONFIGS[name]), device, None, dtype).load(w))
    return _made[key]


def reference(name, toks, seed=3):
    """Plain logits of every position (cached: several tests share prompts)."""
    key = (name, tuple(toks), seed)
    if key not in _want:
        _want[key] = plain.forward(CONFIGS[name], Weights(name, seed).t, toks)[0]
    return _want[key]


def write_model(path, name, seed=3):
    from volta_engine_b200.models.siditar import save_checkpoint
    save_checkpoint(path, CONFIGS[name], seed, tensors=Weights(name, seed).t, **SHAPES[name])
    return json.loads((path / "config.json").read_text())
