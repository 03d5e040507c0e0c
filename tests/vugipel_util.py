"""Small Vugipel configurations for the tests."""
import json

import torch

import vugipel_plain as plain
from listed_util import DEVICES, DTYPES, TOL, engine, off, one_thread, tokens  # noqa: F401
from volta_engine_b200.models.vugipel import RandomSource, VugipelConfig, VugipelModel


def gru(width, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def side_by_side(left, right, scales=(0.9, 0.7), mlp=None):
    """left = (heads, kv heads, dim, vdim, scale, window, first tokens kept, rotated columns, base, cap), right = (heads, dim, vdim, decays)."""
    H, G, d, dv, scale, window, first, dims, base, cap = left
    h, rd, rv, decay = right
    return {"type": "parallel", "mlp": mlp,
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": scale, "softcap": cap, "mask": {"size": window, "keep_first": first},
                               "rot": {"base": base, "dims": dims}},
                      "right": {"heads": h, "dim": rd, "vdim": rv, "decay": decay}, "left_scale": scales[0], "right_scale": scales[1]}}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(width, vocab, layers, eps=1e-5):
    return {"architecture": "Vugipel", "width": width, "vocab": vocab, "layers": layers, "norm": {"eps": eps}}


CONFIGS = {
    # widths that are multiples of 8 but of little else; unlike layers share one pool; a layer without feed-forward
    "eights": config(104, 328, [gru(88, moe(6, 1, 40)),
                                side_by_side((4, 2, 24, 40, 0.4, 37, 5, 16, 500.0, 9.0), (3, 16, 24, [0.9, 0.99, 0.7]), mlp=moe(4, 3, 24)), gru(136),
                                side_by_side((6, 3, 40, 16, 0.3, 70, 1, 40, 9000.0, 4.0), (2, 40, 48, [0.998, 0.5]), (0.6, 1.2)),
                                side_by_side((2, 2, 16, 72, 0.5, 8, 66, 8, 77.0, 30.0), (1, 56, 16, [0.97]), (1.0, 1.0), moe(3, 2, 88))]),
    # odd widths: no 16-byte rows anywhere
    "odd": config(75, 131, [gru(53, moe(7, 2, 19)), side_by_side((3, 3, 21, 14, 0.45, 19, 2, 10, 400.0, 6.0), (2, 9, 21, [0.95, 0.99]), mlp=moe(4, 3, 33)), gru(37),
                            side_by_side((2, 1, 9, 18, 0.6, 100, 3, 6, 50.0, 12.0), (3, 13, 10, [0.9, 1.0, 0.6]), (1.3, 0.4))], 3e-4),
    # widths of a larger model; windows of whole pages and one off; kept tokens up to a page border and across it
    "wide": config(256, 512, [side_by_side((8, 2, 128, 128, 0.1, 128, 64, 64, 1e4, 15.0), (2, 128, 128, [0.99, 0.9]), mlp=moe(16, 2, 72)), gru(320, moe(24, 1, 136)),
                              side_by_side((4, 4, 64, 96, 0.15, 63, 65, 64, 1e5, 8.0), (4, 64, 96, [0.5, 0.9, 0.99, 0.999]), (0.5, 0.8)), gru(200, moe(8, 4, 64))]),
    # one head, one kv head for many heads, widths outside the tensor-core kernels' range, a window of one key, one beyond every prompt
    "edges": config(64, 96, [side_by_side((18, 1, 16, 8, 0.6, 1, 1, 2, 10.0, 5.0), (1, 40, 136, [0.99]), mlp=moe(3, 3, 8)),
                             side_by_side((1, 1, 264, 24, 0.08, 1000, 4, 264, 1e4, 20.0), (1, 200, 8, [0.9]), (0.3, 1.0)), gru(8, moe(40, 1, 16)),
                             side_by_side((2, 1, 24, 160, 0.4, 45, 130, 12, 200.0, 7.0), (2, 8, 8, [0.0, 0.97])), gru(1)]),
}
NAMES = list(CONFIGS)


class Weights:
    """Random weights; gates of all kinds (channels that never forget, channels that keep nothing); routers that are sure of their best
    expert, so that a rounded input changes the choice of the last one only."""

    def __init__(self, name, seed):
        self.src = RandomSource(VugipelConfig.from_dict(CONFIGS[name]), seed)
        self.t = {}
        for n in self.src.shapes:
            t = self.src.tensor(n).float()
            if n.endswith(".router"):
                t = t * 4.0
            if n.endswith(".z.b"):
                t[::5] -= 6.0
                t[1::5] += 9.0
            self.t[n] = t.to(torch.bfloat16)

    def has(self, name):
        return name in self.t

    def tensor(self, name, device=None, dtype=None):
        return self.t[name].to(device=device or "cpu", dtype=dtype or torch.bfloat16)


def wrong(got, want, dtype):
    """Row errors as ``off`` has them: the largest in fp32; in bf16, where a close call of a router may fall the other way on a few
    rows, the one that 85 % of the rows stay below."""
    g, w = got.double().cpu(), want.double()
    e = (g - w).pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().mean()
    return (e.max() if dtype == "fp32" else e.quantile(0.85)).item()


_made, _want = {}, {}


def make(name, device, dtype, seed=3):
    """-> (config, plain weights, model)."""
    key = (name, device, dtype, seed)
    if key not in _made:
        w = Weights(name, seed)
        _made[key] = (CONFIGS[name], w.t, VugipelModel(VugipelConfig.from_dict(CONFIGS[name]), device, None, dtype).load(w))
    return _made[key]


def reference(name, toks, seed=3):
    """Plain logits of every position (cached: several tests share prompts)."""
    key = (name, tuple(toks), seed)
    if key not in _want:
        _want[key] = plain.forward(CONFIGS[name], Weights(name, seed).t, toks)[0]
    return _want[key]


def write_model(path, name, seed=3):
    from volta_engine_b200.models.vugipel import save_checkpoint
    save_checkpoint(path, CONFIGS[name], seed, tensors=Weights(name, seed).t)
    return json.loads((path / "config.json").read_text())
