"""Small Kutolix configurations for the tests."""
import json

import torch

import kutolix_plain as plain
from listed_util import DEVICES, DTYPES, TOL, engine, off, one_thread, tokens  # noqa: F401
from volta_engine_b200.models.kutolix import KutolixConfig, KutolixModel, RandomSource


def attention(heads, kv_heads, dim, vdim, scale, window, dims, base, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": window},
                                                       "rot": {"base": base, "dims": dims}}}


def latent(heads, dim, rot, vdim, rank, scale, window, base, scaling, mlp=None):
    """scaling = (factor, original, fast, slow)."""
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale,
                                                              "mask": {"size": window},
                                                              "rot": {"base": base, "dims": rot, "scaling": dict(zip(("factor", "original", "fast", "slow"), scaling))}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, limit, count=1, keep=1):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top, "groups": {"count": count, "keep": keep}}}


def config(width, vocab, layers, scale, mult, cap, eps=1e-5):
    return {"architecture": "Kutolix", "width": width, "vocab": vocab, "layers": layers, "embedding": {"scale": scale}, "residual_mult": mult, "logit_softcap": cap,
            "norm": {"eps": eps}}


CONFIGS = {
    # widths that are multiples of 8 but of little else; unlike layers share one pool; latent first; a layer without feed-forward
    "eights": config(104, 328, [latent(3, 16, 8, 24, 40, 0.3, 27, 300.0, (8.0, 64, 6.0, 1.0), moe(12, 3, 40, 0.8, 3, 2)),
                                attention(4, 1, 24, 40, 0.31, 37, 16, 500.0, dense(88)), attention(6, 2, 40, 16, 0.2, 70, 40, 9000.0),
                                latent(2, 40, 16, 8, 24, 0.2, 64, 2000.0, (2.5, 200, 20.0, 2.0), dense(200)), attention(2, 2, 16, 72, 0.4, 8, 8, 77.0, moe(6, 2, 24, 2.0, 6, 3))],
                     8.0, 0.8, 9.0),
    # odd widths: no 16-byte rows anywhere; no groups
    "odd": config(75, 131, [attention(3, 3, 21, 13, 0.3, 19, 10, 400.0, moe(7, 2, 19, 1.1)), latent(2, 9, 6, 7, 21, 0.35, 33, 90.0, (3.0, 40, 4.0, 1.0), dense(53)),
                            attention(2, 1, 9, 18, 0.5, 100, 6, 50.0, moe(5, 4, 33, 0.5, 5, 4))], 4.0, 0.9, 6.0, 3e-4),
    # widths of a larger model; windows of whole pages and one off
    "wide": config(192, 512, [attention(8, 2, 128, 64, 0.1, 128, 64, 1e4, dense(320)), latent(4, 64, 32, 128, 128, 0.13, 64, 1e4, (4.0, 256, 16.0, 1.0), moe(16, 4, 64, 3.0, 4, 2)),
                              attention(4, 4, 64, 128, 0.15, 129, 64, 1e5, moe(32, 5, 72, 1.5, 2, 1)), latent(17, 32, 16, 24, 64, 0.2, 63, 500.0, (16.0, 128, 8.0, 0.5), dense(96))],
                   14.0, 0.6, 12.0),
    # one head, one kv head for many heads, widths outside the tensor-core kernels' range, a window of one key, one beyond every prompt
    "edges": config(64, 96, [attention(18, 1, 16, 8, 0.5, 1, 2, 10.0, dense(64)), attention(1, 1, 264, 24, 0.05, 1000, 264, 1e4, moe(3, 3, 8, 0.7)),
                             latent(1, 200, 64, 160, 536, 0.06, 45, 1e4, (2.0, 100, 9.0, 1.0)), latent(2, 12, 4, 12, 12, 0.4, 2, 30.0, (1.0, 50, 3.0, 1.0), moe(40, 1, 16, 5.0, 8, 1))],
                    1.5, 0.5, 30.0),
}


# the first one again with a quieter embedding: a tied head would repeat the last token for ever
CONFIGS["quiet"] = dict(CONFIGS["eights"], embedding={"scale": 0.8}, residual_mult=1.1)
NAMES = ["eights", "odd", "wide", "edges"]


class Weights:
    """Random weights; sinks that count; routers that are sure of their best expert, so that a rounded input changes the choice of the
    last one only."""

    def __init__(self, name, seed):
        self.src = RandomSource(KutolixConfig.from_dict(CONFIGS[name]), seed)
        self.t = {}
        for n in self.src.shapes:
            t = self.src.tensor(n).float()
            if n.endswith(".router"):
                t = t * 4.0
            if n == "embed":
                t = t * 4.0 * CONFIGS[name]["width"] ** -0.5          # logits within the soft cap's bend
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
        _made[key] = (CONFIGS[name], w.t, KutolixModel(KutolixConfig.from_dict(CONFIGS[name]), device, None, dtype).load(w))
    return _made[key]


def reference(name, toks, seed=3):
    """Plain logits of every position (cached: several tests share prompts)."""
    key = (name, tuple(toks), seed)
    if key not in _want:
        _want[key] = plain.forward(CONFIGS[name], Weights(name, seed).t, toks)[0]
    return _want[key]


def write_model(path, name, seed=3):
    from volta_engine_b200.models.kutolix import save_checkpoint
    save_checkpoint(path, CONFIGS[name], seed, tensors=Weights(name, seed).t)
    return json.loads((path / "config.json").read_text())
