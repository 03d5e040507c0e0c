"""Fofosun: a decoder whose configuration lists its layers one by one. Every layer has a token mixer of its own type and sizes
(HGRN2, lightning attention, latent attention) and an optional feed-forward; Dynamic-Tanh norms in front of the sublayers,
an element-wise layer scale on their results, an fp32 residual stream, a PolyNorm feed-forward.

The mixers are those of :mod:`.mixers`, norms and activations the row operators of :mod:`..ops.rowops`; cache, state slots,
scheduling and sampling are the engine's. A model runs in bf16 (matrix products and activations; scores, gates, states,
norms and the residual in fp32) or, with ``dtype="fp32"``, in fp32 throughout.
"""
from __future__ import annotations

import json
from dataclasses import dataclass, field
from pathlib import Path

import torch

from ..ops.rowops import DynamicTanh, PolyNorm, embed_rows, fused_fits, gemv_rows
from ..runtime.batch import BatchRows
from .dense import DenseConfig, DenseModel
from .mixers import MIXERS, apply_linear, make_linear
from .slot_state import SlotStates

# CUDA sources whose kernels this model and its sampling launch
KERNEL_SOURCES = ("gemm_bf16_wide.cu", "gemm_tcgen05.cu", "gemv_rows.cu", "latent.cu", "linattn.cu", "mla.cu", "rowops.cu", "sampling.cu")
DTYPES = {"bf16": torch.bfloat16, "bfloat16": torch.bfloat16, "fp32": torch.float32, "float32": torch.float32}


@dataclass
class FofosunConfig(DenseConfig):
    layers: list = field(default_factory=list)      # [{"type", "mixer": {sizes}, "mlp": {"kind", "ff"} | None}]
    residual: str = "fp32"
    model_type: str = "fofosun"

    @classmethod
    def from_dict(cls, c: dict) -> "FofosunConfig":
        layers = [dict(L) for L in c["layers"]]
        for i, L in enumerate(layers):
            if L["type"] not in MIXERS:
                raise NotImplementedError(f"layer {i}: no mixer {L['type']!r} in this build")
            if L.get("mlp") is not None and L["mlp"].get("kind", "dense") != "dense":
                raise NotImplementedError(f"layer {i}: no feed-forward {L['mlp']['kind']!r} in this build")
        cfg = cls(n_layers=len(layers), hidden=int(c["width"]), vocab=int(c["vocab"]), rms_eps=float(c["norm"]["eps"]), layers=layers,
                  n_q=1, n_kv=1, ffn=max([int(L["mlp"]["ff"]) for L in layers if L.get("mlp") is not None] or [1]), quant="bf16")
        cfg.head_dim = cfg.cache_width()
        return cfg

    def cache_width(self) -> int:
        """Elements of a paged cache row: the widest latent row of any layer."""
        from ..ops.latent import LatentSpec
        w = [LatentSpec(1, 1, int(m["rot_dim"]), 1, int(m["kv_rank"]), 1.0, 1.0, 1e-5).width
             for m in (L["mixer"] for L in self.layers if L["type"] == "latent_attention")]
        return max(w or [64])


class FofosunLayer:
    __slots__ = ("mixer", "norm1", "ls1", "norm2", "ls2", "up", "act", "down")


class FofosunModel(SlotStates, DenseModel):
    prefix_resume = "kv+state"
    supports_mixed = True           # prompt portions and decode rows of several sequences run in one forward

    def __init__(self, cfg: FofosunConfig, device, comm=None, dtype="bf16"):
        super().__init__(cfg, device, comm)
        if self.comm.size != 1:
            raise NotImplementedError("this model runs on one GPU (its norms over all heads and over the feed-forward width are not split)")
        self.dtype = DTYPES[dtype] if isinstance(dtype, str) else dtype
        self.vocab_pad = self.vocab_local = cfg.vocab
        self.layer_tap = None       # a list that receives the residual after every layer (tests, inspection)

    # ------------------------------------------------------------------------------------------ weights
    def load(self, src) -> "FofosunModel":
        """``src``: has ``tensor(name, device, dtype)`` (a checkpoint's tensor source, or :class:`RandomSource`)."""
        cfg, dev, dt, eps = self.cfg, self.device, self.dtype, self.cfg.rms_eps
        f32 = lambda name: src.tensor(name, dev, torch.float32).contiguous()
        self.embed = src.tensor("embed", dev, dt).contiguous()
        self.layers, n_cached = [], 0
        for i, spec in enumerate(cfg.layers):
            p, L = f"l{i}.", FofosunLayer()
            L.mixer = MIXERS[spec["type"]](spec["type"], spec["mixer"], eps, src, p + "mix.", dev, dt)
            if L.mixer.cached:
                L.mixer.cache_index = n_cached
                n_cached += 1
            L.norm1, L.ls1 = DynamicTanh.load(src, p + "norm1", dev), f32(p + "ls1")
            L.norm2 = L.ls2 = L.up = L.act = L.down = None
            if spec.get("mlp") is not None:
                L.norm2, L.ls2 = DynamicTanh.load(src, p + "norm2", dev), f32(p + "ls2")
                L.up, L.down = make_linear(src, p + "mlp.up", dev, dt), make_linear(src, p + "mlp.down", dev, dt)
                L.act = PolyNorm(f32(p + "mlp.act"), eps)
            self.layers.append(L)
        self.kv_layers = n_cached
        self.final_norm = DynamicTanh.load(src, "final.norm", dev)
        self.lm_head = make_linear(src, "head", dev, dt)
        return self

    def init_random(self, seed: int = 1, std: float = 0.02, search: bool = False):
        return self.load(RandomSource(self.cfg, seed, self.device, std))

    kv_layers = 0
    kv_v_dim = 8                    # the cache has one row per token: the value pool is a stub

    def link_prefetch(self) -> None:
        pass

    def ensure_workspace(self, max_rows: int, max_splits: int):
        pass

    def decode_bytes_per_token(self) -> int:
        n = self.lm_head.nbytes()
        for L in self.layers:
            n += sum(lin.nbytes() for lin in L.mixer.linears()) + (L.mixer.extra_bytes() if L.mixer.cached else 0)
            if L.up is not None:
                n += L.up.nbytes() + L.down.nbytes()
        return n

    def weight_bytes(self) -> int:
        return self.decode_bytes_per_token() + self.embed.numel() * self.embed.element_size()

    # ------------------------------------------------------------------------------------------ state slots
    def _states(self, kv) -> list:
        return [L.mixer.bind(kv) if not L.mixer.cached else None for L in self.layers]

    def layer_states(self) -> list:
        return [L.mixer.state for L in self.layers]

    def reset_states(self) -> None:
        """Forget the slots' states (an engine with another slot count is about to be built on this model)."""
        for L in self.layers:
            L.mixer.state = None
        for name in ("_jsets", "_shadows"):
            if hasattr(self, name):
                delattr(self, name)

    def state_bytes_per_slot(self) -> int:
        return sum(4 * m.spec.heads * m.spec.dk * m.spec.dv for m in (L.mixer for L in self.layers) if not m.cached)

    # ------------------------------------------------------------------------------------------ forward
    def forward(self, b: BatchRows, kv) -> torch.Tensor | None:
        if self.kv_layers and kv.k.dtype != self.dtype:
            raise ValueError(f"cache of {kv.k.dtype} under a model of {self.dtype}")
        h = embed_rows(b.ids, self.embed)
        if h.is_cuda and self.dtype == torch.bfloat16 and fused_fits(self._widest(), b.n):
            return self._forward_fused(b, kv, h)
        dt, part, scale = self.dtype, None, None
        for li, L in enumerate(self.layers):
            x = L.norm1.rows(h, dt, part, scale)
            part, scale = L.mixer.rows(x, b, kv, self._journal(li, L, b, kv)), L.ls1
            if L.up is not None:
                x = L.norm2.rows(h, dt, part, scale)
                z = apply_linear(L.up, x, out_f32=b.row_path)
                part, scale = apply_linear(L.down, L.act.rows(z, dt)), L.ls2
            if self.layer_tap is not None:
                self.layer_tap.append(h + part.float() * scale)
        x = self.final_norm.rows(h, dt, part, scale)
        self.last_hidden, self.last_residual = x, h
        x = b.select_logits(x)
        return None if x is None else apply_linear(self.lm_head, x, out_f32=True)

    def _forward_fused(self, b: BatchRows, kv, h):
        """A few decode rows: norms, activations, layer scales and residual adds ride in the linears' launches."""
        for li, L in enumerate(self.layers):
            L.mixer.step(L.norm1.prologue(h), (h, L.ls1), b, kv, self._journal(li, L, b, kv))
            if L.up is not None:
                z = gemv_rows(L.up, b.n, out_f32=True, **L.norm2.prologue(h))
                gemv_rows(L.down, b.n, residual=(h, L.ls2), **L.act.prologue(z))
            if self.layer_tap is not None:
                self.layer_tap.append(h.clone())
        self.last_residual = h
        h = b.select_logits(h)
        return None if h is None else gemv_rows(self.lm_head, h.shape[0], out_f32=True, **self.final_norm.prologue(h))

    def _journal(self, li, L, b, kv):
        return (None, None) if L.mixer.cached else self.journal_of(li, L.mixer.bind(kv), b)

    def _widest(self):
        """The linear with the longest input rows of those that take a prologue."""
        w = getattr(self, "_widest_lin", None)
        if w is None:
            lins = [self.lm_head] + [x for L in self.layers for x in (*L.mixer.linears(), L.up, L.down) if x is not None]
            w = self._widest_lin = max(lins, key=lambda x: x.weight.shape[1])
        return w


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


class RandomSource:
    """Random weights under the checkpoint names: N(0, std) matrices, norms near the identity, forget gates spread over
    (lower, 1). Every tensor has a generator of its own, so any subset can be drawn in any order."""

    def __init__(self, cfg: FofosunConfig, seed: int, device="cpu", std: float | None = None):
        self.shapes, self.seed, self.device, self.std = tensor_shapes(cfg), seed, torch.device(device), std
        self.order = {n: i for i, n in enumerate(sorted(self.shapes))}

    def has(self, name: str) -> bool:
        return name in self.shapes

    def tensor(self, name: str, device=None, dtype=None):
        shape = self.shapes[name]
        g = torch.Generator(device=self.device).manual_seed(self.seed * 1000003 + self.order[name])

        def rnd():
            return torch.randn(shape, generator=g, device=self.device)
        leaf = name.rsplit(".", 1)[-1]
        if len(shape) == 2:
            t = rnd() * (self.std if self.std is not None else shape[1] ** -0.5 if name != "embed" else 1.0)
        elif leaf == "alpha":
            t = torch.full(shape, 0.5, device=self.device)
        elif leaf == "lower":
            t = 0.9 * torch.rand(shape, generator=g, device=self.device)
        elif name.endswith("f.b"):
            t = 2.0 + rnd()
        elif leaf == "b":
            t = 0.05 * rnd()
        elif leaf == "act":
            t = torch.tensor([0.6, 0.3, 0.2, 0.05], device=self.device)
        elif leaf in ("ls1", "ls2"):
            t = 0.7 + 0.1 * rnd()
        else:
            t = 1.0 + 0.1 * rnd()
        t = t.to(torch.bfloat16)                 # what a checkpoint would hold
        return t.to(device=device or self.device, dtype=dtype or t.dtype)


def save_checkpoint(model_dir, config: dict, seed: int = 0, tensors: dict | None = None):
    """Write a model directory (config.json + model.safetensors) with random weights; ``tensors`` replaces some of them."""
    from ..loader.safetensors import write_safetensors
    d = Path(model_dir)
    d.mkdir(parents=True, exist_ok=True)
    (d / "config.json").write_text(json.dumps(config, indent=1))
    src = RandomSource(FofosunConfig.from_dict(config), seed)
    out = {n: src.tensor(n) for n in src.shapes}
    out.update({n: t.to(torch.bfloat16) for n, t in (tensors or {}).items()})
    write_safetensors(d / "model.safetensors", out)


def load_fofosun(hf: dict, src, device, comm=None, dtype="bf16", **_):
    return FofosunModel(FofosunConfig.from_dict(hf), device, comm, dtype).load(src)
