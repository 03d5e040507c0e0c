"""Rotary positions with their constants as parameters: which columns form a pair, and frequencies that are scaled for contexts
longer than the trained one (YaRN: B. Peng, J. Quesnelle, H. Fan, E. Shippole, "YaRN: Efficient Context Window Extension of Large
Language Models"). The kernels read half turns per position in double, reduce them to one turn and take sine and cosine in fp32, so
angles are exact at any position.
"""
from __future__ import annotations

import math
from dataclasses import dataclass

import torch

MAX_PAIRS = 256                 # of the kernels' angle tables


@dataclass
class Rotation:
    """Turns the first ``dims`` columns of a vector; column 2i pairs with 2i + 1 (``neighbours``) or i with i + dims / 2.
    ``scaling``: {"factor", "original", "fast", "slow"} or None: pairs that turn fewer than ``slow`` times over ``original`` positions are
    slowed by ``factor``, those above ``fast`` turns are kept, the ones in between are blended; sine and cosine are multiplied by
    ``mul`` = 0.1 ln(factor) + 1."""
    dims: int
    base: float
    neighbours: bool = True
    scaling: dict | None = None

    def __post_init__(self):
        if self.dims % 2 or self.dims < 0:
            raise ValueError("the rotated width is a number of pairs")
        if self.dims > 2 * MAX_PAIRS:
            raise NotImplementedError(f"{self.dims} rotated columns (at most {2 * MAX_PAIRS})")
        i = torch.arange(self.dims // 2, dtype=torch.float64)
        self.freq = torch.pow(torch.tensor(self.base, dtype=torch.float64), -2.0 * i / max(1, self.dims))
        self.mul = 1.0
        if self.scaling:
            factor, original = float(self.scaling["factor"]), float(self.scaling["original"])

            def pair(turns):
                return self.dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
            lo, hi = max(math.floor(pair(float(self.scaling["fast"]))), 0), min(math.ceil(pair(float(self.scaling["slow"]))), self.dims - 1)
            slowed = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
            self.freq = self.freq * (slowed / factor + 1.0 - slowed)
            self.mul = 0.1 * math.log(factor) + 1.0
        self.half_turns = self.freq / torch.pi

    @classmethod
    def from_config(cls, rot: dict, neighbours: bool) -> "Rotation":
        return cls(int(rot["dims"]), float(rot["base"]), neighbours, rot.get("scaling"))

    def bind(self, device) -> "Rotation":
        self.half_turns = self.half_turns.to(device)
        return self

    @property
    def pairs(self) -> int:
        return self.dims // 2

    def turn(self, v, pos):
        """CPU statement: v [rows, ..., width] (fp32) of the rows' positions, turned."""
        ang = (pos.double()[:, None] * self.freq).reshape(len(pos), *[1] * (v.dim() - 2), self.pairs)
        c, s = (ang.cos() * self.mul).float(), (ang.sin() * self.mul).float()
        out = v.float().clone()
        if self.neighbours:
            x, y = slice(0, self.dims, 2), slice(1, self.dims, 2)
        else:
            x, y = slice(0, self.pairs), slice(self.pairs, self.dims)
        a, b = v[..., x].float(), v[..., y].float()
        out[..., x], out[..., y] = a * c - b * s, b * c + a * s
        return out
