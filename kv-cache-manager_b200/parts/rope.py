"""Position encodings a mixer can be given.

``RotaryEmbedding``: angle(pos, j) = pos * inv_freq[j], inv_freq[j] = theta^(-2j / rotary_dim),
applied to pairs (j, j + rotary_dim/2) ("half", the reference's pairing,
``src/cuda/kernels.cu:51-70``) or (2j, 2j+1) ("interleaved") of the first ``rotary_dim``
elements of every q and k head.  The frequency table is float32, computed once on the host in
float64; a scaled variant only needs another table.  ``NoPositionEncoding`` leaves q and k as
they are.

``scaling`` (YaRN): {factor, original, fast, slow}.  With turns(t) = rotary_dim ln(original / (2 pi t)) / (2 ln theta), the
pair index at which a wave makes t turns over ``original`` positions, the frequencies between lo = max(floor(turns(fast)), 0)
and hi = min(ceil(turns(slow)), rotary_dim - 1) pass linearly from f_i to f_i / factor, and cosines and sines are multiplied
by ``amplitude`` = 0.1 ln(factor) + 1.
"""
from __future__ import annotations

import math
from typing import Optional

import torch

from ..kernels import library as K
from .base import POSITION_ENCODINGS, PositionEncoding


STEP_TABLE_ROWS = 256        # steps with that many rows of portions form their cosines and sines once for all layers


@POSITION_ENCODINGS.register("rope")
class RotaryEmbedding(PositionEncoding):
    def __init__(self, head_dim: int, theta: float, rotary_dim: Optional[int] = None,
                 pairing: str = "half", scaling: Optional[dict] = None) -> None:
        super().__init__()
        self.head_dim = head_dim
        self.theta = float(theta)
        self.rotary_dim = head_dim if rotary_dim is None else int(rotary_dim)
        if self.rotary_dim % 2 or not (0 < self.rotary_dim <= head_dim):
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and within head_dim {head_dim}")
        if pairing not in ("half", "interleaved"):
            raise ValueError(f"unknown rotary pairing '{pairing}'")
        self.interleaved = pairing == "interleaved"
        self.scaling = dict(scaling) if scaling else None
        self.amplitude = 0.1 * math.log(self.scaling["factor"]) + 1.0 if self.scaling else 1.0
        self.inv_freq: Optional[torch.Tensor] = None

    def frequency_table(self) -> torch.Tensor:
        j = torch.arange(self.rotary_dim // 2, dtype=torch.float64)
        f = 1.0 / torch.pow(torch.tensor(self.theta, dtype=torch.float64), 2.0 * j / self.rotary_dim)
        if self.scaling:
            def turns(t: float) -> float:
                return self.rotary_dim * math.log(self.scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(self.theta))
            lo = max(math.floor(turns(self.scaling["fast"])), 0)
            hi = min(math.ceil(turns(self.scaling["slow"])), self.rotary_dim - 1)
            ramp = ((j - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
            f = f / self.scaling["factor"] * ramp + f * (1.0 - ramp)
        return f.to(torch.float32)

    def prepare(self, device, dtype) -> None:
        self.inv_freq = self.frequency_table().to(device)

    def step_table(self, ctx) -> torch.Tensor:
        """The step's cosines and sines (float32 [rows, rotary_dim], without the amplitude), formed once per step for all layers
        with these frequencies."""
        key = ("rope_table", self.theta, self.rotary_dim, repr(self.scaling))
        table = ctx.shared.get(key)
        if table is None:
            table = ctx.shared[key] = torch.empty((ctx.rows, self.rotary_dim), dtype=torch.float32, device=self.inv_freq.device)
            K.rope_table(ctx.positions, self.inv_freq, table)
        return table


@POSITION_ENCODINGS.register("none")
class NoPositionEncoding(PositionEncoding):
    def __init__(self, head_dim: int = 0, **_) -> None:
        super().__init__()
        self.rotary_dim = 0
        self.interleaved = False
        self.amplitude = 1.0
        self.inv_freq = None
