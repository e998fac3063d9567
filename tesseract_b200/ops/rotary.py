"""Rotary positions. The pairs are halves of a range (coordinate i of the first ``dims`` turns with coordinate i + dims / 2) or,
with ``neighbours``, coordinates 2 i and 2 i + 1.

Kernels read a head stored as [u: hp | v: hp | rest], pair i = (u_i, v_i), with hp = dims / 2 rounded up to a multiple of 8
(a permutation with zero padding, the same for queries and keys, so no score sees it), and a table of (cos, sin) per
position and pair.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Optional

import torch


@dataclass(frozen=True)
class Yarn:
    """Frequencies between their own value and that over ``factor``, by how often a pair turns over ``original`` positions
    (more than ``fast`` turns: kept, fewer than ``slow``: divided), and a factor on cos and sin."""
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotary:
    dims: int
    base: float
    scaling: Optional[Yarn] = None
    neighbours: bool = False

    def __post_init__(self):
        if self.dims < 0 or self.dims % 2 or self.base <= 0:
            raise ValueError("rotary: dims is even, base positive")
        if self.scaling is not None and (self.dims == 0 or self.base == 1 or min(self.scaling.factor, self.scaling.original,
                                                                                 self.scaling.fast, self.scaling.slow) <= 0):
            raise ValueError("rotary: scaling needs rotated dims, a base other than 1 and positive constants")

    @property
    def half(self) -> int:
        return self.dims // 2

    @property
    def hp(self) -> int:
        return (self.half + 7) // 8 * 8

    def columns(self, dim: int) -> torch.Tensor:
        """Column of each of a head's ``dim`` coordinates in the stored layout."""
        if dim < self.dims:
            raise ValueError(f"rotary: {self.dims} rotated dims in a head of {dim}")
        i = torch.arange(dim)
        if self.neighbours:
            return torch.where(i < self.dims, i // 2 + i % 2 * self.hp, i - self.dims + 2 * self.hp)
        return torch.where(i < self.half, i, torch.where(i < self.dims, i - self.half + self.hp, i - self.dims + 2 * self.hp))

    def stored(self, dim: int, multiple: int = 8) -> int:
        """Columns of a head of ``dim`` coordinates in the stored layout."""
        n = 2 * self.hp + dim - self.dims
        return (n + multiple - 1) // multiple * multiple

    def frequencies(self):
        """(fp64 [half] angle per position, factor on cos and sin)."""
        i = torch.arange(self.half, dtype=torch.float64)
        f = torch.pow(torch.tensor(self.base, dtype=torch.float64), -2.0 * i / max(self.dims, 1))
        s = self.scaling
        if s is None:
            return f, 1.0

        def pair(turns):
            return self.dims * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.base))
        lo, hi = max(math.floor(pair(s.fast)), 0), min(math.ceil(pair(s.slow)), self.dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return f / s.factor * ramp + f * (1.0 - ramp), 0.1 * math.log(s.factor) + 1.0

    def table(self, positions: int, device=None) -> torch.Tensor:
        """fp32 [positions, hp, 2] of (cos, sin); computed in fp64, so a far position is as exact as a near one."""
        f, mult = self.frequencies()
        out = torch.zeros(positions, self.hp, 2, dtype=torch.float32, device=device)
        for p0 in range(0, positions, 65536):            # (bounds the fp64 intermediates)
            a = torch.arange(p0, min(p0 + 65536, positions), dtype=torch.float64)[:, None] * f
            out[p0:p0 + a.shape[0], :self.half] = (torch.stack((a.cos(), a.sin()), dim=-1) * mult).float().to(out.device)
        return out


def rotate_stored(x: torch.Tensor, table: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
    """x [T, ..., stored columns] (fp32) -> rotated, in the stored layout (the torch restatement of the kernels' loads)."""
    hp = table.shape[1]
    cs = table[positions.long()]
    shape = (x.shape[0],) + (1,) * (x.dim() - 2) + (hp,)
    c, s = cs[..., 0].reshape(shape), cs[..., 1].reshape(shape)
    u, v = x[..., :hp], x[..., hp:2 * hp]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * hp:]], dim=-1)
