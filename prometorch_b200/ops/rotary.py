"""Interleaved rotary positions: neighbours (2i, 2i + 1) of the first ``dims`` entries of a head turn by pos * base^(-2i / dims).

:class:`Rotary` holds the cosines and sines of every position (angles in fp64, stored in fp32); the kernels that write q and the
pages apply them (csrc/rotary_write.cu)."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch


@dataclass
class Rotary:
    dims: int
    base: float
    positions: int
    device: object = "cpu"
    cos: Optional[torch.Tensor] = field(default=None, repr=False)      # [positions, dims / 2] fp32
    sin: Optional[torch.Tensor] = field(default=None, repr=False)

    def __post_init__(self):
        if self.cos is None:
            i = torch.arange(self.dims // 2, dtype=torch.float64, device=self.device)
            freq = torch.pow(torch.tensor(self.base, dtype=torch.float64, device=self.device), -2.0 * i / max(self.dims, 1))
            a = torch.arange(self.positions, dtype=torch.float64, device=self.device)[:, None] * freq
            self.cos, self.sin = a.cos().float().contiguous(), a.sin().float().contiguous()

    def apply(self, x: torch.Tensor, pos: torch.Tensor) -> torch.Tensor:
        """``x [n, heads, size]`` fp32 at the positions ``pos [n]`` (plain math)."""
        if not self.dims:
            return x
        c, s = self.cos[pos.long()][:, None, :], self.sin[pos.long()][:, None, :]
        u, v = x[..., 0:self.dims:2], x[..., 1:self.dims:2]
        y = x.clone()
        y[..., 0:self.dims:2], y[..., 1:self.dims:2] = u * c - v * s, v * c + u * s
        return y
