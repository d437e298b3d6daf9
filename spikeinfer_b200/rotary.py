"""Rotary position factors: configuration and table."""
from __future__ import annotations

from dataclasses import dataclass

import torch


@dataclass(frozen=True)
class RotaryConfig:
    dims: int
    base: float
    factor: float = 1.0
    """Linear scaling: every frequency is divided by it."""

    @classmethod
    def from_dict(cls, d: dict | None) -> "RotaryConfig | None":
        if not d or not d["dims"]:
            return None
        return cls(dims=d["dims"], base=float(d["base"]), factor=float((d.get("scaling") or {}).get("factor", 1.0)))

    def table(self, positions: int, device) -> torch.Tensor:
        """fp32 ``[positions, dims / 2, 2]`` of (cos, sin); the angles are evaluated in double precision."""
        i = torch.arange(self.dims // 2, dtype=torch.float64, device=device)
        freq = self.base ** (-2.0 * i / self.dims) / self.factor
        angle = torch.arange(positions, dtype=torch.float64, device=device)[:, None] * freq[None, :]
        return torch.stack((angle.cos(), angle.sin()), dim=-1).to(torch.float32).contiguous()
