"""Position encodings. A position encoding hands its mixer a table of angles' cosines and sines per position;
the mixer's fused kernel rotates q and k with it.

Rope: inv_freq_i = θ^(−2i/rotary_dim), angle = position · inv_freq in 32-bit, half-split pairs (i, i + rotary_dim/2);
dimensions past `rotary_dim` pass through (std/holon_std/ops/units.py:38-63; std/holon_std/ops/reference.py:21-30).
With `interleaved` the pairs are neighbours (2i, 2i + 1) instead; the table is the same, and a mixer whose kernel knows
both layouts passes the flag on. With `factor` f every frequency is divided by f (positions stretched f-fold: linear scaling).
With `yarn` = (factor, original, fast, slow) only the slow pairs are stretched: with dim(t) = rotary_dim · ln(original / (2π t))
/ (2 ln θ), the number of the pair that turns t times over `original` positions, lo = max(⌊dim(fast)⌋, 0) and hi =
min(⌈dim(slow)⌉, rotary_dim − 1), pair i keeps its frequency up to lo, has it divided by `factor` from hi on, and between them
takes a mixture, linear in i; cosines and sines are all multiplied by 0.1 ln(factor) + 1 (Peng et al., YaRN: Efficient Context
Window Extension of Large Language Models).
"""
from __future__ import annotations

import math

import torch

from .base import BuildContext, Part


class Rope(Part):
    def __init__(self, ctx: BuildContext, *, theta: float, rotary_dim: int, head_dim: int, interleaved: bool = False,
                 factor: float = 1.0, yarn: tuple[float, float, float, float] | None = None) -> None:
        super().__init__()
        if rotary_dim % 2 or not 0 <= rotary_dim <= head_dim:
            raise ValueError(f"rope: rotary_dim {rotary_dim} must be even and at most head_dim {head_dim}")
        if not factor > 0:
            raise ValueError(f"rope: factor {factor} must be positive")
        if yarn is not None and (factor != 1.0 or not (yarn[0] > 0 and yarn[1] > 0 and yarn[2] > 0 and yarn[3] > 0 and theta > 1)):
            raise ValueError(f"rope: yarn {yarn} needs positive numbers, a base above 1 and no linear factor beside it")
        self.yarn = tuple(float(v) for v in yarn) if yarn is not None else None
        self.theta, self.rotary_dim, self.interleaved, self.factor = float(theta), rotary_dim, bool(interleaved), float(factor)
        self.table = self.angles(ctx.max_positions).to(ctx.device)

    def angles(self, positions: int) -> torch.Tensor:
        """[positions, rotary_dim] 32-bit: cosines of the rotary_dim/2 angles, then their sines."""
        rd = self.rotary_dim
        inv_freq = 1.0 / (self.theta ** (torch.arange(0, rd, 2, dtype=torch.float32) / rd))
        if self.factor != 1.0:
            inv_freq = inv_freq / self.factor
        size = 1.0
        if self.yarn is not None and rd:
            factor, original, fast, slow = self.yarn
            turns = lambda t: rd * math.log(original / (2 * math.pi * t)) / (2 * math.log(self.theta))      # noqa: E731
            lo, hi = max(math.floor(turns(fast)), 0), min(math.ceil(turns(slow)), rd - 1)
            i = torch.arange(rd // 2, dtype=torch.float64)
            ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
            freq = self.theta ** (-2.0 * i / rd)
            inv_freq = (freq / factor * ramp + freq * (1.0 - ramp)).to(torch.float32)
            size = 0.1 * math.log(factor) + 1.0
        angle = torch.arange(positions, dtype=torch.float32)[:, None] * inv_freq[None, :]
        return (torch.cat((angle.cos(), angle.sin()), dim=-1) * size).contiguous()
