"""Rotary position encodings.

The reference receives a ready ``inv_freq`` table computed in Python by another
package's rope functions and drops the attention factor they return
(cpmcu/llm.py:181-192); its kernel rotates half-split pairs by position * inv_freq
(src/model/rotary.cuh:6-34).  Here the table and the factor are computed from the
configuration's own keys:

    inv_freq[c] = 1 / (factor[c] * theta^(2c/d))
    factor      = long_factor if max_positions > original_max_positions else short_factor
    magnitude   = sqrt(1 + ln(max_positions/original_max_positions) / ln(original_max_positions))
                  if max_positions > original_max_positions else 1

The factor set is chosen once per model, never per call, so cached keys stay valid
however the tokens are cut into steps.  cos and sin are multiplied by the magnitude.
"""
from __future__ import annotations

import math
from typing import Optional, Sequence, Tuple

import torch

from .base import POSITIONS, PositionEncoding


@POSITIONS.register("none")
class NoPosition(PositionEncoding):
    """No position information: queries and keys pass unchanged."""

    recordable_prompt = True

    def __init__(self, ops):
        super().__init__(ops)

    def rotary(self):
        return (None, 1.0, 0)


@POSITIONS.register("rope")
class Rotary(PositionEncoding):
    recordable_prompt = True
    adjacent = False            # which channels form a pair: (i, i + rot_dim/2), or with ``adjacent`` (2i, 2i + 1)

    def __init__(self, ops, head_dim: int, theta: float, rot_dim: Optional[int] = None):
        super().__init__(ops)
        self.rot_dim = int(rot_dim if rot_dim is not None else head_dim)
        if self.rot_dim % 2 or self.rot_dim > head_dim:
            raise ValueError(f"rotary dimension {self.rot_dim} must be even and at most head_dim {head_dim}")
        self.magnitude = 1.0
        self.inv_freq = self._table(theta, [1.0] * (self.rot_dim // 2))

    def _table(self, theta: float, factors: Sequence[float]) -> torch.Tensor:
        # fp32 arithmetic on the host, in the order the formula is written
        exponent = torch.arange(0, self.rot_dim, 2, dtype=torch.int64).to(torch.float32) / self.rot_dim
        f = torch.tensor([float(x) for x in factors], dtype=torch.float32)
        inv_freq = 1.0 / (f * (float(theta) ** exponent))
        return inv_freq.to(torch.float32).to(self.ops.device if self.ops is not None else "cpu")

    def rotary(self) -> Tuple[torch.Tensor, float, int]:
        return (self.inv_freq, self.magnitude, self.rot_dim)


@POSITIONS.register("scaled_rope")
class LinearlyScaledRotary(Rotary):
    """A rotation of the first ``rot_dim`` channels of a head whose frequencies are all divided by one ``factor``
    (positions stretched by it): inv_freq[i] = theta^(-2i/rot_dim) / factor.  The table is formed in 64-bit on the
    host and rounded once to 32-bit; angles are 32-bit on the device."""

    def __init__(self, ops, head_dim: int, theta: float, rot_dim: Optional[int] = None, factor: float = 1.0):
        super().__init__(ops, head_dim, theta, rot_dim)
        if not factor > 0:
            raise ValueError(f"scaled_rope: the scaling factor must be positive, got {factor}")
        self.factor = float(factor)
        i = torch.arange(self.rot_dim // 2, dtype=torch.float64)
        table = torch.pow(torch.tensor(float(theta), dtype=torch.float64), -2.0 * i / max(self.rot_dim, 1)) / self.factor
        self.inv_freq = table.to(torch.float32).to(self.ops.device if self.ops is not None else "cpu")


@POSITIONS.register("wavelength_scaled_rope")
class WavelengthScaledRotary(Rotary):
    """A rotation of the first ``rot_dim`` channels of a head in adjacent pairs (2i, 2i + 1) (``adjacent`` False: pairs
    (i, i + rot_dim/2)), f_i = theta^(-2i/rot_dim), with the frequencies stretched by wavelength when ``factor`` is given:
    with l = 2 pi / f, a wave shorter than original / high keeps f, one longer than original / low gets f / factor, and
    between the two f becomes (1 - s) f / factor + s f with s = (original / l - low) / (high - low).  The table is formed
    in 64-bit on the host and rounded once to 32-bit; angles are 32-bit on the device."""

    def __init__(self, ops, head_dim: int, theta: float, rot_dim: Optional[int] = None, factor: Optional[float] = None,
                 low: float = 1.0, high: float = 4.0, original: int = 8192, adjacent: bool = True):
        super().__init__(ops, head_dim, theta, rot_dim)
        self.adjacent = bool(adjacent)
        i = torch.arange(self.rot_dim // 2, dtype=torch.float64)
        f = torch.pow(torch.tensor(float(theta), dtype=torch.float64), -2.0 * i / max(self.rot_dim, 1))
        if factor is not None:
            factor, low, high, original = float(factor), float(low), float(high), float(original)
            if not (factor > 0 and high > low and original > 0):
                raise ValueError("wavelength_scaled_rope: needs factor > 0, high > low and original > 0")
            wave = 2.0 * math.pi / f
            blend = (original / wave - low) / (high - low)
            mid = (1.0 - blend) * f / factor + blend * f
            f = torch.where(wave < original / high, f, torch.where(wave > original / low, f / factor, mid))
        self.inv_freq = f.to(torch.float32).to(self.ops.device if self.ops is not None else "cpu")


@POSITIONS.register("yarn_rope")
class YarnRotary(Rotary):
    """A rotation of the first ``rot_dim`` channels of a head in pairs (i, i + rot_dim/2), f_i = theta^(-2i/rot_dim), with
    the slow frequencies stretched when ``factor`` is given: with place(t) = rot_dim ln(original / (2 pi t)) / (2 ln theta),
    the (fractional) i whose wave makes t turns over ``original`` positions, the ramp

        r_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1),    lo = max(floor(place(fast)), 0),  hi = min(ceil(place(slow)), rot_dim - 1)

    blends f_i / factor (r = 1) with f_i (r = 0), and cosine and sine are multiplied by 0.1 ln(factor) + 1.  The table is
    formed in 64-bit on the host and rounded once to 32-bit; angles are 32-bit on the device."""

    def __init__(self, ops, head_dim: int, theta: float, rot_dim: Optional[int] = None, factor: Optional[float] = None,
                 original: int = 8192, fast: float = 32.0, slow: float = 1.0):
        super().__init__(ops, head_dim, theta, rot_dim)
        theta = float(theta)
        i = torch.arange(self.rot_dim // 2, dtype=torch.float64)
        f = torch.pow(torch.tensor(theta, dtype=torch.float64), -2.0 * i / max(self.rot_dim, 1))
        if factor is not None:
            factor, original, fast, slow = float(factor), float(original), float(fast), float(slow)
            if not (factor > 0 and original > 0 and fast > 0 and slow > 0 and theta > 0 and theta != 1.0):
                raise ValueError("yarn_rope: needs positive factor, original, fast and slow, and a base other than 1")
            place = lambda turns: self.rot_dim * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
            lo = max(math.floor(place(fast)), 0)
            hi = min(math.ceil(place(slow)), self.rot_dim - 1)
            ramp = torch.clamp((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
            f = f / factor * ramp + f * (1.0 - ramp)
            self.magnitude = 0.1 * math.log(factor) + 1.0
        self.inv_freq = f.to(torch.float32).to(self.ops.device if self.ops is not None else "cpu")


@POSITIONS.register("longrope")
class LongRotary(Rotary):
    def __init__(self, ops, head_dim: int, theta: float, long_factor: Sequence[float],
                 short_factor: Sequence[float], original_max_positions: int, max_positions: int):
        super().__init__(ops, head_dim, theta)
        extended = max_positions > original_max_positions
        factors = long_factor if extended else short_factor
        if len(factors) != self.rot_dim // 2:
            raise ValueError(f"longrope needs {self.rot_dim // 2} factors, got {len(factors)}")
        self.inv_freq = self._table(theta, factors)
        if extended:
            self.magnitude = math.sqrt(1.0 + math.log(max_positions / original_max_positions)
                                       / math.log(original_max_positions))
