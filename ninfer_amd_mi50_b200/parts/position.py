"""Rotary position embedding, half-split pairing.

For ``i < D/2``: ``angle = float(pos) * inv_freq[i]``, ``inv_freq[i] = theta^(-2i/D)``
evaluated in single precision on the host (src/models/model.hip:636-639);
``x'[i] = x[i] cos - x[i + D/2] sin``, ``x'[i + D/2] = x[i] sin + x[i + D/2] cos``
(src/ops/kernels.hip:73-94).  Applied to every query and key head, never to values.
The rotation itself runs inside the fused rotate-and-append kernel; this part owns the
table and the parameters.
"""

from __future__ import annotations

from typing import Optional, Tuple

import numpy as np
import torch

from ..registry import register_part
from .base import PositionEncoding


def rotary_inverse_frequencies(head_dim: int, theta: float, rotary_dim: Optional[int] = None
                               ) -> torch.Tensor:
    """float32 [rotary_dim / 2]: powf(theta, -2 i / D) with float operands."""
    rot = head_dim if rotary_dim is None else rotary_dim
    i = np.arange(rot // 2, dtype=np.float32)
    expo = (np.float32(-2.0) * i / np.float32(rot)).astype(np.float32)
    inv = np.power(np.float64(np.float32(theta)), expo.astype(np.float64)).astype(np.float32)
    return torch.from_numpy(inv)


def double_inverse_frequencies(rotary_dim: int, theta: float) -> torch.Tensor:
    """float32 [rotary_dim / 2]: theta^(-2i / rot), evaluated in double precision and rounded once."""
    i = np.arange(int(rotary_dim) // 2, dtype=np.float64)
    return torch.from_numpy(np.power(float(theta), -2.0 * i / int(rotary_dim)).astype(np.float32))


def banded_inverse_frequencies(rotary_dim: int, theta: float, factor: float, low: float, high: float,
                               original: float) -> torch.Tensor:
    """float32 [rotary_dim / 2]: the plain frequencies f_i = theta^(-2i / rot) by bands of their wavelength
    l = 2 pi / f (the Llama 3.1 rule): kept where l < original / high, divided by `factor` where
    l > original / low, and between the two blended, (1 - s) f / factor + s f with
    s = (original / l - low) / (high - low).  Evaluated in double precision, rounded once."""
    import math
    out = []
    for i in range(int(rotary_dim) // 2):
        f = float(theta) ** (-2.0 * i / int(rotary_dim))
        wave = 2.0 * math.pi / f
        if wave > original / low:
            f = f / factor
        elif wave >= original / high:
            s = (original / wave - low) / (high - low) if high != low else 1.0
            f = (1.0 - s) * f / factor + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64).to(torch.float32)


@register_part("position", "rotary_half_split")
class RotaryHalfSplit(PositionEncoding):
    def __init__(self, head_dim: int, theta: float, rotary_dim: Optional[int] = None, double: bool = False):
        """`double`: the frequencies are evaluated in double precision and rounded once."""
        self.head_dim, self.theta, self.double = int(head_dim), float(theta), bool(double)
        self.rotary_dim = int(head_dim if rotary_dim is None else rotary_dim)
        if self.rotary_dim % 2 or not 0 < self.rotary_dim <= self.head_dim:
            raise ValueError(f"rotary_dim={self.rotary_dim} must be even and in (0, {head_dim}]")
        self._table = {}

    def rotary_table(self, device: torch.device) -> Optional[Tuple[torch.Tensor, int]]:
        key = str(device)
        if key not in self._table:
            table = (double_inverse_frequencies(self.rotary_dim, self.theta) if self.double
                     else rotary_inverse_frequencies(self.head_dim, self.theta, self.rotary_dim))
            self._table[key] = table.to(device)
        return self._table[key], self.rotary_dim


def blended_inverse_frequencies(rotary_dim: int, theta: float, factor: float, original: float, fast: float,
                                slow: float) -> torch.Tensor:
    """float32 [rotary_dim / 2]: the plain frequencies f_i = theta^(-2i / rot) blended with the stretched
    ones f_i / factor by a ramp over the pair index.  With dim(t) = rot ln(original / (2 pi t)) / (2 ln theta)
    - the index whose wave turns t times over `original` positions - lo = max(floor(dim(fast)), 0),
    hi = min(ceil(dim(slow)), rot - 1) and ramp_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1):
    ``f_i / factor * ramp_i + f_i * (1 - ramp_i)``.  Evaluated in double precision, rounded once."""
    import math
    rot = int(rotary_dim)
    i = np.arange(rot // 2, dtype=np.float64)
    f = np.power(float(theta), -2.0 * i / rot)

    def dim_of(turns: float) -> float:
        return rot * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))

    lo = max(math.floor(dim_of(fast)), 0)
    hi = min(math.ceil(dim_of(slow)), rot - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return torch.from_numpy((f / factor * ramp + f * (1.0 - ramp)).astype(np.float32))


@register_part("position", "rotary_half_split_blended")
class RotaryHalfSplitBlended(RotaryHalfSplit):
    """The half-split rotation with frequencies stretched for contexts longer than the `original` one
    (the YaRN scheme): fast waves keep their frequency, slow ones are divided by `factor`, those between
    are blended (`blended_inverse_frequencies`), and cosine and sine are both multiplied by
    ``0.1 ln(factor) + 1`` (`magnitude`)."""

    def __init__(self, head_dim: int, theta: float, factor: float, original: float, fast: float, slow: float,
                 rotary_dim: Optional[int] = None):
        super().__init__(head_dim, theta, rotary_dim)
        self.factor, self.original, self.fast, self.slow = float(factor), float(original), float(fast), float(slow)
        if not (self.factor >= 1.0 and self.original > 0 and self.fast > 0 and self.slow > 0 and self.theta > 1.0):
            raise ValueError("stretched rotation: factor >= 1, original, fast and slow positive, base above 1")
        import math
        self.magnitude = 0.1 * math.log(self.factor) + 1.0

    def rotary_table(self, device: torch.device) -> Optional[Tuple[torch.Tensor, int]]:
        key = str(device)
        if key not in self._table:
            self._table[key] = blended_inverse_frequencies(self.rotary_dim, self.theta, self.factor, self.original,
                                                           self.fast, self.slow).to(device)
        return self._table[key], self.rotary_dim


@register_part("position", "rotary_half_split_banded")
class RotaryHalfSplitBanded(RotaryHalfSplit):
    """The half-split rotation with frequencies scaled by bands of their wavelength
    (`banded_inverse_frequencies`); cosine and sine are not scaled."""

    def __init__(self, head_dim: int, theta: float, factor: float, low: float, high: float, original: float,
                 rotary_dim: Optional[int] = None):
        super().__init__(head_dim, theta, rotary_dim)
        self.factor, self.low, self.high, self.original = float(factor), float(low), float(high), float(original)
        if not (self.factor > 0 and self.low > 0 and self.high >= self.low and self.original > 0 and self.theta > 0):
            raise ValueError("banded rotation: factor, original and base positive, 0 < low <= high")

    def rotary_table(self, device: torch.device) -> Optional[Tuple[torch.Tensor, int]]:
        key = str(device)
        if key not in self._table:
            self._table[key] = banded_inverse_frequencies(self.rotary_dim, self.theta, self.factor, self.low, self.high,
                                                          self.original).to(device)
        return self._table[key], self.rotary_dim


@register_part("position", "rotary_interleaved")
class RotaryInterleaved(PositionEncoding):
    """The rotation whose pairs are neighbours: dimension 2i with 2i + 1, by pos * theta^(-2i / rot).  For
    kernels that take a layout of pairs (`pair_table`); `rotary_table` promises half-split pairs and gives None."""

    def __init__(self, head_dim: int, theta: float, rotary_dim: Optional[int] = None):
        self.head_dim, self.theta = int(head_dim), float(theta)
        self.rotary_dim = int(head_dim if rotary_dim is None else rotary_dim)
        if self.rotary_dim % 2 or not 0 < self.rotary_dim <= self.head_dim:
            raise ValueError(f"rotary_dim={self.rotary_dim} must be even and in (0, {head_dim}]")
        self._table = {}

    def pair_table(self, device: torch.device) -> Optional[Tuple[torch.Tensor, int, bool]]:
        key = str(device)
        if key not in self._table:
            self._table[key] = double_inverse_frequencies(self.rotary_dim, self.theta).to(device)
        return self._table[key], self.rotary_dim, True


@register_part("position", "none")
class NoPosition(PositionEncoding):
    """No position information enters queries or keys."""

    def __init__(self, head_dim: int = 0):
        self.head_dim = head_dim

    def apply(self, q, k, positions) -> None:
        return None
