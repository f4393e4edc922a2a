"""Rotary position encoding: inv_freq[j] = 1 / theta^(2j/dim) / scaling_factor, j < dim/2, in 32-bit
(jllm/model/common.py:51-55; the factor is linear scaling of positions).  With `bands` = (factor, low, high, original) a
frequency is scaled by its wavelength l = 2 pi / f instead: kept where l < original/high, divided by the factor where
l > original/low, and between the two (1 - s) f / factor + s f with s = (original/l - low) / (high - low).  With `yarn` =
(factor, original, fast, slow) (YaRN, Peng et al.) by the pair's number i: with d(t) = dim ln(original / (2 pi t)) / (2 ln theta),
lo = max(floor d(fast), 0), hi = min(ceil d(slow), dim - 1) and r = clamp((i - lo) / max(hi - lo, 0.001), 0, 1) the frequency
is f r / factor + f (1 - r), and `gain` = 0.1 ln(factor) + 1 multiplies the cosines and sines.  `layout` names the pairs that turn together:
"halves" (element i with i + dim/2) or "interleaved" (2i with 2i + 1); a mixer's preparation kernel must know it.  The part only owns the table; the rotation
itself is applied to queries and keys inside the mixer's preparation kernel (csrc/rope_kv.cu), which
forms the angle position * inv_freq[j] and its cos and sin in 32-bit."""

from __future__ import annotations

import math

import torch

from .base import Part
from .registry import register_position


class Rope(Part):
    def __init__(self, spec, prefix, ctx):
        if spec.dim % 2 or spec.dim < 2:
            raise ValueError(f"rotary dim must be even and positive, got {spec.dim}")
        self.dim, self.theta = int(spec.dim), float(spec.theta)
        self.layout = getattr(spec, "layout", "halves")
        self.factor = float(getattr(spec, "scaling_factor", 1.0))
        if self.layout not in ("halves", "interleaved") or not self.factor > 0:
            raise ValueError(f"rotation: layout {self.layout!r} or scaling factor {self.factor} is not built")
        self.bands = getattr(spec, "bands", None)
        if self.bands is not None:
            self.bands = tuple(float(v) for v in self.bands)
            factor, low, high, original = self.bands
            if not (factor > 0 and low > 0 and high >= low and original > 0):
                raise ValueError(f"rotation: bands {self.bands} (factor, low, high, original) do not fit")
        self.yarn = getattr(spec, "yarn", None)
        self.gain = 1.0
        if self.yarn is not None:
            self.yarn = tuple(float(v) for v in self.yarn)
            factor, original, fast, slow = self.yarn
            if self.bands is not None or not min(factor, original, fast, slow) > 0 or not self.theta > 1:
                raise ValueError(f"rotation: yarn {self.yarn} (factor, original, fast, slow) does not fit")
            self.gain = 0.1 * math.log(factor) + 1.0
        self.wide = torch.float64 if getattr(spec, "exact_table", False) else torch.float32
        self.inv_freq = (self.frequencies(self.dim, self.factor) if self.yarn is None else self._yarn_frequencies()).to(ctx.device)

    def _yarn_frequencies(self) -> torch.Tensor:
        factor, original, fast, slow = self.yarn
        d = lambda t: self.dim * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(self.theta))
        lo, hi = max(math.floor(d(fast)), 0), min(math.ceil(d(slow)), self.dim - 1)
        freq = self.theta ** (-torch.arange(0, self.dim, 2, dtype=torch.float64) / self.dim) / self.factor
        r = ((torch.arange(self.dim // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return (freq / factor * r + freq * (1.0 - r)).to(torch.float32)

    def frequencies(self, dim: int, factor: float = 1.0) -> torch.Tensor:
        """theta^(-2j/dim) / factor (scaled by bands, if there are any) for j < dim/2, as float32 on the CPU."""
        exponents = torch.arange(0, dim, 2, dtype=self.wide) / dim
        freq = 1.0 / (self.theta ** exponents) / factor
        if self.bands is not None:
            div, low, high, original = self.bands
            wavelength = 2.0 * math.pi / freq
            s = (original / wavelength - low) / (high - low)
            mixed = (1.0 - s) * freq / div + s * freq
            freq = torch.where(wavelength < original / high, freq, torch.where(wavelength > original / low, freq / div, mixed))
        return freq.to(torch.float32)

    def table(self):
        return self.inv_freq


register_position("rope", Rope)
