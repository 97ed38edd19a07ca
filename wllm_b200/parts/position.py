"""Rotary position encoding: the table of inverse frequencies.

spec options: theta, head_dim, rotary_dim (defaults to head_dim; 0: nothing turns), exact_table (the table worked
out in 64-bit and rounded once), frequency_divisor (every frequency is divided by it: positions stretched by that
factor; absent: as they are), scaling (absent: none; {"factor": F, "original": L, "fast": a, "slow": b}: a long context
reached from one of L positions, band by band.  Pair j makes L f_j / (2 pi) turns over the original context; t(n) =
rotary_dim ln(L / (2 pi n)) / (2 ln theta) is the pair index that makes n turns.  Pairs up to floor(t(a)) keep their
frequency, pairs from ceil(t(b)) have it divided by F, those between are blended linearly, and sines and cosines are
multiplied by 1 + ln(F) / 10, which the part hands on as `turn_scale`), pairing ('half', the default: element j
turns with j + rotary_dim/2, src/wllm/models/llama.py:47-49; 'interleaved': 2j with 2j + 1).  The table is
inv_freq[j] = theta^(-2j / rotary_dim) in 32-bit (src/wllm/models/llama.py:55) and
never leaves 32-bit; angles are position * inv_freq, computed in the kernel from the
token's absolute position, so no table length limits the context.  Pairs are
(j, j + rotary_dim/2) (src/wllm/models/llama.py:47-49).
"""
from __future__ import annotations

import math

import torch

from .base import POSITIONS


@POSITIONS.register("rope")
class RotaryPosition:
    def __init__(self, spec, device=None):
        self.head_dim = int(spec.head_dim)
        self.rotary_dim = int(spec.options.get("rotary_dim", self.head_dim))
        self.theta = float(spec.theta)
        self.pairing = spec.options.get("pairing", "half")
        if self.pairing not in ("half", "interleaved"):
            raise ValueError(f"rotary pairing {self.pairing!r}: 'half' or 'interleaved'")
        if self.rotary_dim % 2 or self.rotary_dim > self.head_dim or self.rotary_dim < 0:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {self.head_dim}")
        if spec.options.get("exact_table", False):
            # every frequency is the 32-bit number nearest to theta^(-2j / rotary_dim): worked out in 64-bit, rounded once
            exponent = torch.arange(0, self.rotary_dim, 2, dtype=torch.float64) / max(1, self.rotary_dim)
            self.inv_freq = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -exponent).to(torch.float32)
        else:
            exponent = torch.arange(0, self.rotary_dim, 2, dtype=torch.float32) / max(1, self.rotary_dim)
            self.inv_freq = (1.0 / (self.theta ** exponent)).to(torch.float32)
        divisor = spec.options.get("frequency_divisor")
        if divisor is not None:
            if not float(divisor) > 0:
                raise ValueError(f"frequency_divisor {divisor!r} must be positive")
            # theta^(-2j / rotary_dim) / divisor in 64-bit, rounded once
            exponent = torch.arange(0, self.rotary_dim, 2, dtype=torch.float64) / max(1, self.rotary_dim)
            exact = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -exponent) / float(divisor)
            self.inv_freq = exact.to(torch.float32) if spec.options.get("exact_table", False) else self.inv_freq / float(divisor)
        self.turn_scale = 1.0            # factor on the sines and cosines
        scaling = spec.options.get("scaling")
        if scaling is not None and self.rotary_dim > 0:
            if divisor is not None:
                raise ValueError("frequencies are either divided by one number or scaled band by band, not both")
            self._scale_bands(**{k: float(scaling[k]) for k in ("factor", "original", "fast", "slow")})
        if device is not None:
            self.inv_freq = self.inv_freq.to(device)

    def _scale_bands(self, factor: float, original: float, fast: float, slow: float) -> None:
        """Worked out in 64-bit, rounded once."""
        if not (factor > 0 and original > 0 and fast > 0 and slow > 0 and self.theta > 0 and self.theta != 1.0):
            raise ValueError(f"scaling factor {factor}, original {original}, fast {fast}, slow {slow}, theta {self.theta}: all must be "
                             f"positive, theta not 1")
        dims = self.rotary_dim

        def pair_of(turns: float) -> float:
            return dims * math.log(original / (2 * math.pi * turns)) / (2 * math.log(self.theta))
        first, last = max(math.floor(pair_of(fast)), 0), min(math.ceil(pair_of(slow)), dims - 1)
        j = torch.arange(dims // 2, dtype=torch.float64)
        ramp = ((j - first) / max(last - first, 0.001)).clamp(0.0, 1.0)
        plain = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -2.0 * j / dims)
        self.inv_freq = (plain / factor * ramp + plain * (1.0 - ramp)).to(torch.float32)
        self.turn_scale = 0.1 * math.log(factor) + 1.0

    def to(self, device):
        self.inv_freq = self.inv_freq.to(device)
        return self
