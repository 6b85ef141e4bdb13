"""Rotary position encoding (crates/cellm-kernels/src/cpu_kernels.rs:264-292):
pairs (i, i + rot/2) ("half") or (2i, 2i+1) ("interleaved") of the first
`rotary_dim` values of a head turn by pos * theta^(-2i/rotary_dim).

With `scaling` {factor, low, high, original} the frequencies are stretched by wavelength: a frequency f whose
wavelength l = 2 pi / f is shorter than original / high stays; one longer than original / low becomes f / factor;
between the two, with s = (original / l - low) / (high - low), it becomes (1 - s) f / factor + s f.

With `scaling` {factor, original, fast, slow} they are stretched by their place instead (YaRN): with
d(t) = rotary_dim ln(original / (2 pi t)) / (2 ln theta), lo = max(floor(d(fast)), 0), hi = min(ceil(d(slow)), rotary_dim - 1)
and r_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1), frequency i becomes f_i / factor * r_i + f_i (1 - r_i), and cos and sin
are both multiplied by 0.1 ln(factor) + 1 (`amplitude`)."""
from __future__ import annotations

import torch

from ..config.errors import ConfigError
from .base import Position
from .registry import register_position


def scale_by_wavelength(inv: torch.Tensor, scaling: dict) -> torch.Tensor:
    """64-bit frequencies stretched by wavelength (see the module's text)."""
    import math
    factor, low, high, original = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
    if factor <= 0 or high <= low or original <= 0:
        raise ConfigError(f"rope: scaling {scaling!r} needs factor > 0, high > low and original > 0")
    wavelength = 2.0 * math.pi / inv
    s = ((original / wavelength - low) / (high - low)).clamp(0.0, 1.0)
    mixed = (1.0 - s) * inv / factor + s * inv
    return torch.where(wavelength < original / high, inv, torch.where(wavelength > original / low, inv / factor, mixed))


def scale_by_place(inv: torch.Tensor, theta: float, rotary_dim: int, scaling: dict) -> torch.Tensor:
    """64-bit frequencies stretched by their place among them (see the module's text)."""
    import math
    factor, original, fast, slow = (float(scaling[k]) for k in ("factor", "original", "fast", "slow"))
    if min(factor, original, fast, slow) <= 0 or theta <= 0 or theta == 1.0:
        raise ConfigError(f"rope: scaling {scaling!r} needs positive numbers and a base other than 1")
    at = lambda t: rotary_dim * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(theta))
    lo, hi = max(math.floor(at(fast)), 0), min(math.ceil(at(slow)), rotary_dim - 1)
    ramp = ((torch.arange(inv.numel(), dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return inv / factor * ramp + inv * (1.0 - ramp)


def split_inv_freq(theta: float, rotary_dim: int, scaling: dict | None = None) -> torch.Tensor:
    """theta^(-2i/rotary_dim) for i < rotary_dim/2 (stretched by `scaling` if given), computed in 64-bit and given
    as [rotary_dim/2, 2] float32: the nearest float and the remainder, so that the
    kernel can form pos * inv_freq without losing the low bits."""
    i = torch.arange(rotary_dim // 2, dtype=torch.float64)
    inv = float(theta) ** (-(2.0 * i) / max(rotary_dim, 1))
    if scaling:
        inv = scale_by_place(inv, float(theta), rotary_dim, scaling) if "fast" in scaling else scale_by_wavelength(inv, scaling)
    hi = inv.to(torch.float32)
    lo = (inv - hi.to(torch.float64)).to(torch.float32)
    return torch.stack([hi, lo], dim=1).contiguous()


class RotaryEmbedding(Position):
    graph_safe = True

    """params: head_dim, rotary_dim, theta, layout ("half" | "interleaved"), scaling (None, {factor, low, high, original} or
    {factor, original, fast, slow}). `amplitude` multiplies cos and sin; rotation() leaves it to the caller, and a part that
    knows no amplitude must refuse one other than 1 (rotation(amplitude=False), the default, does)."""

    def __init__(self, params: dict, device):
        self.head_dim = int(params["head_dim"])
        self.rotary_dim = int(params.get("rotary_dim", self.head_dim))
        self.theta = float(params["theta"])
        self.layout = params.get("layout", "half")
        if self.layout not in ("half", "interleaved"):
            raise ConfigError(f"rope: layout {self.layout!r} is neither 'half' nor 'interleaved'")
        if self.rotary_dim % 2 or not 0 <= self.rotary_dim <= self.head_dim:
            raise ConfigError(f"rope: rotary_dim {self.rotary_dim} must be even and at most head_dim {self.head_dim}")
        self.scaling = params.get("scaling")
        self.amplitude = 1.0
        if self.scaling and "fast" in self.scaling:
            import math
            self.amplitude = 0.1 * math.log(float(self.scaling["factor"])) + 1.0
        self.inv_freq = split_inv_freq(self.theta, self.rotary_dim, self.scaling).to(device)

    def rotation(self, amplitude: bool = False):
        if not amplitude and self.amplitude != 1.0:
            raise ConfigError("rope: this part takes no amplitude on cos and sin")
        return self.rotary_dim, self.layout == "interleaved", self.inv_freq


register_position("rope", RotaryEmbedding)
