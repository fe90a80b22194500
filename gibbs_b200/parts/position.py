"""Position encodings.  Rotary encodings hand their table to the mixer, whose
kernel applies it to q and k together with the per-head norm."""
from __future__ import annotations

import math

import numpy as np
import torch

from .base import PositionEncoding, Rotary, register_part


def _inv_freq_f32(rotary_dim: int, theta: float) -> np.ndarray:
    """inv_freq[j] = 1 / theta^(2j / rotary_dim), every step in 32-bit
    (MisterTK/gibbs src/arch/gen.rs:137-164, precision 'f32';
    arch/families/lfm2.json5:63-65)."""
    j = np.arange(rotary_dim // 2, dtype=np.float32)
    expo = (np.float32(2.0) * j) / np.float32(rotary_dim)
    return (np.float32(1.0) / np.power(np.float32(theta), expo, dtype=np.float32)).astype(np.float32)


def stretched_inv_freq(rotary_dim: int, base: float, scaling=None) -> np.ndarray:
    """f_i = base^(-2i / rotary_dim) in 64-bit, rounded once to 32-bit.  ``scaling`` = {factor, low, high,
    original} stretches long wavelengths (the rule Llama 3.1 introduced): with l = 2 pi / f, f stays where
    l < original / high, becomes f / factor where l > original / low, and in between is
    (1 - s) f / factor + s f with s = (original / l - low) / (high - low)."""
    i = np.arange(rotary_dim // 2, dtype=np.float64)
    f = np.power(float(base), -2.0 * i / max(rotary_dim, 1))
    if scaling:
        factor, low, high, orig = (float(scaling[k]) for k in ("factor", "low", "high", "original"))
        wl = 2.0 * np.pi / f
        s = (orig / wl - low) / (high - low) if high != low else np.ones_like(f)
        mid = (1.0 - s) * f / factor + s * f
        f = np.where(wl < orig / high, f, np.where(wl > orig / low, f / factor, mid))
    return f.astype(np.float32)


def yarn_inv_freq(rotary_dim: int, base: float, factor: float, original: float, fast: float, slow: float):
    """(frequencies, factor on cosines and sines) of a context stretched by ``factor`` the way YaRN (Peng et al.) does it:
    pairs that turn more than ``fast`` times within ``original`` positions keep f_i = base^(-2i / rotary_dim), those that turn
    less than ``slow`` times get f_i / factor, with a linear ramp over the pair's index in between.  64-bit, rounded once."""
    i = np.arange(rotary_dim // 2, dtype=np.float64)
    f = np.power(float(base), -2.0 * i / max(rotary_dim, 1))

    def index_of(turns: float) -> float:          # the index whose pair turns this many times
        return rotary_dim * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(index_of(fast)), 0), min(math.ceil(index_of(slow)), rotary_dim - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return (f / factor * ramp + f * (1.0 - ramp)).astype(np.float32), 0.1 * math.log(factor) + 1.0


class RotaryHalfSplit(PositionEncoding):
    """Rotates the pairs (j, j + rotary_dim/2) by pos * inv_freq[j]
    (MisterTK/gibbs src/graph/cpu.rs:688-697)."""
    adjacent = False

    def __init__(self, params, tensors, rt):
        super().__init__(params, tensors, rt)
        self.head_dim = int(params["head_dim"])
        self.rotary_dim = int(params.get("rotary_dim", self.head_dim))
        if self.rotary_dim % 2 or not 0 < self.rotary_dim <= self.head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and at most head_dim {self.head_dim}")
        self.inv_freq = torch.from_numpy(_inv_freq_f32(self.rotary_dim, float(params["theta"]))).to(rt.device)
        # the factor on cosines and sines (MisterTK/gibbs src/graph/cpu.rs:674-675); 1 unless given
        self._rotary = Rotary(self.inv_freq, self.rotary_dim, self.adjacent, float(params.get("mscale", 1.0)))

    def rotary(self):
        return self._rotary


class RotaryAdjacent(RotaryHalfSplit):
    """Rotates the pairs (2j, 2j + 1) (MisterTK/gibbs src/graph/cpu.rs:678-687)."""
    adjacent = True


class NoPosition(PositionEncoding):
    pass


register_part("position", "rope_half_split", RotaryHalfSplit)
register_part("position", "rope_adjacent", RotaryAdjacent)
register_part("position", "none", NoPosition)
