"""Position encodings.  Rotary: per-pair frequencies built once in float32.

inv_freq[j] = theta^(-2j / rotary_dim) (float32 `powf`, src/model.c:288-289), divided by the
model's per-frequency factors where it has them (src/model.c:291-297).  The reference reads those
factors from a tensor its converter wrote; for ``rope_scaling`` of type llama3 they are computed
here from the four numbers of the configuration: with wavelength lam = 2*pi/f,
``lam < orig/high`` keeps f, ``lam > orig/low`` divides f by ``factor``, and between the two
f' = (1-s) f/factor + s f with s = (orig/lam - low) / (high - low).  ``rope_scaling`` of type linear divides
every frequency by ``factor`` (src/model.c:361-362).  The rotation itself (angle =
position * inv_freq in float32, pairs (j, j + rotary_dim/2), src/model.c:3514-3532) happens in the
kernel that also stores K and V.
"""
from __future__ import annotations

import math
from fractions import Fraction
from typing import Optional

import numpy as np
import torch

from .base import PositionEncoding, Rotary, register_position


def llama3_divisors(inv_freq: np.ndarray, factor: float, low: float, high: float, orig: float, dtype=np.float32) -> np.ndarray:
    out = np.ones_like(inv_freq, dtype=dtype)
    for j, f in enumerate(inv_freq.tolist()):
        lam = 2.0 * math.pi / f
        if lam < orig / high:
            d = 1.0
        elif low > 0 and lam > orig / low or high <= low:
            d = factor
        else:
            s = (orig / lam - low) / (high - low)
            d = f / ((1.0 - s) * f / factor + s * f)
        out[j] = d
    return out


class DistanceBuckets:
    """Which row of a bias table of `rows` rows a distance from query to key takes: the distance itself below h = rows // 2, then
    steps that grow logarithmically up to the distance `far`, the last row from there on,
        min(rows - 1, h + floor(ln(n / h) / ln(far / h) (rows - h)))       for n >= h.
    ``table()`` lists the rows of the distances 0, 1, ... up to the first that takes the last row (which every larger one takes too)."""

    def __init__(self, rows: int, far: float):
        self.rows, self.far, self.half = int(rows), Fraction(far), int(rows) // 2
        if self.half < 1 or self.far <= self.half:
            raise ValueError(f"distance buckets: {rows} rows up to the distance {far}: at least two rows, and a distance above half of them")

    def _start(self, k: int) -> int:
        """The first distance of step k: the smallest n with (n / h)^steps >= (far / h)^k, compared in whole numbers, so that a
        distance right on a step takes it."""
        h, steps = self.half, self.rows - self.half
        reached = lambda n: Fraction(n, h) ** steps >= (self.far / h) ** k
        n = max(h, int(h * float(self.far / h) ** (k / steps)))
        while not reached(n):
            n += 1
        while n > h and reached(n - 1):
            n -= 1
        return n

    def table(self) -> np.ndarray:
        h, steps = self.half, self.rows - self.half
        starts = np.asarray([self._start(k) for k in range(1, steps)], dtype=np.int64)     # (the last row is rows - 1 = h + steps - 1)
        last = int(starts[-1]) if len(starts) else h
        n = np.arange(last + 1, dtype=np.int64)
        return np.where(n < h, n, h + np.searchsorted(starts, n, side="right"))


class Rope(PositionEncoding):
    def __init__(self, head_dim: int, theta: float, rotary_dim: Optional[int] = None, scaling=None,
                 pairing: str = "half", mscale: float = 1.0):
        """pairing "half" rotates elements (j, j + rotary_dim/2), the layout of a config.json + safetensors
        checkpoint; "adjacent" rotates (2j, 2j + 1), the layout the reference's llama files carry
        (src/model.c:1464-1466).  mscale multiplies every cosine and sine (src/model.c:283, 375)."""
        self.head_dim = head_dim
        self.pairing, self.mscale = pairing, float(mscale)
        self.rotary_dim = head_dim if rotary_dim is None else rotary_dim
        if self.rotary_dim % 2 or self.rotary_dim > head_dim or self.rotary_dim < 0:
            raise ValueError("rotary_dim must be even and at most head_dim")
        half = self.rotary_dim // 2
        j = np.arange(half, dtype=np.float32)
        expo = (np.float32(-2.0) * j / np.float32(self.rotary_dim)).astype(np.float32) if half else j
        inv = np.power(np.float32(theta), expo).astype(np.float32)
        if scaling is not None and getattr(scaling, "rope_type", "llama3") == "linear":
            inv = (inv / np.float32(scaling.factor)).astype(np.float32)          # src/model.c:361-362
        elif scaling is not None:
            div = llama3_divisors(inv, scaling.factor, scaling.low_freq_factor, scaling.high_freq_factor,
                                  scaling.original_max_position_embeddings)
            inv = (inv / div).astype(np.float32)
        self.inv_freq_host = inv
        self.inv_freq = None
        # the same frequencies in float64, for kernels that take the angle in float64
        self.inv_freq64_host = None
        linear = scaling is not None and getattr(scaling, "rope_type", "llama3") == "linear"
        if half:
            self.inv_freq64_host = np.power(float(theta), -2.0 * np.arange(half, dtype=np.float64) / float(self.rotary_dim))
            if linear:
                self.inv_freq64_host = self.inv_freq64_host / float(scaling.factor)
            elif scaling is not None:
                self.inv_freq64_host = self.inv_freq64_host / llama3_divisors(
                    self.inv_freq64_host, scaling.factor, scaling.low_freq_factor, scaling.high_freq_factor,
                    scaling.original_max_position_embeddings, np.float64)

    def prepare(self, rt):
        self.inv_freq = torch.from_numpy(self.inv_freq_host.copy()).to(rt.device)

    def rotary(self):
        return Rotary(self.rotary_dim, self.inv_freq if self.rotary_dim else None, self.pairing, self.mscale)


class YarnRope(PositionEncoding):
    """Rotation with frequencies interpolated by wavelength ("YaRN") and cosines and sines scaled for it.

    With f_i = base^(-2i/dims) and where(t) = dims ln(original / (2 pi t)) / (2 ln base), the pair index whose wavelength fits
    `original` positions t times:  lo = max(floor(where(fast)), 0), hi = min(ceil(where(slow)), dims - 1),
    ramp_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1), frequency_i = f_i / factor * ramp_i + f_i (1 - ramp_i); every cosine
    and sine is multiplied by 0.1 ln(factor) + 1.  Without `factor` the frequencies are f_i and the multiplier is one."""

    def __init__(self, head_dim: int, base: float, rotary_dim: int, factor: Optional[float] = None, original: float = 0.0,
                 fast: float = 32.0, slow: float = 1.0, pairing: str = "half"):
        if rotary_dim % 2 or rotary_dim > head_dim or rotary_dim < 0:
            raise ValueError("rotary_dim must be even and at most head_dim")
        self.head_dim, self.rotary_dim, self.pairing = head_dim, rotary_dim, pairing
        half = rotary_dim // 2
        i = np.arange(half, dtype=np.float64)
        f = np.power(float(base), -2.0 * i / float(rotary_dim)) if half else i
        self.mscale = 1.0
        if factor is not None and half:
            where = lambda turns: rotary_dim * math.log(float(original) / (2.0 * math.pi * turns)) / (2.0 * math.log(float(base)))
            lo, hi = max(math.floor(where(fast)), 0), min(math.ceil(where(slow)), rotary_dim - 1)
            ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
            f = f / float(factor) * ramp + f * (1.0 - ramp)
            self.mscale = 0.1 * math.log(float(factor)) + 1.0
        self.inv_freq64_host = f
        self.inv_freq_host = f.astype(np.float32)
        self.inv_freq = None

    def prepare(self, rt):
        self.inv_freq = torch.from_numpy(self.inv_freq_host.copy()).to(rt.device)

    def rotary(self):
        return Rotary(self.rotary_dim, self.inv_freq if self.rotary_dim else None, self.pairing, self.mscale)


class NoPosition(PositionEncoding):
    """No position signal of its own (order comes from the causal mask alone)."""

    def rotary(self):
        return None


register_position("rope", Rope)
register_position("yarn", YarnRope)
register_position("none", NoPosition)
