"""Position encodings of attention mixers.

"rope": rotation of pairs of q and k elements by position-dependent angles
(src/kernels/rotary_embedding.cu:18-33).  The angle of pair j at position p is
p / theta^(2j / rotary_dim), evaluated in float as the reference's table is
(src/model/qwen.cpp:119-128: ``pos / powf(theta, 2i/d)``).  The divisors are
computed once on the host; the kernel divides and calls sincosf per element, so
no table grows with the context length.  ``pairing`` "half" pairs element j with
j + rotary_dim/2 (what the reference does), "interleaved" pairs 2j with 2j+1.
``rotary_dim`` below the head size leaves the rest of each head unrotated.

"none": no position information is added.
"""
from __future__ import annotations

from typing import Optional

import numpy as np
import torch

from .base import PositionEncoding, register_position_encoding

PAIRINGS = {"half": 0, "interleaved": 1}


@register_position_encoding("rope")
class RotaryEmbedding(PositionEncoding):
    def __init__(self, theta: float, rotary_dim: int, pairing: str = "half", dtype=None, device=None):
        if pairing not in PAIRINGS:
            raise ValueError(f"rope pairing {pairing!r}; known: {sorted(PAIRINGS)}")
        if rotary_dim <= 0 or rotary_dim % 2:
            raise ValueError(f"rope rotary_dim {rotary_dim} must be positive and even")
        if not theta > 0:
            raise ValueError(f"rope theta {theta} must be positive")
        self.theta, self.rotary_dim, self.pairing = float(theta), rotary_dim, pairing
        j = np.arange(rotary_dim // 2, dtype=np.float32)
        exponent = (np.float32(2.0) * j) / np.float32(rotary_dim)
        # theta and the exponent as the reference has them, in float (src/model/qwen.cpp:124); the power itself in
        # double and then rounded, so that every host that computes it gets the same float (powf differs from one
        # library to the next in the last bit, which is enough to move a sampled token)
        denom = np.power(np.float64(np.float32(theta)), exponent.astype(np.float64)).astype(np.float32)
        self.denom = torch.from_numpy(denom).to(device)

    magnitude = 1.0          # factor of cosine and sine

    def fused(self) -> Optional[dict]:
        return {"rotary_dim": self.rotary_dim, "pairing": PAIRINGS[self.pairing], "denom": self.denom}


def rescale_by_wavelength(freq: np.ndarray, factor: float, low: float, high: float, original: float) -> np.ndarray:
    """Frequencies (float64) rescaled by wavelength l = 2 pi / f, as contexts are stretched beyond ``original`` positions:
    short waves (l < original / high) stay, long ones (l > original / low) are divided by ``factor``, and between the two
    the frequency is (1 - s) f / factor + s f with s = (original / l - low) / (high - low)."""
    if not (factor > 0 and original > 0 and high > low >= 0):
        raise ValueError(f"frequency scaling: factor {factor}, low {low} < high {high}, original {original}")
    wavelength = 2.0 * np.pi / freq
    s = (original / wavelength - low) / (high - low)
    between = (1.0 - s) * freq / factor + s * freq
    return np.where(wavelength < original / high, freq, np.where(wavelength > original / low, freq / factor, between))


def stretch_by_ramp(freq: np.ndarray, theta: float, factor: float, original: float, fast: float, slow: float) -> np.ndarray:
    """Frequencies (float64, f_i = theta^(-2i / dims)) rescaled by how often they turn within ``original`` positions: those that turn
    more than ``fast`` times stay, those below ``slow`` are divided by ``factor``, with a linear ramp over the index i between the two
    borders (rounded outwards to whole indices, and kept inside 0 .. dims - 1)."""
    if not (factor > 0 and original > 0 and fast > 0 and slow > 0 and theta > 1):
        raise ValueError(f"frequency scaling: factor {factor}, original {original}, fast {fast}, slow {slow}, base {theta}")
    dims = 2 * len(freq)
    border = lambda turns: dims * np.log(original / (2.0 * np.pi * turns)) / (2.0 * np.log(theta))
    lo, hi = max(np.floor(border(fast)), 0.0), min(np.ceil(border(slow)), dims - 1.0)
    ramp = np.clip((np.arange(len(freq)) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return freq / factor * ramp + freq * (1.0 - ramp)


@register_position_encoding("scaled_rope")
class ScaledRotaryEmbedding(RotaryEmbedding):
    """"rope" whose frequencies f_i = theta^(-2i / rotary_dim) are rescaled by wavelength (``scaling``: None, or
    {"factor", "low", "high", "original"}; rescale_by_wavelength) or by a ramp over their index ({"factor", "fast", "slow",
    "original"}; stretch_by_ramp), in which case cosine and sine are also multiplied by ``magnitude`` = 0.1 ln(factor) + 1 (a mixer
    whose kernel has no such factor refuses an encoding with a magnitude other than 1).  The frequencies are computed in double and rounded
    once; ``inv_freq`` (float32 [rotary_dim / 2]) is what a kernel multiplies a position by, ``denom`` its reciprocal
    for kernels that divide."""

    def __init__(self, theta: float, rotary_dim: int, pairing: str = "half", scaling: Optional[dict] = None, dtype=None, device=None):
        super().__init__(theta, rotary_dim, pairing, dtype=dtype, device=device)
        i = np.arange(rotary_dim // 2, dtype=np.float64)
        freq = np.power(float(theta), -2.0 * i / rotary_dim)
        self.magnitude = 1.0
        if scaling is not None and "fast" in scaling:
            missing = [k for k in ("factor", "fast", "slow", "original") if k not in scaling]
            if missing:
                raise ValueError(f"scaled_rope: scaling lacks {missing}")
            freq = stretch_by_ramp(freq, float(theta), *(float(scaling[k]) for k in ("factor", "original", "fast", "slow")))
            self.magnitude = 0.1 * float(np.log(float(scaling["factor"]))) + 1.0
        elif scaling is not None:
            missing = [k for k in ("factor", "low", "high", "original") if k not in scaling]
            if missing:
                raise ValueError(f"scaled_rope: scaling lacks {missing}")
            freq = rescale_by_wavelength(freq, float(scaling["factor"]), float(scaling["low"]), float(scaling["high"]),
                                         float(scaling["original"]))
        self.scaling = dict(scaling) if scaling is not None else None
        self.inv_freq = torch.from_numpy(freq.astype(np.float32)).to(device)
        self.denom = torch.from_numpy((1.0 / freq).astype(np.float32)).to(device)


@register_position_encoding("none")
class NoPosition(PositionEncoding):
    def __init__(self, dtype=None, device=None):
        pass

    def fused(self) -> Optional[dict]:
        return {"rotary_dim": 0, "pairing": 0, "denom": None}
