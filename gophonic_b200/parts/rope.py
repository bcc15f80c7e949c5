"""Position encodings owned by a mixer.

``RotaryEmbedding``: rotate-half rotary embedding over the first ``rotary_dim`` elements of a head.
inv_freq_i = theta^(-2i/rotary_dim) and the angles pos * inv_freq_i are computed in float64, their
cosines and sines rounded to fp32 tables (internal/qwen3lm/weights.go:681-688;
internal/qwen3lm/evaluator.go:847-858).  The tables are consumed by the fused
norm + rotation + cache-write kernel; this part only owns them.

With ``scaling`` in the spec the slow frequencies are stretched for long contexts (``scaled_frequencies``); a
scaling may also multiply all cosines and sines by a constant (``scaled_magnitude``), which the tables then hold.

``NoPosition``: nothing is applied.
"""
from __future__ import annotations

import math
from typing import Optional, Tuple

import numpy as np
import torch

from ..config.spec import LinearStretch, RampStretch
from .base import PositionEncoding, Runtime


def ramp_frequencies(freq: np.ndarray, scaling: RampStretch, theta: float) -> np.ndarray:
    """``RampStretch`` applied to the frequencies theta^(-2i/dims), i < dims / 2."""
    dims = 2 * len(freq)

    def channel(turns: float) -> float:
        return dims * math.log(scaling.original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
    lo = max(math.floor(channel(scaling.fast)), 0)
    hi = min(math.ceil(channel(scaling.slow)), dims - 1)
    blend = np.clip((np.arange(len(freq), dtype=np.float64) - lo) / max(hi - lo, 1e-3), 0.0, 1.0)
    return freq * (blend / scaling.factor + (1.0 - blend))


def scaled_magnitude(scaling) -> float:
    """The constant a scaling multiplies cosines and sines by."""
    return 0.1 * math.log(scaling.factor) + 1.0 if isinstance(scaling, RampStretch) else 1.0


def scaled_frequencies(freq: np.ndarray, scaling, theta: float = 0.0) -> np.ndarray:
    """Frequencies stretched for long contexts: ``scaling`` = (factor, low, high, original).  A frequency whose
    wavelength is longer than original / low is divided by factor, one whose wavelength is shorter than
    original / high stays, and between the two s = (original / wavelength - low) / (high - low) blends the divided
    and the plain frequency, (1 - s) f / factor + s f.  float64; None: as they are.  A ``LinearStretch`` divides every
    frequency, a ``RampStretch`` (which needs the base ``theta``) blends along the channels."""
    if scaling is None:
        return freq
    if isinstance(scaling, LinearStretch):
        return freq / float(scaling.factor)
    if isinstance(scaling, RampStretch):
        return ramp_frequencies(freq, scaling, float(theta))
    factor, low, high, original = (float(v) for v in scaling)
    wave = 2.0 * np.pi / freq
    s = (original / wave - low) / (high - low)
    out = np.where(wave < original / high, freq, np.where(wave > original / low, freq / factor, (1.0 - s) * freq / factor + s * freq))
    return out


class RotaryEmbedding(PositionEncoding):
    def __init__(self, spec, prefix, tensors, runtime: Runtime):
        if spec.rotary_dim <= 0 or spec.rotary_dim % 2 or spec.rotary_dim > spec.head_dim:
            raise ValueError(f"rotary width {spec.rotary_dim} must be even and in (0, head_dim={spec.head_dim}]")
        self.spec = spec
        self.rt = runtime
        self.cos: Optional[torch.Tensor] = None
        self.sin: Optional[torch.Tensor] = None
        self.capacity = 0

    def prepare(self, capacity: int) -> None:
        if capacity <= self.capacity:
            return
        rot = self.spec.rotary_dim
        i = np.arange(rot // 2, dtype=np.float64)
        scaling = getattr(self.spec, "scaling", None)
        inv_freq = scaled_frequencies(1.0 / np.power(float(self.spec.theta), 2.0 * i / float(rot)), scaling, self.spec.theta)
        ang = np.arange(capacity, dtype=np.float64)[:, None] * inv_freq[None, :]
        mag = scaled_magnitude(scaling)
        self.cos = torch.from_numpy((mag * np.cos(ang)).astype(np.float32)).to(self.rt.device)
        self.sin = torch.from_numpy((mag * np.sin(ang)).astype(np.float32)).to(self.rt.device)
        self.capacity = capacity

    def kernel_args(self) -> Tuple[Optional[torch.Tensor], Optional[torch.Tensor], int]:
        return self.cos, self.sin, self.spec.rotary_dim


class NoPosition(PositionEncoding):
    def __init__(self, spec, prefix, tensors, runtime: Runtime):
        self.spec = spec
        self.capacity = 1 << 62

    def kernel_args(self):
        return None, None, 0


class PairRotaryEmbedding(RotaryEmbedding):
    """Rotary embedding in which channels 2i and 2i + 1 turn together by pos * theta^(-2i/rotary_dim)
    (``RotaryEmbedding`` pairs i with i + rotary_dim / 2).  The angle tables are the same; the kernel
    is told which channels belong together (``pairs``).  A rotary width of 0 rotates nothing."""
    pairs = True

    def __init__(self, spec, prefix, tensors, runtime: Runtime):
        if spec.rotary_dim < 0 or spec.rotary_dim % 2 or spec.rotary_dim > spec.head_dim:
            raise ValueError(f"rotary width {spec.rotary_dim} must be even and in [0, head_dim={spec.head_dim}]")
        self.spec = spec
        self.rt = runtime
        self.cos = self.sin = None
        self.capacity = 0

    def prepare(self, capacity: int) -> None:
        if self.spec.rotary_dim > 0:
            super().prepare(capacity)
