"""Position-encoding parts.  ``rotary``: andre-fu/prism's RoPE
(engine/executor.py:45-57): ``inv_freq_j = theta^(-2j/hd)``, rotate-half
pairing ``(j, j + hd/2)``, the whole head rotated, no scaling.  The table of
inverse frequencies is float32 and angles are formed from the position in the
kernel, so there is neither a rounded table nor a cap on positions."""

from __future__ import annotations

import math

import torch

from .base import PositionEncoding, RotaryParams, register_part


_INV_FREQ = {}      # (device, theta, rotary_dim) -> float32 inverse frequencies on that device


@register_part("position", "rotary")
class RotaryEmbedding(PositionEncoding):
    def __init__(self, head_dim: int, theta: float, rotary_dim: int = None):
        self.head_dim = int(head_dim)
        self.theta = float(theta)
        self.rotary_dim = int(rotary_dim if rotary_dim is not None else head_dim)
        if self.rotary_dim % 2 or self.rotary_dim > self.head_dim:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even and <= head_dim {self.head_dim}")
        self._params = None

    def on_bound(self):
        rd = self.rotary_dim
        # the formula of executor.py:50, evaluated in float32 on the host
        # layers with the same constants share one device table, so the per-step cos/sin table that
        # the kernels build from it is built once per step, not once per layer
        key = (str(self.device), self.theta, rd)
        inv = _INV_FREQ.get(key)
        if inv is None:
            inv = (1.0 / (self.theta ** (torch.arange(0, rd, 2, dtype=torch.float32) / rd))).to(self.device)
            _INV_FREQ[key] = inv
        self._params = RotaryParams(inv, rd)

    def rotary(self):
        return self._params


@register_part("position", "rotary_scaled")
class ScaledRotaryEmbedding(PositionEncoding):
    """Rotation of the first ``rotary_dim`` entries of a head in interleaved pairs (2i, 2i + 1) - or, with
    ``interleaved`` False, in pairs (i, i + rotary_dim / 2) - by ``position * f_i``, ``f_i = theta^(-2i /
    rotary_dim)``, with the frequencies rescaled in three bands by wavelength ``l = 2 pi / f`` (``scaling``: a dict
    ``factor, low, high, original``, or None): unchanged where ``l < original / high``, divided by ``factor`` where
    ``l > original / low``, and ``(1 - s) f / factor + s f`` with ``s = (original / l - low) / (high - low)`` in
    between.  The table is float32; the kernels form the angles from it in float32."""

    def __init__(self, rotary_dim: int, theta: float, scaling: dict = None, interleaved: bool = True):
        self.rotary_dim, self.theta, self.interleaved = int(rotary_dim), float(theta), bool(interleaved)
        if self.rotary_dim % 2 or self.rotary_dim < 0:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even")
        self.scaling = None
        if scaling:
            self.scaling = tuple(float(scaling[k]) for k in ("factor", "low", "high", "original"))
            if self.scaling[2] == self.scaling[1]:
                raise ValueError("frequency scaling: 'high' must differ from 'low'")
        self._params = None

    def frequencies(self) -> torch.Tensor:
        import math
        rd = self.rotary_dim
        f = self.theta ** (-torch.arange(0, rd, 2, dtype=torch.float32) / max(rd, 1))
        if self.scaling is None:
            return f
        factor, low, high, original = self.scaling
        vals = []
        for fi in f.tolist():
            wavelength = 2.0 * math.pi / fi
            if wavelength < original / high:
                vals.append(fi)
            elif wavelength > original / low:
                vals.append(fi / factor)
            else:
                s = (original / wavelength - low) / (high - low)
                vals.append((1.0 - s) * fi / factor + s * fi)
        return torch.tensor(vals, dtype=torch.float32)

    def on_bound(self):
        self._params = RotaryParams(self.frequencies().to(self.device), self.rotary_dim, self.interleaved)

    def rotary(self):
        return self._params


@register_part("position", "rotary_yarn")
class YarnRotaryEmbedding(PositionEncoding):
    """Rotation of the first ``rotary_dim`` entries of a head by ``position * f_i``, ``f_i = theta^(-2i / rotary_dim)``, in
    interleaved pairs (2i, 2i + 1) or, with ``interleaved`` False, in pairs (i, i + rotary_dim / 2).  ``scaling`` (a dict
    ``factor, original, fast, slow``, or None): with ``dim(t) = rotary_dim ln(original / (2 pi t)) / (2 ln theta)``, ``lo =
    max(floor(dim(fast)), 0)``, ``hi = min(ceil(dim(slow)), rotary_dim - 1)`` and ``ramp_i = clamp((i - lo) / max(hi - lo,
    0.001), 0, 1)`` the frequency becomes ``f_i / factor * ramp_i + f_i (1 - ramp_i)``, and cosine and sine are multiplied
    by ``0.1 ln(factor) + 1``.  The table is made on the host in float64 and kept in float32."""

    def __init__(self, rotary_dim: int, theta: float, scaling: dict = None, interleaved: bool = True):
        self.rotary_dim, self.theta, self.interleaved = int(rotary_dim), float(theta), bool(interleaved)
        if self.rotary_dim % 2 or self.rotary_dim < 0:
            raise ValueError(f"rotary_dim {self.rotary_dim} must be even")
        if self.theta <= 0:
            raise ValueError(f"the rotation's base must be positive, got {theta}")
        self.scaling = None
        if scaling:
            self.scaling = tuple(float(scaling[k]) for k in ("factor", "original", "fast", "slow"))
            if min(self.scaling) <= 0 or self.theta == 1.0:
                raise ValueError("frequency scaling: factor, original, fast and slow must be positive and the base not 1")
        self._params = None

    def amplitude(self) -> float:
        return 1.0 if self.scaling is None else 0.1 * math.log(self.scaling[0]) + 1.0

    def frequencies(self) -> torch.Tensor:
        rd, half = self.rotary_dim, self.rotary_dim // 2
        f = self.theta ** (-2.0 * torch.arange(half, dtype=torch.float64) / max(rd, 1))
        if self.scaling is None or not half:
            return f.to(torch.float32)
        factor, original, fast, slow = self.scaling

        def dim(t):
            return rd * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(self.theta))
        lo, hi = max(math.floor(dim(fast)), 0), min(math.ceil(dim(slow)), rd - 1)
        ramp = ((torch.arange(half, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return (f / factor * ramp + f * (1.0 - ramp)).to(torch.float32)

    def on_bound(self):
        key = (str(self.device), "yarn", self.theta, self.rotary_dim, self.scaling)
        inv = _INV_FREQ.get(key)          # layers with the same constants share one device table
        if inv is None:
            inv = _INV_FREQ[key] = self.frequencies().to(self.device)
        self._params = RotaryParams(inv, self.rotary_dim, self.interleaved, self.amplitude())

    def rotary(self):
        return self._params


@register_part("position", "none")
class NoPositionEncoding(PositionEncoding):
    """Keys and queries are used as projected."""

    def __init__(self, head_dim: int = 0):
        self.head_dim = head_dim

    def rotary(self):
        return None

    def apply(self, ctx, q, k):
        return None
