"""Rotary position encoding with the base scaled by dynamic-NTK alpha.

inv_freq[j] = 1 / base^(2j/d), base = theta * alpha^(d/(d-2)) when alpha > 0;
the power in float64, rounded to float32, the reciprocal a float32 division;
angle[p, j] = float32(p) * inv_freq[j] as a float32 product; tables
[positions, d/2] of cos and sin in float32
(crane-core/src/models/hunyuan_dense/modeling.rs:197-239).  The reference
rounds the tables to the model dtype before use (modeling.rs:1004-1009); here
the angles stay 32-bit on every path.
"""
from __future__ import annotations

import numpy as np
import torch

from .base import Part, register_part

_TABLES = {}


@register_part("position", "rope")
class Rope(Part):
    """params: ``head_dim``, ``theta``, ``alpha`` (<= 0: none), ``max_positions``,
    ``rotary_dim`` (the rotated width of a head; default: all of it, which is
    what the reference does).  No tensors.  ``tables(rt, limit)`` gives (cos,
    sin) [positions < limit, rotary_dim / 2]."""
    kind = "position"

    def width(self) -> int:
        return int(self.params.get("rotary_dim") or self.params["head_dim"])

    def inv_freq(self) -> np.ndarray:
        d = self.width()
        base = float(self.params["theta"])
        alpha = float(self.params.get("alpha") or 0.0)
        if alpha > 0.0:
            # a head of 2 elements: the reference's float division gives an infinite exponent, the base
            # becomes infinite (or 0, or stays), and its power 0 is 1 either way
            base = base * alpha ** (d / (d - 2.0) if d != 2 else float("inf"))
        powers = np.array([base ** (i / d) for i in range(0, d, 2)], dtype=np.float64)
        return (np.float32(1.0) / powers.astype(np.float32)).astype(np.float32)

    def tables(self, rt, limit: int):
        n = min(int(self.params["max_positions"]), int(limit))
        key = (self.width(), float(self.params["theta"]),
               float(self.params.get("alpha") or 0.0), n, str(rt.device))
        if key not in _TABLES:
            pos = np.arange(n, dtype=np.float32)[:, None]
            angles = (pos * self.inv_freq()[None, :]).astype(np.float32)   # float32 product
            cos = np.cos(angles.astype(np.float64)).astype(np.float32)
            sin = np.sin(angles.astype(np.float64)).astype(np.float32)
            _TABLES[key] = (torch.from_numpy(cos).to(rt.device), torch.from_numpy(sin).to(rt.device))
        return _TABLES[key]


@register_part("position", "yarn_rope")
class YarnRope(Part):
    """Rotary angles a = p * f_i over ``dims`` rotated elements, f_i = base^(-2i/dims), with YaRN
    scaling (``scaling``: factor, original, fast, slow; or None):
    dim(t) = dims ln(original / (2 pi t)) / (2 ln base), lo = max(floor(dim(fast)), 0),
    hi = min(ceil(dim(slow)), dims - 1), ramp_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1),
    f_i <- f_i / factor * ramp_i + f_i (1 - ramp_i), and cos and sin times 0.1 ln(factor) + 1.
    params: ``dims``, ``base``, ``scaling``, ``max_positions``.  No tensors.  ``tables(rt, limit)``
    gives (cos, sin) [positions < limit, dims / 2] in float, the factor folded in; the angles are
    formed in 64-bit on the host and rounded once."""
    kind = "position"

    def width(self) -> int:
        return int(self.params["dims"])

    def frequencies(self):
        dims, base = self.width(), float(self.params["base"])
        i = np.arange(dims // 2, dtype=np.float64)
        f = base ** (-2.0 * i / dims) if dims else i
        sc = self.params.get("scaling")
        mult = 1.0
        if sc and dims:
            def dim_of(t):
                return dims * np.log(float(sc["original"]) / (2.0 * np.pi * float(t))) / (2.0 * np.log(base))
            lo = max(int(np.floor(dim_of(sc["fast"]))), 0)
            hi = min(int(np.ceil(dim_of(sc["slow"]))), dims - 1)
            ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
            f = f / float(sc["factor"]) * ramp + f * (1.0 - ramp)
            mult = 0.1 * float(np.log(float(sc["factor"]))) + 1.0
        return f, mult

    def tables(self, rt, limit: int):
        n = min(int(self.params["max_positions"]), int(limit))
        sc = self.params.get("scaling") or {}
        key = ("yarn", self.width(), float(self.params["base"]),
               tuple(sorted((k, float(v)) for k, v in sc.items())), n, str(rt.device))
        if key not in _TABLES:
            f, mult = self.frequencies()
            angles = np.arange(n, dtype=np.float64)[:, None] * f[None, :]
            cos = (np.cos(angles) * mult).astype(np.float32).reshape(n, -1)
            sin = (np.sin(angles) * mult).astype(np.float32).reshape(n, -1)
            if cos.shape[1] == 0:           # nothing is rotated: a column that no kernel reads
                cos, sin = np.ones((n, 1), np.float32), np.zeros((n, 1), np.float32)
            _TABLES[key] = (torch.from_numpy(cos).to(rt.device), torch.from_numpy(sin).to(rt.device))
        return _TABLES[key]


@register_part("position", "wavelength_rope")
class WavelengthRope(Part):
    """Rotary angles a = p * f_i over ``dims`` rotated elements, f_i = base^(-2i/dims), scaled by wavelength
    l = 2 pi / f_i as Llama 3.1 does (``scaling``: factor, low, high, original; or None): f_i stays where
    l < original / high, becomes f_i / factor where l > original / low, and in between
    (1 - s) f_i / factor + s f_i with s = (original / l - low) / (high - low).
    params: ``dims``, ``base``, ``scaling``, ``max_positions``.  No tensors.  ``tables(rt, limit)`` gives (cos, sin)
    [positions < limit, dims / 2] in float; the angles are formed in 64-bit on the host and rounded once."""
    kind = "position"

    def width(self) -> int:
        return int(self.params["dims"])

    def frequencies(self):
        dims, base = self.width(), float(self.params["base"])
        f = base ** (-2.0 * np.arange(dims // 2, dtype=np.float64) / dims)
        sc = self.params.get("scaling")
        if not sc:
            return f
        factor, low, high, original = (float(sc[k]) for k in ("factor", "low", "high", "original"))
        wavelength = 2.0 * np.pi / f
        s = (original / wavelength - low) / (high - low) if high != low else np.zeros_like(f)
        between = (1.0 - s) * f / factor + s * f
        return np.where(wavelength < original / high, f, np.where(wavelength > original / low, f / factor, between))

    def tables(self, rt, limit: int):
        n = min(int(self.params["max_positions"]), int(limit))
        sc = self.params.get("scaling") or {}
        key = ("wavelength", self.width(), float(self.params["base"]),
               tuple(sorted((k, float(v)) for k, v in sc.items())), n, str(rt.device))
        if key not in _TABLES:
            angles = np.arange(n, dtype=np.float64)[:, None] * self.frequencies()[None, :]
            _TABLES[key] = tuple(torch.from_numpy(t.astype(np.float32)).to(rt.device) for t in (np.cos(angles), np.sin(angles)))
        return _TABLES[key]
