"""Rotary position encoding: the constants the attention kernels use.

Formula (src/cloud_engine/attention.py:60-85): ``inv_freq[j] = theta^(-2j/R)`` for
j < R/2, angle = position * inv_freq[j]; element j pairs with element j + R/2:
``x'[j] = x[j] cos - x[j+R/2] sin``, ``x'[j+R/2] = x[j+R/2] cos + x[j] sin``.  The
reference builds a cos/sin table of 32768 rows (model.py:190-192) and rotates in the
model dtype; here the kernel computes the angle and the rotation in float32 from
``inv_freq`` and rounds once.  ``rotary_dim`` may be smaller than ``head_dim`` (the rest
of the head passes through).

Beyond the reference (which has exactly the above):

* ``pairing="interleaved"`` pairs element 2j with element 2j + 1 instead.  The kernels keep the
  one pairing they have: the mixer permutes the q and k rows of its weights at load time
  (``row_order``) so that element 2j lands at j and element 2j + 1 at j + R/2.  Scores are dot
  products of q and k, which the same permutation of both leaves unchanged, and nobody else
  reads q or k.
* ``position_scale`` divides positions (linear position scaling); ``attention_factor`` multiplies
  the softmax scale of the mixer that owns this encoding.
* ``ramp`` = (factor, original, fast, slow) blends every frequency f_i between itself and
  f_i / factor: with ``d(t) = R ln(original / (2 pi t)) / (2 ln theta)`` (the pair index at which
  ``original`` positions make ``t`` turns), ``lo = max(floor(d(fast)), 0)``, ``hi = min(ceil(d(slow)),
  R - 1)`` and ``r_i = clamp((i - lo) / max(hi - lo, 0.001), 0, 1)`` the frequency is
  ``f_i / factor * r_i + f_i * (1 - r_i)``; cos and sin are then both multiplied by
  ``magnitude = 0.1 ln(factor) + 1`` (a mixer that rotates with kernels of its own reads
  ``magnitude``; the softmax scale is left alone).
* ``bands`` = (factor, low, high, original) scales frequencies by wavelength: with ``l = 2 pi / f``, f stays where
  ``l < original / high``, becomes ``f / factor`` where ``l > original / low``, and between the two, with
  ``s = (original / l - low) / (high - low)``, ``(1 - s) f / factor + s f``; no magnitude factor.
* ``keep_pairing``: ``row_order`` answers None although the pairing is interleaved, for a mixer whose
  kernels rotate either pairing themselves (``pairing`` tells them which).
"""

from __future__ import annotations

import math

from .base import PositionEncoding, register_part


class RopeNeox(PositionEncoding):
    style = "neox"

    def __init__(self, head_dim: int, rotary_dim: int, theta: float, max_positions: int,
                 pairing: str = "half", position_scale: float = 1.0, attention_factor: float = 1.0,
                 ramp: tuple[float, float, float, float] | None = None, keep_pairing: bool = False,
                 bands: tuple[float, float, float, float] | None = None) -> None:
        if rotary_dim % 2 or rotary_dim > head_dim or rotary_dim < 2:
            raise ValueError(f"rotary_dim {rotary_dim} must be even and within head_dim {head_dim}")
        if pairing not in ("half", "interleaved"):
            raise ValueError(f"pairing must be 'half' or 'interleaved', got {pairing!r}")
        if position_scale <= 0 or attention_factor <= 0:
            raise ValueError("position_scale and attention_factor must be positive")
        self.head_dim = int(head_dim)
        self.rotary_dim = int(rotary_dim)
        self.theta = float(theta)
        self.max_positions = int(max_positions)
        self.pairing = pairing
        self.position_scale = float(position_scale)
        self.attention_factor = float(attention_factor)
        self.ramp = tuple(float(value) for value in ramp) if ramp is not None else None
        if self.ramp is not None and (len(self.ramp) != 4 or min(self.ramp) <= 0):
            raise ValueError("ramp must be (factor, original, fast, slow), all positive")
        self.magnitude = 0.1 * math.log(self.ramp[0]) + 1.0 if self.ramp is not None else 1.0
        self.keep_pairing = bool(keep_pairing)
        self.bands = tuple(float(value) for value in bands) if bands is not None else None
        if self.bands is not None and (len(self.bands) != 4 or min(self.bands) <= 0 or self.ramp is not None):
            raise ValueError("bands must be (factor, low, high, original), all positive, and exclude a ramp")

    def frequencies(self) -> list[float]:
        """f_i for i < rotary_dim / 2, in double precision."""
        dims, half = self.rotary_dim, self.rotary_dim // 2
        plain = [self.theta ** (-2.0 * i / dims) / self.position_scale for i in range(half)]
        if self.bands is not None:
            factor, low, high, original = self.bands

            def banded(f: float) -> float:
                turns = original * f / (2.0 * math.pi)          # original / wavelength
                if turns > high:
                    return f
                if turns < low:
                    return f / factor
                s = (turns - low) / (high - low) if high != low else 1.0
                return (1.0 - s) * f / factor + s * f

            return [banded(f) for f in plain]
        if self.ramp is None:
            return plain
        factor, original, fast, slow = self.ramp

        def pair_index(turns: float) -> float:
            return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.theta))

        lo = max(math.floor(pair_index(fast)), 0)
        hi = min(math.ceil(pair_index(slow)), dims - 1)
        width = max(hi - lo, 0.001)
        blend = [min(max((i - lo) / width, 0.0), 1.0) for i in range(half)]
        return [f / factor * r + f * (1.0 - r) for f, r in zip(plain, blend)]

    def row_order(self) -> list[int] | None:
        """For a mixer: the order in which the elements of a q or k head are to be stored so that
        this encoding's pairs are (j, j + rotary_dim/2) for the kernels; None if they are already."""
        if self.pairing == "half" or self.keep_pairing:
            return None
        half = self.rotary_dim // 2
        order = [2 * j for j in range(half)] + [2 * j + 1 for j in range(half)]
        return order + list(range(self.rotary_dim, self.head_dim))

    def bind(self, tensors, runtime) -> None:
        import torch

        self.runtime = runtime
        if self.ramp is None and self.bands is None:
            exponent = torch.arange(0, self.rotary_dim, 2, dtype=torch.float32) / self.rotary_dim
            inv_freq = 1.0 / (self.theta ** exponent) / self.position_scale
        else:
            inv_freq = torch.tensor(self.frequencies(), dtype=torch.float64).to(torch.float32)
        self.inv_freq = inv_freq.to(runtime.device).contiguous()


register_part("position", "rope_neox", RopeNeox, replace=True)
