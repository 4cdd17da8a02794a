"""Position encodings that a mixer applies to its queries and keys.

``rope``: rotary over the first ``rotary_dim`` dims of a head: for
k < rotary_dim/2, angle = position * theta^(-2k/rotary_dim), and a pair of
dimensions turns by it: (k, k + rotary_dim/2) with ``pairing="half"``,
(2k, 2k + 1) with ``pairing="adjacent"`` (which kernels take which pairing is
the mixers' business: grouped-query attention takes "half", latent attention
either) (berniehans/titan:
engine/engine-core/src/forward_cpu.rs:226-241; rotary_dim = head_dim,
forward_driver.rs:608).  ``scaling`` = (factor, low, high, original) changes a frequency f by its wavelength 2 pi / f:
below original / high it stays, above original / low it becomes f / factor, between them
(1 - s) f / factor + s f with s = (original / wavelength - low) / (high - low).  The inverse frequencies are computed in float64 on the
host and rounded once to float32; the angle and its sine and cosine are float32
in the kernel.

``none``: no table; the mixer's kernel then leaves the heads as they are.
"""
from __future__ import annotations

import math
from typing import Dict

import torch

from .base import POSITIONS, PositionEncoding


def scaled_frequencies(inv: torch.Tensor, factor: float, low: float, high: float, original: float) -> torch.Tensor:
    """Frequencies (float64) scaled by wavelength; with low = high there is no stretch between the two."""
    waves = original * inv / (2.0 * math.pi)                 # original / wavelength
    s = ((waves - low) / (high - low if high != low else 1.0)).clamp(0.0, 1.0)
    blended = (1.0 - s) * inv / factor + s * inv
    return torch.where(waves > high, inv, torch.where(waves < low, inv / factor, blended))


class Rotary(PositionEncoding):
    def __init__(self, spec):
        if spec.pairing not in ("half", "adjacent"):
            raise ValueError(f"rotary pairing '{spec.pairing}' is not supported ('half' or 'adjacent')")
        if spec.rotary_dim <= 0 or spec.rotary_dim % 2:
            raise ValueError(f"rotary_dim {spec.rotary_dim} must be positive and even")
        self.spec = spec
        self._tables: Dict[str, torch.Tensor] = {}

    @property
    def rotary_dim(self) -> int:
        return self.spec.rotary_dim

    def kernel_args(self, device):
        args = super().kernel_args(device)
        args.adjacent = int(self.spec.pairing == "adjacent")
        return args

    def tables(self, device) -> Dict[str, torch.Tensor]:
        if not self._tables:
            rot = self.spec.rotary_dim
            k = torch.arange(rot // 2, dtype=torch.float64)
            inv = torch.tensor(self.spec.theta, dtype=torch.float64) ** (-2.0 * k / rot)
            if self.spec.scaling is not None:
                inv = scaled_frequencies(inv, *self.spec.scaling)
            self._tables = {"inv_freq": inv.to(torch.float32).to(device)}
        return self._tables


class NoPosition(PositionEncoding):
    def __init__(self, spec):
        self.spec = spec


POSITIONS.register("rope", Rotary)
POSITIONS.register("none", NoPosition)
