"""Position encodings of the attention mixer.

``rope_neox``: rotary embedding with half-split pairs (x[i], x[i + rot/2]);
``rope_interleaved``: pairs (x[2i], x[2i+1]).  Frequencies follow the
reference: freq_i = theta^((-1/rot) * 2i) evaluated in 32-bit
(src/backend/cpu.rs:1276-1282); the angle pos * freq_i and its sine and
cosine are taken in 32-bit inside the kernel (csrc/rope_cache.cu).
``scaling_factor`` (default 1) divides every frequency: positions stretched linearly.
``yarn`` {factor, original, fast, slow}: pairs that turn often within ``original`` positions keep
their frequency, pairs that turn rarely are slowed down by ``factor``, with a ramp over the
pair's index between the indices that make ``fast`` and ``slow`` turns; cosines and sines are
multiplied by 0.1 ln(factor) + 1 (``magnitude``).
``llama3`` {factor, low, high, original} (the frequency scaling of Llama 3.1): with L = 2 pi / f a
pair's wavelength, f stays where L < original / high, becomes f / factor where L > original / low,
and between the two a mean of both, weighed by how many turns it makes in ``original`` positions.
``frequencies: "float64"`` evaluates theta^(-2i/rot) in 64-bit and rounds once to 32-bit.
``none``: no encoding.

A position part offers ``rotary()`` -> (inv_freq, rotary_dim, style) for the
fused rotate-and-store kernel, and ``magnitude``, the factor on cosine and sine (1 as a rule; only
head_prepare applies another).  A part without ``rotary`` must offer
``apply(q, k, ctx)`` instead, which rotates the ``[rows, heads, head_dim]``
views in place before keys are stored.
"""

from __future__ import annotations

import math
from typing import Dict, Mapping, Optional, Tuple

import torch

from ..config.spec import ConfigError
from ..kernels import native
from ..weights.loader import TensorDecl
from .registry import register_position


def yarn(freqs: torch.Tensor, rotary_dim: int, theta: float, scaling: Mapping) -> Tuple[torch.Tensor, float]:
    """(slowed-down 64-bit frequencies, factor on cosine and sine).  A pair's (real) index at which
    the plain frequencies make ``t`` turns in ``original`` positions is
    dims ln(original / (2 pi t)) / (2 ln theta)."""
    factor, original = float(scaling["factor"]), float(scaling["original"])

    def index(turns: float) -> float:
        return rotary_dim * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
    lo = max(math.floor(index(float(scaling["fast"]))), 0)
    hi = min(math.ceil(index(float(scaling["slow"]))), rotary_dim - 1)
    ramp = ((torch.arange(freqs.numel(), dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
    return freqs / factor * ramp + freqs * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def llama3(freqs: torch.Tensor, scaling: Mapping) -> torch.Tensor:
    """Frequencies (64-bit) with the long wavelengths slowed down by ``factor``."""
    factor, original = float(scaling["factor"]), float(scaling["original"])
    low, high = float(scaling["low"]), float(scaling["high"])
    length = 2.0 * math.pi / freqs
    turns = original / length
    share = (turns - low) / (high - low) if high != low else torch.zeros_like(freqs)
    between = (1.0 - share) * freqs / factor + share * freqs
    return torch.where(length < original / high, freqs,
                       torch.where(length > original / low, freqs / factor, between))


class Rope:
    style = native.ROPE_HALF_SPLIT
    magnitude = 1.0

    @staticmethod
    def tensors(params: Mapping, head_dim: int) -> Dict[str, TensorDecl]:
        return {}

    def __init__(self, params: Mapping, head_dim: int, weights: Mapping[str, torch.Tensor], rt):
        self.theta = float(params["theta"])
        self.rotary_dim = int(params.get("rotary_dim") or head_dim)
        if self.rotary_dim % 2 or not 0 < self.rotary_dim <= head_dim:
            raise ConfigError(f"rotary_dim {self.rotary_dim} must be even and at most "
                              f"head_dim {head_dim}")
        if params.get("yarn") and params.get("llama3"):
            raise ConfigError("rope: 'yarn' and 'llama3' scale the same frequencies; one of them at most")
        if params.get("frequencies") == "float64" or params.get("yarn") or params.get("llama3"):
            two_i = torch.arange(self.rotary_dim // 2, dtype=torch.float64) * 2.0
            freqs = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -two_i / self.rotary_dim)
            if params.get("yarn"):
                freqs, self.magnitude = yarn(freqs, self.rotary_dim, self.theta, params["yarn"])
            if params.get("llama3"):
                freqs = llama3(freqs, params["llama3"])
            freqs = freqs.to(torch.float32)
        else:
            inv_ndims = torch.tensor(-1.0 / self.rotary_dim, dtype=torch.float32)
            two_i = torch.arange(self.rotary_dim // 2, dtype=torch.float32) * 2.0
            freqs = torch.pow(torch.tensor(self.theta, dtype=torch.float32), inv_ndims * two_i)
        self.scaling_factor = float(params.get("scaling_factor") or 1.0)
        if self.scaling_factor <= 0:
            raise ConfigError(f"scaling_factor {self.scaling_factor} must be positive")
        if self.scaling_factor != 1.0:
            freqs = freqs / self.scaling_factor
        self.inv_freq = freqs.to(rt.device).contiguous()

    def rotary(self) -> Tuple[Optional[torch.Tensor], int, int]:
        return self.inv_freq, self.rotary_dim, self.style


class RopeInterleaved(Rope):
    style = native.ROPE_INTERLEAVED


class NoPosition:
    magnitude = 1.0

    @staticmethod
    def tensors(params: Mapping, head_dim: int) -> Dict[str, TensorDecl]:
        return {}

    def __init__(self, params: Mapping, head_dim: int, weights, rt):
        pass

    def rotary(self):
        return None, 0, native.ROPE_HALF_SPLIT


register_position("rope_neox", Rope)
register_position("rope_interleaved", RopeInterleaved)
register_position("none", NoPosition)
