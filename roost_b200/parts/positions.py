"""Position encodings a mixer can be given.

The attention mixer's fused kernel rotates the first ``rotary_dim`` elements of every query and key head by
the angle position * inv_freq[i], pairing element i with i + rotary_dim/2 (NeoX form,
src/Starlings.Roost.Ops/CpuOps.cs:111-177). A position encoding therefore hands the mixer a table of
frequencies in double precision and a rotary width; ``rotary_dim`` 0 means no rotation. Frequency-scaled
variants (``PositionSpec.scaling``) are other tables behind the same interface; one that also scales cosines and sines says so in
``amplitude``, and a mixer whose kernel does not take that refuses it (``require_plain_amplitude``). An encoding whose angles are not position x frequency (several
position axes, angles looked up in a table) gives the step's cosines and sines itself (``step_table``); the pairing of
elements stays the kernel's.
"""
from __future__ import annotations

import math

import torch

from ..config.spec import PositionSpec, RotationScaling
from .base import Part, Runtime, register_position


class PositionEncoding(Part):
    def rotation(self) -> tuple[torch.Tensor | None, int]:
        """(inv_freq: float64 [rotary_dim / 2] on the device, rotary_dim)."""
        raise NotImplementedError

    def step_table(self, batch) -> torch.Tensor | None:
        """Optional: the cosines and sines of this step's tokens, float32 [T, rotary_dim / 2, 2] on the device, made from
        the step's device tables (``batch.positions``: -1 for the padding tokens of a captured step). None (the default):
        the kernels form position * inv_freq themselves."""
        return None

    max_positions: int = 0  # 0: unbounded
    amplitude: float = 1.0  # the factor on cosines and sines


def require_plain_amplitude(position, what: str) -> None:
    if position is not None and getattr(position, "amplitude", 1.0) != 1.0:
        raise ValueError(f"{what}: the kernel does not scale cosines and sines (the position encoding asks for a factor of {position.amplitude})")


def scaled_frequencies(theta: float, rotary_dim: int, scaling: RotationScaling | None) -> tuple[list, float]:
    """(the frequencies theta^(-2i / rotary_dim) as ``scaling`` changes them, the factor on cosines and sines), formed in double."""
    freqs = [float(theta) ** (-2.0 * i / rotary_dim) for i in range(rotary_dim // 2)]
    if scaling is None:
        return freqs, 1.0
    s = scaling
    if not s.factor > 0 or not s.original > 0:
        raise ValueError(f"rotation scaling: factor {s.factor} and original {s.original} must be positive")
    if s.kind == "llama3":
        if not 0 < s.low < s.high:
            raise ValueError(f"rotation scaling: low {s.low} and high {s.high} must be positive, low below high")

        def stretched(f):
            turns = s.original * f / (2.0 * math.pi)          # original / wavelength
            if turns > s.high:
                return f
            if turns < s.low:
                return f / s.factor
            mix = (turns - s.low) / (s.high - s.low)
            return (1.0 - mix) * f / s.factor + mix * f

        return [stretched(f) for f in freqs], 1.0
    if s.kind == "yarn":
        if not s.fast > 0 or not s.slow > 0 or theta == 1.0:
            raise ValueError(f"rotation scaling: fast {s.fast} and slow {s.slow} must be positive and theta not one")
        at = lambda turns: rotary_dim * math.log(s.original / (2.0 * math.pi * turns)) / (2.0 * math.log(theta))
        lo, hi = max(math.floor(at(s.fast)), 0), min(math.ceil(at(s.slow)), rotary_dim - 1)
        ramp = lambda i: min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        return [f / s.factor * ramp(i) + f * (1.0 - ramp(i)) for i, f in enumerate(freqs)], 0.1 * math.log(s.factor) + 1.0
    raise ValueError(f"rotation scaling: kind '{s.kind}' is not one of llama3, yarn")


_FREQUENCIES: dict = {}   # (theta, rotary_dim, scaling, device) -> the frequency table that equal encodings share


class RopeNeox(PositionEncoding):
    """f_i = theta^(-2i / rotary_dim), changed by ``scaling`` where the spec has one, computed in double once at build. Encodings of
    equal theta, width and scaling on one device
    hand out the same tensor: a step keeps its table of cosines and sines by that tensor, so that the layers of a model,
    each with an encoding of its own, share one table a step."""

    pairing = "halves"

    def __init__(self, spec: PositionSpec, runtime: Runtime):
        if spec.rotary_dim <= 0 or spec.rotary_dim % 2:
            raise ValueError(f"rope_neox: rotary_dim {spec.rotary_dim} must be positive and even")
        if spec.theta <= 0:
            raise ValueError(f"rope_neox: theta {spec.theta} must be positive")
        self.spec = spec
        self.max_positions = spec.max_positions
        key = (float(spec.theta), spec.rotary_dim, spec.scaling, str(torch.device(runtime.device)))
        freqs, self.amplitude = scaled_frequencies(spec.theta, spec.rotary_dim, spec.scaling)
        if key not in _FREQUENCIES:
            _FREQUENCIES[key] = torch.tensor(freqs, dtype=torch.float64).to(runtime.device)
        self.inv_freq = _FREQUENCIES[key]

    def rotation(self):
        return self.inv_freq, self.spec.rotary_dim


class RopeInterleaved(RopeNeox):
    """The same angles as ``rope_neox`` with element 2i paired with element 2i + 1: the pair (u, v) at position p becomes
    (u cos a - v sin a, v cos a + u sin a), a = p f_i. The pairing is the mixer's kernel's; a mixer that takes this encoding
    says so (``pairing``)."""
    pairing = "interleaved"


class NoPosition(PositionEncoding):
    def __init__(self, spec: PositionSpec, runtime: Runtime):
        self.spec = spec

    def rotation(self):
        return None, 0


register_position("rope_neox", RopeNeox)
register_position("rope_interleaved", RopeInterleaved)
register_position("none", NoPosition)
