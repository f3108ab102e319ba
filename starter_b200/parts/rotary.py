"""Rotary position tables: cos and sin of ``position * theta ** (-2j / head_dim)``.

The angles are formed in float32 exactly as the reference forms them
(engine/engine.py:240-259): exponent ``arange(0, D, 2) / D``, ``inv_freq = 1 /
theta ** exponent``, ``outer(position, inv_freq)``.  The two halves of the
reference's ``[positions, D]`` table are equal, so only ``D / 2`` columns are kept.
The tables stay float32; the kernel that applies them rounds to the working type
where the reference casts (before any multiply).  Tables are computed on the host
so that they are the same bits on every machine, and grow on demand.
"""

from __future__ import annotations

import math
from dataclasses import dataclass

import torch

from .base import Part


@dataclass(frozen=True)
class Rotation:
    """What a mixer needs to rotate queries and keys: float32 tables ``[positions, rotary_dim / 2]``,
    how many leading dimensions of a head they turn, and how the two halves of a pair lie in a head
    (``"half_split"``: element ``j`` with element ``j + rotary_dim / 2``; ``"interleaved"``: ``2j``
    with ``2j + 1``).  The kernels say which of these they take (``ops.rotation_tables``)."""

    cos: torch.Tensor
    sin: torch.Tensor
    rotary_dim: int
    layout: str = "half_split"


class RotaryTable(Part):
    MIN_POSITIONS = 4096

    def __init__(self, spec, dtype, device="cuda"):
        super().__init__(spec, dtype)
        self.device = device
        self.length = 0
        self.cos = None
        self.sin = None

    @staticmethod
    def angles(theta: float, head_dim: int, length: int) -> torch.Tensor:
        exponent = torch.arange(0, head_dim, 2, dtype=torch.int64).float() / head_dim
        inv_freq = 1.0 / (theta ** exponent)
        pos = torch.arange(length, dtype=torch.int64).float()
        return torch.outer(pos, inv_freq)

    def rotation(self) -> Rotation:
        """The tables as they are now (call ``ensure`` first): the whole head, half-split."""
        return Rotation(self.cos, self.sin, self.spec.head_dim, "half_split")

    def ensure(self, length: int) -> bool:
        """Make the tables cover positions ``[0, length)``; True if they moved (captured graphs that
        read the old tables must then be dropped)."""
        if length <= self.length:
            return False
        size = max(self.MIN_POSITIONS, self.length)
        while size < length:
            size *= 2
        freqs = self.angles(self.spec.theta, self.spec.head_dim, size)
        self.cos = freqs.cos().contiguous().to(self.device)
        self.sin = freqs.sin().contiguous().to(self.device)
        self.length = size
        return True


class InterleavedRotaryTable(RotaryTable):
    """Tables for a rotation of entry ``2i`` with entry ``2i + 1`` over the first ``dims`` entries of a
    vector: ``[positions, dims / 2]`` of ``cos`` and ``sin`` of ``position * base ** (-2i / dims)``.  The spec's ``scaling``
    changes the frequencies (and, for YaRN, multiplies cos and sin).  The angles are formed in float64 on the host and
    the tables rounded to float32 once."""

    LAYOUT = "interleaved"

    def rotation(self) -> Rotation:
        return Rotation(self.cos, self.sin, self.spec.dims, self.LAYOUT)

    def frequencies(self):
        """``(float64 [dims / 2], multiplier of cos and sin)``."""
        dims, base, scaling = self.spec.dims, float(self.spec.base), self.spec.scaling
        i = torch.arange(dims // 2, dtype=torch.float64)
        freq = torch.pow(torch.tensor(base, dtype=torch.float64), -2.0 * i / dims)
        if scaling is None:
            return freq, 1.0
        if not hasattr(scaling, "original"):
            return freq / scaling.factor, 1.0

        def index_of(turns: float) -> float:
            # the (fractional) frequency that makes that many turns over the original length
            return dims * math.log(scaling.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

        lo = max(math.floor(index_of(scaling.fast)), 0)
        hi = min(math.ceil(index_of(scaling.slow)), dims - 1)
        stretched = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        return freq / scaling.factor * stretched + freq * (1.0 - stretched), 0.1 * math.log(scaling.factor) + 1.0

    def ensure(self, length: int) -> bool:
        if length <= self.length:
            return False
        size = max(self.MIN_POSITIONS, self.length)
        while size < length:
            size *= 2
        freq, mult = self.frequencies()
        angles = torch.outer(torch.arange(size, dtype=torch.float64), freq)
        self.cos = (angles.cos() * mult).float().contiguous().to(self.device)
        self.sin = (angles.sin() * mult).float().contiguous().to(self.device)
        self.length = size
        return True


class PartialRotaryTable(InterleavedRotaryTable):
    """Tables for a rotation of entry ``i`` with entry ``i + dims / 2`` over the first ``dims`` entries of a
    vector: the same angles as the interleaved tables, paired half-split."""

    LAYOUT = "half_split"
