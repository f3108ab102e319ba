"""RMSNorm with a plain gain, alone or fused with the residual sum that always precedes it."""

from __future__ import annotations

import torch

from .. import ops
from .base import ParamSpec, Part, bytes_of


class RMSNorm(Part):
    """``y = gain * round(x * rsqrt(mean(x^2) + eps))``; reduce and scale in float
    (engine/engine.py:75-88, engine/kernels/rmsnorm.py:21-45)."""

    def param_specs(self):
        if getattr(self.spec, "unit_offset", False):
            return {"weight": ParamSpec((self.spec.size,), "gain_offset")}
        if getattr(self.spec, "gain_32bit", False):
            return {"weight": ParamSpec((self.spec.size,), "gain32")}
        return {"weight": ParamSpec((self.spec.size,), "gain")}

    def set_params(self, params):
        self.weight = params["weight"]
        if getattr(self.spec, "unit_offset", False):
            # stored around zero: the gain is formed once, in float32, and the kernels see a plain gain
            self.weight = (1.0 + self.weight.float()).contiguous()

    def parameters(self):
        """``(gain, eps)`` for the kernel that reads several residual streams and norms what it read; None when the
        gain is not held in float32 (the norm then runs as a kernel of its own)."""
        return (self.weight, self.spec.eps) if self.weight.dtype == torch.float32 else None

    def __call__(self, x):
        return ops.rmsnorm(x, self.weight, self.spec.eps)

    def add(self, residual, delta):
        """``residual += delta`` in place, then the norm of the sum (engine/kernels/fused.py:115-144)."""
        if delta is None or delta is ops.ADDED:      # nothing open, or the part before added it itself
            return ops.rmsnorm(residual, self.weight, self.spec.eps)
        return ops.rmsnorm(residual, self.weight, self.spec.eps, delta=delta)

    def add_rows(self, residual, delta, rows):
        """The norm of ``(residual + delta)[rows]`` without touching ``residual``."""
        if delta is ops.ADDED:
            delta = None
        return ops.rmsnorm(residual, self.weight, self.spec.eps, delta=delta, rows=rows)

    def weight_bytes(self):
        return bytes_of(self.weight)
