"""What may stand between two layers of the run order (family ``junction``).

``EmbeddingJoin``: the embedding output is brought back into a float32 residual stream, ``x <- W [x ; x0]``.  The sum that
closes the sublayer before it and the row ``[x | x0]`` the product reads are one kernel (``ops.residual_join``: ``x0`` is
looked up again, nothing of it is kept); the product's float32 result is the new stream.
"""

from __future__ import annotations

from .. import ops
from .base import ParamSpec, Part, bytes_of


class EmbeddingJoin(Part):
    #: the residual streams it stands in (see the arrangements' ``residual_kind``)
    residual_kind = "float32"

    def param_specs(self):
        w = self.spec.width
        return {"weight": ParamSpec((w, 2 * w))}

    def set_params(self, params):
        self.weight = params["weight"].contiguous()

    def __call__(self, residual, pending, ctx, table, scale):
        """The new stream; ``pending`` (or None) is taken in first, ``table`` and ``scale`` give the embedding output."""
        rows = ops.residual_join(residual, pending.for_kernel() if pending is not None else None, ctx.tokens, table, scale)
        return ops.linear(rows, self.weight, out_float=True, status=ctx.status)

    def weight_bytes(self):
        return bytes_of(self.weight)
