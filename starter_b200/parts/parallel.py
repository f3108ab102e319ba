"""Two mixers side by side that read the same input, joined as the spec says: ``"norm_mean"``, half the sum of their
outputs, each first RMS-normed over the model width with a plain gain of its own (``ops.norm_pair_mean``);
``"scaled_sum"``, their sum with two constants (``ops.scaled_sum``).

The two sides are built from their own specs through the registry, so any mixer can stand on either side.  The
layer's cache entry serves both: at most one side may keep keys and values; when both keep a float32 state, a slot
holds the left side's floats, then the right side's (``state_at`` tells a side where its own begin).
"""

from __future__ import annotations

from .. import ops
from ..cache.layout import StateNeed
from .base import ParamSpec, Part, bytes_of

JOINS = ("norm_mean", "scaled_sum")


class ParallelMixer(Part):
    SIDES = ("left", "right")

    def __init__(self, spec, dtype, position=None):
        super().__init__(spec, dtype)
        from .registry import lookup

        if spec.join not in JOINS:
            raise ValueError(f"no join {spec.join!r} of two mixers (known: {', '.join(JOINS)})")
        self.sides = {}
        for name in self.SIDES:
            side = getattr(spec, name)
            wants = getattr(side, "position", None) is not None
            self.sides[name] = lookup("mixer", side.kind)(side, dtype, position if wants else None)
        if sum(m.kv_need() is not None for m in self.sides.values()) > 1:
            raise ValueError("both sides of a parallel mixer keep keys and values; a layer has one cache entry")
        needs = {n: m.state_need() for n, m in self.sides.items() if m.state_need() is not None}
        self.state_floats = 0
        if len(needs) > 1:
            for name, need in needs.items():
                if len(need.shape) != 1 or need.dtype != "float32" or not hasattr(self.sides[name], "state_at"):
                    raise ValueError(f"both sides of a parallel mixer keep a per-sequence state, and the {name} side's cannot "
                                     f"share a slot")
                self.sides[name].state_at = self.state_floats
                self.state_floats += -(-need.shape[0] // 4) * 4          # a side's state starts on a 16-byte boundary

    def kv_need(self):
        return next((n for n in (m.kv_need() for m in self.sides.values()) if n is not None), None)

    def state_need(self):
        if self.state_floats:
            return StateNeed((self.state_floats,), "float32")
        return next((n for n in (m.state_need() for m in self.sides.values()) if n is not None), None)

    def param_specs(self):
        out = {}
        for name, mixer in self.sides.items():
            out.update({f"{name}.{k}": v for k, v in mixer.param_specs().items()})
            if self.spec.join == "norm_mean":
                out[f"{name}_out"] = ParamSpec((self.spec.hidden_size,), "gain32")
        return out

    def set_params(self, params):
        for name, mixer in self.sides.items():
            mixer.set_params({k[len(name) + 1:]: v for k, v in params.items() if k.startswith(name + ".")})
        self.gains = {}
        if self.spec.join == "norm_mean":
            self.gains = {name: params[f"{name}_out"].float().contiguous() for name in self.sides}

    def prepare(self, max_position: int) -> bool:
        moved = False
        for mixer in self.sides.values():
            moved = bool(mixer.prepare(max_position)) or moved
        return moved

    def __call__(self, x, ctx, entry, writes_cache=True):
        left, right = (self.sides[n](x, ctx, entry, writes_cache) for n in self.SIDES)
        if self.spec.join == "scaled_sum":
            return ops.scaled_sum(left, right, self.spec.left_scale, self.spec.right_scale)
        return ops.norm_pair_mean(left, right, self.gains["left"], self.gains["right"], self.spec.norm_eps)

    def weight_bytes(self):
        return sum(m.weight_bytes() for m in self.sides.values()) + bytes_of(*self.gains.values())
