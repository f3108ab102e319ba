"""What every layer part has in common: named parameters with stated shapes, set once after loading.

A part is built from its spec and a working dtype, says which tensors it wants
(``param_specs``), receives them (``set_params``) and then computes.  It never
learns which model it sits in: tensor names in a checkpoint are the layer spec's
business, sizes and constants arrive through the part's own spec.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch


@dataclass(frozen=True)
class Role:
    """What a kind of tensor is drawn from in the random-weights mode (``mean``, ``std``) and how it is
    placed on the device: ``keep_32bit`` tensors that the checkpoint stores in 32-bit stay so (the
    others are cast to the working type); ``always_32bit`` tensors are float32 on the device however
    they are stored (what enters a 32-bit computation: norm parameters, stream weights, biases that a
    kernel adds in float)."""

    mean: float
    std: float
    keep_32bit: bool = False
    always_32bit: bool = False


#: the roles a parameter can have.  ``matrix``: a projection, N(0, 0.02), working type.  ``gain``: a
#: norm's scale, 1 + N(0, 0.1).  ``bias``: an additive term, N(0, 0.02).  ``state``: a per-channel
#: constant of a recurrence (a decay, a time step, a short convolution), N(0, 0.1), kept in 32-bit when
#: stored so.  A part with another kind of tensor registers its role; an unknown role is an error,
#: never silently a matrix.
ROLES = {
    "matrix": Role(0.0, 0.02),
    "gain": Role(1.0, 0.1, keep_32bit=True),
    "bias": Role(0.0, 0.02, keep_32bit=True),
    "state": Role(0.0, 0.1, keep_32bit=True),
    # float32 on the device whatever the checkpoint stores
    "gain32": Role(1.0, 0.1, always_32bit=True),
    "bias32": Role(0.0, 0.02, always_32bit=True),
    "slope": Role(0.5, 0.1, always_32bit=True),          # the scalar inside a Dynamic Tanh
    "vector32": Role(0.0, 0.1, always_32bit=True),       # small learnt vectors (lambda's factors)
    "stream_weight": Role(0.25, 0.2, always_32bit=True),  # how streams are read, written and mixed
    "gain_offset": Role(0.0, 0.1, always_32bit=True),    # a norm's gain stored around zero (gain - 1)
    "shift": Role(0.5, 0.2, always_32bit=True),          # how much of the previous token a mix takes
    "floor": Role(0.4, 0.1, always_32bit=True),          # the lower bound of a forget gate
    "matrix32": Role(0.0, 0.02, always_32bit=True),      # a small projection computed in 32-bit (a router)
}


def register_role(name: str, role: Role) -> None:
    ROLES[name] = role


def role_of(name: str) -> Role:
    try:
        return ROLES[name]
    except KeyError:
        raise ValueError(f"no tensor role {name!r} is registered (known: {', '.join(sorted(ROLES))})") from None


@dataclass(frozen=True)
class ParamSpec:
    """A parameter's shape and its ``role`` (see ``ROLES``)."""

    shape: tuple
    role: str = "matrix"

    def __post_init__(self):
        role_of(self.role)


class Part:
    def __init__(self, spec, dtype):
        self.spec = spec
        self.dtype = dtype

    def param_specs(self) -> dict:
        return {}

    def set_params(self, params: dict) -> None:
        if params:
            raise ValueError(f"{type(self).__name__} takes no parameters")

    def weight_bytes(self) -> int:
        """Bytes of parameters one step reads (for the bandwidth account)."""
        return 0


def bytes_of(*tensors) -> int:
    return sum(t.numel() * t.element_size() for t in tensors if isinstance(t, torch.Tensor))
