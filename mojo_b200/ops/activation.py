"""Activations with constants that differ between models."""
from __future__ import annotations

from typing import NamedTuple


class Glu(NamedTuple):
    """Gated linear unit g * sigmoid(alpha g) * (u + up_bias), after g = min(g, limit) and u = clamp(u, -limit, limit)."""
    limit: float = float("inf")
    alpha: float = 1.0
    up_bias: float = 0.0


SWIGLU = Glu()
# max(g, 0) * u: so steep a sigmoid is a step
REGLU = Glu(alpha=1e30)
