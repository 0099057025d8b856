"""Position encodings. A position part owns a float32 table of inverse frequencies
that the rotation kernel multiplies by each token's position; no table means the
layer sees no positions at all (NoPE).

Reference: per-layer base with 0 = no rotation
(src/mlx_omnia/engine/models/muse_glimmer/layers/attention.py:39-40); half-split pairing
(i, i + d/2), angle pos * theta^(-2i/d), scale 1
(src/mlx_omnia/engine/core/attention.py:587-599,
src/mlx_omnia/engine/core/kernels/qkv_rope/epilogue.py:56-63).
"""

from __future__ import annotations

import math

import torch

from mlx_omnia_b200.parts.base import Position, register_position


_TABLES: dict[tuple, torch.Tensor] = {}


@register_position("rotary")
class Rotary(Position):
    """Rotary embedding over the first `dims` dims of each head.

    theta:   the base; inverse frequency i is theta^(-2i/dims), computed in float64 and
             rounded once to float32, so every consumer multiplies the same constants.
    pairing: which dims turn together: "half" pairs dim i with i + dims/2, "interleaved" pairs
             2i with 2i + 1. The table is the same; the mixer's kernel does the pairing, and a
             mixer says which one it implements.
    scaling: None, or YaRN's constants (factor, original, fast, slow): a pair that turns at least `fast` times
             over `original` positions keeps its frequency, one that turns at most `slow` times has it divided
             by `factor`, pairs in between are blended linearly by their index; cosine and sine are then
             multiplied by `amount` = 0.1 ln(factor) + 1 (a mixer says whether it applies an amount).
    """

    def __init__(self, dims: int, theta: float, pairing: str = "half",
                 scaling: tuple[float, float, float, float] | None = None) -> None:
        if pairing not in ("half", "interleaved"):
            raise ValueError(f"rotary pairing {pairing!r}")
        self.pairing = pairing
        if dims % 2 or dims <= 0:
            raise ValueError(f"rotary dims must be even and positive, got {dims}")
        if theta <= 0:
            raise ValueError(f"rotary theta must be positive, got {theta}")
        self.dims, self.theta = dims, float(theta)
        self.scaling = None if scaling is None else tuple(float(v) for v in scaling)
        if self.scaling is not None and (min(self.scaling) <= 0 or theta == 1):
            raise ValueError(f"rotary scaling takes positive numbers (and a theta other than 1), got {scaling}")
        self.amount = 1.0 if self.scaling is None else 0.1 * math.log(self.scaling[0]) + 1.0
        self._table = None

    def _inverse_frequencies(self) -> torch.Tensor:
        exponent = torch.arange(self.dims // 2, dtype=torch.float64) * (2.0 / self.dims)
        inv = torch.pow(torch.tensor(self.theta, dtype=torch.float64), -exponent)
        if self.scaling is None:
            return inv
        factor, original, fast, slow = self.scaling

        def index_of(turns: float) -> float:  # the (fractional) pair that turns so often over `original` positions
            return self.dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(self.theta))

        low = max(math.floor(index_of(fast)), 0)
        high = min(math.ceil(index_of(slow)), self.dims - 1)
        blend = ((torch.arange(self.dims // 2, dtype=torch.float64) - low) / max(high - low, 0.001)).clamp(0.0, 1.0)
        return inv / factor * blend + inv * (1.0 - blend)

    def load(self, tensors, runtime) -> None:
        super().load(tensors, runtime)
        # Layers of one base share one tensor: what kernels make from a table once per pass over the
        # layers (the angles of a step's positions) is then made once, not once per layer.
        key = (self.dims, self.theta, self.scaling, str(runtime.device))
        if key not in _TABLES:
            _TABLES[key] = self._inverse_frequencies().to(torch.float32).to(runtime.device)
        self._table = _TABLES[key]

    def table(self) -> torch.Tensor | None:
        return self._table


@register_position("none")
class NoPosition(Position):
    """The layer is not told where a token is."""

    def __init__(self) -> None:
        pass

    def table(self) -> None:
        return None
