"""Average over depth: behind every layer the residual becomes a learned weighted sum of all states so far.

With ``X_0`` the embedding output and ``X_(i+1)`` the result of the i-th layer of the run order (before its average)::

    x <- sum_(j = 0 .. i+1) w_i[j] * X_j

``w_i`` (``i + 2`` numbers) is the tensor that :attr:`LayerSpec.average` names.  The states are those of the step's own
tokens: nothing is carried from one step to the next.  They live in one float32 buffer ``[layers, T, hidden]``; the sum
itself is left pending (:class:`~distie_b200.kernels.interface.Averaged`) and done by the norm kernel that follows.
"""

from __future__ import annotations

import torch

from ..config.model_spec import ModelSpec
from ..kernels.interface import Averaged
from .base import BuildContext, ResidualStream, TensorSpec


class DepthAverage:
    def __init__(self, weights: list[torch.Tensor]) -> None:
        self.weights = weights  # in the run order
        self._history: torch.Tensor | None = None

    @staticmethod
    def tensor_specs(spec: ModelSpec) -> list[TensorSpec]:
        if not spec.depth_averaged:
            return []
        return [TensorSpec(spec.layers[call.layer].average, (index + 2,), "average") for index, call in enumerate(spec.order)]

    @classmethod
    def build(cls, spec: ModelSpec, ctx: BuildContext) -> "DepthAverage":
        return cls([ctx.weights.vector(t.name) for t in cls.tensor_specs(spec)])

    def start(self, stream: ResidualStream) -> None:
        """The embedding output becomes the first state of the step."""
        first = stream.settle()
        self._history = torch.empty((len(self.weights), *first.shape), dtype=torch.float32, device=first.device)
        self._history[0].copy_(first)

    def after(self, index: int, stream: ResidualStream) -> None:
        stream.pending = Averaged(stream.pending, self._history, index + 1, self.weights[index])
        if index + 1 == len(self.weights):
            self._history = None  # what is pending holds on to it
