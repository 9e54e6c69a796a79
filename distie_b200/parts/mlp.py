"""Dense feed-forwards, no biases: SwiGLU ``down(silu(gate(x)) * up(x))``, its capped form, and ``activated``
``down(act(up(x)))``.

Formula of the reference (worker/src/inference/qwen2/model.py:228-236).  Gate and
up are one product against the row-stacked weight ``[2 * inter, hidden]``.
``none`` is the feed-forward of a layer that has none: it declares nothing and adds nothing.
"""

from __future__ import annotations

import math

import torch

from ..config.model_spec import PartSpec
from .base import FEED_FORWARDS, BuildContext, LayerRun, TensorSpec
from .linear import Linear, fuse_rows


@FEED_FORWARDS.register("swiglu")
class SwiGluFeedForward:
    """params: ``intermediate_size``; optional ``names``: what the names of the gate, up and down matrices add to
    the prefix (default ``gate_proj.weight``, ``up_proj.weight``, ``down_proj.weight``); ``limit`` (None: none): the
    hidden activation is the capped form ``g' sigmoid(1.702 g') (u' + 1)`` with ``g' = min(g, limit)`` and ``u' = clamp(u,
    -limit, limit)`` (see :meth:`KernelSet.linear_glu`)."""

    _NAMES = ("gate_proj.weight", "up_proj.weight", "down_proj.weight")

    def __init__(self, gate_up: Linear, down: Linear, inter: int, kernels, limit: float | None = None) -> None:
        self.gate_up = gate_up
        self.down = down
        self.inter = inter
        self.limit = limit
        self.kernels = kernels

    @classmethod
    def tensor_specs(cls, spec: PartSpec, hidden_size: int) -> list[TensorSpec]:
        p, inter = spec.prefix, int(spec.params["intermediate_size"])
        gate, up, down = spec.params.get("names", cls._NAMES)
        return [
            TensorSpec(p + gate, (inter, hidden_size)),
            TensorSpec(p + up, (inter, hidden_size)),
            TensorSpec(p + down, (hidden_size, inter)),
        ]

    @classmethod
    def build(cls, spec: PartSpec, ctx: BuildContext) -> "SwiGluFeedForward":
        p, w = spec.prefix, ctx.weights
        gate, up, down = spec.params.get("names", cls._NAMES)
        gate_up = fuse_rows([w.matrix(p + gate), w.matrix(p + up)])
        return cls(
            Linear(gate_up, None, ctx.kernels),
            Linear(w.matrix(p + down), None, ctx.kernels),
            int(spec.params["intermediate_size"]),
            ctx.kernels,
            cls._limit(spec),
        )

    @staticmethod
    def _limit(spec: PartSpec) -> float | None:
        limit = spec.params.get("limit")
        if limit is not None and float(limit) <= 0:
            raise ValueError(f"limit must be positive, got {limit}")
        return float(limit) if limit is not None else None

    def forward(self, x: torch.Tensor, run: LayerRun) -> torch.Tensor:
        # The down product's float32 slices are summed by the norm that follows (or by the stream).
        k = self.kernels
        hidden = k.linear_swiglu(x, self.gate_up.weight) if self.limit is None else k.linear_glu(x, self.gate_up.weight, self.limit)
        return k.linear_split(hidden, self.down.weight)


def _softplus(z: float) -> float:
    return max(z, 0.0) + math.log1p(math.exp(-abs(z)))


@FEED_FORWARDS.register("activated")
class ActivatedFeedForward:
    """``down(act(up(x)))`` with the activation on the product's float32 accumulators.  params:
    ``intermediate_size``, ``activation`` (``"relu2"``: the square of ReLU; ``"gelu"``: the exact one; ``"xielu"``: a
    parabola right of zero and an exponential left of it, see :meth:`KernelSet.linear_act`); optional ``names``: what
    the names of the up and down matrices add to the prefix (default ``up_proj.weight``, ``down_proj.weight``);
    ``numbers`` (xielu): what the name of its two learned numbers ``[p, q]`` adds to the prefix, whose factors are
    ``softplus(p)`` and ``1/2 + softplus(q)``."""

    _NAMES = ("up_proj.weight", "down_proj.weight")
    _ACTIVATIONS = ("relu2", "gelu", "xielu")

    def __init__(self, up: torch.Tensor, down: torch.Tensor, activation: str, kernels, numbers=None) -> None:
        self.up, self.down, self.activation, self.kernels, self.numbers = up, down, activation, kernels, numbers

    @classmethod
    def _check(cls, spec: PartSpec) -> None:
        if spec.params.get("activation") not in cls._ACTIVATIONS:
            raise ValueError(f"activation {spec.params.get('activation')!r}: one of {cls._ACTIVATIONS}")
        if (spec.params["activation"] == "xielu") != bool(spec.params.get("numbers")):
            raise ValueError("xielu, and no other activation, has two learned numbers")

    @classmethod
    def tensor_specs(cls, spec: PartSpec, hidden_size: int) -> list[TensorSpec]:
        cls._check(spec)
        p, inter = spec.prefix, int(spec.params["intermediate_size"])
        up, down = spec.params.get("names", cls._NAMES)
        specs = [TensorSpec(p + up, (inter, hidden_size)), TensorSpec(p + down, (hidden_size, inter))]
        if spec.params.get("numbers"):
            specs.append(TensorSpec(p + spec.params["numbers"], (2,), "bias"))
        return specs

    @classmethod
    def build(cls, spec: PartSpec, ctx: BuildContext) -> "ActivatedFeedForward":
        cls._check(spec)
        p, w = spec.prefix, ctx.weights
        up, down = spec.params.get("names", cls._NAMES)
        numbers = None
        if spec.params.get("numbers"):
            right, left = w.vector(p + spec.params["numbers"]).double().tolist()
            numbers = (_softplus(right), 0.5 + _softplus(left))
        return cls(w.matrix(p + up), w.matrix(p + down), spec.params["activation"], ctx.kernels, numbers)

    def forward(self, x: torch.Tensor, run: LayerRun) -> torch.Tensor:
        return self.kernels.linear_split(self.kernels.linear_act(x, self.up, self.activation, self.numbers), self.down)


@FEED_FORWARDS.register("none")
class NoFeedForward:
    @classmethod
    def tensor_specs(cls, spec: PartSpec, hidden_size: int) -> list[TensorSpec]:
        return []

    @classmethod
    def build(cls, spec: PartSpec, ctx: BuildContext) -> "NoFeedForward":
        return cls()

    def forward(self, x: torch.Tensor, run: LayerRun):
        return None
