"""Mixers with a recurrent state whose decay varies by channel and token.

``selective_scan`` (Mamba): one input projection laid out ``[x | z]``; x passes a short causal convolution (with bias)
and SiLU; from it come a low-rank step size, an input and an output vector, ``W_x x = [d | B | C]``,
``dt = softplus(W_dt d + b_dt)`` per channel.  Per channel c and state n, with ``A = -exp(A_log)``::

    S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c x_c B_n;   y_c = sum_n S[c, n] C_n + D_c x_c

The read-out is gated by ``silu(z)`` and projected.

``channel_delta`` (a delta rule with a decay and a removal rate per key channel): per head, with r, k, v projections of
the input, ``w = exp(-exp(-1/2) sigmoid(W_w2 tanh(W_w1 h) + w0))``, ``a = sigmoid(W_a h + b_a)`` and the unit key
``u = k / sqrt(sum(k^2) + 1e-6)``::

    S <- diag(w) S - (a * u) (u^T S) + k v^T   (the old S on the right);   o = S^T r

The read-out is RMS-normed per head, scaled by a weight over all heads, gated by ``sigmoid(W_g h)`` and projected.

Projections leave float32 (the products' accumulators); everything between them and the next product's input is
float32: convolution, activations, step sizes, decays, rates, unit norms, the state, gates and norms.  Both keep their
state in the cache manager's state slots and a step moves it on by the tokens it brings, however a prompt was cut.
"""

from __future__ import annotations

import torch

from ..config.model_spec import PartSpec
from .base import MIXERS, BuildContext, FreeSize, LayerRun, StateNeed, TensorSpec
from .linear import Linear, fuse_rows


@MIXERS.register("selective_scan")
class SelectiveScan:
    """params: ``inner`` (channels), ``state`` (numbers a channel keeps), ``dt_rank``, ``taps``.

    tensors (prefix +): ``in [2 inner, hidden]``, ``conv [inner, taps]``, ``conv.b [inner]``, ``x [dt_rank + 2 state,
    inner]``, ``dt [inner, dt_rank]``, ``dt.b [inner]``, ``A_log [inner, state]``, ``D [inner]``, ``o [hidden, inner]``."""

    graph_safe = True

    def __init__(self, proj, conv, conv_bias, select, step_up, vectors: dict, out, prm: dict, kernels) -> None:
        self.proj, self.conv, self.conv_bias, self.select, self.step_up = proj, conv, conv_bias, select, step_up
        self.vectors, self.out, self.kernels = vectors, out, kernels
        self.inner, self.state, self.rank, self.taps = self._sizes(prm)

    @staticmethod
    def _sizes(prm) -> tuple[int, int, int, int]:
        inner, state, rank, taps = (int(prm[n]) for n in ("inner", "state", "dt_rank", "taps"))
        if inner < 1 or rank < 1 or not 1 <= state <= 256:
            raise ValueError(f"inner {inner}, dt_rank {rank}, state {state}: at least 1 each, state at most 256")
        if taps < 1 or taps > 16:
            raise ValueError("the short convolution takes 1 to 16 taps")
        return inner, state, rank, taps

    @classmethod
    def tensor_specs(cls, spec: PartSpec, hidden_size: int) -> list[TensorSpec]:
        p = spec.prefix
        inner, state, rank, taps = cls._sizes(spec.params)
        return [
            TensorSpec(p + "in", (2 * inner, hidden_size)),
            TensorSpec(p + "conv", (inner, taps), "bias"), TensorSpec(p + "conv.b", (inner,), "bias"),
            TensorSpec(p + "x", (rank + 2 * state, inner)),
            TensorSpec(p + "dt", (inner, rank)), TensorSpec(p + "dt.b", (inner,), "bias"),
            TensorSpec(p + "A_log", (inner, state), "bias"), TensorSpec(p + "D", (inner,), "bias"),
            TensorSpec(p + "o", (hidden_size, inner)),
        ]

    @classmethod
    def cache_need(cls, spec: PartSpec):
        return None

    @classmethod
    def state_need(cls, spec: PartSpec):
        inner, state, _, taps = cls._sizes(spec.params)
        need = {"channels": StateNeed((state, inner), torch.float32)}
        if taps > 1:
            need["conv"] = StateNeed((taps - 1, inner), torch.float32)
        return need

    @classmethod
    def build(cls, spec: PartSpec, ctx: BuildContext) -> "SelectiveScan":
        p, w = spec.prefix, ctx.weights
        vectors = {n: w.vector(p + n) for n in ("dt.b", "D")}
        vectors["rates"] = (-torch.exp(w.vector(p + "A_log"))).t().contiguous()  # [state, inner]: channels side by side
        return cls(w.matrix(p + "in"), w.vector(p + "conv"), w.vector(p + "conv.b"), w.matrix(p + "x"), w.matrix(p + "dt"),
                   vectors, w.matrix(p + "o"), dict(spec.params), ctx.kernels)

    def forward(self, x: torch.Tensor, run: LayerRun):
        k = self.kernels
        tokens, inner, state, rank = x.shape[0], self.inner, self.state, self.rank
        y = k.linear_split(x, self.proj)  # float32 slices [S, T, 2 inner], added up by what reads them
        conv, conv_typed = k.short_conv(y[:, :, :inner], self.conv, self.conv_bias, run.state["conv"] if self.taps > 1 else None,
                            run.step, "silu", typed=True)
        select = k.linear_split(conv_typed, self.select)
        low = k.activation(select[:, :, :rank], "none", out_dtype=x.dtype)
        dt = k.linear_split(low, self.step_up)
        gated = torch.empty((tokens, inner), dtype=x.dtype, device=x.device)
        k.selective_scan(conv, dt, select[:, :, rank : rank + state], select[:, :, rank + state : rank + 2 * state],
                         y[:, :, inner:], self.vectors["rates"], self.vectors["D"], self.vectors["dt.b"],
                         run.state["channels"], run.step, gated)
        return k.linear_split(gated, self.out)


@MIXERS.register("channel_delta")
class ChannelDelta:
    """params: ``heads``, ``dim`` (of keys and values), ``eps`` (of the read-out norm).  The rank of the decay's
    projection is the checkpoint's.

    tensors (prefix +): ``r, k, v, g, a [heads * dim, hidden]``, ``a.b [heads * dim]``, ``w1 [rank, hidden]``,
    ``w2 [heads * dim, rank]``, ``w0 [heads * dim]``, ``norm [heads * dim]``, ``o [hidden, heads * dim]``."""

    graph_safe = True
    DEFAULT_RANK = 64

    def __init__(self, proj, decay_up, vectors: dict, out, prm: dict, kernels) -> None:
        self.proj, self.decay_up, self.vectors, self.out, self.kernels = proj, decay_up, vectors, out, kernels
        self.heads, self.dim = self._sizes(prm)
        self.eps = float(prm["eps"])

    @staticmethod
    def _sizes(prm) -> tuple[int, int]:
        heads, dim = int(prm["heads"]), int(prm["dim"])
        if heads < 1 or not 1 <= dim <= 256:
            raise ValueError(f"heads {heads}, dim {dim}: at least 1 each, dim at most 256")
        return heads, dim

    @classmethod
    def tensor_specs(cls, spec: PartSpec, hidden_size: int) -> list[TensorSpec]:
        p = spec.prefix
        heads, dim = cls._sizes(spec.params)
        n, rank = heads * dim, FreeSize(p + "rank", cls.DEFAULT_RANK)
        return [TensorSpec(p + name, (n, hidden_size)) for name in ("r", "k", "v", "g", "a")] + [
            TensorSpec(p + "a.b", (n,), "bias"), TensorSpec(p + "w1", (rank, hidden_size)), TensorSpec(p + "w2", (n, rank)),
            TensorSpec(p + "w0", (n,), "bias"), TensorSpec(p + "norm", (n,), "norm"), TensorSpec(p + "o", (hidden_size, n)),
        ]

    @classmethod
    def cache_need(cls, spec: PartSpec):
        return None

    @classmethod
    def state_need(cls, spec: PartSpec):
        heads, dim = cls._sizes(spec.params)
        return {"matrix": StateNeed((heads, dim, dim), torch.float32)}

    @classmethod
    def build(cls, spec: PartSpec, ctx: BuildContext) -> "ChannelDelta":
        p, w = spec.prefix, ctx.weights
        # One product for everything that reads the mixer's input: [r | k | v | rate | gate | low-rank decay].
        proj = fuse_rows([w.matrix(p + n) for n in ("r", "k", "v", "a", "g", "w1")])
        vectors = {n: w.vector(p + n) for n in ("a.b", "w0", "norm")}
        return cls(proj, w.matrix(p + "w2"), vectors, w.matrix(p + "o"), dict(spec.params), ctx.kernels)

    def forward(self, x: torch.Tensor, run: LayerRun):
        k = self.kernels
        n = self.heads * self.dim
        y = k.linear_split(x, self.proj)  # float32 slices [S, T, 5 n + rank], added up by what reads them
        low = k.activation(y[:, :, 5 * n :], "tanh", out_dtype=x.dtype)
        decay = k.linear_split(low, self.decay_up)
        read = k.channel_delta(y[:, :, : 4 * n], decay, self.vectors["w0"], self.vectors["a.b"], run.state["matrix"], run.step,
                               self.heads, self.dim)
        normed = torch.empty((x.shape[0], n), dtype=x.dtype, device=x.device)
        k.gated_rmsnorm(read, y[:, :, 4 * n : 5 * n], self.vectors["norm"], self.eps, self.dim, False, normed, activation="sigmoid")
        return k.linear_split(normed, self.out)
