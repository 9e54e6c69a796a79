"""The set of operations the parts are written against.

Parts never call a kernel by name; they are handed a :class:`KernelSet` when they
are built.  The engine has two of them, both in :mod:`distie_b200.kernels.device`:
the bfloat16 set that serving uses and the float32 set in which every product,
sum and exponential is a true 32-bit operation.  Tests pass a third, written with
plain tensor operations, to check each kernel against and to run the engine's
bookkeeping on a machine without a GPU; the product never falls back to it.

Shapes (``T`` tokens of this step, ``B`` requests of this step):

``StepTensors``   the step's metadata on the device, all int32
    token_ids [T], positions [T], token_seq [T] (batch row of each token),
    seq_seat [B] (seat = row of the block tables and of the state slots).
``KvSlot``        one cache slot of one group
    k  [pages, kv_heads, page_size, head_dim], v  [pages, kv_heads, page_size, value_dim];
    block_table [seats, width] int32.  In a group whose values lie inside its keys (attention through
    a latent) ``v`` is a view of the first ``value_dim`` columns of ``k``.

Which keys a token sees: all keys up to its own position (``first_visible``), the last
``window`` of them, or those of its own ``chunk`` (positions ``chunk * n .. chunk * (n + 1) - 1``);
beside a window, the request's first ``keep_first`` positions when a layer keeps them.
"""

from __future__ import annotations

from abc import ABC, abstractmethod
from dataclasses import dataclass, field

import torch


Q_TILE = 128  # tokens per tile of StepTensors.q_tiles


@dataclass
class StepTensors:
    token_ids: torch.Tensor
    positions: torch.Tensor
    token_seq: torch.Tensor
    seq_seat: torch.Tensor
    num_tokens: int
    num_seqs: int
    num_decode_tokens: int  # the first this-many tokens are single-token rows
    max_kv_len: int = 0  # bound on the keys any token sees; a captured step uses a fixed bound
    q_tiles: torch.Tensor | None = None  # [n, 2] int32: (first token, rows <= Q_TILE) of each tile of the
    num_q_tiles: int = 0                 # multi-token entries; a tile holds consecutive tokens of one request
    derived: dict = field(default_factory=dict)  # what a kernel set made of this step once and its layers share


@dataclass
class KvSlot:
    k: torch.Tensor
    v: torch.Tensor
    block_table: torch.Tensor
    page_size: int
    num_pages: int


def first_visible(position: int, window: int | None = None, chunk: int | None = None) -> int:
    """The oldest key the token at ``position`` sees (it sees every key from there to itself)."""
    first = 0
    if window:
        first = max(first, position - int(window) + 1)
    if chunk:
        first = max(first, position // int(chunk) * int(chunk))
    return first


@dataclass
class Terms:
    """A sum that is still to be done: ``sum_i scale_i * tensor_i``, each tensor ``[T, hidden]`` or float32
    slices ``[S, T, hidden]`` (see :meth:`KernelSet.linear_split`).  A block whose sublayers all read one norm
    hands its sublayers' outputs over like this, and the norm kernel that follows adds them to the residual."""

    items: list  # of (tensor, scale)

    @classmethod
    def of(cls, value, scale: float = 1.0) -> "Terms":
        if isinstance(value, Terms):
            return cls([(t, s * scale) for t, s in value.items])
        return cls([(value, float(scale))])

    def __add__(self, other: "Terms") -> "Terms":
        return Terms(self.items + Terms.of(other).items)

    def flat(self) -> list:
        """``(float32 [T, hidden] matrix, scale)`` pairs: every slice on its own."""
        out = []
        for tensor, scale in self.items:
            if tensor.dim() == 3:
                out += [(tensor[i], scale) for i in range(tensor.shape[0])]
            else:
                out.append((tensor if tensor.dtype == torch.float32 else tensor.float(), scale))
        return out

    def total(self) -> torch.Tensor:
        """The sum itself, float32 ``[T, hidden]``, in the order of the items."""
        total = None
        for tensor, scale in self.flat():
            part = tensor if scale == 1.0 else tensor * scale
            total = part if total is None else total + part
        return total


@dataclass
class Normed:
    """A sublayer's output that is normalised before it joins the residual: ``rms_norm(sum of terms) * weight``.

    ``value`` is what a mixer or feed-forward returns (a matrix, float32 slices or :class:`Terms`); ``weight`` is
    the float32 scale of the norm (an offset the checkpoint leaves out is already added) and ``eps`` its epsilon.
    The norm kernel that follows does the sum, this norm, the addition to the residual and its own norm in one pass."""

    value: object
    weight: torch.Tensor
    eps: float


@dataclass
class Averaged:
    """A layer's end in a decoder that averages over depth.  ``value`` (a :class:`Normed`, :class:`Terms`, a tensor or
    None) is still to be added to the residual, which gives the layer's own result ``X``; ``X`` is then kept as
    ``history[count]`` (when there is room: the last one is read by nobody) and the residual becomes
    ``sum_(j < count) weights[j] * history[j] + weights[count] * X``.  ``history [slots, T, hidden]`` is float32, like
    ``weights [count + 1]``.  The norm kernel that follows does all of it beside its own norm."""

    value: object
    history: torch.Tensor
    count: int
    weights: torch.Tensor

    def close(self, state: torch.Tensor) -> torch.Tensor:
        """The average, given the layer's own result (plain tensor operations)."""
        if self.count < self.history.shape[0]:
            self.history[self.count].copy_(state)
        out = self.weights[self.count] * state
        for j in range(self.count):
            out = out + self.weights[j] * self.history[j]
        return out


@dataclass(frozen=True)
class RotaryTable:
    """What the fused rotation kernel needs of a rotary position encoding."""

    inv_freq: torch.Tensor  # [rotary_dim / 2] float32
    rotary_dim: int
    interleaved: bool = False
    factor: float = 1.0  # cos and sin are multiplied by it (the attention factor of scaled rotary encodings)


class KernelSet(ABC):
    dtype: torch.dtype
    device: torch.device

    @abstractmethod
    def embed(self, step: StepTensors, table: torch.Tensor, residual: torch.Tensor) -> None:
        """residual[t] = table[token_ids[t]] as float32."""

    @abstractmethod
    def add_rmsnorm(self, delta, residual, weight, eps: float, out, rows_index=None) -> None:
        """residual += delta (float32, kept), out = weight * cast(residual * rsqrt(mean sq + eps)).

        ``delta`` is ``[T, hidden]`` in the set's dtype, or ``[S, T, hidden]`` float32 slices as
        :meth:`linear_split` returns them, which are added up in the same kernel.
        """

    @abstractmethod
    def linear(self, x, weight, bias=None, out_dtype=None):
        """x @ weight.T (+ bias); weight is [out, in]."""

    def linear_split(self, x, weight):
        """``x @ weight.T`` as float32 slices ``[S, T, out]`` whose sum over ``S`` is the product.

        A set that splits the reduction of a skinny product over several thread blocks returns
        the slices as they are and leaves the sum to the consumer (``add_rmsnorm``,
        ``rope_kv_write``), which saves the product a round of synchronisation.  The default is
        one slice.
        """
        return self.linear(x, weight, None, torch.float32).unsqueeze(0)

    @abstractmethod
    def swiglu(self, gate_up, out) -> None:
        """out = silu(gate_up[:, :I]) * gate_up[:, I:]."""

    def linear_swiglu(self, x, weight):
        """silu(x Wg^T) * (x Wu^T) for weight = [Wg; Wu] stacked along the rows; sets may fuse it."""
        gate_up = self.linear(x, weight)
        out = torch.empty((x.shape[0], weight.shape[0] // 2), dtype=gate_up.dtype, device=x.device)
        self.swiglu(gate_up, out)
        return out

    @abstractmethod
    def rope_kv_write(self, qkv, step: StepTensors, kv: KvSlot | None, rotary: RotaryTable | None,
                      num_heads: int, num_kv_heads: int, head_dim: int, bias=None, q_out=None) -> None:
        """Rotate q and k, store k and v of the new tokens in their pages (if kv).

        ``qkv`` is ``[T, (heads + 2 kv_heads) * head_dim]`` in the set's dtype with q rotated in
        place, or float32 slices ``[S, T, ...]`` of the projection (see :meth:`linear_split`), in
        which case the slices are summed, ``bias`` is added and the rotated q is written to
        ``q_out [T, heads * head_dim]``.
        """

    def qkv_rope_write(self, x, weight, bias, step: StepTensors, kv: KvSlot | None, rotary: RotaryTable | None,
                       num_heads: int, num_kv_heads: int, head_dim: int, q_out) -> None:
        """The q/k/v projection with what follows it: ``x @ weight.T + bias``, q and k rotated, q to
        ``q_out`` and k and v into their pages (if kv).  The default is the two ops after one another;
        a set may do it in the product's epilogue."""
        slices = self.linear_split(x, weight)
        self.rope_kv_write(slices, step, kv, rotary, num_heads, num_kv_heads, head_dim, bias=bias, q_out=q_out)

    def qkv_attention(self, x, weight, bias, step: StepTensors, kv: KvSlot, writes_cache: bool,
                      rotary: RotaryTable | None, num_heads: int, num_kv_heads: int, head_dim: int,
                      window: int | None, scale: float, out, chunk: int | None = None) -> None:
        """From the mixer's input to the attention's output: the q/k/v projection, bias, rotation, the new
        keys and values into their pages (if ``writes_cache``) and attention over the pages into ``out``.
        The default is the ops after one another; a set may merge them for some steps."""
        q = torch.empty((x.shape[0], num_heads * head_dim), dtype=out.dtype, device=x.device)
        self.qkv_rope_write(x, weight, bias, step, kv if writes_cache else None, rotary, num_heads, num_kv_heads,
                            head_dim, q)
        self.attention(q, out, step, kv, num_heads, num_kv_heads, head_dim, window, scale, chunk)

    @abstractmethod
    def attention(self, qkv, out, step: StepTensors, kv: KvSlot, num_heads: int, num_kv_heads: int,
                  head_dim: int, window: int | None, scale: float, chunk: int | None = None,
                  keep_first: int = 0, softcap: float = 0.0, sink=None) -> None:
        """Causal attention of every token over its request's pages, optionally only over the last
        ``window`` keys or over the keys of the token's own ``chunk``.  With a window, ``keep_first`` keeps
        the request's first that-many positions visible to every later token, at their true positions.
        The size of a value is the last dimension of ``kv.v`` and may differ from ``head_dim``; ``out`` is
        ``[T, heads * value size]``.  ``softcap > 0``: a score ``s = q . k * scale`` becomes ``softcap * tanh(s /
        softcap)``.  ``sink [heads]`` (float32): the softmax's denominator also holds ``exp(sink_h)``, a term with
        no key and no value that is neither scaled nor capped."""

    def qkv_norm_write(self, qkv, bias, step: StepTensors, kv: KvSlot | None, rotary: RotaryTable | None,
                       num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int, norm_eps: float | None,
                       q_weight, k_weight, q_temp, q_out) -> None:
        """``qkv`` is the float32 projection ``[T, heads * head_dim + kv_heads * (head_dim + value_dim)]`` (or the
        slices of a split product; more columns behind these are not read) and ``bias`` its float32 bias or None.
        With ``norm_eps`` every head of q and k is divided by its root mean square over ``head_dim`` (eps inside
        the root) and, with ``q_weight`` / ``k_weight`` (float32 ``[head_dim]``), multiplied by it; THEN q and k are
        rotated (``rotary``); with ``q_temp = (coef, every)`` q at position p is multiplied by
        ``1 + coef * ln(floor((p + 1) / every) + 1)`` (``every`` a positive number).  k and v go to their pages (if ``kv``; values may have
        another size than keys) and q to ``q_out [T, heads * head_dim]`` in the set's dtype.  All float32."""
        raise NotImplementedError

    # -- norms around a sublayer, keys that are their own values, routed feed-forwards -----------------------------
    def norm_add_rmsnorm(self, delta, delta_weight, delta_eps: float, residual, weight, eps: float, out,
                         rows_index=None) -> None:
        """``d = sum of delta's terms`` (float32); ``residual += d * rsqrt(mean(d^2) + delta_eps) * delta_weight``
        (kept); ``out = cast(residual * rsqrt(mean(residual^2) + eps) * weight)``, everything in float32 up to the
        one cast.  ``delta``: None (nothing is added), a matrix, float32 slices or :class:`Terms`; with
        ``delta_weight`` None the sum is added as it is.  With ``rows_index`` only those rows are made and the
        residual stays as it is.  ``out`` None: only the residual is moved on."""
        raise NotImplementedError

    def average_add_rmsnorm(self, ahead: Averaged, residual, weight, eps: float, out, rows_index=None) -> None:
        """What :class:`Averaged` describes, then ``out = cast(residual * rsqrt(mean(residual^2) + eps) * weight)`` of
        the averaged residual (kept), all float32 up to the one cast.  With ``rows_index`` only those rows are made and
        residual and history stay as they are.  ``out`` None: only residual and history are moved on."""
        raise NotImplementedError

    def qk_rope_norm_write(self, qk, bias, step: StepTensors, kv: KvSlot | None, rotary: RotaryTable | None,
                           num_heads: int, num_kv_heads: int, head_dim: int, norm_eps: float | None, q_out) -> None:
        """For layers whose values are their keys: ``qk`` is the projection ``[T, (heads + kv_heads) * head_dim]``
        (float32, or the float32 slices of a split product) and ``bias`` its float32 bias or None.  The key with
        its bias, before anything else is done to it, is stored as the value; q and k are rotated (``rotary``),
        then, with ``norm_eps`` not None, each head is divided by its root mean square over ``head_dim``; k goes to
        its page (if ``kv``) and q to ``q_out [T, heads * head_dim]`` in the set's dtype.  All arithmetic float32."""
        raise NotImplementedError

    def activation(self, x, kind: str = "silu", scale: float = 1.0, scaled_columns: int = 0, out_dtype=None):
        """A matrix ``[T, n]`` (float32, or of ``out_dtype``) out of ``x`` (float32, any row stride, or slices):
        ``act(x)`` with ``kind`` ``"silu"``, ``"tanh"`` or ``"none"``, the first ``scaled_columns`` columns also times
        ``scale``."""
        raise NotImplementedError

    def exp_gate_scan(self, log_in, log_forget, in_bias, forget_bias, cap: float, state, step: StepTensors):
        """Exponential gates with a running maximum, per head and request, float32:

        ``i = cap * tanh((log_in + in_bias) / cap)``; ``f = logsigmoid(cap * tanh((log_forget + forget_bias) / cap))``;
        ``m_t = max(f_t + m_(t-1), i_t)``; returns ``(keep, take, floor)``, each ``[T, heads]``:
        ``keep = exp(f + m_(t-1) - m_t)``, ``take = exp(i - m_t)``, ``floor = exp(-m_t)``.
        ``log_in, log_forget [T, heads]`` float32 (or slices); ``state [seats, heads]`` holds m (0 at a request's
        start) and is moved on by the step's tokens."""
        raise NotImplementedError

    def stabilized_readout(self, read, floor, heads: int, value_dim: int):
        """``read [T, heads * (value_dim + 1)]`` is the read-out of a recurrence whose last column per head is the
        normaliser ``n . q``: returns float32 ``[T, heads * value_dim]`` with head h of token t divided by
        ``max(|n . q|, floor[t, h]) + 1e-6``."""
        raise NotImplementedError

    def route_top(self, x, router, top: int, scoring: str = "sigmoid", groups: tuple[int, int] | None = None,
                  weight_scale: float = 1.0, extra_rows: int = 0, correction=None, normalise: bool = False,
                  logit_bias=None):
        """The ``top`` experts of every token: logits ``x @ router.T`` (``router [experts, hidden]``) accumulated in
        float32 -> ``(ids [T, top] int32, weights [T, top] float32)``, ``weights`` the chosen experts' scores
        (``sigmoid(logit)``, not renormalised) times ``weight_scale``, the largest first, ties to the lower index.

        ``groups = (count, keep)``: the experts form ``count`` equal groups of neighbours; a group's score is the
        sum of its two largest scores (of its one score, for groups of one), and only experts of the ``keep`` groups
        with the largest scores (ties to the lower group) can be chosen.  With ``extra_rows`` the router matrix has
        that many more rows below the experts', which are no experts: their float32 logits ``[T, extra_rows]`` are
        returned as a third value (a gate that reads the same input, made in the same pass).

        ``scoring="softmax"``: the scores are a softmax over all experts' logits.  ``correction [experts]``
        (float32) is added to the scores for the choice only; the weights are the plain scores.  ``normalise``:
        the chosen scores are divided by their sum (+ 1e-20) before ``weight_scale``.
        ``scoring="softmax_chosen"``: the choice is made on the logits and the weights are the softmax over the chosen
        logits alone.  ``logit_bias [experts]`` (float32) is part of the logits."""
        raise NotImplementedError

    def routed_swiglu(self, x, ids, weights, gate_up, down, scale_input: bool = True, limit: float | None = None,
                      identity: int = 0):
        """Every token through its chosen experts: ``gate_up [experts, 2 ff, hidden]`` (gate rows, then up rows),
        ``down [experts, hidden, ff]``; expert e of pair (t, j) computes ``down_e (silu(gate_e z) * (up_e z))`` with
        ``z = weights[t, j] * x[t]`` (``scale_input``) or on ``x[t]`` with the result times the weight.  With a
        ``limit`` the hidden activation is the capped form of :meth:`linear_glu`.  Returns
        float32 slices ``[top, T, hidden]`` whose sum over the first axis is the routed output.  With ``identity = n``
        ids ``experts .. experts + n - 1`` stand for experts that return their input: such a pair's slice row is
        ``weights[t, j] * x[t]`` (``scale_input`` False only)."""
        raise NotImplementedError

    def linear_glu(self, x, weight, limit: float | None = None, row_gate=None):
        """A gated hidden layer: ``weight = [Wg; Wu]`` stacked along the rows, ``g = x Wg^T``, ``u = x Wu^T``
        (float32 accumulators).  ``limit`` None: ``silu(g) * u``; a number: the capped form
        ``g' = min(g, limit)``, ``u' = clamp(u, -limit, limit)``, ``g' * sigmoid(1.702 g') * (u' + 1)``.
        ``row_gate`` (float32 ``[T]`` logits, any stride, or slices ``[S, T]``): row t also times
        ``sigmoid(row_gate[t])``.  Returns ``[T, rows / 2]`` in the set's dtype."""
        raise NotImplementedError

    def linear_act(self, x, weight, kind: str = "relu2", numbers: tuple[float, float] | None = None):
        """``act(x @ weight.T)`` in the set's dtype, the activation applied to the float32 accumulators:
        ``"relu2"`` is ``max(z, 0)^2``; ``"gelu"`` is ``z (1 + erf(z / sqrt 2)) / 2``; ``"xielu"`` with ``numbers = (a,
        b)`` is ``a z^2 + z / 2`` right of zero and ``b (exp(z) - 1 - z) + z / 2`` left of it."""
        raise NotImplementedError

    def routed_act(self, x, ids, weights, up, down, kind: str = "gelu", numbers: tuple[float, float] | None = None):
        """Every token through its chosen experts of two matrices: ``up [experts, ff, hidden]``, ``down [experts,
        hidden, ff]``; pair (t, j) with expert e computes ``weights[t, j] * down_e act(up_e x[t])`` (``kind`` and
        ``numbers`` as in :meth:`linear_act`).  Returns float32 slices ``[top, T, hidden]`` whose sum over the first
        axis is the routed output."""
        raise NotImplementedError

    # -- attention through a latent: one shared key/value row per token, queries folded into the latent's space ------
    def latent_kv_write(self, proj, step: StepTensors, kv: KvSlot | None, rotary: RotaryTable | None, q_rank: int,
                        q_norm, kv_rank: int, kv_norm, rot_dim: int, eps: float, q_latent_out) -> None:
        """``proj`` is the float32 projection ``[T, q_rank (+ kv_rank + rot_dim)]`` (or its slices).  Columns
        ``[0, q_rank)`` divided by their root mean square (``eps`` inside the root) times ``q_norm`` go to
        ``q_latent_out [T, q_rank]`` in the set's dtype.  With ``kv`` the next ``kv_rank`` columns, normed the same
        way with ``kv_norm``, and the last ``rot_dim`` columns, rotated by ``rotary`` at the token's position and not
        normed, are stored side by side as the token's one row ``[kv_rank + rot_dim]`` of ``kv.k``.  All float32
        up to the stores.  Without ``kv`` the projection has the query columns only.  ``q_rank`` 0 (with ``q_norm`` and
        ``q_latent_out`` None): there is no query latent and the projection starts with the ``kv_rank`` columns."""
        raise NotImplementedError

    def latent_queries(self, q, up_keys, step: StepTensors, rotary: RotaryTable | None, num_heads: int, dim: int,
                       rot_dim: int):
        """``q`` is the float32 query projection ``[T, heads * (dim + rot_dim)]`` (or its slices), per head ``dim``
        plain columns and ``rot_dim`` columns to rotate; ``up_keys [heads, dim, kv_rank]`` maps a latent to a
        head's plain key.  Returns ``(folded [heads, T, kv_rank], rotated [T, heads, rot_dim])`` in the set's
        dtype: ``folded[h, t] = q_plain[t, h] @ up_keys[h]`` (so that ``folded . latent == q_plain . key``)."""
        raise NotImplementedError

    def latent_attention(self, folded, rotated, step: StepTensors, kv: KvSlot, num_heads: int, kv_rank: int,
                         rot_dim: int, scale: float, sink, out, window: int | None = None) -> None:
        """Causal softmax attention of every token over its request's rows ``[latent | rotated key part]`` of
        ``kv.k``, shared by all heads: score ``(folded[h, t] . latent_j + rotated[t, h] . part_j) * scale`` for every
        ``j <= position``; with ``sink [heads]`` (float32) the denominator also holds ``exp(sink_h)``;
        ``out[h, t] = sum_j weight_j latent_j`` (``[heads, T, kv_rank]``, the set's dtype).  Scores, softmax and the
        sum are float32.  With a ``window`` a token sees itself and the ``window - 1`` positions before it."""
        raise NotImplementedError

    def latent_values(self, mixed, up_values, gate, num_heads: int, value_dim: int):
        """``mixed [heads, T, kv_rank]`` (what :meth:`latent_attention` left), ``up_values [heads, kv_rank,
        value_dim]`` -> ``[T, heads * value_dim]`` in the set's dtype: head h of token t is ``mixed[h, t] @
        up_values[h]`` times ``sigmoid(gate[t, h])`` (``gate`` float32 ``[T, heads]``, any stride, or slices; None:
        no gate)."""
        raise NotImplementedError

    def latent_heads(self, q, up_keys, up_values, up_rows, gate, step: StepTensors, seqs, kv: KvSlot, rotary: RotaryTable | None,
                     num_heads: int, dim: int, rot_dim: int, value_dim: int, kv_rank: int, scale: float, sink,
                     window: int | None = None):
        """From the float32 query projection (as :meth:`latent_queries` takes it) to what the output projection reads,
        ``[T, heads * value_dim]``; the step's rows are in the cache already.  ``up_rows [heads * (dim + value_dim),
        kv_rank]``: all heads' key rows, then all heads' value rows (``up_keys`` and ``up_values`` hold the same numbers);
        ``seqs``: the step's requests as the host knows them (or None).  The default folds the queries into the latent's
        space; a set may instead expand the latents of long portions to keys and values of every head."""
        folded, rotated = self.latent_queries(q, up_keys, step, rotary, num_heads, dim, rot_dim)
        mixed = torch.empty((num_heads, step.num_tokens, kv_rank), dtype=folded.dtype, device=folded.device)
        self.latent_attention(folded, rotated, step, kv, num_heads, kv_rank, rot_dim, scale, sink, mixed, window)
        return self.latent_values(mixed, up_values, gate, num_heads, value_dim)

    # -- layer norm, gates, short convolutions and linear recurrences (layers with per-request state) --------
    # Where a float32 input is marked "or slices" it may also be ``[S, T, n]``, the slices of a split product
    # (:meth:`linear_split`) or a view of their columns: the op adds them up while it loads.
    def add_layernorm(self, delta, residual, weight, bias, eps: float, out, rows_index=None) -> None:
        """residual += delta (float32, kept); out = (residual - mean) / sqrt(var + eps) * weight + bias, with the
        variance the mean of the squared deviations.  ``delta``: None, ``[T, hidden]``, float32 slices
        ``[S, T, hidden]`` or :class:`Terms`.  With ``rows_index`` only those rows, residual kept."""
        raise NotImplementedError

    def add_dynamic_tanh(self, delta, residual, alpha: float, weight, bias, out, rows_index=None) -> None:
        """residual += delta (float32, kept); out = cast(tanh(alpha * residual) * weight + bias), float32 up to the one
        cast.  ``delta``: None, ``[T, hidden]``, float32 slices ``[S, T, hidden]`` or :class:`Terms`.  With ``rows_index``
        only those rows, residual kept."""
        raise NotImplementedError

    def kv_write(self, k, v, step: StepTensors, kv: KvSlot) -> None:
        """Store the new tokens' keys ``[T, kv_heads * head_dim]`` and values ``[T, kv_heads * value_dim]``
        (any float type, any row stride) in their pages: the write of layers that rotate nothing."""
        raise NotImplementedError

    def head_gate(self, x, logits, num_heads: int) -> None:
        """x ``[T, heads * d]`` in place: head h of token t times sigmoid(logits[t, h]) (float32 logits, or slices).
        With ``num_heads`` the number of columns (``d = 1``) the gate is element by element."""
        raise NotImplementedError

    def short_conv(self, x, weight, bias, state, step: StepTensors, activation: str = "silu", input_bias=None, typed: bool = False):
        """Causal convolution over time, per channel and per request: ``x [T, C]`` float32 (any row stride; or slices),
        ``weight [C, taps]`` whose last column multiplies the current token, ``state [seats, taps - 1, C]`` the
        request's last inputs (oldest first; zeros at a request's start), which the call moves on by the
        step's tokens.  Returns float32 ``[T, C]`` after the activation (``"silu"`` or ``"none"``).  ``input_bias [C]``
        (float32) is added to every input of the step before anything else (the state holds the sums; before a
        request's start the inputs are zeros, not the bias).  ``typed``: returns a pair, the same values
        in the set's dtype as the second, for a product that reads them."""
        raise NotImplementedError

    # -- recurrences whose decay varies by channel ------------------------------------------------------------------
    def selective_scan(self, x, dt, B, C, gate, rates, skip, dt_bias, state, step: StepTensors, out) -> None:
        """A diagonal state per channel and request, moved on token by token in float32: with ``d =
        softplus(dt[t, c] + dt_bias[c])``

        ``S[n, c] <- exp(d rates[n, c]) S[n, c] + d x[t, c] B[t, n]``;
        ``out[t, c] = (sum_n S[n, c] C[t, n] + skip[c] x[t, c]) * silu(gate[t, c])`` in the set's dtype.

        ``x [T, channels]``, ``dt, gate [T, channels]`` and ``B, C [T, states]`` float32 (any row stride; ``dt``, ``B``,
        ``C`` and ``gate`` or slices; ``B`` and ``C`` are views of one projection), ``rates [states, channels]`` the
        (negative) rates of decay, ``state [seats, states, channels]`` float32, read and written through each token's
        seat."""
        raise NotImplementedError

    def channel_delta(self, proj, decay, decay_bias, rate_bias, state, step: StepTensors, heads: int, dim: int):
        """A matrix state ``S [dim, dim]`` per head and request with a decay and a removal rate per key channel:

        ``S <- diag(w) S - (a * u) (u^T S) + k v^T`` (the old S on the right), ``o = S^T r``, ``u = k / sqrt(sum(k^2) +
        1e-6)``, ``w = exp(-exp(-1/2) sigmoid(decay + decay_bias))``, ``a = sigmoid(rate + rate_bias)``.

        ``proj [T, 4 * heads * dim (+ more)]`` float32 (or slices) holds ``[r | k | v | rate]``, each head by head;
        ``decay [T, heads * dim]`` float32 (or slices); the biases ``[heads * dim]``; ``state [seats, heads, dim, dim]``
        float32 (S transposed: value element, then key channel).  Returns float32 ``[T, heads * dim]``."""
        raise NotImplementedError

    def linear_recurrence(self, rule: str, q, k, v, decay, write, state, step: StepTensors, heads: int, groups: int,
                          key_dim: int, value_dim: int, decay_rate=None, decay_bias=None, skip=None,
                          unit_column: bool = False):
        """A matrix state ``S [key_dim, value_dim]`` per head and request, moved on token by token in float32:

        ``S <- g S;  u = write-term;  S <- S + k u^T;  o = S^T q (+ skip * v)``

        Head h reads q and k of group ``h // (heads / groups)``.  ``q, k [T, groups * key_dim]``,
        ``v [T, heads * value_dim]``, ``decay, write [T, heads]`` (or slices), all float32 with any row stride.

        ``rule="delta"``: q and k are made unit vectors per head first (``x / sqrt(sum x^2 + 1e-6)``, q also
        times ``key_dim**-0.5``); ``g = exp(-exp(decay_rate) * softplus(decay + decay_bias))``;
        ``u = sigmoid(write) * (v - S^T k)`` with the decayed S.
        ``rule="ssd"``: ``dt = softplus(write + decay_bias)``; ``g = exp(-exp(decay_rate) * dt)``; ``u = dt * v``;
        ``skip [heads]`` adds ``skip_h * v`` to the read-out (``decay`` is not read).
        ``rule="gated"``: nothing is normalised; ``g = decay[t, h]`` as given, or with ``decay`` None the constant
        ``decay_rate[h]``; ``u = write[t, h] * v``, or ``v`` with ``write`` None.  With ``unit_column`` the state has
        one more column per head than ``v`` has elements (``value_dim`` counts it), whose value is 1 for every
        token: it carries ``n <- g n + write k`` and its read-out ``n . q`` is the last column of each head.

        ``state`` is ``[seats, heads, value_dim, key_dim]`` float32 (S transposed), read and written through
        each token's seat.  Returns float32 ``[T, heads * value_dim]``.  A set may overwrite ``q`` and ``k``
        (with their unit vectors): the caller hands over buffers it no longer needs."""
        raise NotImplementedError

    def gated_rmsnorm(self, x, gate, weight, eps: float, group: int, gate_first: bool, out,
                      activation: str = "silu") -> None:
        """Root-mean-square norm over groups of ``group`` neighbouring columns of ``x [T, n]`` (float32) with
        a gate (float32, or slices; written ``silu`` below, ``activation="sigmoid"`` makes it ``sigmoid(gate)``): ``gate_first``: ``norm(x * silu(gate)) * weight``; else ``norm(x) * weight * silu(gate)``.
        ``weight`` is float32 of ``n`` elements, or fewer, then repeated (``weight[column % len]``); None: no weight."""
        raise NotImplementedError

    def rotate_heads(self, qk, step: StepTensors, rotary: RotaryTable | None, heads: int, key_dim: int, key_scale: float = 1.0):
        """``qk [T, 2 * heads * key_dim (+ more)]`` float32 (any row stride, or slices): q head by head, then k.  Returns
        float32 ``[T, n]`` of as many columns: q and k with each head's first ``rotary_dim`` elements rotated at the
        token's position, k then times ``key_scale``; the columns behind them as they are."""
        raise NotImplementedError

    def retention(self, qkv, gate, rotary: RotaryTable | None, key_scale: float, decay, state, step: StepTensors, heads: int,
                  key_dim: int, value_dim: int, weight, eps: float, activation: str, out) -> None:
        """From the float32 projection ``qkv [T, 2 * heads * key_dim + heads * value_dim]`` (or slices) of a linear
        attention with the constant ``decay [heads]`` to what its output projection reads: q and k rotated and k scaled
        (:meth:`rotate_heads`), the state moved on and read (:meth:`linear_recurrence`, rule ``"gated"``), the read-out
        normed and gated (:meth:`gated_rmsnorm`) into ``out [T, heads * value_dim]``.  ``weight`` None: every head is
        normed by itself and has no weight; else all heads are normed together and multiplied by it.  The default is
        the ops after one another; a set may merge them."""
        qk = heads * key_dim
        turned = self.rotate_heads(qkv, step, rotary, heads, key_dim, key_scale)
        read = self.linear_recurrence("gated", turned[:, :qk], turned[:, qk : 2 * qk], turned[:, 2 * qk :], None, None, state, step,
                                      heads, heads, key_dim, value_dim, decay_rate=decay)
        group = value_dim if weight is None else heads * value_dim
        self.gated_rmsnorm(read, gate, weight, eps, group, False, out, activation=activation)

    @abstractmethod
    def sample(self, logits, temperatures, uniforms, out_tokens) -> None:
        """Arg-max for rows with temperature <= 0, inverse-CDF draw at uniforms[row] otherwise."""

    def check_errors(self) -> None:
        """Raise if a kernel of an earlier launch reported a bad index (after a synchronise)."""
