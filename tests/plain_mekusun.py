"""A plain, slow Mekusun decoder: one function per mechanism, whole sequences, no cache.

Written from the design's equations only; it shares no code with the engine.  A sequence is run from its first
token, token by token where the design has a recurrence, so it is the oracle for every way of cutting and batching.

Notation: ``h`` is a mixer's input ``[T, width]``; weights are ``[out, in]`` and applied as ``h @ W.T``; ``w`` maps a
tensor name to its tensor; ``cfg`` is the dictionary of ``config.json``.
"""

from __future__ import annotations

import math

import torch


STORED = None  # a torch dtype: what an engine of that type hands from one product to the next is rounded to it


def stored(x):
    """``x`` as a 16-bit engine stores it between two products; unchanged unless :func:`stored_as` is active."""
    return x if STORED is None else x.to(STORED).to(x.dtype)


class stored_as:
    """``with stored_as(torch.bfloat16): forward(...)``: the plain implementation with the roundings of a 16-bit engine
    (everything else stays in the precision of the call): what such an engine may lose, and nothing more."""

    def __init__(self, dtype):
        self.dtype = dtype

    def __enter__(self):
        global STORED
        self.before, STORED = STORED, self.dtype

    def __exit__(self, *exc):
        global STORED
        STORED = self.before


# -- element by element ---------------------------------------------------------------------------------------
def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.where(z > 0, z + torch.log1p(torch.exp(-z.abs())), torch.log1p(torch.exp(torch.minimum(z, torch.zeros_like(z)))))


def erf_gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def xielu(z, p, q):
    """Two learned numbers: the quadratic part right of zero has factor ``softplus(p)``, the exponential part left of
    zero ``1/2 + softplus(q)``; both branches have slope 1/2 at zero."""
    right = softplus(p) * z * z + 0.5 * z
    left = (0.5 + softplus(q)) * (torch.expm1(torch.clamp(z, max=0.0)) - z) + 0.5 * z
    return torch.where(z > 0, right, left)


# -- norms ------------------------------------------------------------------------------------------------------
def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def zero_centred_norm(x, weight, eps):
    """RMS norm whose weight is stored around zero."""
    return rms_unit(x, eps) * (1.0 + weight)


def normed_input(x, weight, eps):
    """What a sublayer reads: the norm of the residual, as the engine stores it."""
    return stored(zero_centred_norm(x, weight, eps))


def depth_average(states, weights):
    """``sum_j weights[j] * states[j]`` over the embedding output and every layer's result so far."""
    out = torch.zeros_like(states[0])
    for j, state in enumerate(states):
        out = out + weights[j] * state
    return out


# -- selective scan -----------------------------------------------------------------------------------------------
def causal_conv(x, weight, bias):
    """``y[t, c] = bias[c] + sum_j weight[c, taps-1-j] x[t-j, c]``; inputs before the start are zero."""
    taps = weight.shape[1]
    out = torch.zeros_like(x) + bias
    for t in range(x.shape[0]):
        for j in range(min(taps, t + 1)):
            out[t] = out[t] + weight[:, taps - 1 - j] * x[t - j]
    return out


def selective_scan(x, dt, B, C, A, D):
    """``x, dt [T, channels]``, ``B, C [T, state]``, ``A [channels, state]`` (negative), ``D [channels]``."""
    S = torch.zeros_like(A)
    out = torch.zeros_like(x)
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out[t] = S @ C[t] + D * x[t]
    return out


def mamba_mixer(h, w, p, m, eps):
    inner, rank, state = m["inner"], m["dt_rank"], m["state"]
    both = h @ w[p + "in"].T
    x = silu(causal_conv(both[:, :inner], w[p + "conv"], w[p + "conv.b"]))
    z = both[:, inner:]
    proj = stored(x) @ w[p + "x"].T
    dt = softplus(stored(proj[:, :rank]) @ w[p + "dt"].T + w[p + "dt.b"])
    y = selective_scan(x, dt, proj[:, rank : rank + state], proj[:, rank + state :], -torch.exp(w[p + "A_log"]), w[p + "D"])
    return stored(y * silu(z)) @ w[p + "o"].T


# -- attention through a latent ------------------------------------------------------------------------------------
def rotate_half(x, positions, base, dims):
    """``x [T, n, d]``: dimension i of the first ``dims`` is paired with i + dims/2."""
    i = torch.arange(dims // 2, dtype=x.dtype)
    angles = positions.to(x.dtype)[:, None] * (base ** (-2.0 * i / dims))[None, :]
    cos, sin = angles.cos()[:, None, :], angles.sin()[:, None, :]
    u, v = x[..., : dims // 2], x[..., dims // 2 : dims]
    out = x.clone()
    out[..., : dims // 2] = u * cos - v * sin
    out[..., dims // 2 : dims] = v * cos + u * sin
    return out


def causal_softmax_attention(q, k, v, scale):
    """``q, k [T, heads, d]``, ``v [T, heads, vdim]`` -> ``[T, heads, vdim]``."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=q.dtype)
    for i in range(q.shape[0]):
        scores = torch.einsum("hd,jhd->hj", q[i], k[: i + 1]) * scale
        out[i] = torch.einsum("hj,jhv->hv", torch.softmax(scores, -1), v[: i + 1])
    return out


def latent_mixer(h, w, p, m, eps):
    tokens = h.shape[0]
    heads, dim, rot_dim, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions = torch.arange(tokens)
    q = (h @ w[p + "q"].T).reshape(tokens, heads, dim + rot_dim)
    q_rot = rotate_half(q[..., dim:], positions, m["rot"]["base"], m["rot"]["dims"])
    down = h @ w[p + "dkv"].T
    c = stored(rms_unit(down[:, :rank], eps) * w[p + "dkv.norm"])
    part = stored(rotate_half(down[:, None, rank:], positions, m["rot"]["base"], m["rot"]["dims"]))
    k = (c @ w[p + "uk"].T).reshape(tokens, heads, dim)
    v = (c @ w[p + "uv"].T).reshape(tokens, heads, vdim)
    q_all = torch.cat([stored(q[..., :dim]), stored(q_rot)], -1)
    k_all = torch.cat([k, part.expand(tokens, heads, rot_dim)], -1)
    o = causal_softmax_attention(q_all, k_all, v, m["scale"])
    return stored(o.reshape(tokens, heads * vdim)) @ w[p + "o"].T


# -- generalized delta rule ------------------------------------------------------------------------------------------
def channel_decay(h, w, p):
    """Between ``exp(-exp(-1/2))`` and 1, a number per head and key channel, through a low-rank projection."""
    low = torch.tanh(h @ w[p + "w1"].T)
    return torch.exp(-math.exp(-0.5) * torch.sigmoid(stored(low) @ w[p + "w2"].T + w[p + "w0"]))


def delta_rule(r, k, v, decay, rate):
    """All ``[T, heads, dim]``: ``S <- diag(decay) S - (rate * u) (u^T S) + k v^T`` with ``u`` the unit key and the old
    S on the right, ``o = S^T r``."""
    tokens, heads, dim = r.shape
    out = torch.zeros_like(v)
    for head in range(heads):
        S = torch.zeros(dim, v.shape[2], dtype=r.dtype)
        for t in range(tokens):
            key = k[t, head]
            u = key / torch.sqrt((key * key).sum() + 1e-6)
            S = decay[t, head][:, None] * S - torch.outer(rate[t, head] * u, u @ S) + torch.outer(key, v[t, head])
            out[t, head] = S.T @ r[t, head]
    return out


def delta_mixer(h, w, p, m, eps):
    tokens, heads, dim = h.shape[0], m["heads"], m["dim"]
    r, k, v = ((h @ w[p + n].T).reshape(tokens, heads, dim) for n in ("r", "k", "v"))
    decay = channel_decay(h, w, p).reshape(tokens, heads, dim)
    rate = torch.sigmoid(h @ w[p + "a"].T + w[p + "a.b"]).reshape(tokens, heads, dim)
    o = rms_unit(delta_rule(r, k, v, decay, rate), eps).reshape(tokens, heads * dim)
    return stored(o * w[p + "norm"] * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


# -- feed-forwards ----------------------------------------------------------------------------------------------------
def dense_ff(h, w, p):
    act = w[p + "act"]
    return stored(xielu(h @ w[p + "up"].T, act[0], act[1])) @ w[p + "down"].T


def expert(h, w, p):
    return stored(erf_gelu(h @ w[p + "up"].T)) @ w[p + "down"].T


def route(logits, top):
    """Per token the indices of the ``top`` largest logits and the softmax over those alone."""
    picked = torch.topk(logits, top, dim=-1)
    return picked.indices, torch.softmax(picked.values, -1)


def routed_ff(h, w, p, mlp, margins=None):
    """``margins`` (a list) receives, per token, the gap between the logits of the last expert chosen and the first
    one left out (infinite when every expert is chosen)."""
    experts, top = mlp["router"]["experts"], mlp["router"]["top"]
    logits = h @ w[p + "router"].T + w[p + "router.b"]
    if margins is not None:
        ranked = torch.sort(logits, dim=-1, descending=True).values
        margins.append(ranked[:, top - 1] - ranked[:, top] if top < experts else torch.full_like(ranked[:, 0], float("inf")))
    ids, weights = route(logits, top)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, s in zip(ids[t].tolist(), weights[t]):
            out[t] += s * expert(h[t : t + 1], w, f"{p}e{e}.")[0]
    return out


# -- the model ----------------------------------------------------------------------------------------------------------
MIXERS = {"mamba1": mamba_mixer, "latent_attention": latent_mixer, "general_delta": delta_mixer}


def forward(cfg, w, tokens, dtype=torch.float64, trace=None, margins=None):
    """Logits ``[T, vocab]`` of one sequence; ``trace`` (a list) receives the residual after every layer's average,
    ``margins`` (a list) every router's margins."""
    w = {name: t.to(dtype) for name, t in w.items()}
    eps = float(cfg["norm"]["eps"])
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    states = [x]
    for index, layer in enumerate(cfg["layers"]):
        p = f"l{index}."
        mixed = MIXERS[layer["type"]](normed_input(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
        x = x + zero_centred_norm(mixed, w[p + "norm1b"], eps) * w[p + "ls1"]
        mlp = layer.get("mlp")
        if mlp is not None:
            h = normed_input(x, w[p + "norm2"], eps)
            fed = dense_ff(h, w, p + "mlp.") if mlp["kind"] == "dense" else routed_ff(h, w, p + "mlp.", mlp, margins)
            x = x + zero_centred_norm(fed, w[p + "norm2b"], eps) * w[p + "ls2"]
        states.append(x)
        x = depth_average(states, w[p + "dwa"])
        if trace is not None:
            trace.append(x.clone())
    logits = normed_input(x, w["final.norm"], eps) @ w["head"].T
    cap = float(cfg["logit_softcap"])
    return cap * torch.tanh(logits / cap)


# -- tensors of a configuration, and random ones --------------------------------------------------------------------------
def tensor_shapes(cfg, decay_rank=8):
    """``decay_rank``: the rank of a delta layer's decay projection, which the configuration does not give (a number,
    or one per layer by index)."""
    width = cfg["width"]
    shapes = {"embed": (cfg["vocab"], width)}
    for index, layer in enumerate(cfg["layers"]):
        p, m = f"l{index}.", layer["mixer"]
        shapes.update({p + "norm1": (width,), p + "norm1b": (width,), p + "ls1": (width,), p + "dwa": (index + 2,)})
        q = p + "mix."
        if layer["type"] == "mamba1":
            inner, rank, state = m["inner"], m["dt_rank"], m["state"]
            shapes.update({q + "in": (2 * inner, width), q + "conv": (inner, m["conv"]), q + "conv.b": (inner,),
                           q + "x": (rank + 2 * state, inner), q + "dt": (inner, rank), q + "dt.b": (inner,),
                           q + "A_log": (inner, state), q + "D": (inner,), q + "o": (width, inner)})
        elif layer["type"] == "latent_attention":
            heads, dim, rot, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            shapes.update({q + "q": (heads * (dim + rot), width), q + "dkv": (rank + rot, width), q + "dkv.norm": (rank,),
                           q + "uk": (heads * dim, rank), q + "uv": (heads * vdim, rank), q + "o": (width, heads * vdim)})
        else:
            n = m["heads"] * m["dim"]
            low = decay_rank[index] if isinstance(decay_rank, dict) else decay_rank
            shapes.update({q + name: (n, width) for name in ("r", "k", "v", "g", "a")})
            shapes.update({q + "a.b": (n,), q + "w1": (low, width), q + "w2": (n, low), q + "w0": (n,), q + "norm": (n,),
                           q + "o": (width, n)})
        mlp = layer.get("mlp")
        if mlp is not None:
            shapes.update({p + "norm2": (width,), p + "norm2b": (width,), p + "ls2": (width,)})
            q = p + "mlp."
            if mlp["kind"] == "dense":
                shapes.update({q + "up": (mlp["ff"], width), q + "down": (width, mlp["ff"]), q + "act": (2,)})
            else:
                experts, ff = mlp["router"]["experts"], mlp["expert"]["ff"]
                shapes.update({q + "router": (experts, width), q + "router.b": (experts,)})
                for e in range(experts):
                    shapes.update({f"{q}e{e}.up": (ff, width), f"{q}e{e}.down": (width, ff)})
    shapes["final.norm"] = (width,)
    shapes["head"] = (cfg["vocab"], width)
    return shapes


def random_weights(cfg, seed, decay_rank=8, router_gain=6.0):
    """Weights rounded to bfloat16 (as checkpoints store them), sized so that activations stay of order one, states
    remember for many tokens and every layer's average leans on all of the states before it."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, decay_rank).items():
        leaf = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = torch.randn(shape, generator=g) / cfg["embedding"]["scale"]
        elif leaf == "router":
            t = torch.randn(shape, generator=g) * router_gain / math.sqrt(shape[1])  # logits well apart: few close calls
        elif leaf in ("ls1", "ls2"):
            t = 0.6 + torch.randn(shape, generator=g) * 0.2
        elif leaf == "dwa":
            t = torch.randn(shape, generator=g) * 0.3
            t[-1] = 1.0
        elif leaf == "act":
            t = torch.randn(shape, generator=g)
        elif leaf == "A_log":  # decays from slow to fast along the state
            t = torch.log(torch.arange(1, shape[1] + 1).float()) - 2.0 + 0.3 * torch.randn(shape, generator=g)
        elif leaf == "D":
            t = torch.randn(shape, generator=g)
        elif name.endswith("dt.b"):
            t = -1.5 + torch.randn(shape, generator=g)
        elif leaf == "w0":
            t = -2.5 + torch.randn(shape, generator=g) * 1.5
        elif leaf == "conv":
            t = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        elif name.endswith("router.b"):
            t = torch.randn(shape, generator=g)
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) / math.sqrt(shape[1])
        elif leaf == "b":
            t = torch.randn(shape, generator=g) * 0.5
        elif name.endswith(("mix.norm", "dkv.norm")):
            t = 1.0 + torch.randn(shape, generator=g) * 0.2
        else:  # norm scales stored around zero
            t = torch.randn(shape, generator=g) * 0.2
        out[name] = t.to(torch.bfloat16).float()
    return out
