"""A plain, slow Labolix decoder: one function per mechanism, whole sequences, no cache.

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


# -- norms ------------------------------------------------------------------------------------------------------
def squash(x, alpha, weight, bias):
    """The norm that measures nothing: every element on its own."""
    return torch.tanh(alpha * x) * weight + bias


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


# -- rotations ----------------------------------------------------------------------------------------------------
def plain_frequencies(base, dims):
    return [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]


def frequencies_by_wavelength(base, dims, factor, low, high, original):
    """Short waves stay, long ones are slowed by ``factor``, a straight blend between the two."""
    out = []
    for f in plain_frequencies(base, dims):
        wave = 2.0 * math.pi / f
        if wave < original / high:
            out.append(f)
        elif wave > original / low:
            out.append(f / factor)
        else:
            s = (original / wave - low) / (high - low)
            out.append((1.0 - s) * f / factor + s * f)
    return out


def frequencies_by_ramp(base, dims, factor, original, fast, slow):
    """Slowed along a ramp over the pair index; returns the frequencies and the factor on cos and sin."""

    def place(turns):
        return dims * math.log(original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo = max(math.floor(place(fast)), 0)
    hi = min(math.ceil(place(slow)), dims - 1)
    out = []
    for i, f in enumerate(plain_frequencies(base, dims)):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * ramp + f * (1.0 - ramp))
    return out, 0.1 * math.log(factor) + 1.0


def turn(x, positions, freqs, pairs, strength=1.0):
    """``x [T, n, d]``: pair i is the two indices ``pairs(i)``; everything else passes unchanged."""
    out = x.clone()
    for i, f in enumerate(freqs):
        a, b = pairs(i)
        angle = positions.to(x.dtype) * f
        cos, sin = (torch.cos(angle) * strength)[:, None], (torch.sin(angle) * strength)[:, None]
        u, v = x[..., a], x[..., b]
        out[..., a] = u * cos - v * sin
        out[..., b] = v * cos + u * sin
    return out


def neighbours(i):
    return 2 * i, 2 * i + 1


def halves(dims):
    return lambda i: (i, i + dims // 2)


# -- softmax attention ----------------------------------------------------------------------------------------------
def attend(q, k, v, scale, sink, window=None):
    """``q, k [T, heads, d]``, ``v [T, heads, vdim]``, ``sink [heads]`` (the score of a term of the denominator that has
    no value) -> ``[T, heads, vdim]``; with a window a token sees itself and the ``window - 1`` tokens before it."""
    out = torch.zeros(q.shape[0], q.shape[1], v.shape[2], dtype=q.dtype)
    for i in range(q.shape[0]):
        first = 0 if window is None else max(0, i - window + 1)
        scores = torch.einsum("hd,jhd->hj", q[i], k[first : i + 1]) * scale
        top = torch.maximum(scores.max(-1).values, sink)
        e = torch.exp(scores - top[:, None])
        weights = e / (e.sum(-1) + torch.exp(sink - top))[:, None]
        out[i] = torch.einsum("hj,jhv->hv", weights, v[first : i + 1])
    return out


def attention_mixer(h, w, p, m, eps):
    tokens, heads, kv_heads = h.shape[0], m["heads"], m["kv_heads"]
    positions, rot = torch.arange(tokens), m["rot"]
    scaling = rot.get("scaling")
    freqs = plain_frequencies(rot["base"], rot["dims"]) if scaling is None else frequencies_by_wavelength(
        rot["base"], rot["dims"], scaling["factor"], scaling["low"], scaling["high"], scaling["original"])
    q = stored(turn((h @ w[p + "q"].T).reshape(tokens, heads, m["dim"]), positions, freqs, neighbours))
    k = stored(turn((h @ w[p + "k"].T).reshape(tokens, kv_heads, m["dim"]), positions, freqs, neighbours))
    v = stored((h @ w[p + "v"].T).reshape(tokens, kv_heads, m["vdim"]))
    of = [head // (heads // kv_heads) for head in range(heads)]
    o = attend(q, k[:, of], v[:, of], m["scale"], torch.zeros(heads, dtype=h.dtype))
    return stored(o.reshape(tokens, heads * m["vdim"])) @ w[p + "o"].T


def latent_mixer(h, w, p, m, eps):
    tokens = h.shape[0]
    heads, dim, rot_dim, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    positions, rot = torch.arange(tokens), m["rot"]
    scaling = rot.get("scaling")
    freqs, strength = plain_frequencies(rot["base"], rot["dims"]), 1.0
    if scaling is not None:
        freqs, strength = frequencies_by_ramp(rot["base"], rot["dims"], scaling["factor"], scaling["original"],
                                              scaling["fast"], scaling["slow"])
    q = (h @ w[p + "q"].T).reshape(tokens, heads, dim + rot_dim)
    down = h @ w[p + "dkv"].T
    c = stored(rms_unit(down[:, :rank], eps) * w[p + "dkv.norm"])
    part = stored(turn(down[:, None, rank:], positions, freqs, neighbours, strength))
    k = (c @ w[p + "uk"].T).reshape(tokens, heads, dim)
    v = (c @ w[p + "uv"].T).reshape(tokens, heads, vdim)
    q_all = torch.cat([stored(q[..., :dim]), stored(turn(q[..., dim:], positions, freqs, neighbours, strength))], -1)
    k_all = torch.cat([k, part.expand(tokens, heads, rot_dim)], -1)
    o = attend(q_all, k_all, v, m["scale"], w[p + "sink"], m["mask"]["size"])
    return stored(o.reshape(tokens, heads * vdim)) @ w[p + "o"].T


# -- retention --------------------------------------------------------------------------------------------------------
def retain(q, k, v, decay):
    """``q, k [T, heads, dim]``, ``v [T, heads, vdim]``, ``decay`` a number per head: the state forgets at a fixed rate,
    takes in the outer product of key and value, and is read by the query; nothing is divided."""
    tokens, heads, dim = q.shape
    out = torch.zeros_like(v)
    for head in range(heads):
        S = torch.zeros(dim, v.shape[2], dtype=q.dtype)
        for t in range(tokens):
            S = decay[head] * S + torch.outer(k[t, head], v[t, head])
            out[t, head] = S.T @ q[t, head]
    return out


def retention_mixer(h, w, p, m, eps):
    tokens, heads, dim, vdim = h.shape[0], m["heads"], m["dim"], m["vdim"]
    positions, rot = torch.arange(tokens), m["rot"]
    freqs, pairs = plain_frequencies(rot["base"], rot["dims"]), halves(rot["dims"])
    q = turn((h @ w[p + "q"].T).reshape(tokens, heads, dim), positions, freqs, pairs)
    k = turn((h @ w[p + "k"].T).reshape(tokens, heads, dim), positions, freqs, pairs) * dim ** -0.5
    v = (h @ w[p + "v"].T).reshape(tokens, heads, vdim)
    o = rms_unit(retain(q, k, v, m["decay"]), eps).reshape(tokens, heads * vdim)
    g = h @ w[p + "g"].T
    return stored(o * g * torch.sigmoid(g)) @ w[p + "o"].T


# -- feed-forward -------------------------------------------------------------------------------------------------------
def capped_glu(gate, up, limit):
    g, u = torch.clamp(gate, max=limit), torch.clamp(up, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, w, p, mlp):
    return stored(capped_glu(h @ w[p + "gate"].T, h @ w[p + "up"].T, mlp["limit"])) @ w[p + "down"].T


# -- the model ----------------------------------------------------------------------------------------------------------
MIXERS = {"latent_attention": latent_mixer, "retention": retention_mixer, "attention": attention_mixer}


def owner(cfg, index):
    """The layer whose tensors layer ``index`` uses."""
    while cfg["layers"][index].get("weights_of") is not None:
        index = cfg["layers"][index]["weights_of"]
    return index


def forward(cfg, w, tokens, dtype=torch.float64, trace=None):
    """Logits ``[T, vocab]`` of one sequence; ``trace`` (a list) receives the residual after every layer that runs."""
    w = {name: t.to(dtype) for name, t in w.items()}
    eps = float(cfg["norm"]["eps"])

    def normed(x, name):
        return stored(squash(x, w[name + ".alpha"], w[name], w[name + ".b"]))

    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for index, layer in enumerate(cfg["layers"]):
        p = f"l{owner(cfg, index)}."
        x = x + MIXERS[layer["type"]](normed(x, p + "norm1"), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + dense_ff(normed(x, p + "norm2"), w, p + "mlp.", layer["mlp"])
        if trace is not None:
            trace.append(x.clone())
    logits = normed(x, "final.norm") @ w["embed"].T
    cap = cfg.get("logit_softcap")
    return logits if cap is None else cap * torch.tanh(logits / cap)


# -- tensors of a configuration, and random ones --------------------------------------------------------------------------
def tensor_shapes(cfg):
    width = cfg["width"]

    def norm(name):
        return {name: (width,), name + ".b": (width,), name + ".alpha": ()}

    shapes = {"embed": (cfg["vocab"], width)}
    for index, layer in enumerate(cfg["layers"]):
        if owner(cfg, index) != index:
            continue
        p, m = f"l{index}.", layer["mixer"]
        shapes.update(norm(p + "norm1"))
        q, heads = p + "mix.", m["heads"]
        if layer["type"] == "latent_attention":
            dim, rot, vdim, rank = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            shapes.update({q + "q": (heads * (dim + rot), width), q + "dkv": (rank + rot, width), q + "dkv.norm": (rank,),
                           q + "uk": (heads * dim, rank), q + "uv": (heads * vdim, rank), q + "sink": (heads,),
                           q + "o": (width, heads * vdim)})
        else:
            kv = m["kv_heads"] if layer["type"] == "attention" else heads
            shapes.update({q + "q": (heads * m["dim"], width), q + "k": (kv * m["dim"], width),
                           q + "v": (kv * m["vdim"], width), q + "o": (width, heads * m["vdim"])})
            if layer["type"] == "retention":
                shapes[q + "g"] = (heads * m["vdim"], width)
        mlp = layer.get("mlp")
        if mlp is not None:
            shapes.update(norm(p + "norm2"))
            q = p + "mlp."
            shapes.update({q + "gate": (mlp["ff"], width), q + "up": (mlp["ff"], width), q + "down": (width, mlp["ff"])})
    shapes.update(norm("final.norm"))
    return shapes


def random_weights(cfg, seed, gain=1.2):
    """Weights rounded to bfloat16 (as checkpoints store them), sized so that activations stay of order one, the norms
    bend, a feed-forward's limits are met and sinks take a share.  A retention layer's keys lean towards its queries: a
    read-out that is almost nothing would be blown up to full size by its norm, rounding and all."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        leaf = name.rsplit(".", 1)[-1]
        if name == "embed":
            t = torch.randn(shape, generator=g)
        elif leaf == "alpha":
            t = 0.4 + 0.4 * torch.rand(shape, generator=g)
        elif leaf == "b":
            t = torch.randn(shape, generator=g) * 0.2
        elif leaf == "sink":
            t = torch.randn(shape, generator=g) * 1.5
        elif len(shape) == 2:
            t = torch.randn(shape, generator=g) * gain / math.sqrt(shape[1])
            layer = cfg["layers"][int(name.split(".", 1)[0][1:])] if name.startswith("l") else None
            if layer is not None and layer["type"] == "retention" and name.endswith("mix.k"):
                t = 0.8 * out[name[:-1] + "q"] + 0.6 * t
        else:
            t = 1.0 + torch.randn(shape, generator=g) * 0.3
        out[name] = t.to(torch.bfloat16).float()
    return out
