"""Recipe of the Labolix decoder: typed configuration -> parts and run order.

The design: token embeddings; layers in the order the configuration lists them, each a ``pre_norm`` block whose norms
measure nothing (``tanh(alpha x) * w + b``): ``x += mixer(norm_1(x))``, ``x += ff(norm_2(x))`` (a layer may have no
feed-forward); a final norm of the same kind; the embedding table as the head, logits capped by ``cap * tanh(z / cap)``.
An entry may run another entry's weights again: in the run order that layer is named once more, with a cache slot (and
state slot) of its own.  Mixers:

* ``latent_attention``: attention through a cached latent over a window of positions, a learned sink per head in the
  softmax's denominator, queries straight from the input, the rotated part's long waves slowed along a ramp over the
  pair index, with a factor on cos and sin;
* ``retention``: a matrix state per head with a constant decay, q and k rotated, the read-out divided by its root mean
  square per head and gated by ``silu(W_g h)``;
* ``attention``: grouped-query softmax attention with one added to the denominator, q and k rotated in neighbouring
  pairs whose long waves are slowed by their wavelength, values of a size of their own.

Feed-forward: gated, with capped halves (``g' sigmoid(1.702 g') (u' + 1)``).

Tensor names: ``embed``; ``l<i>.norm1|norm2`` (+ ``.alpha``, ``.b``); ``l<i>.mix.q|dkv|dkv.norm|uk|uv|sink|o``
(latent_attention), ``l<i>.mix.q|k|v|g|o`` (retention), ``l<i>.mix.q|k|v|o`` (attention); ``l<i>.mlp.gate|up|down``;
``final.norm`` (+ ``.alpha``, ``.b``).  Layers that run another's weights have no tensors.
"""

from __future__ import annotations

import math

from ..config.labolix_config import LabolixConfig, RetentionSizes, Rotation, WindowedLatentSizes
from ..config.model_spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from ..config.registry import register_architecture


def _norm(prefix: str, name: str) -> PartSpec:
    return PartSpec("dynamic_tanh", {"weight": name, "bias": name + ".b", "alpha": name + ".alpha"}, prefix)


def _rotation(rot: Rotation, head_dim: int, interleaved: bool) -> PartSpec:
    factor = 0.1 * math.log(rot.scaling["factor"]) + 1.0 if rot.scaling and "fast" in rot.scaling else 1.0
    return PartSpec("rotary", {"head_dim": head_dim, "rotary_dim": rot.dims, "theta": rot.base, "interleaved": interleaved,
                               "factor": factor, "scaling": dict(rot.scaling) if rot.scaling else None})


def _mixer(m, prefix: str, eps: float) -> PartSpec:
    if isinstance(m, RetentionSizes):
        return PartSpec(
            "decay_attention",
            {"heads": m.heads, "key_dim": m.dim, "value_dim": m.vdim, "decay": m.decay, "eps": eps, "activation": "none",
             "position": _rotation(m.rot, m.dim, False), "key_scale": m.dim ** -0.5, "norm": "head", "gate": "silu"},
            prefix,
        )
    if isinstance(m, WindowedLatentSizes):
        return PartSpec(
            "latent_attention",
            {"num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim, "kv_rank": m.kv_rank,
             "q_rank": None, "scale": m.scale, "eps": eps, "position": _rotation(m.rot, m.rot_dim, True), "sink": True,
             "window": m.window},
            prefix,
        )
    return PartSpec(
        "gqa_attention",
        {"num_heads": m.heads, "num_kv_heads": m.kv_heads, "head_dim": m.dim, "value_dim": m.vdim, "scale": m.scale,
         "names": {"q": "q", "k": "k", "v": "v", "o": "o"}, "sink_score": 0.0, "position": _rotation(m.rot, m.dim, True)},
        prefix,
    )


def labolix_recipe(cfg: LabolixConfig) -> ModelSpec:
    layers, place = [], {}  # place: entry of the configuration -> index among the layers that have weights
    for i, layer in enumerate(cfg.layers):
        if cfg.weights_of[i] != i:
            continue
        p = f"l{i}."
        norms = {"input": _norm(p, "norm1")}
        feed_forward = PartSpec("none")
        if layer.mlp is not None:
            norms["post_mixer"] = _norm(p, "norm2")
            feed_forward = PartSpec("swiglu", {"intermediate_size": layer.mlp.ff, "names": ("gate", "up", "down"),
                                               "limit": layer.mlp.limit}, p + "mlp.")
        place[i] = len(layers)
        layers.append(LayerSpec("pre_norm", _mixer(layer.mixer, p + "mix.", cfg.eps), feed_forward, norms))
    return ModelSpec(
        architecture="Labolix",
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        layers=tuple(layers),
        order=tuple(LayerCall(place[owner], slot, True) for slot, owner in enumerate(cfg.weights_of)),
        final_norm=_norm("final.", "norm"),
        embedding_name="embed",
        head_name=None,
        eos_token_id=cfg.eos_token_id,
        logit_softcap=cfg.logit_softcap,
        # a layer without a feed-forward reads no second norm; a checkpoint may carry one all the same
        tolerated=tuple(f"l{i}.norm2{s}" for i in place if cfg.layers[i].mlp is None for s in ("", ".b", ".alpha")),
    )


register_architecture("Labolix", LabolixConfig, labolix_recipe)
