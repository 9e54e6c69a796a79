"""Recipe of the Mekusun decoder: typed configuration -> parts and run order.

The design: token embeddings times a constant; layers in the order the configuration lists them, each a ``sandwich``
block (RMS norms with scales stored around zero before and after each sublayer, the latter times a learned vector:
``x += ls_1 * norm_1b(mixer(norm_1(x)))``, ``x += ls_2 * norm_2b(ff(norm_2(x)))``; a layer may have no feed-forward);
behind every layer the residual becomes a learned weighted sum of the embedding output and of all layers' results so
far; a final norm; an untied head whose logits are capped by ``cap * tanh(z / cap)``.  Mixers:

* ``mamba1``: a selective scan (a diagonal state per channel, step sizes, inputs and outputs made from the token);
* ``latent_attention``: attention through a cached latent, queries straight from the input, no sink, no gate;
* ``general_delta``: a matrix state per head with a decay and a removal rate per key channel.

Feed-forwards: dense with the xIELU activation, or routed over experts of two matrices with the exact GELU, chosen
and weighted by a softmax over the chosen logits (with a bias per expert).

Tensor names: ``embed``; ``l<i>.norm1|norm1b|norm2|norm2b|ls1|ls2|dwa``; ``l<i>.mix.in|conv|conv.b|x|dt|dt.b|A_log|D|o``
(mamba1), ``l<i>.mix.q|dkv|dkv.norm|uk|uv|o`` (latent_attention), ``l<i>.mix.r|k|v|g|a|a.b|w1|w2|w0|norm|o``
(general_delta); ``l<i>.mlp.up|down|act`` (dense) or ``l<i>.mlp.router|router.b``, ``l<i>.mlp.e<j>.up|down``;
``final.norm``; ``head``.
"""

from __future__ import annotations

from ..config.mekusun_config import ChannelDeltaSizes, DenseSizes, MekusunConfig, SelectiveScanSizes
from ..config.model_spec import LayerCall, LayerSpec, ModelSpec, PartSpec
from ..config.registry import register_architecture


def _norm(eps: float, prefix: str, name: str, times: str | None = None) -> PartSpec:
    return PartSpec("rmsnorm", {"eps": eps, "name": name, "offset": 1.0, "times": times}, prefix)


def _mixer(m, prefix: str, eps: float) -> PartSpec:
    if isinstance(m, SelectiveScanSizes):
        return PartSpec("selective_scan", {"inner": m.inner, "state": m.state, "dt_rank": m.dt_rank, "taps": m.conv}, prefix)
    if isinstance(m, ChannelDeltaSizes):
        return PartSpec("channel_delta", {"heads": m.heads, "dim": m.dim, "eps": eps}, prefix)
    position = PartSpec("rotary", {"head_dim": m.rot_dim, "rotary_dim": m.rot_dims, "theta": m.rot_base})
    return PartSpec(
        "latent_attention",
        {"num_heads": m.heads, "head_dim": m.dim, "rot_dim": m.rot_dim, "value_dim": m.vdim, "kv_rank": m.kv_rank,
         "q_rank": None, "scale": m.scale, "eps": eps, "position": position},
        prefix,
    )


def _feed_forward(mlp, prefix: str) -> PartSpec:
    if mlp is None:
        return PartSpec("none")
    if isinstance(mlp, DenseSizes):
        return PartSpec("activated", {"intermediate_size": mlp.ff, "activation": "xielu", "names": ("up", "down"),
                                      "numbers": "act"}, prefix)
    return PartSpec("routed_activated", {"experts": mlp.experts, "top": mlp.top, "intermediate_size": mlp.ff,
                                         "activation": "gelu", "scoring": "softmax_chosen", "router_bias": "router.b"}, prefix)


def mekusun_recipe(cfg: MekusunConfig) -> ModelSpec:
    layers = []
    for i, layer in enumerate(cfg.layers):
        p = f"l{i}."
        norms = {"input": _norm(cfg.eps, p, "norm1"), "mixer_out": _norm(cfg.eps, p, "norm1b", "ls1")}
        if layer.mlp is not None:
            norms.update(post_mixer=_norm(cfg.eps, p, "norm2"), ff_out=_norm(cfg.eps, p, "norm2b", "ls2"))
        layers.append(LayerSpec("sandwich", _mixer(layer.mixer, p + "mix.", cfg.eps), _feed_forward(layer.mlp, p + "mlp."), norms,
                                average=p + "dwa"))
    return ModelSpec(
        architecture="Mekusun",
        vocab_size=cfg.vocab,
        hidden_size=cfg.width,
        layers=tuple(layers),
        order=tuple(LayerCall(i, i, True) for i in range(len(layers))),
        final_norm=_norm(cfg.eps, "final.", "norm"),
        embedding_name="embed",
        head_name="head",
        eos_token_id=cfg.eos_token_id,
        embedding_scale=cfg.embedding_scale,
        logit_softcap=cfg.logit_softcap,
        # a layer without a feed-forward reads no second pair of norms; a checkpoint may carry them all the same
        tolerated=tuple(f"l{i}.{n}" for i, layer in enumerate(cfg.layers) if layer.mlp is None for n in ("norm2", "norm2b", "ls2")),
    )


register_architecture("Mekusun", MekusunConfig, mekusun_recipe)
