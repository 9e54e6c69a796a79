"""Typed configuration of the Mekusun decoder, read from ``config.json`` keys.

``config.json`` gives ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``logit_softcap`` and ``layers``, a
list in which every entry names its ``type``, the sizes and constants of its ``mixer`` and its feed-forward ``mlp``.

Mixer keys.  ``"mamba1"``: ``inner``, ``state``, ``dt_rank``, ``conv`` (taps of the short convolution).
``"latent_attention"``: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``rot: {base, dims}``.
``"general_delta"``: ``heads``, ``dim`` (the rank of its decay projection is the checkpoint's).  Feed-forwards:
``{"kind": "dense", "ff"}``, ``{"kind": "moe", "router": {"experts", "top"}, "expert": {"ff"}}``, or null for a
layer without one.  Nothing has a default: a key that is missing is an error that names it.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

from .qwen2_config import ConfigError
from .zelasun_config import _count, _get, _number


@dataclass(frozen=True)
class SelectiveScanSizes:
    """A recurrence with a diagonal state per channel whose step size, input and output vary with the token."""

    inner: int
    state: int
    dt_rank: int
    conv: int

    @classmethod
    def read(cls, raw, where: str) -> "SelectiveScanSizes":
        return cls(_count(raw, "inner", where), _count(raw, "state", where), _count(raw, "dt_rank", where),
                   _count(raw, "conv", where))


@dataclass(frozen=True)
class PlainLatentAttentionSizes:
    """Softmax attention whose keys and values are made from one latent per token; queries come from the input."""

    heads: int
    dim: int        # plain (unrotated) query/key dimensions per head
    rot_dim: int    # rotated query/key dimensions per head; the key's are one vector shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    rot_base: float
    rot_dims: int

    @classmethod
    def read(cls, raw, where: str) -> "PlainLatentAttentionSizes":
        rot = _get(raw, "rot", where)
        out = cls(_count(raw, "heads", where), _count(raw, "dim", where), _count(raw, "rot_dim", where),
                  _count(raw, "vdim", where), _count(raw, "kv_rank", where), _number(raw, "scale", where),
                  _number(rot, "base", where + "rot."), _count(rot, "dims", where + "rot."))
        if out.rot_dims % 2 or out.rot_dims > out.rot_dim:
            raise ConfigError(f"{where}rot.dims ({out.rot_dims}) must be even and at most rot_dim ({out.rot_dim})")
        return out


@dataclass(frozen=True)
class ChannelDeltaSizes:
    """A matrix state per head with a decay and a removal rate per key channel."""

    heads: int
    dim: int

    @classmethod
    def read(cls, raw, where: str) -> "ChannelDeltaSizes":
        return cls(_count(raw, "heads", where), _count(raw, "dim", where))


_MIXERS = {"mamba1": SelectiveScanSizes, "latent_attention": PlainLatentAttentionSizes, "general_delta": ChannelDeltaSizes}


@dataclass(frozen=True)
class DenseSizes:
    ff: int


@dataclass(frozen=True)
class UngatedRoutedSizes:
    """Experts of two matrices, weighted by a softmax over the chosen experts' logits."""

    experts: int
    top: int
    ff: int

    @classmethod
    def read(cls, raw, where: str) -> "UngatedRoutedSizes":
        router = _get(raw, "router", where)
        out = cls(_count(router, "experts", where + "router."), _count(router, "top", where + "router."),
                  _count(_get(raw, "expert", where), "ff", where + "expert."))
        if out.top > out.experts:
            raise ConfigError(f"{where}router.top ({out.top}) exceeds router.experts ({out.experts})")
        return out


def _read_mlp(raw, where: str):
    if raw is None:
        return None
    kind = _get(raw, "kind", where)
    if kind == "dense":
        return DenseSizes(_count(raw, "ff", where))
    if kind == "moe":
        return UngatedRoutedSizes.read(raw, where)
    raise ConfigError(f"{where}kind {kind!r}: this design has 'dense' and 'moe' feed-forwards")


@dataclass(frozen=True)
class MekusunLayer:
    type: str    # a key of _MIXERS
    mixer: Any   # SelectiveScanSizes | PlainLatentAttentionSizes | ChannelDeltaSizes
    mlp: Any     # DenseSizes | UngatedRoutedSizes | None


@dataclass(frozen=True)
class MekusunConfig:
    vocab: int
    width: int
    eps: float
    embedding_scale: float
    logit_softcap: float
    layers: tuple[MekusunLayer, ...]
    eos_token_id: int | None = None
    architecture: str = "Mekusun"
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "MekusunConfig":
        listed = _get(raw, "layers", "")
        if not isinstance(listed, (list, tuple)) or not listed:
            raise ConfigError("layers must be a non-empty list")
        layers = []
        for index, entry in enumerate(listed):
            where = f"layers[{index}]."
            kind = _get(entry, "type", where)
            if kind not in _MIXERS:
                raise ConfigError(f"{where}type {kind!r}: this design has {', '.join(sorted(_MIXERS))} layers")
            mixer = _MIXERS[kind].read(_get(entry, "mixer", where), where + "mixer.")
            layers.append(MekusunLayer(kind, mixer, _read_mlp(entry.get("mlp"), where + "mlp.")))
        eos = raw.get("eos_token_id")
        cap = _number(raw, "logit_softcap", "")
        if cap <= 0:
            raise ConfigError(f"logit_softcap must be positive, got {cap}")
        known = {"architecture", "architectures", "layers", "norm", "vocab", "width", "embedding", "logit_softcap", "eos_token_id"}
        return cls(
            vocab=_count(raw, "vocab", ""),
            width=_count(raw, "width", ""),
            eps=_number(_get(raw, "norm", ""), "eps", "norm."),
            embedding_scale=_number(_get(raw, "embedding", ""), "scale", "embedding."),
            logit_softcap=cap,
            layers=tuple(layers),
            eos_token_id=int(eos) if eos is not None else None,
            extra={k: v for k, v in raw.items() if k not in known},
        )
