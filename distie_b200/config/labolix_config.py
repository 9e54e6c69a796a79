"""Typed configuration of the Labolix decoder, read from ``config.json`` keys.

``config.json`` gives ``vocab``, ``width``, ``norm.eps``, ``logit_softcap`` and ``layers``, a list in which every entry
names its ``type``, the sizes and constants of its ``mixer`` and its feed-forward ``mlp`` (``{"kind": "dense", "ff",
"limit"}``, or null for a layer without one).  An entry with ``weights_of: j`` runs layer j's weights once more.

Mixer keys.  ``"latent_attention"``: ``heads``, ``dim``, ``rot_dim``, ``vdim``, ``kv_rank``, ``scale``, ``mask: {size}``,
``rot: {base, dims, scaling: {factor, original, fast, slow}}``.  ``"retention"``: ``heads``, ``dim``, ``vdim``, ``decay``
(a number per head), ``rot: {base, dims}``.  ``"attention"``: ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``,
``rot: {base, dims, scaling: {factor, low, high, original}}``.  ``scaling`` and ``logit_softcap`` may be absent; any other
missing key is an error that names it.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping

from .qwen2_config import ConfigError
from .zelasun_config import _count, _divides, _get, _number


@dataclass(frozen=True)
class Rotation:
    """A rotary encoding of the first ``dims`` elements, its long waves slowed by ``scaling`` (see ``parts/position.py``)."""

    base: float
    dims: int
    scaling: Mapping[str, float] | None = None

    @classmethod
    def read(cls, raw, room: int, where: str, scaling_keys: tuple[str, ...] = ()) -> "Rotation":
        rot = _get(raw, "rot", where)
        where = where + "rot."
        base, dims = _number(rot, "base", where), _count(rot, "dims", where)
        if dims % 2 or dims > room:
            raise ConfigError(f"{where}dims ({dims}) must be even and at most the {room} dimensions it turns a part of")
        if base <= 0:
            raise ConfigError(f"{where}base must be positive, got {base}")
        scaling = rot.get("scaling")
        if scaling is not None:
            if not scaling_keys:
                raise ConfigError(f"{where}scaling: this kind of layer has none")
            scaling = {key: _number(scaling, key, where + "scaling.") for key in scaling_keys}
            if min(scaling.values()) <= 0:
                raise ConfigError(f"{where}scaling: {', '.join(scaling_keys)} must be positive")
        return cls(base, dims, scaling)


@dataclass(frozen=True)
class WindowedLatentSizes:
    """Softmax attention over a window, through one latent per token, with a learned sink per head."""

    heads: int
    dim: int        # plain (unrotated) query/key dimensions per head
    rot_dim: int    # rotated query/key dimensions per head; the key's are one vector shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    window: int
    rot: Rotation

    @classmethod
    def read(cls, raw, where: str) -> "WindowedLatentSizes":
        rot_dim = _count(raw, "rot_dim", where)
        return cls(_count(raw, "heads", where), _count(raw, "dim", where), rot_dim, _count(raw, "vdim", where),
                   _count(raw, "kv_rank", where), _number(raw, "scale", where),
                   _count(_get(raw, "mask", where), "size", where + "mask."),
                   Rotation.read(raw, rot_dim, where, ("factor", "original", "fast", "slow")))


@dataclass(frozen=True)
class RetentionSizes:
    """Linear attention with a fixed decay per head."""

    heads: int
    dim: int
    vdim: int
    decay: tuple[float, ...]
    rot: Rotation

    @classmethod
    def read(cls, raw, where: str) -> "RetentionSizes":
        heads, dim = _count(raw, "heads", where), _count(raw, "dim", where)
        decay = _get(raw, "decay", where)
        if not isinstance(decay, (list, tuple)) or len(decay) != heads or not all(
                isinstance(d, (int, float)) and not isinstance(d, bool) for d in decay):
            raise ConfigError(f"{where}decay must list one number per head ({heads})")
        return cls(heads, dim, _count(raw, "vdim", where), tuple(float(d) for d in decay), Rotation.read(raw, dim, where))


@dataclass(frozen=True)
class UnitSinkAttentionSizes:
    """Grouped-query softmax attention with one added to the denominator."""

    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation

    @classmethod
    def read(cls, raw, where: str) -> "UnitSinkAttentionSizes":
        dim = _count(raw, "dim", where)
        out = cls(_count(raw, "heads", where), _count(raw, "kv_heads", where), dim, _count(raw, "vdim", where),
                  _number(raw, "scale", where), Rotation.read(raw, dim, where, ("factor", "low", "high", "original")))
        _divides(out.kv_heads, out.heads, where + "heads / kv_heads")
        return out


_MIXERS = {"latent_attention": WindowedLatentSizes, "retention": RetentionSizes, "attention": UnitSinkAttentionSizes}


@dataclass(frozen=True)
class CappedDenseSizes:
    ff: int
    limit: float


def _read_mlp(raw, where: str) -> CappedDenseSizes | None:
    if raw is None:
        return None
    kind = _get(raw, "kind", where)
    if kind != "dense":
        raise ConfigError(f"{where}kind {kind!r}: this design has dense feed-forwards only")
    out = CappedDenseSizes(_count(raw, "ff", where), _number(raw, "limit", where))
    if out.limit <= 0:
        raise ConfigError(f"{where}limit must be positive, got {out.limit}")
    return out


@dataclass(frozen=True)
class LabolixLayer:
    type: str                      # a key of _MIXERS
    mixer: Any                     # WindowedLatentSizes | RetentionSizes | UnitSinkAttentionSizes
    mlp: CappedDenseSizes | None


@dataclass(frozen=True)
class LabolixConfig:
    vocab: int
    width: int
    eps: float
    logit_softcap: float | None
    layers: tuple[LabolixLayer, ...]     # every entry of the file
    weights_of: tuple[int, ...]          # whose weights each entry runs: its own index, or an entry's that has its own
    eos_token_id: int | None = None
    architecture: str = "Labolix"
    extra: Mapping[str, Any] = field(default_factory=dict, compare=False)

    @staticmethod
    def _owners(listed) -> tuple[int, ...]:
        named = [entry.get("weights_of") if isinstance(entry, Mapping) else None for entry in listed]
        for index, j in enumerate(named):
            if j is not None and (isinstance(j, bool) or not isinstance(j, int) or not 0 <= j < len(named)):
                raise ConfigError(f"layers[{index}].weights_of must be a layer's index, got {j!r}")
        out = []
        for index in range(len(named)):
            at, seen = index, {index}
            while named[at] is not None:
                at = named[at]
                if at in seen:
                    raise ConfigError(f"layers[{index}].weights_of leads back to itself: no layer on the way has weights")
                seen.add(at)
            out.append(at)
        return tuple(out)

    @classmethod
    def from_dict(cls, raw: Mapping[str, Any]) -> "LabolixConfig":
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
            layers.append(LabolixLayer(kind, mixer, _read_mlp(entry.get("mlp"), where + "mlp.")))
        owners = cls._owners(listed)
        for index, j in enumerate(owners):
            if layers[index] != layers[j]:
                raise ConfigError(f"layers[{index}] runs the weights of layer {j} and must equal it in everything else")
        eos, cap = raw.get("eos_token_id"), raw.get("logit_softcap")
        if cap is not None and _number(raw, "logit_softcap", "") <= 0:
            raise ConfigError(f"logit_softcap must be positive, got {cap}")
        known = {"architecture", "architectures", "layers", "norm", "vocab", "width", "logit_softcap", "eos_token_id"}
        return cls(
            vocab=_count(raw, "vocab", ""),
            width=_count(raw, "width", ""),
            eps=_number(_get(raw, "norm", ""), "eps", "norm."),
            logit_softcap=float(cap) if cap is not None else None,
            layers=tuple(layers),
            weights_of=owners,
            eos_token_id=int(eos) if eos is not None else None,
            extra={k: v for k, v in raw.items() if k not in known},
        )
