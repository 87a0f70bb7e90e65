"""Typed configuration of the Letanex decoder.

Its config.json lists the layers one by one: ``layers`` is a list of objects with
``type``, ``mixer`` (that mixer's sizes) and ``mlp`` (or null for a layer without a
feed-forward).  The mixers:

* ``attention``: ``heads``, ``kv_heads``, ``dim`` (channels of one map of a query or key
  head), ``vdim``, ``scale``, ``diff``, and optionally ``rot`` (``dims``, ``base`` and
  optionally ``scaling.factor``) and ``kv_from``: j for a layer that has no key and value
  projections and reads layer j's cache;
* ``lightning``: ``heads``, ``dim``, ``vdim``, ``decay`` (one number a head).

The feed-forwards: ``{"kind": "dense", "ff"}`` and ``{"kind": "moe", "expert": {"ff",
"limit"}, "router": {"experts", "top", "identity", "scale"}, "shared": {"ff", "limit"}}``
(``identity``, ``scale`` and ``shared`` may be missing: none, 1 and none).

Further keys: ``vocab``, ``width``, ``norm.eps``.  Every size and every constant a model
of this design may choose comes from there; nothing here names a model size.  The
reference has no such architecture.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple, Union

from .llama import ConfigError
from .ropovik import DenseMlp, _get

MIXER_TYPES = ("attention", "lightning")
MLP_KINDS = ("dense", "moe")


@dataclass(frozen=True)
class LinearRotation:
    dims: int
    base: float
    factor: Optional[float] = None

    def to_json(self) -> dict:
        out = {"dims": self.dims, "base": self.base}
        if self.factor is not None:
            out["scaling"] = {"factor": self.factor}
        return out


@dataclass(frozen=True)
class DifferentialMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    rot: Optional[LinearRotation]
    kv_from: Optional[int] = None

    def to_json(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale, "diff": self.diff}
        if self.rot is not None:
            out["rot"] = self.rot.to_json()
        if self.kv_from is not None:
            out["kv_from"] = self.kv_from
        return out


@dataclass(frozen=True)
class LightningMixer:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]

    def to_json(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "decay": list(self.decay)}


@dataclass(frozen=True)
class ClampedExpert:
    ff: int
    limit: float

    def to_json(self) -> dict:
        return {"ff": self.ff, "limit": self.limit}


@dataclass(frozen=True)
class MixtureMlp:
    expert: ClampedExpert
    experts: int
    top: int
    identity: int
    scale: float
    shared: Optional[ClampedExpert]

    def to_json(self) -> dict:
        out = {"kind": "moe", "expert": self.expert.to_json(),
               "router": {"experts": self.experts, "top": self.top, "identity": self.identity, "scale": self.scale}}
        if self.shared is not None:
            out["shared"] = self.shared.to_json()
        return out


@dataclass(frozen=True)
class LetanexLayer:
    type: str                          # "attention" | "lightning"
    mixer: Union[DifferentialMixer, LightningMixer]
    mlp: Optional[Union[DenseMlp, MixtureMlp]]

    def to_json(self) -> dict:
        return {"type": self.type, "mixer": self.mixer.to_json(), "mlp": self.mlp.to_json() if self.mlp else None}


def _block(m: Mapping[str, Any], key: str, where: str) -> Mapping[str, Any]:
    if not isinstance(m.get(key), Mapping):
        raise ConfigError(f"config.json: {where} lacks {key!r}")
    return m[key]


def _read_rotation(r: Any, where: str, most: int) -> Optional[LinearRotation]:
    if r is None:
        return None
    dims, base = _get(r, "dims", where), _get(r, "base", where, float)
    if dims % 2 or dims > most:
        raise ConfigError(f"config.json: {where}.dims must be even and at most {most}, got {dims}")
    if base <= 1.0:
        raise ConfigError(f"config.json: {where}.base must exceed 1, got {base}")
    factor = None
    if r.get("scaling") is not None:
        factor = _get(r["scaling"], "factor", where + ".scaling", float)
    return LinearRotation(dims, base, factor)


def _read_attention(m: Mapping[str, Any], where: str, index: int) -> DifferentialMixer:
    heads, kv = _get(m, "heads", where), _get(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}: {heads} query heads cannot share {kv} key/value heads")
    dim = _get(m, "dim", where)
    source = m.get("kv_from")
    if source is not None and (isinstance(source, bool) or not isinstance(source, int) or not 0 <= source < index):
        raise ConfigError(f"config.json: {where}.kv_from must name an earlier layer, got {source!r}")
    return DifferentialMixer(heads, kv, dim, _get(m, "vdim", where), _get(m, "scale", where, float),
                             _get(m, "diff", where, float, positive=False), _read_rotation(m.get("rot"), where + ".rot", dim), source)


def _read_lightning(m: Mapping[str, Any], where: str) -> LightningMixer:
    heads = _get(m, "heads", where)
    decay = m.get("decay")
    if (not isinstance(decay, (list, tuple)) or len(decay) != heads
            or any(isinstance(a, bool) or not isinstance(a, (int, float)) or not 0.0 <= a <= 1.0 for a in decay)):
        raise ConfigError(f"config.json: {where}.decay must list {heads} numbers between 0 and 1, got {decay!r}")
    return LightningMixer(heads, _get(m, "dim", where), _get(m, "vdim", where), tuple(float(a) for a in decay))


def _read_expert(m: Mapping[str, Any], where: str) -> ClampedExpert:
    return ClampedExpert(_get(m, "ff", where), _get(m, "limit", where, float))


def _read_mlp(m: Any, where: str) -> Optional[Union[DenseMlp, MixtureMlp]]:
    if m is None:
        return None
    if not isinstance(m, Mapping) or m.get("kind", "dense") not in MLP_KINDS:
        raise ConfigError(f"config.json: {where}.kind is not known: {', '.join(map(repr, MLP_KINDS))}")
    if m.get("kind", "dense") == "dense":
        return DenseMlp(_get(m, "ff", where))
    router, w = _block(m, "router", where), where + ".router"
    experts, top = _get(router, "experts", w), _get(router, "top", w)
    identity = router.get("identity") or 0
    if isinstance(identity, bool) or not isinstance(identity, int) or identity < 0:
        raise ConfigError(f"config.json: {w}.identity must be a number of experts, got {identity!r}")
    if top > experts + identity:
        raise ConfigError(f"config.json: {w}: a token cannot use {top} of {experts + identity} experts")
    scale = _get(router, "scale", w, float) if router.get("scale") is not None else 1.0
    shared = _read_expert(_block(m, "shared", where), where + ".shared") if m.get("shared") is not None else None
    return MixtureMlp(_read_expert(_block(m, "expert", where), where + ".expert"), experts, top, identity, scale, shared)


@dataclass(frozen=True)
class LetanexConfig:
    vocab: int
    width: int
    layers: Tuple[LetanexLayer, ...]
    norm_eps: float

    @staticmethod
    def from_json(raw: Mapping[str, Any]) -> "LetanexConfig":
        vocab, width = _get(raw, "vocab", "the model"), _get(raw, "width", "the model")
        if not isinstance(raw.get("layers"), (list, tuple)) or not raw["layers"]:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw["layers"]):
            where = f"layers[{i}]"
            if not isinstance(entry, Mapping):
                raise ConfigError(f"config.json: {where} must be an object")
            kind = entry.get("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not known: {', '.join(map(repr, MIXER_TYPES))}")
            m, w = _block(entry, "mixer", where), where + ".mixer"
            mixer = _read_attention(m, w, i) if kind == "attention" else _read_lightning(m, w)
            source = getattr(mixer, "kv_from", None)
            if source is not None:
                src = layers[source]
                if src.type != "attention" or src.mixer.kv_from is not None:
                    raise ConfigError(f"config.json: {w}.kv_from names layer {source}, which has no keys and values of its own for this "
                                      f"layer to read")
                if (src.mixer.kv_heads, src.mixer.dim, src.mixer.vdim, src.mixer.rot) != (mixer.kv_heads, mixer.dim, mixer.vdim, mixer.rot):
                    raise ConfigError(f"config.json: {w} reads layer {source}'s keys and values, so kv_heads, dim, vdim and rot must equal "
                                      f"that layer's")
            layers.append(LetanexLayer(kind, mixer, _read_mlp(entry.get("mlp"), where + ".mlp")))
        return LetanexConfig(vocab, width, tuple(layers), _get(raw.get("norm") or {}, "eps", "norm", float))

    def to_json(self) -> dict:
        return {"architecture": "Letanex", "vocab": self.vocab, "width": self.width,
                "layers": [layer.to_json() for layer in self.layers], "norm": {"eps": self.norm_eps}}
