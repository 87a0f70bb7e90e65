"""Typed configuration of the Mererax decoder.

Its config.json lists the layers one by one: ``layers`` is a list of objects with
``type``, ``mixer`` (that mixer's sizes), ``mlp`` (``{"kind": "dense", "ff": n}`` or
null for a layer without a feed-forward) and optionally ``weights_of``: j for a
layer that has no tensors of its own and runs layer j's (whose entry its own must
equal) on a cache and state of its own.  The mixers:

* ``parallel``: ``left`` (``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale`` and
  optionally ``q_temp`` with ``coef`` and ``every``) and ``right`` (``heads``, ``dim``,
  ``vdim``, ``gate_cap``);
* ``mamba1``: ``inner``, ``state``, ``dt_rank``, ``conv``.

Further keys: ``vocab``, ``width``, ``norm.eps`` and ``embedding.scale``.  Every size
and every constant a model of this design may choose comes from there; nothing
here names a model size.  The reference has no such architecture.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Mapping, Optional, Tuple

from .llama import ConfigError
from .ropovik import DenseMlp, _get

MIXER_TYPES = ("parallel", "mamba1")


@dataclass(frozen=True)
class QueryTemperature:
    coef: float
    every: float

    def to_json(self) -> dict:
        return {"coef": self.coef, "every": self.every}


@dataclass(frozen=True)
class SlopedAttention:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    q_temp: Optional[QueryTemperature]

    def to_json(self) -> dict:
        out = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.q_temp is not None:
            out["q_temp"] = self.q_temp.to_json()
        return out


@dataclass(frozen=True)
class MatrixMemory:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    def to_json(self) -> dict:
        return {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "gate_cap": self.gate_cap}


@dataclass(frozen=True)
class ParallelMixer:
    left: SlopedAttention
    right: MatrixMemory

    def to_json(self) -> dict:
        return {"left": self.left.to_json(), "right": self.right.to_json()}


@dataclass(frozen=True)
class Mamba1Mixer:
    inner: int
    state: int
    dt_rank: int
    conv: int

    def to_json(self) -> dict:
        return {"inner": self.inner, "state": self.state, "dt_rank": self.dt_rank, "conv": self.conv}


@dataclass(frozen=True)
class MereraxLayer:
    type: str                          # "parallel" | "mamba1"
    mixer: Any                         # ParallelMixer | Mamba1Mixer
    mlp: Optional[DenseMlp]
    weights_of: Optional[int] = None

    def to_json(self) -> dict:
        out = {"type": self.type, "mixer": self.mixer.to_json(), "mlp": self.mlp.to_json() if self.mlp else None}
        if self.weights_of is not None:
            out["weights_of"] = self.weights_of
        return out


def _read_left(m: Any, where: str) -> SlopedAttention:
    heads, kv = _get(m, "heads", where), _get(m, "kv_heads", where)
    if heads % kv:
        raise ConfigError(f"config.json: {where}: {heads} query heads cannot share {kv} key/value heads")
    dim = _get(m, "dim", where)
    vdim = _get(m, "vdim", where) if m.get("vdim") is not None else dim
    if vdim != dim:
        raise ConfigError(f"config.json: {where}: the values are the keys, so vdim ({vdim}) must equal dim ({dim})")
    temp = None
    if m.get("q_temp") is not None:
        w = where + ".q_temp"
        temp = QueryTemperature(_get(m["q_temp"], "coef", w, float, positive=False), _get(m["q_temp"], "every", w, float))
    return SlopedAttention(heads, kv, dim, vdim, _get(m, "scale", where, float), temp)


def _read_right(m: Any, where: str) -> MatrixMemory:
    return MatrixMemory(_get(m, "heads", where), _get(m, "dim", where), _get(m, "vdim", where), _get(m, "gate_cap", where, float))


def _read_mixer(kind: str, m: Mapping[str, Any], where: str):
    if kind == "parallel":
        for side in ("left", "right"):
            if not isinstance(m.get(side), Mapping):
                raise ConfigError(f"config.json: {where} lacks {side!r}")
        return ParallelMixer(_read_left(m["left"], where + ".left"), _read_right(m["right"], where + ".right"))
    return Mamba1Mixer(_get(m, "inner", where), _get(m, "state", where), _get(m, "dt_rank", where), _get(m, "conv", where))


@dataclass(frozen=True)
class MereraxConfig:
    vocab: int
    width: int
    layers: Tuple[MereraxLayer, ...]
    norm_eps: float
    embedding_scale: float

    @staticmethod
    def from_json(raw: Mapping[str, Any]) -> "MereraxConfig":
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
            if not isinstance(entry.get("mixer"), Mapping):
                raise ConfigError(f"config.json: {where} lacks 'mixer'")
            mlp = None
            if entry.get("mlp") is not None:
                if not isinstance(entry["mlp"], Mapping) or entry["mlp"].get("kind", "dense") != "dense":
                    raise ConfigError(f"config.json: {where}.mlp.kind is not known: 'dense'")
                mlp = DenseMlp(_get(entry["mlp"], "ff", where + ".mlp"))
            source = entry.get("weights_of")
            if source is not None and (isinstance(source, bool) or not isinstance(source, int)
                                       or not 0 <= source < len(raw["layers"]) or source == i):
                raise ConfigError(f"config.json: {where}.weights_of must name another layer, got {source!r}")
            layers.append(MereraxLayer(kind, _read_mixer(kind, entry["mixer"], where + ".mixer"), mlp, source))
        scale = 1.0
        if raw.get("embedding") is not None:
            scale = _get(raw["embedding"], "scale", "embedding", float)
        cfg = MereraxConfig(vocab, width, tuple(layers), _get(raw.get("norm") or {}, "eps", "norm", float), scale)
        for i, layer in enumerate(cfg.layers):
            src = cfg.layers[cfg.source_of(i)]
            if (src.type, src.mixer, src.mlp) != (layer.type, layer.mixer, layer.mlp):
                raise ConfigError(f"config.json: layers[{i}] runs the tensors of layer {cfg.source_of(i)}, so the rest of its entry "
                                  f"must equal that layer's")
        return cfg

    def source_of(self, i: int) -> int:
        """The layer whose tensors layer i runs (itself, where it has its own)."""
        seen = set()
        while self.layers[i].weights_of is not None:
            if i in seen:
                raise ConfigError(f"config.json: layers[{i}].weights_of leads back to itself")
            seen.add(i)
            i = self.layers[i].weights_of
        return i

    def to_json(self) -> dict:
        return {"architecture": "Mererax", "vocab": self.vocab, "width": self.width,
                "layers": [layer.to_json() for layer in self.layers], "norm": {"eps": self.norm_eps},
                "embedding": {"scale": self.embedding_scale}}
