"""Typed configuration of the Biropel decoder.

Its config.json is nested: ``architecture`` (the name), ``vocab``, ``width``, ``streams`` (residual streams), ``norm.eps`` and ``layers``, a list whose entries give
``type`` (``attention``, ``parallel`` or ``parallel_2``), the mixer's sizes under ``mixer`` and the feed-forward under ``mlp`` (``{"kind": "dense", "ff": n}`` or null).
An attention's sizes are ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale`` and, each optional, ``mask.size`` (a window), ``rot`` (``dims``, ``base`` and perhaps
``scaling``: ``factor``, ``original``, ``fast``, ``slow``), ``softcap`` and ``q_temp`` (``coef``, ``every``).  An ``attention`` mixer may name another layer under
``kv_from``: it has no keys and values of its own then and reads that layer's.  The other two types hold such an attention under ``left`` and, under ``right``, a
state-space mixer (``parallel``: ``heads``, ``vdim``, ``state``, ``groups``, ``norm_groups``, ``conv``) or a matrix memory (``parallel_2``: ``heads``, ``dim``,
``vdim``, ``gate_cap``).  Every size and constant is read from there; nothing is assumed equal between layers.  A key that is missing or of the
wrong kind is refused by name.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Optional

from .base import ConfigError
from .nunivik import _get, _positive_int, _positive_number

ARCHITECTURE = "Biropel"


@dataclass(frozen=True)
class RotationScaling:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    scaling: Optional[RotationScaling] = None


@dataclass(frozen=True)
class QueryTemperature:
    coef: float
    every: int


@dataclass(frozen=True)
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int = 0  # 0: every earlier key is seen
    softcap: float = 0.0  # 0: scores are not capped
    rot: Optional[Rotation] = None
    q_temp: Optional[QueryTemperature] = None
    kv_from: Optional[int] = None  # the layer whose keys and values are read


@dataclass(frozen=True)
class StateSpaceSizes:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int


@dataclass(frozen=True)
class MatrixMemorySizes:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class ParallelMixer:
    left: AttentionSizes
    right: Any  # StateSpaceSizes or MatrixMemorySizes


@dataclass(frozen=True)
class BiropelLayer:
    type: str
    mixer: Any  # AttentionSizes or ParallelMixer
    ff: Optional[int]  # the feed-forward's inner width, None: no feed-forward


@dataclass(frozen=True)
class BiropelConfig:
    vocab: int
    width: int
    streams: int
    eps: float
    layers: tuple[BiropelLayer, ...]
    eos_token_ids: tuple[int, ...] = ()
    architecture: str = field(default=ARCHITECTURE)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def cache_window(self, index: int) -> int:
        """The widest window that reads the keys and values of the ``attention`` layer ``index`` (0: one of them sees every key)."""
        readers = [layer.mixer.window for i, layer in enumerate(self.layers) if layer.type == "attention" and (i == index or layer.mixer.kv_from == index)]
        return 0 if 0 in readers else max(readers)

    @classmethod
    def from_dict(cls, document: dict[str, Any]) -> "BiropelConfig":
        if not isinstance(document, dict):
            raise ConfigError("<root>", "must be a JSON object")
        if document.get("architecture") != ARCHITECTURE:
            raise ConfigError("architecture", f"must be {ARCHITECTURE!r}, got {document.get('architecture')!r}")
        entries = _get(document, "", "layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("layers", "must be a non-empty list")
        layers: list[BiropelLayer] = []
        for index, entry in enumerate(entries):
            path = f"layers[{index}]."
            kind = _get(entry, path, "type")
            mixer = _get(entry, path, "mixer")
            if kind == "attention":
                parsed: Any = _attention(mixer, path + "mixer.")
            elif kind in ("parallel", "parallel_2"):
                left = _attention(_get(mixer, path + "mixer.", "left"), path + "mixer.left.")
                if left.kv_from is not None:
                    raise ConfigError(path + "mixer.left.kv_from", "only a layer of type 'attention' reads another layer's keys and values")
                right = _get(mixer, path + "mixer.", "right")
                parsed = ParallelMixer(left, (_state_space if kind == "parallel" else _matrix_memory)(right, path + "mixer.right."))
            else:
                raise ConfigError(path + "type", f"{kind!r} is not a mixer of this design (attention, parallel, parallel_2)")
            layers.append(BiropelLayer(kind, parsed, _feed_forward(entry.get("mlp"), path + "mlp.")))
        for index, layer in enumerate(layers):
            source = layer.mixer.kv_from if layer.type == "attention" else None
            if source is None:
                continue
            path = f"layers[{index}].mixer.kv_from"
            if not 0 <= source < index:
                raise ConfigError(path, f"must name an earlier layer, got {source}")
            lender = layers[source]
            if lender.type != "attention" or lender.mixer.kv_from is not None:
                raise ConfigError(path, f"layer {source} has no keys and values of this mixer's kind to lend")
            if any(getattr(lender.mixer, name) != getattr(layer.mixer, name) for name in ("kv_heads", "dim", "vdim")):
                raise ConfigError(path, f"layer {source} has key/value heads of another number or size")
        eos = document.get("eos_token_id")
        eos_ids = tuple(eos if isinstance(eos, list) else [eos]) if eos is not None else ()
        return cls(vocab=_positive_int(document, "", "vocab"), width=_positive_int(document, "", "width"), streams=_positive_int(document, "", "streams"),
                   eps=_positive_number(_get(document, "", "norm"), "norm.", "eps"), layers=tuple(layers), eos_token_ids=eos_ids)

    def to_dict(self) -> dict[str, Any]:
        """The config.json document this configuration is read back from."""
        layers = []
        for layer in self.layers:
            if layer.type == "attention":
                mixer: dict[str, Any] = _attention_document(layer.mixer)
            else:
                right = layer.mixer.right
                names = ("heads", "vdim", "state", "groups", "norm_groups", "conv") if layer.type == "parallel" else ("heads", "dim", "vdim", "gate_cap")
                mixer = {"left": _attention_document(layer.mixer.left), "right": {name: getattr(right, name) for name in names}}
            layers.append({"type": layer.type, "mixer": mixer, "mlp": {"kind": "dense", "ff": layer.ff} if layer.ff is not None else None})
        document: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams, "norm": {"eps": self.eps},
                                    "layers": layers}
        if self.eos_token_ids:
            document["eos_token_id"] = list(self.eos_token_ids)
        return document


def _number(mapping: Any, path: str, key: str) -> float:
    value = _get(mapping, path, key)
    if isinstance(value, bool) or not isinstance(value, (int, float)) or not math.isfinite(value):
        raise ConfigError(path + key, f"must be a number, got {value!r}")
    return float(value)


def _rotation(rot: Any, path: str, dim: int) -> Optional[Rotation]:
    if rot is None:
        return None
    dims = _get(rot, path, "dims")
    if isinstance(dims, bool) or not isinstance(dims, int) or dims < 0 or dims % 2 or dims > dim:
        raise ConfigError(path + "dims", f"must be even and at most dim {dim}, got {dims!r}")
    scaling = rot.get("scaling")
    base = _positive_number(rot, path, "base")
    if scaling is not None:
        if base == 1.0:
            raise ConfigError(path + "base", "must not be 1 where the frequencies are scaled")
        names = ("factor", "original", "fast", "slow")
        scaling = RotationScaling(*(_positive_number(scaling, path + "scaling.", name) for name in names))
    return Rotation(dims, base, scaling)


def _attention(m: Any, path: str) -> AttentionSizes:
    heads, kv_heads = _positive_int(m, path, "heads"), _positive_int(m, path, "kv_heads")
    if heads % kv_heads:
        raise ConfigError(path + "kv_heads", f"{kv_heads} does not divide heads {heads}")
    dim = _positive_int(m, path, "dim")
    mask, temp, source = m.get("mask"), m.get("q_temp"), m.get("kv_from")
    if source is not None and (isinstance(source, bool) or not isinstance(source, int)):
        raise ConfigError(path + "kv_from", f"must name a layer of the model, got {source!r}")
    return AttentionSizes(heads=heads, kv_heads=kv_heads, dim=dim, vdim=_positive_int(m, path, "vdim"), scale=_number(m, path, "scale"),
                          window=_positive_int(mask, path + "mask.", "size") if mask is not None else 0,
                          softcap=_positive_number(m, path, "softcap") if m.get("softcap") is not None else 0.0,
                          rot=_rotation(m.get("rot"), path + "rot.", dim),
                          q_temp=QueryTemperature(_number(temp, path + "q_temp.", "coef"), _positive_int(temp, path + "q_temp.", "every")) if temp is not None else None,
                          kv_from=source)


def _attention_document(m: AttentionSizes) -> dict[str, Any]:
    document: dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
    if m.window:
        document["mask"] = {"size": m.window}
    if m.softcap:
        document["softcap"] = m.softcap
    if m.rot is not None:
        document["rot"] = {"dims": m.rot.dims, "base": m.rot.base}
        if m.rot.scaling is not None:
            s = m.rot.scaling
            document["rot"]["scaling"] = {"factor": s.factor, "original": s.original, "fast": s.fast, "slow": s.slow}
    if m.q_temp is not None:
        document["q_temp"] = {"coef": m.q_temp.coef, "every": m.q_temp.every}
    if m.kv_from is not None:
        document["kv_from"] = m.kv_from
    return document


def _state_space(m: Any, path: str) -> StateSpaceSizes:
    sizes = StateSpaceSizes(**{name: _positive_int(m, path, name) for name in ("heads", "vdim", "state", "groups", "norm_groups", "conv")})
    if sizes.heads % sizes.groups:
        raise ConfigError(path + "groups", f"{sizes.groups} does not divide heads {sizes.heads}")
    if sizes.heads * sizes.vdim % sizes.norm_groups:
        raise ConfigError(path + "norm_groups", f"{sizes.norm_groups} does not divide the inner width {sizes.heads * sizes.vdim}")
    return sizes


def _matrix_memory(m: Any, path: str) -> MatrixMemorySizes:
    return MatrixMemorySizes(heads=_positive_int(m, path, "heads"), dim=_positive_int(m, path, "dim"), vdim=_positive_int(m, path, "vdim"),
                             gate_cap=_positive_number(m, path, "gate_cap"))


def _feed_forward(mlp: Any, path: str) -> Optional[int]:
    if mlp is None:
        return None
    kind = _get(mlp, path, "kind")
    if kind != "dense":
        raise ConfigError(path + "kind", f"{kind!r} is not supported ('dense')")
    return _positive_int(mlp, path, "ff")
