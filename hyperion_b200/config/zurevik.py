"""Typed configuration of the Zurevik decoder.

Its config.json is nested: ``architecture`` (the name), ``vocab``, ``width``, ``embedding.scale``, ``norm.eps``, ``logit_softcap`` and ``layers``, a list
whose entries give ``type`` (``attention`` or ``attention_2``), the mixer's sizes under ``mixer`` and the feed-forward under ``mlp``
(``{"kind": "moe", "expert": {"ff": n}, "router": {"experts": n, "top": k}}`` or null).  An ``attention_2`` mixer may name another layer under
``kv_from``: it has no keys and values of its own then and reads that layer's.  Every size and constant is read from there; nothing is
assumed equal between layers.  A key that is missing or of the wrong kind is refused by name.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any, Optional

from .base import ConfigError
from .nunivik import _get, _positive_int, _positive_number

ARCHITECTURE = "Zurevik"


@dataclass(frozen=True)
class DifferentialSizes:
    heads: int
    kv_heads: int
    dim: int  # of a query or key of one of the two maps
    vdim: int
    scale: float
    diff: float
    window: int  # 0: every earlier key is seen
    keep_first: int  # the first positions that are seen beside the window


@dataclass(frozen=True)
class SinkAttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int  # 0: every earlier key is seen
    kv_from: Optional[int] = None  # the layer whose keys and values are read


@dataclass(frozen=True)
class ExpertsFF:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class ZurevikLayer:
    type: str
    mixer: Any
    mlp: Optional[ExpertsFF]


@dataclass(frozen=True)
class ZurevikConfig:
    vocab: int
    width: int
    embedding_scale: float
    eps: float
    logit_softcap: float  # 0: none
    layers: tuple[ZurevikLayer, ...]
    eos_token_ids: tuple[int, ...] = ()
    architecture: str = field(default=ARCHITECTURE)

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def cache_window(self, index: int) -> int:
        """The widest window that reads the keys and values of layer ``index`` (0: one of them sees every key)."""
        readers = [layer.mixer.window for i, layer in enumerate(self.layers) if i == index or getattr(layer.mixer, "kv_from", None) == index]
        return 0 if 0 in readers else max(readers)

    @classmethod
    def from_dict(cls, document: dict[str, Any]) -> "ZurevikConfig":
        if not isinstance(document, dict):
            raise ConfigError("<root>", "must be a JSON object")
        if document.get("architecture") != ARCHITECTURE:
            raise ConfigError("architecture", f"must be {ARCHITECTURE!r}, got {document.get('architecture')!r}")
        width = _positive_int(document, "", "width")
        norm = _get(document, "", "norm")
        embedding = document.get("embedding")
        entries = _get(document, "", "layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("layers", "must be a non-empty list")
        layers: list[ZurevikLayer] = []
        for index, entry in enumerate(entries):
            path = f"layers[{index}]."
            kind = _get(entry, path, "type")
            mixer = _get(entry, path, "mixer")
            if kind == "attention":
                parsed: Any = _differential(mixer, path + "mixer.")
            elif kind == "attention_2":
                parsed = _sink_attention(mixer, path + "mixer.")
            else:
                raise ConfigError(path + "type", f"{kind!r} is not a mixer of this design (attention, attention_2)")
            mlp = entry.get("mlp")
            layers.append(ZurevikLayer(kind, parsed, _experts(mlp, path + "mlp.") if mlp is not None else None))
        for index, layer in enumerate(layers):
            source = getattr(layer.mixer, "kv_from", None)
            if source is None:
                continue
            path = f"layers[{index}].mixer.kv_from"
            if not 0 <= source < index:
                raise ConfigError(path, f"must name an earlier layer, got {source}")
            lender = layers[source]
            if lender.type != layer.type or lender.mixer.kv_from is not None:
                raise ConfigError(path, f"layer {source} has no keys and values of this mixer's kind to lend")
            if any(getattr(lender.mixer, name) != getattr(layer.mixer, name) for name in ("kv_heads", "dim", "vdim")):
                raise ConfigError(path, f"layer {source} has key/value heads of another number or size")
        eos = document.get("eos_token_id")
        eos_ids = tuple(eos if isinstance(eos, list) else [eos]) if eos is not None else ()
        return cls(vocab=_positive_int(document, "", "vocab"), width=width,
                   embedding_scale=_number(embedding, "embedding.", "scale") if embedding is not None and embedding.get("scale") is not None else 1.0,
                   eps=_positive_number(norm, "norm.", "eps"),
                   logit_softcap=_positive_number(document, "", "logit_softcap") if document.get("logit_softcap") is not None else 0.0,
                   layers=tuple(layers), eos_token_ids=eos_ids)

    def to_dict(self) -> dict[str, Any]:
        """The config.json document this configuration is read back from."""
        layers = []
        for layer in self.layers:
            m = layer.mixer
            mixer: dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            if m.window:
                mixer["mask"] = {"size": m.window}
            if layer.type == "attention":
                mixer["diff"] = m.diff
                if m.window:
                    mixer["mask"]["keep_first"] = m.keep_first
            elif m.kv_from is not None:
                mixer["kv_from"] = m.kv_from
            f = layer.mlp
            mlp = {"kind": "moe", "expert": {"ff": f.ff}, "router": {"experts": f.experts, "top": f.top}} if f is not None else None
            layers.append({"type": layer.type, "mixer": mixer, "mlp": mlp})
        document: dict[str, Any] = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": {"scale": self.embedding_scale},
                                    "norm": {"eps": self.eps}, "layers": layers}
        if self.logit_softcap:
            document["logit_softcap"] = self.logit_softcap
        if self.eos_token_ids:
            document["eos_token_id"] = list(self.eos_token_ids)
        return document


def _number(mapping: Any, path: str, key: str) -> float:
    value = _get(mapping, path, key)
    if isinstance(value, bool) or not isinstance(value, (int, float)) or not math.isfinite(value):
        raise ConfigError(path + key, f"must be a number, got {value!r}")
    return float(value)


def _heads(m: Any, path: str) -> dict[str, Any]:
    heads, kv_heads = _positive_int(m, path, "heads"), _positive_int(m, path, "kv_heads")
    if heads % kv_heads:
        raise ConfigError(path + "kv_heads", f"{kv_heads} does not divide heads {heads}")
    mask = m.get("mask")
    return {"heads": heads, "kv_heads": kv_heads, "dim": _positive_int(m, path, "dim"), "vdim": _positive_int(m, path, "vdim"), "scale": _number(m, path, "scale"),
            "window": _positive_int(mask, path + "mask.", "size") if mask is not None else 0}


def _differential(m: Any, path: str) -> DifferentialSizes:
    sizes = _heads(m, path)
    keep = (m.get("mask") or {}).get("keep_first") or 0
    if isinstance(keep, bool) or not isinstance(keep, int) or keep < 0:
        raise ConfigError(path + "mask.keep_first", f"must be a non-negative integer, got {keep!r}")
    return DifferentialSizes(**sizes, diff=_number(m, path, "diff"), keep_first=keep)


def _sink_attention(m: Any, path: str) -> SinkAttentionSizes:
    source = m.get("kv_from")
    if source is not None and (isinstance(source, bool) or not isinstance(source, int)):
        raise ConfigError(path + "kv_from", f"must name a layer of the model, got {source!r}")
    return SinkAttentionSizes(**_heads(m, path), kv_from=source)


def _experts(mlp: Any, path: str) -> ExpertsFF:
    kind = _get(mlp, path, "kind")
    if kind != "moe":
        raise ConfigError(path + "kind", f"{kind!r} is not supported ('moe')")
    router = _get(mlp, path, "router")
    experts, top = _positive_int(router, path + "router.", "experts"), _positive_int(router, path + "router.", "top")
    if top > experts:
        raise ConfigError(path + "router.top", f"{top} of {experts} experts")
    return ExpertsFF(ff=_positive_int(_get(mlp, path, "expert"), path + "expert.", "ff"), experts=experts, top=top)
