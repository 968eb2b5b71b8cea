"""Linurax configuration.

config.json of this design is nested: ``vocab``, ``width``, ``embedding.scale``, ``norm.eps`` and one entry per layer under
``layers``: ``type`` ("attention" or "mingru"), the mixer's sizes and constants under ``mixer`` and the feed-forward under
``mlp`` (``kind`` "dense" with ``ff``, or null for none).

An "attention" mixer has heads, kv_heads, dim, vdim (equal to dim: the projected keys are the values), scale and ``rot``
(dims, base; null or absent: no rotation). A "mingru" mixer has ``width``, the number of its recurrent channels. Every size
comes from here or from a tensor's shape; nothing is assumed equal between layers.
"""
from __future__ import annotations

import dataclasses
from typing import Any, Dict, Tuple

from .base import ConfigError, ModelConfig
from .delunex import _number, _positive_int
from .pilonex import _object

MIXER_TYPES = ("attention", "mingru")
MLP_KINDS = ("dense",)


@dataclasses.dataclass(frozen=True)
class LinuraxConfig(ModelConfig):
    architecture = "Linurax"
    model_type = ""

    vocab: int
    width: int
    layers: Tuple[dict, ...]
    embedding: dict
    norm: dict
    max_position_embeddings: int = 65536      # positions the rotation tables are made for
    stop_token_ids: Tuple[int, ...] = ()

    def validate(self) -> None:
        if self.vocab <= 0 or self.width <= 0:
            raise ConfigError(f"vocab and width must be positive, got {self.vocab} and {self.width}")
        if not isinstance(self.norm, dict) or not _number("norm", self.norm, "eps") > 0.0:
            raise ConfigError("norm.eps must be a number > 0")
        if not isinstance(self.embedding, dict):
            raise ConfigError(f"'embedding' must be an object with a 'scale', got {self.embedding!r}")
        _number("embedding", self.embedding, "scale")
        if not self.layers:
            raise ConfigError("'layers' must list at least one layer")
        for i, layer in enumerate(self.layers):
            where = f"layers[{i}]"
            if not isinstance(layer, dict) or not isinstance(layer.get("mixer"), dict):
                raise ConfigError(f"{where}: an object with a 'mixer' object is expected")
            if layer.get("type") not in MIXER_TYPES:
                raise ConfigError(f"{where}: type {layer.get('type')!r} is not known (known: {', '.join(MIXER_TYPES)})")
            m, mw = layer["mixer"], where + ".mixer"
            if layer["type"] == "mingru":
                _positive_int(mw, m, "width")
            else:
                heads, kv = _positive_int(mw, m, "heads"), _positive_int(mw, m, "kv_heads")
                if heads % kv:
                    raise ConfigError(f"{mw}: {heads} heads do not divide into {kv} kv_heads")
                dim = _positive_int(mw, m, "dim")
                if _positive_int(mw, m, "vdim") != dim:
                    raise ConfigError(f"{mw}: vdim {m['vdim']} must equal dim {dim} (the projected keys are the values)")
                _number(mw, m, "scale")
                if m.get("rot") is not None:
                    rot = _object(mw, m, "rot")
                    dims = _positive_int(mw + ".rot", rot, "dims")
                    if dims % 2 or dims > dim:
                        raise ConfigError(f"{mw}.rot: dims {dims} must be even and at most dim {dim}")
                    if not _number(mw + ".rot", rot, "base") > 0.0:
                        raise ConfigError(f"{mw}.rot: base must be > 0")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") not in MLP_KINDS:
                    raise ConfigError(f"{where}.mlp: kind must be one of {', '.join(MLP_KINDS)}, or the mlp null")
                _positive_int(where + ".mlp", mlp, "ff")

    def with_stop_token_ids(self, ids) -> "LinuraxConfig":
        return dataclasses.replace(self, stop_token_ids=tuple(int(i) for i in ids))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": dict(self.embedding),
            "norm": dict(self.norm), "layers": [dict(layer) for layer in self.layers],
        }
        if self.max_position_embeddings != 65536:
            d["max_position_embeddings"] = self.max_position_embeddings
        return d
