"""Rolevik configuration.

config.json of this design is nested: ``vocab``, ``width``, ``embedding.scale``, ``norm.eps``, ``logit_scale`` and one entry per
layer under ``layers``: ``type`` ("parallel" or "rglru"), the mixer's sizes and constants under ``mixer`` and the feed-forward
under ``mlp`` (``kind`` "dense" with ``ff``, ``kind`` "moe", or null for none).

A "parallel" mixer has a ``left`` (attention in chunks: heads, kv_heads, dim, vdim, scale, optional mask.size, optional rot with
dims and base) and a ``right`` (gated delta rule: heads, kv_heads, dim, vdim, conv). An "rglru" mixer has ``width`` (its
recurrent channels), ``blocks`` (equal parts of them) and ``conv``. A "moe" feed-forward has ``expert.ff``, ``router`` (experts, top,
optional scale, identity, and groups with count and keep) and optionally ``shared.ff``. Every size comes from here or from a
tensor's shape; nothing is assumed equal between layers.
"""
from __future__ import annotations

import dataclasses
from typing import Any, Dict, Tuple

from .base import ConfigError, ModelConfig
from .delunex import _number, _positive_int
from .pilonex import _object

MIXER_TYPES = ("parallel", "rglru")
MLP_KINDS = ("dense", "moe")


def _heads(where: str, m: Dict[str, Any]) -> None:
    heads, kv = _positive_int(where, m, "heads"), _positive_int(where, m, "kv_heads")
    if heads % kv:
        raise ConfigError(f"{where}: {heads} heads do not divide into {kv} kv_heads")
    for key in ("dim", "vdim"):
        _positive_int(where, m, key)


def _check_parallel(where: str, m: Dict[str, Any]) -> None:
    left, right = _object(where, m, "left"), _object(where, m, "right")
    lw, rw = where + ".left", where + ".right"
    _heads(lw, left)
    _number(lw, left, "scale")
    if left.get("mask") is not None:
        _positive_int(lw + ".mask", _object(lw, left, "mask"), "size")
    if left.get("rot") is not None:
        rot = _object(lw, left, "rot")
        dims = _positive_int(lw + ".rot", rot, "dims")
        if dims % 2 or dims > int(left["dim"]):
            raise ConfigError(f"{lw}.rot: dims {dims} must be even and at most dim {left['dim']}")
        if not _number(lw + ".rot", rot, "base") > 0.0:
            raise ConfigError(f"{lw}.rot: base must be > 0")
    _heads(rw, right)
    _positive_int(rw, right, "conv")


def _check_moe(where: str, mlp: Dict[str, Any]) -> None:
    _positive_int(where + ".expert", _object(where, mlp, "expert"), "ff")
    router, rw = _object(where, mlp, "router"), where + ".router"
    experts, top = _positive_int(rw, router, "experts"), _positive_int(rw, router, "top")
    identity = router.get("identity") or 0
    if isinstance(identity, bool) or not isinstance(identity, int) or identity < 0:
        raise ConfigError(f"{rw}: identity must be an integer >= 0, got {identity!r}")
    if router.get("scale") is not None:
        _number(rw, router, "scale")
    count = keep = 1
    if router.get("groups") is not None:
        groups = _object(rw, router, "groups")
        count, keep = _positive_int(rw + ".groups", groups, "count"), _positive_int(rw + ".groups", groups, "keep")
    choices = experts + identity
    if keep > count or choices % count or (choices // count) * keep < top:
        raise ConfigError(f"{rw}: {choices} choices in {count} groups of which {keep} are kept cannot give {top}")
    if mlp.get("shared") is not None:
        _positive_int(where + ".shared", _object(where, mlp, "shared"), "ff")


@dataclasses.dataclass(frozen=True)
class RolevikConfig(ModelConfig):
    architecture = "Rolevik"
    model_type = ""

    vocab: int
    width: int
    layers: Tuple[dict, ...]
    embedding: dict
    norm: dict
    logit_scale: float = 1.0
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
            if layer["type"] == "parallel":
                _check_parallel(mw, m)
            else:
                width, blocks = _positive_int(mw, m, "width"), _positive_int(mw, m, "blocks")
                _positive_int(mw, m, "conv")
                if width % blocks:
                    raise ConfigError(f"{mw}: a width of {width} does not divide into {blocks} blocks")
            mlp = layer.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict) or mlp.get("kind") not in MLP_KINDS:
                    raise ConfigError(f"{where}.mlp: kind must be one of {', '.join(MLP_KINDS)}, or the mlp null")
                if mlp["kind"] == "dense":
                    _positive_int(where + ".mlp", mlp, "ff")
                else:
                    _check_moe(where + ".mlp", mlp)

    def with_stop_token_ids(self, ids) -> "RolevikConfig":
        return dataclasses.replace(self, stop_token_ids=tuple(int(i) for i in ids))

    def to_dict(self) -> Dict[str, Any]:
        d: Dict[str, Any] = {
            "architecture": self.architecture, "vocab": self.vocab, "width": self.width, "embedding": dict(self.embedding),
            "norm": dict(self.norm), "logit_scale": self.logit_scale, "layers": [dict(layer) for layer in self.layers],
        }
        if self.max_position_embeddings != 65536:
            d["max_position_embeddings"] = self.max_position_embeddings
        return d
