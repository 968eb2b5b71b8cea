"""Small Rolevik configurations for the tests, and what the tests share: model folders with random weights and the float64
oracle of a whole sequence.

The configurations differ from one another in every size, and none of their sizes coincide by accident: attentions of one to
ten heads in groups of one to eight, keys and values of different sizes, rotated parts from two numbers to the whole head and
none, chunks of one to seventy positions and none, delta rules with groups of their own, filters of one to five taps, recurrent
units narrower and wider than the model in one to several parts, feed-forwards dense, routed and missing, routers with and
without groups, choices that stand for the input, a shared expert and a scale, embeddings and logits scaled by less than one and
by more.
"""
from __future__ import annotations

import json
import os
import random
from typing import Dict, List

import torch
from safetensors import safe_open
from safetensors.torch import save_file


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, groups=None, identity=None, scale=None, shared=None):
    router = {"experts": experts, "top": top}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    if identity is not None:
        router["identity"] = identity
    if scale is not None:
        router["scale"] = scale
    m = {"kind": "moe", "expert": {"ff": ff}, "router": router}
    if shared is not None:
        m["shared"] = {"ff": shared}
    return m


def attn(heads, kv_heads, dim, vdim, scale, chunk=None, rot=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return m


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def par(left, right, mlp=None):
    return {"type": "parallel", "mixer": {"left": left, "right": right}, "mlp": mlp}


def lru(width, blocks, conv, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def model(vocab, width, layers, eps=1e-5, scale=1.0, logit_scale=1.0):
    return {"architecture": "Rolevik", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "logit_scale": logit_scale, "layers": layers}


CASE_A = model(211, 64, [
    lru(40, 5, 4, mlp=moe(24, 6, 2, groups=(4, 2), identity=2, scale=1.7, shared=40)),
    par(attn(4, 2, 16, 24, 0.4, chunk=21, rot=(8, 1000.0)), delta(4, 2, 8, 20, 3), mlp=dense(48)),
    par(attn(3, 1, 24, 8, 0.35, chunk=48, rot=(24, 50.0)), delta(3, 3, 20, 12, 2)),
    lru(96, 3, 2, mlp=moe(16, 5, 3, groups=(3, 2), identity=1, scale=0.6)),
], eps=1e-5, scale=9.0, logit_scale=0.7)
# no mask, no rotation, no groups, no identity choices, one tap, one part, one head, every size unlike its neighbour's
CASE_B = model(97, 48, [
    par(attn(6, 6, 8, 16, 0.7, rot=(2, 7.0)), delta(1, 1, 16, 8, 1), mlp=moe(20, 7, 1, shared=12)),
    par(attn(1, 1, 40, 8, 0.3, chunk=1), delta(6, 2, 12, 4, 5), mlp=moe(12, 4, 4)),
    lru(20, 1, 1, mlp=dense(100)),
    par(attn(5, 5, 16, 16, 0.5, chunk=16, rot=(16, 10000.0)), delta(5, 1, 4, 28, 2)),
    lru(48, 48, 3),
], eps=1e-6, scale=1.0, logit_scale=1.0)
# heads the tensor-core kernels take in bfloat16, one group size each, chunks at and beside the pages' and tiles' edges
CASE_C = model(300, 128, [
    par(attn(6, 2, 32, 32, 0.3, chunk=32, rot=(16, 30000.0)), delta(2, 1, 32, 64, 4), mlp=dense(96)),
    lru(256, 2, 4, mlp=moe(64, 8, 3, groups=(2, 1), scale=2.5, shared=64)),
    par(attn(8, 1, 64, 64, 0.2, chunk=65, rot=(64, 10000.0)), delta(4, 4, 64, 32, 3), mlp=moe(32, 12, 2, groups=(5, 2), identity=3, scale=3.0)),
    par(attn(2, 1, 128, 128, 0.12, chunk=40, rot=(128, 1000000.0)), delta(4, 2, 128, 16, 2), mlp=dense(72)),
    lru(136, 17, 3, mlp=dense(80)),
    par(attn(10, 5, 32, 32, 0.3, chunk=70, rot=(30, 100.0)), delta(2, 2, 40, 40, 4)),
], eps=1e-6, scale=5.0, logit_scale=0.4)
# sizes that are multiples of nothing
CASE_D = model(101, 36, [
    par(attn(3, 1, 10, 6, 0.6, chunk=19, rot=(6, 100.0)), delta(3, 1, 7, 5, 4), mlp=moe(14, 5, 2, groups=(2, 1), identity=3, scale=1.3, shared=9)),
    lru(33, 3, 5, mlp=dense(14)),
    par(attn(10, 5, 6, 10, 0.8, chunk=37, rot=(4, 30.0)), delta(2, 2, 21, 3, 3)),
    lru(5, 5, 2, mlp=moe(6, 9, 3, groups=(3, 2), scale=0.9)),
], eps=1e-4, scale=4.0, logit_scale=2.0)
# one kind of layer alone: a model without pages, a model whose every layer has pages
CASE_E = model(64, 80, [lru(52, 4, 3), lru(130, 10, 4, mlp=dense(44))], eps=1e-5, scale=11.0, logit_scale=0.3)
CASE_F = model(64, 80, [par(attn(12, 3, 32, 32, 0.35, chunk=50, rot=(32, 10000.0)), delta(3, 1, 16, 24, 3), mlp=dense(40)),
                        par(attn(7, 7, 64, 40, 0.25, chunk=33, rot=(8, 99.0)), delta(1, 1, 48, 48, 2), mlp=dense(24))],
               eps=1e-5, scale=2.0, logit_scale=1.5)
CASES = {"A": (CASE_A, 51), "B": (CASE_B, 52), "C": (CASE_C, 53), "D": (CASE_D, 54), "E": (CASE_E, 55), "F": (CASE_F, 56)}


# In 16 bits a router's near tie may rightly fall either way, and the rows behind it differ. Models that run in bfloat16 therefore
# get corrections that lie further apart than scores can (SETTLED): which experts a layer uses then rests on the corrections, the
# groups and the weights, not on a token's scores; models that run in 32-bit get scores that matter (SPREAD).
SPREAD, SETTLED = 0.15, 1.25


def make_folder(path: str, cfg: dict, seed: int, spread: float = SPREAD) -> str:
    from openinfer_b200.config.base import resolve_architecture
    from openinfer_b200.weights import write_random_model

    config = resolve_architecture(cfg).config_cls.from_dict(cfg)
    write_random_model(config, path, seed)
    spread_corrections(path, seed, spread)
    return path


def spread_corrections(path: str, seed: int, spread: float) -> None:
    """The routers' corrections become numbers ``spread`` apart in a random order, and their logits three times as large: a token's scores
    still change the choice where ``spread`` lets them, but few tokens come near a tie."""
    tensors = read_folder(path)[1]
    g = torch.Generator().manual_seed(seed)
    for name, t in tensors.items():
        if name.endswith(".correction"):
            n = t.numel()
            tensors[name] = (spread * (torch.randperm(n, generator=g) - 0.5 * n)).to(t.dtype)
        elif name.endswith(".router"):
            tensors[name] = 3.0 * t
    save_file(tensors, os.path.join(path, "model.safetensors"))


def read_folder(path: str):
    with open(os.path.join(path, "config.json")) as fh:
        cfg = json.load(fh)
    tensors: Dict[str, torch.Tensor] = {}
    with safe_open(os.path.join(path, "model.safetensors"), "pt") as f:
        for k in f.keys():
            tensors[k] = f.get_tensor(k)
    return cfg, tensors


_ORACLE: Dict[tuple, tuple] = {}
CLOSE_CALL = 0.01       # a router's choice nearer than this to another one (in score units) may rightly fall either way in 16 bits


def _evaluate(path: str, tokens: List[int]):
    import plain_rolevik

    key = (path, tuple(tokens))
    if key not in _ORACLE:
        cfg, tensors = read_folder(path)
        margins: list = []
        logits = plain_rolevik.forward(cfg, tensors, list(tokens), dtype=torch.float64, margins=margins)
        size = logits.pow(2).mean().sqrt().item()
        # what rounding alone does in float32, and what 16-bit roundings of the sublayers' inputs, queries, keys and values alone do
        single = plain_rolevik.forward(cfg, tensors, list(tokens), dtype=torch.float32).double()
        # (three roundings on different grids: a read-out that nearly vanishes before it is normed shows in some of them only)
        halves = [(plain_rolevik.forward(cfg, tensors, list(tokens), dtype=torch.float64, round_to=torch.bfloat16, round_scale=c) - logits).abs()
                  for c in (1.0, 1.37, 0.77)]
        close = torch.stack(margins).min(dim=0).values < CLOSE_CALL if margins else torch.zeros(len(tokens), dtype=torch.bool)
        first_close = int(close.nonzero()[0]) if close.any() else len(tokens)
        halves = [h[: max(1, first_close)] for h in halves]
        _ORACLE[key] = (logits, (single - logits).abs().max().item() / size,
                        (max(h.max().item() for h in halves) / size, max(h.mean().item() for h in halves) / size), first_close)
    return _ORACLE[key]


def oracle(path: str, tokens: List[int]) -> torch.Tensor:
    """float64 logits [T, vocab] of the whole sequence by the plain implementation (cached per folder and sequence)."""
    return _evaluate(path, tokens)[0]


def float32_noise(path: str, tokens: List[int]) -> float:
    return _evaluate(path, tokens)[1]


def bfloat16_noise(path: str, tokens: List[int]):
    return _evaluate(path, tokens)[2]


def first_close_call(path: str, tokens: List[int]) -> int:
    """The first row at which some router's choice is a close call (the sequence's length if none is)."""
    return _evaluate(path, tokens)[3]


def tokens_for(cfg: dict, n: int, seed: int) -> List[int]:
    rng = random.Random(seed)
    return [rng.randrange(cfg["vocab"]) for _ in range(n)]


# Errors are measured against the root mean square of the reference logits of the sequence.
# float32 engine against the float64 oracle: 3e-5, or five times what rounding alone does to the plain implementation
# evaluated in float32 on that sequence where that is more.
F32_MAX_REL = 3e-5
F32_NOISE_FACTOR = 5.0
# bfloat16 engine: the bounds below, or four times what the roundings of the sublayers' inputs, queries, keys and values
# alone do to the float64 plain implementation on that sequence where that is more (the engine rounds at more places: the
# projections, the gate and up sums, the recurrences' results). Rows from a sequence's first close router call on are left out
# of the worst-row bound (the engine may rightly choose the other expert there, and state and cache carry the difference on),
# but of all rows at most one in ten may exceed it.
BF16_MAX_REL, BF16_MEAN_REL = 0.10, 0.02
BF16_NOISE_FACTOR = 4.0


def assert_logits(got: torch.Tensor, ref: torch.Tensor, dtype: str, what: str, noise: float = 0.0, noise16=(0.0, 0.0),
                  first_close: int = 1 << 30) -> None:
    got, ref = got.detach().double().cpu(), ref.detach().double().cpu()
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    diff = (got - ref).abs()
    scale = ref.pow(2).mean().sqrt().item()
    worst = diff.max().item() / scale
    row = int(diff.max(dim=1).values.argmax())
    if dtype == "float32":
        bound = max(F32_MAX_REL, F32_NOISE_FACTOR * noise)
        assert worst <= bound, f"{what}: float32 error {worst:.3e} of the logits' size (bound {bound:.3e}), worst row {row}"
        return
    max_bound = max(BF16_MAX_REL, BF16_NOISE_FACTOR * noise16[0])
    mean_bound = max(BF16_MEAN_REL, BF16_NOISE_FACTOR * noise16[1])
    sure, per_row = diff[:first_close] / scale, diff.max(dim=1).values / scale
    assert sure.numel() == 0 or (sure.max().item() <= max_bound and sure.mean().item() <= mean_bound), \
        f"{what}: bfloat16 error max {sure.max().item():.4f} (bound {max_bound:.4f}), mean {sure.mean().item():.5f} (bound {mean_bound:.5f}); " \
        f"worst row {row}, first close call {first_close}"
    assert int((per_row > max_bound).sum()) <= max(1, per_row.numel() // 10), \
        f"{what}: bfloat16: {int((per_row > max_bound).sum())} of {per_row.numel()} rows over {max_bound:.4f}"
