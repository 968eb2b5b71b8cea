"""Small Linurax configurations for the tests, and what the tests share: model folders with random weights and the float64
oracle of a whole sequence.

The configurations differ from one another in every size, and none of their sizes coincide by accident: one to twenty heads
on one to several key heads (groups of one to eight, and groups that fill no power of two), heads of 8 to 128 numbers and of
sizes that are multiples of nothing, rotated parts from two numbers to the whole head and none, recurrences narrower and
wider than the model, layers of either kind with and without a feed-forward, in every order, embeddings scaled by one, by less
and by more. Score scales are about twice 1 / sqrt(dim): a row's weights differ by orders of magnitude.
"""
from __future__ import annotations

import json
import os
import random
from typing import Dict, List

import torch
from safetensors import safe_open


def dense(ff):
    return {"kind": "dense", "ff": ff}


def attn(heads, kv_heads, dim, scale, rot=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale}
    if rot is not None:
        m["rot"] = {"dims": rot[0], "base": rot[1]}
    return {"type": "attention", "mixer": m, "mlp": dense(mlp) if mlp else None}


def gru(width, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": dense(mlp) if mlp else None}


def model(vocab, width, layers, eps=1e-5, scale=1.0):
    return {"architecture": "Linurax", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps}, "layers": layers}


CASE_A = model(211, 64, [
    gru(40), attn(4, 2, 16, 0.4, rot=(8, 1000.0), mlp=48), attn(3, 1, 24, 0.35, rot=(24, 50.0)), gru(96, mlp=72),
], eps=1e-5, scale=30.0)
CASE_B = model(97, 48, [
    attn(6, 6, 8, 0.7, rot=(2, 7.0)), attn(5, 5, 40, 0.3, mlp=30), gru(20, mlp=100), attn(1, 1, 16, 0.5, rot=(16, 10000.0)),
], eps=1e-6, scale=1.0)
# heads the tensor-core kernels take in bfloat16, one group size each
CASE_C = model(300, 128, [
    attn(6, 2, 32, 0.3, rot=(16, 30000.0), mlp=96), gru(256, mlp=64), attn(8, 2, 64, 0.25, rot=(64, 10000.0)),
    attn(16, 2, 64, 0.2, rot=(32, 500.0), mlp=160), attn(2, 1, 128, 0.15, rot=(128, 1000000.0)), gru(33), attn(20, 5, 32, 0.35, rot=(30, 100.0)),
], eps=1e-6, scale=0.7)
# sizes that are multiples of nothing
CASE_D = model(101, 36, [
    attn(3, 1, 10, 0.6, rot=(6, 100.0), mlp=50), gru(33, mlp=14), attn(10, 5, 6, 0.8, rot=(4, 30.0)), gru(5),
], eps=1e-4, scale=5.0)
# one kind of layer alone: a model without pages, a model without state
CASE_E = model(64, 80, [gru(52), gru(130, mlp=44)], eps=1e-5, scale=11.0)
CASE_F = model(64, 80, [attn(12, 3, 32, 0.35, rot=(32, 10000.0), mlp=40), attn(7, 7, 64, 0.25, rot=(8, 99.0), mlp=24)], eps=1e-5, scale=2.0)
CASES = {"A": (CASE_A, 41), "B": (CASE_B, 42), "C": (CASE_C, 43), "D": (CASE_D, 44), "E": (CASE_E, 45), "F": (CASE_F, 46)}


def make_folder(path: str, cfg: dict, seed: int) -> str:
    from openinfer_b200.config.base import resolve_architecture
    from openinfer_b200.weights import write_random_model

    config = resolve_architecture(cfg).config_cls.from_dict(cfg)
    write_random_model(config, path, seed)
    return path


def read_folder(path: str):
    with open(os.path.join(path, "config.json")) as fh:
        cfg = json.load(fh)
    tensors: Dict[str, torch.Tensor] = {}
    with safe_open(os.path.join(path, "model.safetensors"), "pt") as f:
        for k in f.keys():
            tensors[k] = f.get_tensor(k)
    return cfg, tensors


_ORACLE: Dict[tuple, tuple] = {}


def _evaluate(path: str, tokens: List[int]):
    import plain_linurax

    key = (path, tuple(tokens))
    if key not in _ORACLE:
        cfg, tensors = read_folder(path)
        logits = plain_linurax.forward(cfg, tensors, list(tokens), dtype=torch.float64)
        size = logits.pow(2).mean().sqrt().item()
        # what rounding alone does in float32, and what 16-bit roundings of the sublayers' inputs, queries, keys and values alone do
        single = plain_linurax.forward(cfg, tensors, list(tokens), dtype=torch.float32).double()
        half = plain_linurax.forward(cfg, tensors, list(tokens), dtype=torch.float64, round_to=torch.bfloat16)
        _ORACLE[key] = (logits, (single - logits).abs().max().item() / size,
                        ((half - logits).abs().max().item() / size, (half - logits).abs().mean().item() / size))
    return _ORACLE[key]


def oracle(path: str, tokens: List[int]) -> torch.Tensor:
    """float64 logits [T, vocab] of the whole sequence by the plain implementation (cached per folder and sequence)."""
    return _evaluate(path, tokens)[0]


def float32_noise(path: str, tokens: List[int]) -> float:
    return _evaluate(path, tokens)[1]


def bfloat16_noise(path: str, tokens: List[int]):
    return _evaluate(path, tokens)[2]


def tokens_for(cfg: dict, n: int, seed: int) -> List[int]:
    rng = random.Random(seed)
    return [rng.randrange(cfg["vocab"]) for _ in range(n)]


# Errors are measured against the root mean square of the reference logits of the sequence.
# float32 engine against the float64 oracle: 3e-5, or three times what rounding alone does to the plain implementation
# evaluated in float32 on that sequence where that is more.
F32_MAX_REL = 3e-5
F32_NOISE_FACTOR = 3.0
# bfloat16 engine: the bounds below, or four times what the roundings of the sublayers' inputs, queries, keys and
# values alone do to the float64 plain implementation on that sequence where that is more (the engine rounds at more places:
# the projections, the gate and up sums, the weights on their way into the second product).
BF16_MAX_REL, BF16_MEAN_REL = 0.10, 0.02
BF16_NOISE_FACTOR = 4.0


def assert_logits(got: torch.Tensor, ref: torch.Tensor, dtype: str, what: str, noise: float = 0.0, noise16=(0.0, 0.0)) -> None:
    got, ref = got.detach().double().cpu(), ref.detach().double().cpu()
    assert got.shape == ref.shape, f"{what}: shape {tuple(got.shape)} vs {tuple(ref.shape)}"
    assert torch.isfinite(got).all(), f"{what}: non-finite logits"
    diff = (got - ref).abs()
    scale = ref.pow(2).mean().sqrt().item()
    worst, mean = diff.max().item() / scale, diff.mean().item() / scale
    row = int(diff.max(dim=1).values.argmax())
    if dtype == "float32":
        bound = max(F32_MAX_REL, F32_NOISE_FACTOR * noise)
        assert worst <= bound, f"{what}: float32 error {worst:.3e} of the logits' size (bound {bound:.3e}), worst row {row}"
    else:
        max_bound = max(BF16_MAX_REL, BF16_NOISE_FACTOR * noise16[0])
        mean_bound = max(BF16_MEAN_REL, BF16_NOISE_FACTOR * noise16[1])
        assert worst <= max_bound and mean <= mean_bound, \
            f"{what}: bfloat16 error max {worst:.4f} (bound {max_bound:.4f}), mean {mean:.5f} (bound {mean_bound:.5f}); worst row {row}"
