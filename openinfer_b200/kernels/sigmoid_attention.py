"""Dispatch of attention with sigmoid weights to the kernel that takes the shape, and the planning of its work items.

The tensor-core kernels (bfloat16, heads of 32 / 64 / 128 numbers, up to 32 heads, pages that are a multiple of 16 keys) work
on items planned on the host once per step and shared by all layers of one geometry: prompt portions are cut into tiles of a
few tokens (all heads of a token belong together), single tokens go to the decode kernel; the keys of either may be cut into
slices, whose results another kernel adds up. Every other shape, and float32, goes to the general kernel.
"""
from __future__ import annotations

import dataclasses
from typing import Optional, Sequence

import numpy as np
import torch

from . import lib as _lib
from . import ops, policy
from .attention import _sm_count

PAGE_MULTIPLE = 16
KEYS_PER_STEP = 32
MIN_STEPS_PER_SLICE = 8         # a prompt tile's slice is at least 256 keys long
SLICE_SHARE = 0.65              # of an even share of all tiles' keys over the SMs: the longest slice, where there are no more
                                # tiles than SMs (prompts of 1,024 to 4,096 tokens: 5-15 % shorter than a whole share)
DECODE_MIN_KEYS_PER_SLICE = 64  # a step of 16 keys for each of the CTA's four warps
DECODE_MAX_SLICES = 64
DECODE_CTAS_PER_SM = 2
USE_TENSOR_CORES = True         # False: the general kernel takes every shape

_PLAN_RING = ops.UploadRing()


@dataclasses.dataclass
class SigmoidPlan:
    tile_items: torch.Tensor      # int32 [n, 4]: request, first token of the tile, slice, slices
    decode_items: torch.Tensor    # int32 [n, 4]: request, 0, slice, slices
    row_splits: torch.Tensor      # int32 [tokens]
    row_base: torch.Tensor        # int32 [tokens]: where a row's partial results begin
    any_split: bool
    part_rows: int                # partial results of all rows


def decode_slices(rows: int, sm_count: int, longest: int) -> int:
    """Key slices per single-token row: as many as fill the GPU once, each at least 64 keys of the longest row."""
    if policy.batch_invariant():
        return policy.INVARIANT_DECODE_SPLITS
    want = max(1, DECODE_CTAS_PER_SM * sm_count // max(1, rows))
    return max(1, min(want, DECODE_MAX_SLICES, longest // DECODE_MIN_KEYS_PER_SLICE))


def plan_items(q_lens: Sequence[int], kv_lens: Sequence[int], tile_tokens: int, sm_count: int,
               fixed_decode_slices: Optional[int] = None):
    """Work items of one step: (tile_items [n, 4], decode_items [n, 4], row_splits [tokens], row_base [tokens], partial rows).

    A prompt tile's keys are cut so that no item is longer than (SLICE_SHARE of) an even share of all tiles' keys over the
    SMs, or MIN_STEPS_PER_SLICE steps: the last tiles of a long prompt would otherwise still run when the others are done."""
    starts = np.concatenate([[0], np.cumsum(q_lens)]).astype(np.int64)
    tokens = int(starts[-1])
    row_splits = np.ones(tokens, dtype=np.int32)
    decode_reqs = [b for b, n in enumerate(q_lens) if n == 1]
    decode_items = []
    if decode_reqs:
        ns = fixed_decode_slices or decode_slices(len(decode_reqs), sm_count, max(kv_lens[b] for b in decode_reqs))
        for b in decode_reqs:
            row_splits[starts[b]] = ns
            decode_items.extend((b, 0, s, ns) for s in range(ns))
    tiles = []
    for b, (n, kv) in enumerate(zip(q_lens, kv_lens)):
        if n > 1:
            for t0 in range(0, n, tile_tokens):
                toks = min(tile_tokens, n - t0)
                tiles.append((b, t0, toks, -(-(kv - n + t0 + toks) // KEYS_PER_STEP)))
    tiles.sort(key=lambda t: -t[3])
    limit = None
    if tiles and not policy.batch_invariant():
        share = sum(t[3] for t in tiles) / sm_count
        limit = max(MIN_STEPS_PER_SLICE, int((SLICE_SHARE if len(tiles) <= sm_count else 1.0) * share) + 1)
    items = []
    for b, t0, toks, steps in tiles:
        ns = -(-steps // limit) if limit else 1
        row_splits[starts[b] + t0: starts[b] + t0 + toks] = ns
        per = -(-steps // ns)
        items.extend((-min(per, steps - s * per), b, t0, s, ns) for s in range(ns))
    items.sort()                                   # longest first
    cut = np.where(row_splits > 1, row_splits, 0)
    row_base = (np.cumsum(cut) - cut).astype(np.int32)
    tile_items = np.asarray([i[1:] for i in items], dtype=np.int32).reshape(-1, 4)
    return tile_items, np.asarray(decode_items, dtype=np.int32).reshape(-1, 4), row_splits, row_base, int(cut.sum())


def _plan_for(ctx, group_step, nq: int, nkv: int, hd: int, tile_tokens: int, device) -> SigmoidPlan:
    key = ("sigmoid_attention_plan", id(group_step), tile_tokens)
    plan = ctx.scratch.get(key)
    if plan is None:
        sms = _sm_count(device)
        if getattr(ctx, "static_decode", False):
            # recorded once, replayed for other lengths: the slices follow from the batch and the width of the block tables
            # (which serve the lengths in their upper half)
            longest = int(group_step.block_table.shape[1]) * ctx.cache.page_size // 2
            packed = plan_items([1] * ctx.num_requests, [1] * ctx.num_requests, tile_tokens, sms,
                                fixed_decode_slices=decode_slices(ctx.num_requests, sms, longest))
        else:
            packed = plan_items(ctx.q_lens_host, ctx.kv_lens_host, tile_tokens, sms)
        t_items, d_items, splits, base, part_rows = packed
        dev = _PLAN_RING.upload(np.concatenate([t_items.reshape(-1), d_items.reshape(-1), splits, base]).astype(np.int32, copy=False), device)
        nt, nd, T = t_items.shape[0] * 4, d_items.shape[0] * 4, splits.shape[0]
        plan = SigmoidPlan(dev[:nt].view(-1, 4), dev[nt: nt + nd].view(-1, 4), dev[nt + nd: nt + nd + T], dev[nt + nd + T:],
                           part_rows > 0, part_rows)
        ctx.scratch[key] = plan
    return plan


def _general(proj, out, gate, k_cache, v_cache, page_stride, ctx, group_step, nq, nkv, hd, scale, mix, bias) -> None:
    bt = group_step.block_table
    _lib.check(_lib.load().oi_sigmoid_attention(
        proj.data_ptr(), proj.stride(0), out.data_ptr(), out.stride(0), 0 if gate is None else gate.data_ptr(),
        0 if gate is None else gate.stride(0), ops._code(proj, "sigmoid_attention"), k_cache.data_ptr(), v_cache.data_ptr(),
        int(page_stride), ctx.cache.page_size, bt.data_ptr(), bt.stride(0), ctx.token_req.data_ptr(), ctx.positions.data_ptr(),
        out.shape[0], nq, nkv, hd, float(scale), mix.data_ptr(), bias.data_ptr(), _lib.current_stream()), "sigmoid_attention")


def _tensor_cores(proj, out, gate, k_cache, v_cache, page_stride, ctx, group_step, nq, nkv, hd, scale, mix, bias) -> bool:
    """The tensor-core kernels, when they take the shape. Returns whether they ran."""
    if proj.dtype != torch.bfloat16 or ctx.cache.page_size % PAGE_MULTIPLE:
        return False
    L = _lib.load()
    tile_tokens = L.oi_sigmoid_attention_tile_tokens(nq, nkv, hd)
    if not tile_tokens or proj.stride(0) % 8 or out.stride(0) % 8 or (gate is not None and gate.data_ptr() % 16):
        return False
    plan = _plan_for(ctx, group_step, nq, nkv, hd, tile_tokens, proj.device)
    part = torch.empty(plan.part_rows * nq * hd, dtype=torch.float32, device=proj.device) if plan.any_split else None
    bt = group_step.block_table
    g_ptr, g_stride = (0, 0) if gate is None else (gate.data_ptr(), gate.stride(0))
    _lib.check(L.oi_sigmoid_attention_mma(
        proj.data_ptr(), proj.stride(0), out.data_ptr(), out.stride(0), g_ptr, g_stride, k_cache.data_ptr(), v_cache.data_ptr(),
        int(page_stride), ctx.cache.page_size, bt.data_ptr(), bt.stride(0), ctx.cu_seqlens.data_ptr(), group_step.kv_lens.data_ptr(),
        plan.tile_items.data_ptr(), plan.tile_items.shape[0], plan.decode_items.data_ptr(), plan.decode_items.shape[0],
        plan.row_base.data_ptr(), 0 if part is None else part.data_ptr(), nq, nkv, hd, float(scale), mix.data_ptr(), bias.data_ptr(),
        _lib.current_stream()), "sigmoid_attention_mma")
    if part is not None:
        _lib.check(L.oi_slice_sum_gate(part.data_ptr(), plan.row_splits.data_ptr(), plan.row_base.data_ptr(), out.data_ptr(), 1,
                                       out.stride(0), g_ptr, g_stride, out.shape[0], nq * hd, _lib.current_stream()), "slice_sum_gate")
    return True


def sigmoid_attention(proj: torch.Tensor, out: torch.Tensor, gate: Optional[torch.Tensor], k_cache: torch.Tensor,
                      v_cache: torch.Tensor, page_stride: int, ctx, group_step, nq: int, nkv: int, hd: int, scale: float,
                      mix: torch.Tensor, bias: torch.Tensor, mix_is_short: bool = False) -> torch.Tensor:
    """out[t, h] = sigmoid(gate[t, h]) * sum_j sigmoid(scale * sum_g mix[h, g] (q_t,g . k_j,c(g)) + bias[h]) v_j,c(h) over the
    keys j up to the row's own, from the pages ``group_step.block_table`` lists; q are the first nq * hd columns of ``proj``.
    ``mix_is_short``: the mix holds numbers of at most 11 bits of mantissa (bfloat16 ones, say)."""
    if mix.dtype != torch.float32 or tuple(mix.shape) != (nq, nq) or not mix.is_contiguous() or bias.dtype != torch.float32 \
            or bias.numel() != nq or not bias.is_contiguous():
        raise ops.KernelError("sigmoid_attention: the head mix must be float32 [heads, heads] and the bias float32 [heads]")
    if proj.stride(1) != 1 or out.stride(1) != 1 or out.dtype != proj.dtype or k_cache.dtype != proj.dtype \
            or (gate is not None and (gate.dtype != proj.dtype or gate.stride(1) != 1)):
        raise ops.KernelError("sigmoid_attention: q, gate, out and the cache must share one dtype and be rows")
    ops._cuda(proj, out, gate, k_cache, v_cache, mix, bias)
    args = (proj, out, gate, k_cache, v_cache, page_stride, ctx, group_step, nq, nkv, hd, scale, mix, bias)
    if not (USE_TENSOR_CORES and mix_is_short and _tensor_cores(*args)):
        _general(*args)
    return out
