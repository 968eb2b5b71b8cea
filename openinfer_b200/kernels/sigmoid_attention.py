"""Dispatch of attention with sigmoid weights to the kernel that takes the shape."""
from __future__ import annotations

from typing import Optional

import torch

from . import lib as _lib
from . import ops


def sigmoid_attention_general(proj: torch.Tensor, out: torch.Tensor, gate: Optional[torch.Tensor], k_cache: torch.Tensor,
                              v_cache: torch.Tensor, page_stride: int, ctx, group_step, nq: int, nkv: int, hd: int, scale: float,
                              mix: torch.Tensor, bias: torch.Tensor) -> None:
    """The general kernel: one block per row, every shape, float32 or bfloat16."""
    ops._cuda(proj, out, gate, k_cache, v_cache, mix, bias)
    bt = group_step.block_table
    _lib.check(_lib.load().oi_sigmoid_attention(
        proj.data_ptr(), proj.stride(0), out.data_ptr(), out.stride(0), 0 if gate is None else gate.data_ptr(),
        0 if gate is None else gate.stride(0), ops._code(proj, "sigmoid_attention"), k_cache.data_ptr(), v_cache.data_ptr(),
        int(page_stride), ctx.cache.page_size, bt.data_ptr(), bt.stride(0), ctx.token_req.data_ptr(), ctx.positions.data_ptr(),
        out.shape[0], nq, nkv, hd, float(scale), mix.data_ptr(), bias.data_ptr(), _lib.current_stream()), "sigmoid_attention")


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
    sigmoid_attention_general(proj, out, gate, k_cache, v_cache, page_stride, ctx, group_step, nq, nkv, hd, scale, mix, bias)
    return out
