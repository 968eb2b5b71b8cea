"""Attention whose weights are sigmoids, over the paged cache: grouped-query, causal, not normalised over the keys.

score_h(i, j) = scale q_h,i . k_c(h),j;  with ``mix_heads`` score_h <- sum_g T[h, g] score_g over ALL heads;  weight =
sigmoid(score_h + bias_h) for every j <= i;  o_h,i = sum_j weight v_c(h),j;  then, with ``output_gate``, every number times
sigmoid(W_g x), and the output projection.

One fused projection q | k | (v) | gate. A first kernel norms q and k over all their heads together, turns neighbouring
pairs and writes q back and key and value to the row's page; with ``values_from_keys`` the value is the key as it was
projected. Mixing makes every head's weight depend on all heads' scores, so the attention kernels keep all heads of a
query together (csrc/sigmoid_attention_mma.cu, bfloat16); sums need no maximum and no denominator, so the results of key
slices are simply added up. The general kernel (csrc/sigmoid_attention.cu) takes float32 and every size the other refuses.

Heads are cached and multiplied in rows of ``head_dim`` = the next multiple of eight; the projections get zero rows up to it
when they are loaded, which change neither a score nor a value.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..cache.manager import KvNeed
from ..kernels import ops
from ..kernels import sigmoid_attention as kernels
from ..kernels.linear import linear
from .base import CacheBinding, Mixer
from .registry import build_position_encoding, register_mixer
from .spec import ParamInfo, SigmoidAttentionSpec


@register_mixer("sigmoid_attention")
class SigmoidAttention(Mixer):
    graph_safe = True
    takes_out_dtype = True

    def __init__(self, spec: SigmoidAttentionSpec) -> None:
        super().__init__(spec)
        s = spec
        if min(s.num_heads, s.num_kv_heads, s.qk_dim, s.v_dim) <= 0 or s.num_heads % s.num_kv_heads:
            raise ValueError(f"sigmoid_attention: heads {s.num_heads}, kv heads {s.num_kv_heads}, dim {s.qk_dim}, vdim {s.v_dim}")
        if s.values_from_keys and s.v_dim != s.qk_dim:
            raise ValueError(f"sigmoid_attention: values that are the keys have their size, {s.v_dim} is not {s.qk_dim}")
        if s.position.kind != "none" and not s.position.interleaved:
            raise ValueError("sigmoid_attention: the rotation turns neighbouring pairs")
        self.hd = -(-max(s.qk_dim, s.v_dim) // 8) * 8
        if self.hd > 512:
            raise ValueError(f"sigmoid_attention: heads of {self.hd} numbers (at most 512)")
        H, G, hd = s.num_heads, s.num_kv_heads, self.hd
        self.k_off = H * hd
        self.v_off = self.k_off if s.values_from_keys else self.k_off + G * hd
        self.g_off = self.v_off + G * hd
        self.position = build_position_encoding(s.position)
        self.tables = None
        self.w_in = self.w_o = self.q_norm_w = self.k_norm_w = self.mix = self.bias = None

    def kv_need(self) -> Optional[KvNeed]:
        return KvNeed(self.spec.num_kv_heads, self.hd)

    def parameters(self) -> Dict[str, ParamInfo]:
        s = self.spec
        H, G, D, V, W = s.num_heads, s.num_kv_heads, s.qk_dim, s.v_dim, s.hidden_size
        std = W ** -0.5
        p = {s.q_name: ParamInfo((H * D, W), ("normal", std)), s.k_name: ParamInfo((G * D, W), ("normal", std)),
             s.out_name: ParamInfo((W, H * V), ("normal", (H * V) ** -0.5))}
        if not s.values_from_keys:
            p[s.v_name] = ParamInfo((G * V, W), ("normal", std))
        if s.joint_norm_eps > 0.0:
            p[s.q_norm_name] = ParamInfo((H * D,), ("one_plus_normal", 0.1))
            p[s.k_norm_name] = ParamInfo((G * D,), ("one_plus_normal", 0.1))
        if s.mix_heads:
            p[s.mix_name] = ParamInfo((H, H), ("eye_plus_normal", 0.3))
        if s.score_bias:
            p[s.bias_name] = ParamInfo((H,), ("normal_around", 0.3, -4.0))
        if s.output_gate:
            p[s.gate_name] = ParamInfo((H * V, W), ("normal", std))
        return p

    def load(self, tensors: Dict[str, torch.Tensor]) -> None:
        s = self.spec
        hd = self.hd

        def rows_padded(w, heads, size):       # [heads * size, ...] -> [heads * hd, ...], zero rows behind each head's
            if size == hd:
                return w
            out = torch.zeros((heads, hd, *w.shape[1:]), dtype=w.dtype, device=w.device)
            out[:, :size] = w.view(heads, size, *w.shape[1:])
            return out.view(heads * hd, *w.shape[1:])

        fused = [rows_padded(tensors[s.q_name], s.num_heads, s.qk_dim), rows_padded(tensors[s.k_name], s.num_kv_heads, s.qk_dim)]
        if not s.values_from_keys:
            fused.append(rows_padded(tensors[s.v_name], s.num_kv_heads, s.v_dim))
        if s.output_gate:
            fused.append(rows_padded(tensors[s.gate_name], s.num_heads, s.v_dim))
        if len({w.dtype for w in fused}) != 1:
            raise ValueError("the projections of a mixer must be stored in one dtype to be fused")
        self.w_in = torch.cat(fused, dim=0).contiguous()
        o = tensors[s.out_name]
        if s.v_dim != hd:
            wide = torch.zeros((o.shape[0], s.num_heads, hd), dtype=o.dtype, device=o.device)
            wide[:, :, : s.v_dim] = o.view(o.shape[0], s.num_heads, s.v_dim)
            o = wide.view(o.shape[0], s.num_heads * hd)
        self.w_o = o.contiguous()
        if s.joint_norm_eps > 0.0:
            self.q_norm_w = rows_padded(tensors[s.q_norm_name].to(torch.float32), s.num_heads, s.qk_dim).contiguous()
            self.k_norm_w = rows_padded(tensors[s.k_norm_name].to(torch.float32), s.num_kv_heads, s.qk_dim).contiguous()
        if s.mix_heads:
            # (exact in 11 bits of mantissa, as bfloat16 numbers are: the tensor-core kernel multiplies it as it is)
            self.mix_is_short = tensors[s.mix_name].dtype == torch.bfloat16
            self.mix = tensors[s.mix_name].to(torch.float32).contiguous()
        if s.score_bias:
            self.bias = tensors[s.bias_name].to(torch.float32).contiguous()

    def prepare(self, device: torch.device, dtype: torch.dtype) -> None:
        s = self.spec
        self.tables = self.position.rotation_tables(device)
        if self.mix is None:
            self.mix, self.mix_is_short = torch.eye(s.num_heads, dtype=torch.float32, device=device), True
        if self.bias is None:
            self.bias = torch.zeros(s.num_heads, dtype=torch.float32, device=device)

    def forward(self, x: torch.Tensor, ctx, binding: CacheBinding, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
        s = self.spec
        if binding.kv is None or not binding.owns_kv:
            raise RuntimeError("sigmoid_attention needs a cache of its own")
        H, G, hd = s.num_heads, s.num_kv_heads, self.hd
        group = ctx.groups[binding.kv.group]
        k_cache, v_cache, page_stride = ctx.cache.kv_views(binding.kv)
        proj = linear(x, self.w_in)
        cos, sin = self.tables if self.tables is not None else (None, None)
        ops.joint_norm_rope_store(proj, H, G, hd, s.qk_dim, self.k_off, self.v_off, q_norm_w=self.q_norm_w, k_norm_w=self.k_norm_w,
                                  eps=s.joint_norm_eps, cos=cos, sin=sin, positions=ctx.positions, slots=group.slot_mapping,
                                  k_cache=k_cache, v_cache=v_cache, page_stride=page_stride, page_size=ctx.cache.page_size)
        out = torch.empty((x.shape[0], H * hd), dtype=x.dtype, device=x.device)
        gate = proj[:, self.g_off: self.g_off + H * hd] if s.output_gate else None
        kernels.sigmoid_attention(proj, out, gate, k_cache, v_cache, page_stride, ctx, group, H, G, hd, s.score_scale, self.mix,
                                  self.bias, mix_is_short=self.mix_is_short)
        return linear(out, self.w_o, out_dtype=out_dtype)
