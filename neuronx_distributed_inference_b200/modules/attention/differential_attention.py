"""Differential attention on ragged rows and the paged cache: two softmax maps per head over the same values, subtracted.

Every query head ``h`` and every key head ``g`` carries TWO vectors of ``head_dim`` channels (map 1, map 2; laid out head by head), every
value head ONE of ``v_head_dim``.  Map ``m`` is a grouped-query attention of its own (rotate-half rotation on the first ``rot_dims`` channels
of each map, ``scale``, causal, optionally a sliding ``window``); with the two outputs ``a1`` and ``a2`` of a head

    o = a1 - lambda * a2,      o <- o / sqrt(mean(o^2) + eps) * out_scale

where ``lambda`` is one learned number per layer (``lam``; :func:`differential_lambda` forms it from the four vectors checkpoints store).

Data flow (CUDA: csrc/seqmix.cu, one kernel per line after the first):

    p = W_in x                          q | k | v in ONE GEMM
    q = head_norm_rope_append(p)        rotation + paged cache write (2 G key rows, G value rows per token)
    o = paged_diff_attention(q)         both maps of a head in one block, difference, norm and scale in the epilogue
    y = W_o o

The cache row of a token is ``2 G head_dim`` key channels and ``G v_head_dim`` value channels: the values are stored once for both maps.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from ... import ops
from ...parallel.layers import ColumnParallelLinear, RowParallelLinear
from ..rope import compute_inv_freq
from .conv_window_attention import ragged_rope_tables


def differential_lambda(q1, k1, q2, k2, offset: float) -> torch.Tensor:
    """``exp(q1 . k1) - exp(q2 . k2) + offset`` as a one-element fp32 tensor."""
    dot = lambda a, b: (a.double() * b.double()).sum()          # noqa: E731
    return (torch.exp(dot(q1, k1)) - torch.exp(dot(q2, k2)) + offset).float().reshape(1)


class DifferentialAttention(nn.Module):
    def __init__(self, hidden_size: int, num_heads: int, num_kv_heads: int, head_dim: int, v_head_dim: int, *, rot_dims: int, rot_base: float,
                 scale: float, out_scale: float, eps: float, layer_idx: int, window=None, dtype=torch.bfloat16, device=None, tp_group=None):
        super().__init__()
        if tp_group is not None and tp_group.size != 1:
            raise NotImplementedError("differential attention: tensor parallel degree 1")
        if num_heads % num_kv_heads:
            raise ValueError("query heads must be a multiple of key / value heads")
        if rot_dims % 2 or rot_dims > head_dim:
            raise ValueError("rotated channels: an even number, at most the head size")
        self.n_q, self.n_kv, self.head_dim, self.v_head_dim = num_heads, num_kv_heads, head_dim, v_head_dim
        self.rot_dims, self.scale, self.out_scale, self.eps = int(rot_dims), float(scale), float(out_scale), float(eps)
        self.layer_idx, self.window = layer_idx, int(window) if window else None
        width = 2 * head_dim * (num_heads + num_kv_heads) + num_kv_heads * v_head_dim
        self.in_proj = ColumnParallelLinear(hidden_size, width, bias=False, gather_output=False, dtype=dtype, device=device,
                                            tensor_model_parallel_group=tp_group)
        self.o_proj = RowParallelLinear(num_heads * v_head_dim, hidden_size, bias=False, input_is_parallel=True, dtype=dtype, device=device,
                                        tensor_model_parallel_group=tp_group)
        self.lam = nn.Parameter(torch.zeros(1, dtype=torch.float32, device=device), requires_grad=False)
        if self.rot_dims:
            inv, _ = compute_inv_freq(self.rot_dims, float(rot_base), None, dtype=torch.float64)
            self.register_buffer("rope_inv_freq", inv.to(device=device, dtype=torch.float64), persistent=False)
            self.rope_tag = ("half", self.rot_dims, float(rot_base))

    def state_specs(self, cache_index=None):
        return {}

    def kv_shape(self):
        """Key and value heads of a cache row: the layered cache takes one head count, so a row is kept as ``n_kv`` heads of two maps."""
        return (self.n_kv, 2 * self.head_dim, self.v_head_dim)

    def forward(self, x, meta, kv_mgr, cache_index=None):
        p = self.in_proj(x)
        ex = meta.extras
        ctx, qlen = ex["ctx_len"], ex["q_len"]
        cos, sin = ragged_rope_tables(meta, p.shape[1], self.rot_dims, 0.0, self.rope_inv_freq, 1.0, self.rope_tag) if self.rot_dims else (None, None)
        k, v = kv_mgr.get_kv_by_layer_id(self.layer_idx if cache_index is None else cache_index)
        k = k.view(k.shape[0], k.shape[1], 2 * self.n_kv, self.head_dim)
        q = ops.head_norm_rope_append(p, 2 * self.n_q, 2 * self.n_kv, self.head_dim, self.v_head_dim, cos, sin, None, None, 0, self.eps, False,
                                      k, v, meta.block_table, ctx, qlen, n_v=self.n_kv)
        return self.o_proj(ops.paged_diff_attention(q, k, v, meta.block_table, ctx, qlen, self.scale, self.lam, self.out_scale, self.eps,
                                                    self.window or 0))
