"""HGRN2 mixer: linear attention whose forget gate also decides what is written.

    q = silu(W_q x),  v = W_v x,  f = l + (1 - l) sigmoid(W_f x + b)      (per head and channel)
    S_t = diag(f_t) S_(t-1) + (1 - f_t) v_t^T,   o_t = S_t^T q_t,   y = W_o [rmsnorm(o_1) .. rmsnorm(o_H)]

The state S [heads, dim, vdim] is 32-bit and lives in a per-layer pool of the cache manager with one slot per request.
Portions of prompts run one scan kernel for the whole step, decode one step kernel that includes the head norm.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..ops import linear_attn
from .linear import LiteLinear

# from this many tokens the projections that may be 16-bit (q, v) are written as 16-bit values by their own product
_SPLIT_TOKENS = 1024


class Hgrn2(nn.Module):
    def __init__(self, hidden: int, heads: int, dim: int, vdim: int, eps: float, dtype):
        super().__init__()
        self.nh, self.dim, self.vdim, self.eps = heads, dim, vdim, float(eps)
        self.nq, self.nv = heads * dim, heads * vdim
        # rows: query | value | forget gate
        self.in_proj = LiteLinear(hidden, 2 * self.nq + self.nv, dtype=dtype, out_splits=[self.nq, self.nv, self.nq])
        self.f_bias = nn.Parameter(torch.zeros(self.nq, dtype=torch.float32), requires_grad=False)
        self.lower = nn.Parameter(torch.zeros(self.nq, dtype=torch.float32), requires_grad=False)
        self.head_norm = nn.Parameter(torch.ones(vdim, dtype=torch.float32), requires_grad=False)
        self.o_proj = LiteLinear(self.nv, hidden, dtype=dtype)

    def state_shape(self) -> tuple[int, int, int]:
        return self.nh, self.dim, self.vdim

    def forward(self, x, batch, pool):
        """x [T, hidden] -> [T, hidden]; pool: fp32 [slots, heads, dim, vdim]."""
        split = self.nq + self.nv
        w = self.in_proj.weight
        if x.shape[0] >= _SPLIT_TOKENS and x.is_cuda and x.dtype != torch.float32:
            qv = ops.linear(x, w[:split])
            f = ops.linear(x, w[split:], out_dtype=torch.float32)
        else:
            p = self.in_proj(x, out_dtype=torch.float32)
            qv, f = p[:, :split], p[:, split:]
        q, v = qv[:, :self.nq], qv[:, self.nq:]
        slots = batch.extras.get("slot_ids")
        if slots is None:
            raise RuntimeError("the batch carries no slot ids (recurrent state is pooled by slot)")
        if batch.is_decode:
            o = linear_attn.hgrn2_step(q, f, v, self.f_bias, self.lower, pool, slots, batch.seq_lens, self.head_norm,
                                       self.eps, self.nh, self.dim, self.vdim, x.dtype)
        else:
            o = linear_attn.hgrn2_scan(q, f, v, self.f_bias, self.lower, pool, slots, batch.cu_q, batch.seq_lens, self.nh,
                                       self.dim, self.vdim)
            o = linear_attn.head_norm(o, self.head_norm, self.eps, x.dtype)
        return self.o_proj(o)
