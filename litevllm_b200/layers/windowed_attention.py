"""Grouped-head attention over a sliding window whose values are its keys:

    q = R(pos) rmsnorm(W_q x),  k = R(pos) rmsnorm(W_k x)   (norms over the whole projection, all heads at once)
    v = W_k x,   o_h = sum_j p_hj v_j,   p_hj = exp(s_hj) / (exp(sink) + sum_i exp(s_hi)),   s = (q . k) * scale
    y = W_o (o * sigmoid(W_g x))

One product computes [q | k | gate], one kernel turns it into queries and cache rows, and the attention kernels apply the
gate when they store.  Heads are padded with zeros to a kernel head size in the cache.  Sizes, window, rotation, scale, the
sink's score and the gate are parameters.
"""
from __future__ import annotations

import torch
from torch import nn

from ..ops import qk_attn
from .linear import LiteLinear
from .paged import attend, tensor_head_size
from .rope import get_cos_sin


class WindowedAttention(nn.Module):
    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, scale: float, eps: float, dtype, window: int = 0,
                 rope_base: float = 10000.0, rope_dims: int | None = None, sink: float | None = None, gated: bool = True,
                 max_pos: int = 4096):
        super().__init__()
        self.nh, self.nkv, self.dim = heads, kv_heads, dim
        self.scale, self.eps, self.window = float(scale), float(eps), int(window)
        self.rope_base, self.rope_dims, self.max_pos = float(rope_base), dim if rope_dims is None else rope_dims, max_pos
        self.nq, self.nk, self.gated = heads * dim, kv_heads * dim, gated
        splits = [self.nq, self.nk] + ([self.nq] if gated else [])
        self.qkg_proj = LiteLinear(hidden, sum(splits), dtype=dtype, out_splits=splits)
        self.q_norm = nn.Parameter(torch.ones(self.nq, dtype=torch.float32), requires_grad=False)
        self.k_norm = nn.Parameter(torch.ones(self.nk, dtype=torch.float32), requires_grad=False)
        self.o_proj = LiteLinear(self.nq, hidden, dtype=dtype)
        self.sinks = None if sink is None else nn.Parameter(torch.full((heads,), float(sink), dtype=torch.float32),
                                                            requires_grad=False)
        self._cos_sin = None
        hd = tensor_head_size(dtype, dim) if dim % 2 == 0 else 0
        self.tensor, self.hd = hd > 0, hd or dim

    def cache_shape(self) -> tuple[int, int]:
        return self.nkv, self.hd

    def cos_sin(self, device):
        if self._cos_sin is None or self._cos_sin.device != device:
            self._cos_sin = get_cos_sin(self.rope_dims, self.max_pos, self.rope_base, None, device)
        return self._cos_sin

    def forward(self, x, batch, kv):
        """x [T, hidden] -> [T, hidden]; kv: the layer's key and value pages [blocks, kv heads, block size, hd]."""
        k_cache, v_cache = kv
        proj = self.qkg_proj(x)
        gate = proj[:, self.nq + self.nk:] if self.gated else None
        q = qk_attn.prepare(proj, self.q_norm, self.k_norm, self.eps, batch.positions, self.cos_sin(x.device),
                            batch.slot_mapping, k_cache, v_cache, self.nh, self.nkv, self.dim)
        o = attend(q, kv, batch, self.nkv, self.scale, self.window, self.dim, self.tensor, self.sinks, gate)
        return self.o_proj(o)
