"""Grouped-head causal attention without a softmax, inside chunks of positions, over values that carry their position:

    q = R(pos) rmsnorm(W_q x),  k = R(pos) rmsnorm(W_k x)   (norms over the whole projection, all heads at once)
    v = P(pos) W_v x,   o_h = P(pos)^-1 sum_j sigmoid((q_h . k_j) * scale + b_h) v_j,   y = W_o o

The sum runs over the keys j <= i of the query's chunk, floor(j / chunk) = floor(i / chunk); weights are not normalised.  R
turns halves of the first ``rope_dims`` channels of a head, P halves of all value channels.

One product computes [q | k | v], one kernel turns it into queries and cache rows, and the attention kernels turn outputs
back when they store.  Value channels m and m + vdim / 2 of a head lie side by side inside the layer (rows of W_v and columns
of W_o are reordered once after loading), so a pair never leaves a thread.  Heads are padded with zeros to a kernel head size
in the cache.
"""
from __future__ import annotations

import torch
from torch import nn

from ..ops import SigmoidWeights, qk_attn
from .linear import LiteLinear
from .paged import attend, tensor_head_size
from .rope import get_cos_sin


def _vec(n: int) -> nn.Parameter:
    return nn.Parameter(torch.ones(n, dtype=torch.float32), requires_grad=False)


class SigmoidAttention(nn.Module):
    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, dtype, chunk: int = 0,
                 rope_base: float = 10000.0, rope_dims: int | None = None, max_pos: int = 4096):
        super().__init__()
        if vdim % 2:
            raise ValueError("values that turn in pairs need an even number of channels")
        self.nh, self.nkv, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.scale, self.eps, self.chunk = float(scale), float(eps), int(chunk)
        self.rope_base, self.rope_dims, self.max_pos = float(rope_base), dim if rope_dims is None else rope_dims, max_pos
        splits = [heads * dim, kv_heads * dim, kv_heads * vdim]
        self.qkv_proj = LiteLinear(hidden, sum(splits), dtype=dtype, out_splits=splits)
        self.q_norm, self.k_norm, self.bias = _vec(heads * dim), _vec(kv_heads * dim), _vec(heads)
        self.o_proj = LiteLinear(heads * vdim, hidden, dtype=dtype)
        hd = tensor_head_size(dtype, dim, vdim) if dim % 2 == 0 else 0
        self.tensor = hd > 0
        self.key_width, self.value_width = (hd, hd) if self.tensor else (dim, vdim)
        self._tables = None

    def cache_shape(self) -> tuple[int, int, int]:
        """Heads, key and value channels of a cache row."""
        return self.nkv, self.key_width, self.value_width

    def finish_loading(self) -> None:
        half, w, o = self.vdim // 2, self.qkv_proj.weight.data, self.o_proj.weight.data
        v = w[-self.nkv * self.vdim:]
        v.copy_(v.view(self.nkv, 2, half, -1).transpose(1, 2).reshape(v.shape).clone())
        o.copy_(o.view(o.shape[0], self.nh, 2, half).transpose(2, 3).reshape(o.shape).clone())

    def tables(self, device):
        """(cos | sin) rows per position: of queries and keys, of values."""
        if self._tables is None or self._tables[0] != device:
            cs = [get_cos_sin(n, self.max_pos, self.rope_base, None, device) for n in (self.rope_dims, self.vdim)]
            self._tables = (device, cs[0], cs[1], SigmoidWeights(self.bias.data, self.chunk, cs[1]))
        return self._tables[1:]

    def forward(self, x, batch, kv):
        """x [T, hidden] -> [T, hidden]; kv: the layer's key and value pages."""
        cos_sin, v_cos_sin, weights = self.tables(x.device)
        q = qk_attn.prepare(self.qkv_proj(x), self.q_norm, self.k_norm, self.eps, batch.positions, cos_sin, batch.slot_mapping, *kv,
                            self.nh, self.nkv, self.dim, self.vdim, v_cos_sin)
        return self.o_proj(attend(q, kv, batch, self.nkv, self.scale, 0, self.vdim, self.tensor, sigmoid=weights))
