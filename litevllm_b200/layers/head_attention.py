"""Grouped-head causal attention whose queries and keys are normalised head by head:

    q = t(pos) N(R(pos) W_q x),  k = N(R(pos) W_k x),  v = W_v x        (or R after N)
    a_h = sum_j softmax_j((q_h . k_j) * scale) v_j
    y = W_o (a_h * sigmoid((W_g x)_h))_h

with an RMS norm N per head (a weight of the head's channels or none), rotation R over the first channels of a head
(neighbouring channels or halves turn together; optional), a factor t(pos) = 1 + coef ln(1 + floor((pos + 1) / every))
on queries (optional) and one gate value per head (optional).

Differential form: every head has two maps, queries and keys of their own over one value, and

    o_h = a1_h - lambda a2_h,   o_h <- rms(o_h) (1 - init),   lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + init

A cache row holds both keys, [k1 | k2]; queries are [q1 | 0] and [0 | q2], so the paged kernels see plain grouped heads and
take the difference when they store.  One product computes [q | k | v | gate], one kernel turns it into queries and cache
rows.  Heads are padded with zeros to a kernel head size in the cache.
"""
from __future__ import annotations

import torch
from torch import nn

from ..ops import qk_attn
from .linear import LiteLinear
from .paged import attend, tensor_head_size
from .rope import get_cos_sin


def _vec(n: int) -> nn.Parameter:
    return nn.Parameter(torch.ones(n, dtype=torch.float32), requires_grad=False)


def position_factor(max_pos: int, coef: float, every: float, device) -> torch.Tensor:
    """fp32 [max_pos]: 1 + coef ln(1 + floor((p + 1) / every))."""
    p = torch.arange(1, max_pos + 1, dtype=torch.float64, device="cpu")
    return (1.0 + coef * torch.log(torch.floor(p / every) + 1.0)).float().to(device)


class HeadAttention(nn.Module):
    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, eps: float, dtype,
                 norm_weights: bool = True, rope_dims: int = 0, rope_base: float = 10000.0, neighbours: bool = False,
                 norm_last: bool = False, temperature: tuple[float, float] | None = None, head_gate: bool = False,
                 diff_init: float | None = None, max_pos: int = 4096):
        """``norm_last``: the norm's weight multiplies what is already rotated.  ``temperature``: (coef, every).
        ``diff_init``: the differential form's constant (None: ordinary attention)."""
        super().__init__()
        if diff_init is not None and head_gate:
            raise ValueError("the differential form has no output gate")
        self.nh, self.nkv, self.dim, self.vdim, self.scale, self.eps = heads, kv_heads, dim, vdim, float(scale), float(eps)
        self.maps = 1 if diff_init is None else 2
        self.rope_base, self.rope_dims, self.temperature, self.max_pos = float(rope_base), rope_dims, temperature, max_pos
        splits = [heads * self.maps * dim, kv_heads * self.maps * dim, kv_heads * vdim] + ([heads] if head_gate else [])
        self.gated = head_gate
        self.in_proj = LiteLinear(hidden, sum(splits), dtype=dtype, out_splits=splits)
        self.q_norm, self.k_norm = (_vec(dim), _vec(dim)) if norm_weights else (None, None)
        self.o_proj = LiteLinear(heads * vdim, hidden, dtype=dtype)
        hd = tensor_head_size(dtype, self.maps * dim, vdim) if vdim % 2 == 0 else 0
        self.tensor = hd > 0
        self.key_width, self.value_width = (hd, hd) if self.tensor else (self.maps * dim, vdim)
        self.spec = qk_attn.HeadSpec(heads, kv_heads, dim, vdim, self.maps, self.eps, hd if self.tensor else dim,
                                     dim if self.tensor else 0, rope_dims, neighbours, norm_last)
        self.diff_init, self.diff = diff_init, None
        if diff_init is not None:
            self.lq1, self.lk1, self.lq2, self.lk2 = (_vec(dim) for _ in range(4))
        self._tables = None

    def cache_shape(self) -> tuple[int, int, int]:
        """Heads, key and value channels of a cache row."""
        return self.nkv, self.key_width, self.value_width

    def finish_loading(self) -> None:
        if self.diff_init is not None:
            one, two = ((a.double() * b.double()).sum().exp() for a, b in ((self.lq1, self.lk1), (self.lq2, self.lk2)))
            self.diff = (float(one - two) + self.diff_init, 1.0 - self.diff_init, self.eps)

    def tables(self, device):
        """Per position: (cos | sin) rows and the factor of queries."""
        if self._tables is None or self._tables[0] != device:
            cs = get_cos_sin(self.rope_dims, self.max_pos, self.rope_base, None, device) if self.rope_dims else None
            f = position_factor(self.max_pos, *self.temperature, device) if self.temperature else None
            self._tables = (device, cs, f)
        return self._tables[1:]

    def forward(self, x, batch, kv):
        """x [T, hidden] -> [T, hidden]; kv: the layer's key and value pages."""
        proj = self.in_proj(x)
        cos_sin, factor = self.tables(x.device)
        q = qk_attn.prepare_heads(proj, self.q_norm, self.k_norm, self.spec, batch.positions, cos_sin, factor,
                                  batch.slot_mapping, *kv)
        lo = self.spec.v_off + self.nkv * self.vdim
        gate = proj[:, lo:lo + self.nh] if self.gated else None
        return self.o_proj(attend(q, kv, batch, self.nkv, self.scale, 0, self.vdim, self.tensor, gate=gate, diff=self.diff))
