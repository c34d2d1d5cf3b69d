"""Gated delta rule with one decay per head and key channel:

    q, k, v = silu(conv(W_q x)), silu(conv(W_k x)), silu(conv(W_v x))     (short causal convolutions per channel)
    q = q / |q| * dim^-1/2,  k = k / |k|,  beta = sigmoid(W_b x),  g = exp(-exp(A) softplus(W_a2 W_a1 x + bias))
    S <- diag(g) S,   u = beta (v - S^T k),   S <- S + k u^T,   o = S^T q
    y = W_o [rmsnorm(o_h) * sigmoid(W_g2 W_g1 x)_h]

The state S [heads, dim, vdim] is 32-bit and lives, with the last convolution inputs, in per-slot pools of the cache
manager.  One product computes q | k | v and the low-rank halves of decay and gate, a second one (block diagonal) expands
those.  Portions of prompts run the chunked kernels for the whole step, decode one step kernel that includes convolution,
head norm and gate.  The write strength's projection comes from outside: it shares a 32-bit product with the router.
"""
from __future__ import annotations

import torch
from torch import nn

from ..ops import linear_attn
from .linear import LiteLinear

# from this many tokens decay and gate are expanded by products of their own (32-bit decays, gates in the model's type)
_SPLIT_TOKENS = 1024


def _pad8(n: int) -> int:
    return (n + 7) // 8 * 8


class ChannelDelta(nn.Module):
    def __init__(self, hidden: int, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, eps: float, dtype):
        super().__init__()
        self.nh, self.nkv, self.dim, self.vdim, self.taps, self.eps = heads, kv_heads, dim, vdim, taps, float(eps)
        self.nk, self.nv, self.nz = kv_heads * dim, heads * vdim, heads * dim
        self.channels = 2 * self.nk + self.nv
        self.hidden, self.dtype = hidden, dtype
        # rows: query | key | value, then the low-rank halves (decay, gate) once their ranks are known
        self.in_proj = LiteLinear(hidden, self.channels, dtype=dtype, out_splits=[self.nk, self.nk, self.nv])
        self.expand = None
        self.conv = nn.Parameter(torch.zeros(self.channels, taps, dtype=torch.float32), requires_grad=False)
        self.A_log = nn.Parameter(torch.zeros(heads, dtype=torch.float32), requires_grad=False)
        self.dt_bias = nn.Parameter(torch.zeros(self.nz, dtype=torch.float32), requires_grad=False)
        self.head_norm = nn.Parameter(torch.ones(vdim, dtype=torch.float32), requires_grad=False)
        self.o_proj = LiteLinear(self.nv, hidden, dtype=dtype)
        self._low: dict[str, torch.Tensor] = {}
        self.spec = None

    def state_shape(self) -> tuple[int, int, int]:
        return self.nh, self.dim, self.vdim

    def ring_shape(self) -> tuple[int, int]:
        return self.taps, self.channels

    # ------------------------------------------------------------------ loading
    def conv_rows(self, which: str) -> torch.Tensor:
        lo = {"q": 0, "k": self.nk, "v": 2 * self.nk}[which]
        return self.conv[lo:lo + (self.nv if which == "v" else self.nk)]

    def low_rank(self, name: str):
        """Receiver of one factor ("a1", "a2": decay, "g1", "g2": gate); the ranks are the checkpoint's."""
        def take(tensor):
            rows = {"a2": self.nz, "g2": self.nv}.get(name)
            if tensor.dim() != 2 or (rows is None and tensor.shape[1] != self.hidden) or (rows is not None and tensor.shape[0] != rows):
                raise ValueError(f"low-rank factor {name!r} has shape {tuple(tensor.shape)}")
            self._low[name] = tensor.to(device=self.conv.device, dtype=self.dtype)
        return take

    def finish_loading(self) -> None:
        a1, a2, g1, g2 = (self._low[n] for n in ("a1", "a2", "g1", "g2"))
        ra, rg = a1.shape[0], g1.shape[0]
        if a2.shape[1] != ra or g2.shape[1] != rg:
            raise ValueError(f"low-rank factors do not fit: {tuple(a1.shape)} with {tuple(a2.shape)}, {tuple(g1.shape)} with {tuple(g2.shape)}")
        # ranks are padded with zeros to whole 16-byte groups
        self.ra, self.rg = _pad8(ra), _pad8(rg)
        first = _pad8(self.channels)
        w = self.in_proj.weight.data
        merged = torch.zeros(first + self.ra + self.rg, self.hidden, dtype=self.dtype, device=w.device)
        merged[:self.channels], merged[first:first + ra], merged[first + self.ra:first + self.ra + rg] = w, a1, g1
        self.low0 = first
        self.in_proj.weight = nn.Parameter(merged, requires_grad=False)
        self.in_proj.out_features = self.in_proj.full_out = merged.shape[0]
        self.in_proj.out_splits = [self.nk, self.nk, self.nv, merged.shape[0] - self.channels]
        e = torch.zeros(self.nz + self.nv, self.ra + self.rg, dtype=self.dtype, device=w.device)
        e[:self.nz, :ra], e[self.nz:, self.ra:self.ra + rg] = a2, g2
        self.expand = LiteLinear(self.ra + self.rg, self.nz + self.nv, dtype=self.dtype, out_splits=[self.nz, self.nv])
        self.expand.weight = nn.Parameter(e, requires_grad=False)
        self._low.clear()
        self.spec = linear_attn.DeltaSpec(self.nh, self.nkv, self.dim, self.vdim, self.conv.data, torch.exp(self.A_log.data),
                                          self.dt_bias.data)

    # ------------------------------------------------------------------ forward
    def forward(self, x, b, batch, pool, ring):
        """x [T, hidden], b fp32 [T, heads] (projection of the write strength) -> [T, hidden]; pool fp32 [slots, heads,
        dim, vdim], ring fp32 [slots, taps, channels]."""
        from .. import ops
        p = self.in_proj(x)
        qkv, low = p[:, :self.channels], p[:, self.low0:]
        if x.shape[0] >= _SPLIT_TOKENS and x.is_cuda and x.dtype != torch.float32:
            w = self.expand.weight
            z = ops.linear(low[:, :self.ra], w[:self.nz, :self.ra], out_dtype=torch.float32)
            gate = ops.linear(low[:, self.ra:], w[self.nz:, self.ra:])
        else:
            zg = self.expand(low, out_dtype=torch.float32)
            z, gate = zg[:, :self.nz], zg[:, self.nz:]
        slots = batch.extras.get("slot_ids")
        if slots is None:
            raise RuntimeError("the batch carries no slot ids (recurrent state is pooled by slot)")
        if batch.is_decode:
            o = linear_attn.delta_step(qkv, z, b, self.spec, pool, ring, slots, batch.seq_lens, self.head_norm, self.eps, gate,
                                       x.dtype)
        else:
            chunks = batch.extras.get("delta_chunks")
            if chunks is None:
                n = sum(-(-m // linear_attn.DELTA_CHUNK) for m in batch.q_lens_cpu)
                chunks = batch.extras["delta_chunks"] = (linear_attn.delta_chunks(batch.cu_q), n)
            o = linear_attn.delta_portions(qkv, z, b, self.spec, pool, ring, slots, batch.cu_q, batch.seq_lens, *chunks)
            o = linear_attn.head_norm(o, self.head_norm, self.eps, x.dtype, gate)
        return self.o_proj(o)
