"""Mamba-2: a state-space layer with one scalar decay per head.

    [z | x | B | C | dt] = W_in h,   x, B, C <- silu(conv([x | B | C]) + b)       (short causal convolution per channel)
    dt <- softplus(dt + bias),   S[i, :] <- a S[i, :] + dt B_i x  with  ln a = -dt e^A,   then  y = C S + D x     (per head)
    out = W_o [rms over equal parts of (y silu(z))] * norm

B and C [groups, state] are shared by groups of heads.  The state S [heads, state, vdim] is 32-bit and lives, with the last
convolution inputs, in per-slot pools of the cache manager.  Portions of prompts run a convolution, a scan and a norm kernel
for the whole step, decode one step kernel (convolution included) and the norm.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..ops import linear_attn
from .linear import LiteLinear

# from this many tokens the projections that may be 16-bit (z, x, B, C) are written as 16-bit values by their own product
_SPLIT_TOKENS = 1024


def _vec(*shape: int) -> nn.Parameter:
    return nn.Parameter(torch.zeros(*shape, dtype=torch.float32), requires_grad=False)


class Mamba2(nn.Module):
    def __init__(self, hidden: int, heads: int, vdim: int, state: int, groups: int, norm_groups: int, taps: int, eps: float, dtype):
        super().__init__()
        self.nh, self.vdim, self.state, self.groups, self.parts = heads, vdim, state, groups, norm_groups
        self.taps, self.eps, self.inner = taps, float(eps), heads * vdim
        self.channels = self.inner + 2 * groups * state
        self.split = self.inner + self.channels
        # rows: z | x | B | C | dt
        self.in_proj = LiteLinear(hidden, self.split + heads, dtype=dtype)
        self.conv, self.conv_bias = _vec(taps, self.channels), _vec(self.channels)
        self.dt_bias, self.A_log, self.D, self.norm = _vec(heads), _vec(heads), _vec(heads), _vec(self.inner)
        self.o_proj = LiteLinear(self.inner, hidden, dtype=dtype)
        self.rate = None

    def state_shape(self) -> tuple[int, int, int]:
        return self.nh, self.state, self.vdim

    def ring_shape(self) -> tuple[int, int]:
        return self.taps, self.channels

    def destinations(self, prefix: str) -> dict:
        """Checkpoint name -> where its values go."""
        return {prefix + "in": (self.in_proj, 0, "weight"), prefix + "conv": self.conv.data.t(), prefix + "conv.b": self.conv_bias,
                prefix + "dt_bias": self.dt_bias, prefix + "A_log": self.A_log, prefix + "D": self.D, prefix + "norm": self.norm,
                prefix + "o": (self.o_proj, 0, "weight")}

    def finish_loading(self) -> None:
        self.rate = torch.exp(self.A_log.data)

    def forward(self, x, batch, pool, ring):
        """x [T, hidden] -> [T, hidden]; pool fp32 [slots, heads, state, vdim], ring fp32 [slots, taps, channels]."""
        w = self.in_proj.weight
        if x.shape[0] >= _SPLIT_TOKENS and x.is_cuda and x.dtype != torch.float32:
            p = ops.linear(x, w[:self.split])
            dt = ops.linear(x, w[self.split:], out_dtype=torch.float32)
        else:
            p = self.in_proj(x, out_dtype=torch.float32)
            dt = p[:, self.split:]
        y = linear_attn.ssd(p[:, self.inner:self.split], p[:, :self.inner], dt, self.dt_bias, self.rate, self.D, self.conv,
                            self.conv_bias, pool, ring, self.groups, batch, self.norm, self.parts, self.eps, x.dtype)
        return self.o_proj(y)
