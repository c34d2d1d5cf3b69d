"""Time mixing: linear attention with one decay per head and key channel and a bonus for the current token.  r, k, v, the gate
and the decay each read their own blend of the present and the previous input:

    x_i = x_t + (x_(t-1) - x_t) mu_i                                    (i of r, k, v, g, w; formed with the layer's input)
    r, k, v = W_r x_r, W_k x_k, W_v x_v,   gate = silu(W_g x_g),   ln w = -e^z,  z = W_2 tanh(W_1 x_w) + w0
    o = r S + (sum_i r_i u_i k_i) v,   then  S[i, :] <- w_i S[i, :] + k_i v        (per head; i: key channels)
    y = W_o [rms(o_h) norm_h gate_h]

The state S [heads, dim, dim] is 32-bit and lives in a per-layer pool of the cache manager with one slot per request.  The
four square projections run as one grouped product.  Portions of prompts run one scan
kernel for the whole step, decode one step kernel that includes norm and gate.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..ops import linear_attn, moe
from .linear import LiteLinear

BLENDS = "rkvgw"


def _vec(*shape: int) -> nn.Parameter:
    return nn.Parameter(torch.zeros(*shape, dtype=torch.float32), requires_grad=False)


class TimeMix(nn.Module):
    def __init__(self, hidden: int, heads: int, dim: int, eps: float, dtype):
        super().__init__()
        self.nh, self.dim, self.eps, self.hidden, self.dtype = heads, dim, float(eps), hidden, dtype
        n = heads * dim
        self.proj = nn.Parameter(torch.empty(4, n, hidden, dtype=dtype), requires_grad=False)      # r, k, v, g
        self.mu, self.w0, self.u, self.norm = _vec(5, hidden), _vec(n), _vec(heads, dim), _vec(n)
        self.o_proj = LiteLinear(n, hidden, dtype=dtype)
        self.w1 = self.w2 = None
        self._low: dict[str, torch.Tensor] = {}

    def state_shape(self) -> tuple[int, int, int]:
        return self.nh, self.dim, self.dim

    # ------------------------------------------------------------------ loading
    def destinations(self, prefix: str) -> dict:
        """Checkpoint name -> where its values go; the rank of the decay's factors is the checkpoint's."""
        d = {prefix + "mu." + c: self.mu[i] for i, c in enumerate(BLENDS)}
        d.update({prefix + c: self.proj[i] for i, c in enumerate("rkvg")})
        d.update({prefix + "w0": self.w0, prefix + "u": self.u, prefix + "norm": self.norm, prefix + "o": (self.o_proj, 0, "weight")})
        d.update({prefix + n: (lambda t, n=n: self._low.__setitem__(n, t)) for n in ("w1", "w2")})
        return d

    def finish_loading(self) -> None:
        a, b = self._low["w1"], self._low["w2"]
        if a.dim() != 2 or b.dim() != 2 or a.shape[1] != self.hidden or tuple(b.shape) != (self.nh * self.dim, a.shape[0]):
            raise ValueError(f"low-rank factors do not fit: {tuple(a.shape)} with {tuple(b.shape)}")
        rank, dev = a.shape[0], self.proj.device
        padded = (rank + 7) // 8 * 8                   # whole 16-byte groups; tanh keeps the padding zero
        w1 = torch.zeros(padded, self.hidden, dtype=self.dtype, device=dev)
        w2 = torch.zeros(self.nh * self.dim, padded, dtype=self.dtype, device=dev)
        w1[:rank], w2[:, :rank] = a.to(dev, self.dtype), b.to(dev, self.dtype)
        self.w1, self.w2 = (nn.Parameter(w, requires_grad=False) for w in (w1, w2))
        self._low.clear()

    # ------------------------------------------------------------------ forward
    def forward(self, blends, batch, pool):
        """blends [5, T, hidden] -> [T, hidden]; pool: fp32 [slots, heads, dim, dim]."""
        r, k, v, gate = moe.stacked_linear(blends[:4], self.proj)
        z = ops.linear(ops.linear(blends[4], self.w1, act="tanh"), self.w2, out_dtype=torch.float32)
        return self.o_proj(linear_attn.time_mix(r, k, v, gate, z, self.w0, self.u, pool, batch, self.norm, self.eps, blends.dtype))
