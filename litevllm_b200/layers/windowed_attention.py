"""Grouped-head attention over a sliding window whose values are its keys:

    q = R(pos) rmsnorm(W_q x),  k = R(pos) rmsnorm(W_k x)   (norms over the whole projection, all heads at once)
    v = W_k x,   o_h = sum_j p_hj v_j,   p_hj = exp(s_hj) / (exp(sink) + sum_i exp(s_hi)),   s = (q . k) * scale
    y = W_o (o * sigmoid(W_g x))

One product computes [q | k | gate], one kernel turns it into queries and cache rows, and the attention kernels apply the
gate when they store.  Decode and short portions run split-KV / ``mma.sync`` kernels, portions of at least
``LONG_PORTION`` tokens the tcgen05 prefill kernel; 32-bit models and head sizes outside those kernels the general row
kernel.  Heads are padded with zeros to a kernel head size in the cache.  Sizes, window, rotation, scale, the sink's score
and the gate are parameters.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..ops import qk_attn
from .linear import LiteLinear
from .rope import get_cos_sin

LONG_PORTION = 64


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
        # head size of the tensor-core kernels that holds a head; 0: none does
        self.tensor = dtype != torch.float32 and dim % 2 == 0 and dim <= 256
        self.hd = next(hd for hd in (64, 128, 256) if dim <= hd) if self.tensor else dim

    def cache_shape(self) -> tuple[int, int]:
        return self.nkv, self.hd

    def cos_sin(self, device):
        if self._cos_sin is None or self._cos_sin.device != device:
            self._cos_sin = get_cos_sin(self.rope_dims, self.max_pos, self.rope_base, None, device)
        return self._cos_sin

    def _portions(self, q, k_cache, v_cache, batch, gate):
        """Varlen portions on the tensor-core kernels; long ones (at the front of the step) and short ones apart."""
        n = 0
        for m in batch.q_lens_cpu:
            if m < LONG_PORTION:
                break
            n += 1
        B, T = len(batch.q_lens_cpu), q.shape[0]
        out = torch.empty(T, self.nq, dtype=q.dtype, device=q.device)
        t = sum(batch.q_lens_cpu[:n])
        for lo, hi, a, e in ((0, n, 0, t), (n, B, t, T)):
            if lo == hi:
                continue
            cu = batch.cu_q[lo:hi + 1]
            if lo:
                cu = batch.extras.get("short_cu")
                if cu is None:
                    cu = batch.extras["short_cu"] = (batch.cu_q[lo:hi + 1] - t).contiguous()
            ops.paged_attention_prefill(q[a:e].view(e - a, -1), k_cache, v_cache, batch.block_tables[lo:hi],
                                        batch.seq_lens[lo:hi], cu, max(batch.q_lens_cpu[lo:hi]), self.nh, self.nkv, self.hd,
                                        self.scale, self.window, out=out[a:e], sinks=self.sinks, v_dim=self.dim,
                                        gate=None if gate is None else gate[a:e])
        return out

    def forward(self, x, batch, kv):
        """x [T, hidden] -> [T, hidden]; kv: the layer's key and value pages [blocks, kv heads, block size, hd]."""
        k_cache, v_cache = kv
        T = x.shape[0]
        proj = self.qkg_proj(x)
        gate = proj[:, self.nq + self.nk:] if self.gated else None
        q = qk_attn.prepare(proj, self.q_norm, self.k_norm, self.eps, batch.positions, self.cos_sin(x.device),
                            batch.slot_mapping, k_cache, v_cache, self.nh, self.nkv, self.dim)
        if x.is_cuda and self.tensor:
            if batch.is_decode:
                o = ops.paged_attention_decode(q.view(T, -1), k_cache, v_cache, batch.block_tables, batch.seq_lens, self.nh,
                                               self.nkv, self.hd, self.scale, self.window, max_kv_len=batch.max_kv_len,
                                               sinks=self.sinks, v_dim=self.dim, gate=gate)
            else:
                o = self._portions(q, k_cache, v_cache, batch, gate)
        else:
            lens, seq = batch.seq_lens, None
            if not batch.is_decode:
                rows = batch.extras.get("token_rows")
                if rows is None:
                    tok = torch.arange(T, dtype=torch.int32, device=x.device)
                    seq = torch.searchsorted(batch.cu_q[1:].contiguous(), tok, right=True).to(torch.int32)
                    rows = batch.extras["token_rows"] = ((batch.positions + 1).to(torch.int32), seq)
                lens, seq = rows
            o = qk_attn.attend_rows(q, k_cache, v_cache, batch.block_tables, lens, seq, self.scale, self.window, self.sinks,
                                    gate, self.dim)
        return self.o_proj(o)
