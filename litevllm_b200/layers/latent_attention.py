"""Latent attention: keys and values are up-projections of one small normalised latent per token, plus one rotary key
part shared by all heads; only ``[latent | rotary key]`` is cached.

    c = rmsnorm(W_c x),  k_r = R(pos) W_r x,   k_h = [W_uk,h c | k_r],  v_h = W_uv,h c
    o_h = sum_j a_hj v_hj,  a_h = softmax over the visible j of (q_h . k_hj) * scale, with exp(sink_h) added to the
    denominator when the layer has sinks;   y = W_o [o_1 .. o_H]

Two forms of the same result, chosen per part of a step:
  rows     every new token is a row with its own visible length; W_uk is applied to the query and W_uv to the sums of
           latents, so the kernel reads cache rows only (decode, short portions, 32-bit models)
  context  portions of at least ``LONG_PORTION`` tokens: the visible context is gathered, up-projected once and laid
           out as per-head tiles for the prefill attention kernel
Sizes, the window, the rotation base, the scale and the presence of sinks are parameters.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..ops import latent_attn as la
from .linear import LiteLinear
from .rope import get_cos_sin

LONG_PORTION = 64


class LatentAttention(nn.Module):
    def __init__(self, hidden: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int, scale: float, eps: float,
                 dtype, window: int = 0, rope_base: float = 10000.0, rope_dims: int | None = None, sinks: bool = False,
                 max_pos: int = 4096):
        super().__init__()
        self.nh, self.dim, self.rot, self.vdim, self.rank = heads, dim, rot_dim, vdim, kv_rank
        self.scale, self.eps, self.window = float(scale), float(eps), int(window)
        self.rope_base, self.rope_dims, self.max_pos = float(rope_base), rot_dim if rope_dims is None else rope_dims, max_pos
        self.q_size, self.kd = heads * (dim + rot_dim), kv_rank + rot_dim
        self.qkv_proj = LiteLinear(hidden, self.q_size + self.kd, dtype=dtype, out_splits=[self.q_size, self.kd])
        self.latent_norm = nn.Parameter(torch.ones(kv_rank, dtype=torch.float32), requires_grad=False)
        self.up_proj = LiteLinear(kv_rank, heads * (dim + vdim), dtype=dtype, out_splits=[heads * dim, heads * vdim])
        self.o_proj = LiteLinear(heads * vdim, hidden, dtype=dtype)
        self.sinks = nn.Parameter(torch.zeros(heads, dtype=torch.float32), requires_grad=False) if sinks else None
        self._cos_sin = None
        # head size of the prefill kernels that holds both a key and a value; 0: no kernel is that wide
        need = max(dim + rot_dim, vdim)
        self.pool_hd = next((hd for hd in (64, 128, 256) if need <= hd), 0) if vdim % 2 == 0 else 0

    def cache_width(self) -> int:
        return self.kd

    def cos_sin(self, device):
        if self._cos_sin is None or self._cos_sin.device != device:
            self._cos_sin = get_cos_sin(self.rope_dims, self.max_pos, self.rope_base, None, device)
        return self._cos_sin

    def _rows(self, q, dkv, cache, positions, slot_mapping, block_tables, row_lens, seq_of_row, max_len, out):
        T, nh, dim, rank = q.shape[0], self.nh, self.dim, self.rank
        q_cat = torch.empty(T, nh, self.kd, dtype=q.dtype, device=q.device)
        up = self.up_proj.weight
        w_uk = up[:nh * dim].view(nh, dim, rank)
        w_uv = up[nh * dim:].view(nh, self.vdim, rank)
        qn = q.unflatten(1, (nh, dim + self.rot))[..., :dim].transpose(0, 1)
        torch.bmm(qn, w_uk, out=q_cat[..., :rank].transpose(0, 1))
        la.prepare(q, dkv, self.latent_norm, self.eps, positions, self.cos_sin(q.device), slot_mapping, cache, q_cat, nh,
                   dim, self.rot, rank, -1, rank)
        lat = la.attend_rows(q_cat, cache, block_tables, row_lens, seq_of_row, rank, self.scale, self.window, self.sinks,
                             max_len)
        torch.bmm(lat, w_uv.transpose(1, 2), out=out.view(T, nh, self.vdim).transpose(0, 1))

    def _context(self, q, dkv, cache, batch, n_seqs, out):
        T, nh, hd = q.shape[0], self.nh, self.pool_hd
        q_pad = torch.empty(T, nh, hd, dtype=q.dtype, device=q.device)
        la.prepare(q, dkv, self.latent_norm, self.eps, batch.positions[:T], self.cos_sin(q.device), batch.slot_mapping[:T],
                   cache, q_pad, nh, self.dim, self.rot, self.rank, 0, self.dim)
        plans = batch.extras.setdefault("latent_context", {})
        plan = plans.get(self.window)
        if plan is None:
            plan = la.ContextPlan(batch.block_tables, cache.shape[2], batch.seq_lens_cpu[:n_seqs],
                                  batch.q_lens_cpu[:n_seqs], self.window, q.device)
            plans[self.window] = plan
        k_pool, v_pool = la.context_pool(plan, cache, self.up_proj.weight, nh, self.dim, self.rot, self.vdim, self.rank, hd)
        ops.paged_attention_prefill(q_pad.view(T, nh * hd), k_pool, v_pool, plan.table, plan.lens, batch.cu_q[:n_seqs + 1],
                                    max(batch.q_lens_cpu[:n_seqs]), nh, nh, hd, self.scale, self.window, out=out,
                                    sinks=self.sinks, v_dim=self.vdim)

    def _long_prefix(self, batch, x) -> tuple[int, int]:
        """(sequences, tokens) at the front of the step that take the context form."""
        if batch.is_decode or not x.is_cuda or x.dtype == torch.float32 or not self.pool_hd:
            return 0, 0
        n = tokens = 0
        for q in batch.q_lens_cpu:
            if q < LONG_PORTION:
                break
            n, tokens = n + 1, tokens + q
        return n, tokens

    def forward(self, x, batch, cache):
        """x [T, hidden] -> [T, hidden]; cache: the layer's rows [blocks, 1, block size, rank + rot]."""
        T = x.shape[0]
        proj = self.qkv_proj(x)
        q, dkv = proj[:, :self.q_size], proj[:, self.q_size:]
        width = self.nh * self.vdim
        out = torch.empty(T, width, dtype=x.dtype, device=x.device)
        if batch.is_decode:
            self._rows(q, dkv, cache, batch.positions, batch.slot_mapping, batch.block_tables, batch.seq_lens, None,
                       batch.max_kv_len, out)
        else:
            n, t = self._long_prefix(batch, x)
            if n:
                self._context(q[:t], dkv[:t], cache, batch, n, out[:t])
            if t < T:
                rows = batch.extras.get("token_rows")
                if rows is None:
                    lens = batch.positions + 1
                    tok = torch.arange(T, dtype=torch.int32, device=x.device)
                    seq = torch.searchsorted(batch.cu_q[1:].contiguous(), tok, right=True).to(torch.int32)
                    rows = batch.extras["token_rows"] = (lens.to(torch.int32), seq)
                self._rows(q[t:], dkv[t:], cache, batch.positions[t:], batch.slot_mapping[t:], batch.block_tables,
                           rows[0][t:], rows[1][t:], max(batch.seq_lens_cpu[n:]), out[t:])
        return self.o_proj(out)
