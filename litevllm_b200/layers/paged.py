"""Attention of one step over paged keys and values, whatever the step holds: single tokens, portions of prompts, or
both.  Decode and short portions run split-KV / ``mma.sync`` kernels, portions of at least ``LONG_PORTION`` tokens the
tcgen05 prefill kernel; 32-bit models and head sizes outside those kernels the general row kernel."""
from __future__ import annotations

import torch

from .. import ops
from ..ops import qk_attn

LONG_PORTION = 64


def tensor_head_size(dtype, *widths: int) -> int:
    """Head size of the tensor-core kernels that holds rows of all ``widths``; 0: none does."""
    if dtype == torch.float32 or max(widths) > 256:
        return 0
    return next(hd for hd in (64, 128, 256) if max(widths) <= hd)


def _portions(q, k_cache, v_cache, batch, nh, nkv, hd, scale, window, sinks, v_dim, gate, diff, sigmoid):
    """Varlen portions on the tensor-core kernels; long ones (at the front of the step) and short ones apart."""
    n = 0
    for m in batch.q_lens_cpu:
        if m < LONG_PORTION:
            break
        n += 1
    B, T = len(batch.q_lens_cpu), q.shape[0]
    out = torch.empty(T, (nh if diff is None else nh // 2) * v_dim, dtype=q.dtype, device=q.device)
    t = sum(batch.q_lens_cpu[:n])
    for lo, hi, a, e in ((0, n, 0, t), (n, B, t, T)):
        if lo == hi:
            continue
        cu = batch.cu_q[lo:hi + 1]
        if lo:
            cu = batch.extras.get("short_cu")
            if cu is None:
                cu = batch.extras["short_cu"] = (batch.cu_q[lo:hi + 1] - t).contiguous()
        ops.paged_attention_prefill(q[a:e].view(e - a, -1), k_cache, v_cache, batch.block_tables[lo:hi], batch.seq_lens[lo:hi],
                                    cu, max(batch.q_lens_cpu[lo:hi]), nh, nkv, hd, scale, window, out=out[a:e], sinks=sinks,
                                    v_dim=v_dim, gate=None if gate is None else gate[a:e], diff=diff, sigmoid=sigmoid)
    return out


def attend(q, kv, batch, nkv: int, scale: float, window: int, v_dim: int, tensor: bool, sinks=None, gate=None, diff=None,
           sigmoid=None):
    """q [T, query heads, row] of :mod:`ops.qk_attn`; kv: the layer's key and value pages; ``tensor``: rows are padded for
    the tensor-core kernels.  Returns [T, heads * v_dim]; ``sinks``, ``gate``, ``diff``, ``sigmoid`` as in ``ops.paged_attention_decode``."""
    k_cache, v_cache = kv
    T, nh, hd = q.shape
    if q.is_cuda and tensor:
        if batch.is_decode:
            tables, lens = batch.attention_tables(window or (sigmoid.chunk if sigmoid is not None else 0))
            return ops.paged_attention_decode(q.view(T, -1), k_cache, v_cache, tables, lens, nh, nkv, hd, scale, window,
                                              max_kv_len=batch.max_kv_len, sinks=sinks, v_dim=v_dim, gate=gate, diff=diff,
                                              sigmoid=sigmoid)
        return _portions(q, k_cache, v_cache, batch, nh, nkv, hd, scale, window, sinks, v_dim, gate, diff, sigmoid)
    tables, lens, seq = batch.block_tables, batch.seq_lens, None
    if batch.is_decode:
        tables, lens = batch.attention_tables(window or (sigmoid.chunk if sigmoid is not None else 0))
    else:
        rows = batch.extras.get("token_rows")
        if rows is None:
            tok = torch.arange(T, dtype=torch.int32, device=q.device)
            seq = torch.searchsorted(batch.cu_q[1:].contiguous(), tok, right=True).to(torch.int32)
            rows = batch.extras["token_rows"] = ((batch.positions + 1).to(torch.int32), seq)
        lens, seq = rows
    return qk_attn.attend_rows(q, k_cache, v_cache, tables, lens, seq, scale, window, sinks, gate, v_dim, diff, sigmoid)
