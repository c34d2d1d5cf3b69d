"""Grouped-head attention over paged keys and values with a norm over the whole query / key projection, values taken
from the keys before norm and rotation, a constant in the softmax denominator and an output gate.

``prepare`` turns the merged projection of a step into cache rows and rotated queries; ``attend_rows`` is the general
form over flattened query rows (32-bit models, head sizes outside the tensor-core kernels).  Kernels:
csrc/attn/qk_prepare.cu, csrc/attn/latent_rows.cu; the tensor-core forms are ``ops.paged_attention_decode`` and
``ops.paged_attention_prefill``.  CPU tensors run PyTorch forms.
"""
from __future__ import annotations

import torch

from . import _DT, _count, _lib, _p, _stream
from .. import ops as _ops


def _rotate_halves(x, cos, sin):
    """x [T, heads, dim] fp32: channels i and i + half turn together; the rest pass."""
    half = cos.shape[-1]
    out = x.clone()
    u, v = x[..., :half], x[..., half:2 * half]
    out[..., :half] = u * cos - v * sin
    out[..., half:2 * half] = v * cos + u * sin
    return out


def _normed(x, w, eps: float):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w


def prepare(proj, wq, wk, eps: float, positions, cos_sin, slot_mapping, k_cache, v_cache, H: int, G: int, dim: int):
    """proj [T, >= (H + G) * dim] (q | k); caches [blocks, G, block size, hd] with hd >= dim (the rest is cleared); slots
    < 0 write no cache row.  Returns queries [T, H, hd] in the type of ``proj``."""
    T, hd, bs = proj.shape[0], k_cache.shape[3], k_cache.shape[2]
    q_out = torch.empty(T, H, hd, dtype=proj.dtype, device=proj.device)
    if not proj.is_cuda:
        half = cos_sin.shape[1] // 2
        cs = cos_sin[positions.long()][:, None]
        q = _normed(proj[:, :H * dim].float(), wq, eps).view(T, H, dim)
        raw = proj[:, H * dim:(H + G) * dim].float()
        k = _normed(raw, wk, eps).view(T, G, dim)
        q_out.zero_()
        q_out[..., :dim] = _rotate_halves(q, cs[..., :half], cs[..., half:]).to(proj.dtype)
        k = _rotate_halves(k, cs[..., :half], cs[..., half:])
        at = torch.nonzero(slot_mapping >= 0).view(-1)
        slot = slot_mapping[at].long()
        for cache, rows in ((k_cache, k), (v_cache, raw.view(T, G, dim))):
            full = torch.zeros(at.shape[0], G, hd, dtype=cache.dtype)
            full[..., :dim] = rows[at].to(cache.dtype)
            cache[slot // bs, :, slot % bs] = full
        return q_out
    if _ops._BOUNDS_CHECK:
        _ops._check_index("qk_attn.prepare.slot_mapping", slot_mapping, -(1 << 31), k_cache.shape[0] * bs,
                          "flat slots of the cache pool; negative = skip")
        _ops._check_index("qk_attn.prepare.positions", positions, 0, cos_sin.shape[0], "rows of the cos/sin table")
    assert proj.stride(1) == 1 and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert k_cache.dtype == v_cache.dtype == proj.dtype and positions.dtype == slot_mapping.dtype == torch.int32
    rc = _lib.kernels().fi_qk_prepare(_p(proj), proj.stride(0), _p(wq), _p(wk), eps, _p(positions), _p(cos_sin),
                                      cos_sin.shape[0], _p(slot_mapping), _p(q_out), _p(k_cache), _p(v_cache), T, H, G, dim,
                                      hd, cos_sin.shape[1], bs, _DT[proj.dtype], _stream())
    _lib.check(rc, "fi_qk_prepare")
    _count()
    return q_out


def attend_rows(q, k_cache, v_cache, block_tables, row_lens, seq_of_row, scale: float, window: int, sinks, gate, dim: int):
    """q [R, H, hd]; row r sees the first ``row_lens[r]`` tokens (the last ``window`` of them) of sequence
    ``seq_of_row[r]`` (None: sequence r).  Returns [R, H * dim], gated by ``sigmoid(gate)``."""
    R, H, hd = q.shape
    G, bs = k_cache.shape[1], k_cache.shape[2]
    if not q.is_cuda:
        out = torch.zeros(R, H, dim, dtype=q.dtype)
        for r in range(R):
            n = int(row_lens[r])
            if n <= 0:
                continue
            b = r if seq_of_row is None else int(seq_of_row[r])
            pos = torch.arange(max(0, n - window) if window else 0, n)
            blk = block_tables[b].long()[pos // bs]
            k = k_cache[blk, :, pos % bs].float().repeat_interleave(H // G, 1)              # [n, H, hd]
            v = v_cache[blk, :, pos % bs].float().repeat_interleave(H // G, 1)
            s = torch.einsum("hd,nhd->hn", q[r].float(), k) * scale
            if sinks is not None:
                s = torch.cat([s, sinks[:, None]], dim=1)
            a = torch.softmax(s, dim=-1)[:, :k.shape[0]]
            out[r] = torch.einsum("hn,nhd->hd", a, v)[:, :dim].to(out.dtype)
        out = out.reshape(R, H * dim)
        return out if gate is None else (out.float() * torch.sigmoid(gate.float())).to(out.dtype)
    if hd != dim:
        raise ValueError("the general row kernel reads caches without padded channels")
    if _ops._BOUNDS_CHECK:
        _ops._check_index("qk_attn.row_lens", row_lens, 0, block_tables.shape[1] * bs + 1, "tokens per block table row")
        _ops._check_index("qk_attn.block_tables", block_tables, 0, k_cache.shape[0], "blocks of the cache pool")
    assert q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous() and block_tables.is_contiguous()
    out = torch.empty(R, H * dim, dtype=q.dtype, device=q.device)
    rc = _lib.kernels().fi_attn_rows(_p(q), _p(k_cache), _p(v_cache), _p(out), _p(block_tables), _p(row_lens), _p(seq_of_row),
                                     R, H, G, hd, dim, block_tables.shape[1], bs, k_cache.shape[0], int(window), _p(sinks),
                                     _p(gate), gate.stride(0) if gate is not None else 0, scale, _DT[q.dtype], _stream())
    _lib.check(rc, "fi_attn_rows")
    _count()
    return out
