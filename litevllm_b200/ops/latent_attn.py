"""Latent attention over one shared cache row per token, ``[RMS-normed latent (rank) | rotary key (rot)]``.

``prepare`` turns the projections of a step into cache rows and rotated queries; ``attend_rows`` lets flattened query
rows ``[q W_UK | rotated q]`` attend to cache rows (decode, short portions, 32-bit models); ``context`` gathers and
up-projects the visible context of long portions into a temporary per-head pool for the prefill attention kernels.
Kernels: csrc/attn/latent_rows.cu, csrc/attn/mla_decode.cu, csrc/attn/prefill_tc.cu.  CPU tensors run PyTorch forms.
"""
from __future__ import annotations

import torch

from . import _DT, _count, _lib, _p, _stream, scratch
from .. import ops as _ops

POOL_BLOCK = 128        # tokens per block of the temporary pool: one TMA box per key tile


def _rotate_pairs(x, cos, sin):
    """x [..., rot]: channels (2i, 2i + 1), i < cos.shape[-1], turn; the rest pass.  fp32 in, fp32 out."""
    n = 2 * cos.shape[-1]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    out = x.clone()
    out[..., 0:n:2] = u * cos - v * sin
    out[..., 1:n:2] = v * cos + u * sin
    return out


def prepare(q, dkv, norm_w, eps: float, positions, cos_sin, slot_mapping, cache, q_out, nh: int, dim: int, rot: int,
            rank: int, nope_off: int, rot_off: int) -> None:
    """q [T, >= nh * (dim + rot)] (rotary part of a head last), dkv [T, >= rank + rot]; cache [blocks, 1, bs, rank + rot];
    q_out [T, nh, pitch]: rotated parts go to ``rot_off``; with ``nope_off >= 0`` the other dimensions are copied there
    and everything beyond ``dim + rot`` is cleared.  Slots < 0 write no cache row."""
    T = q_out.shape[0]
    kd = rank + rot
    if not q.is_cuda:
        half = cos_sin.shape[1] // 2
        cs = cos_sin[positions.long()]
        cos, sin = cs[:, :half], cs[:, half:]
        c = dkv[:, :rank].float()
        c = c / torch.sqrt(c.pow(2).mean(-1, keepdim=True) + eps) * norm_w
        kr = _rotate_pairs(dkv[:, rank:kd].float(), cos, sin)
        keep = slot_mapping >= 0
        cache.view(-1, kd)[slot_mapping[keep].long()] = torch.cat([c, kr], dim=-1)[keep].to(cache.dtype)
        qh = q[:, :nh * (dim + rot)].reshape(T, nh, dim + rot)
        qr = _rotate_pairs(qh[..., dim:].float(), cos[:, None], sin[:, None])
        if nope_off >= 0:
            q_out.zero_()
            q_out[..., nope_off:nope_off + dim] = qh[..., :dim]
        q_out[..., rot_off:rot_off + rot] = qr.to(q_out.dtype)
        return
    if _ops._BOUNDS_CHECK:
        _ops._check_index("latent_attn.prepare.slot_mapping", slot_mapping, -(1 << 31), cache.shape[0] * cache.shape[2],
                          "flat slots of the cache pool; negative = skip")
        _ops._check_index("latent_attn.prepare.positions", positions, 0, cos_sin.shape[0], "rows of the cos/sin table")
    assert q.stride(1) == dkv.stride(1) == 1 and q_out.is_contiguous() and cache.is_contiguous()
    assert cache.dtype == q.dtype == dkv.dtype == q_out.dtype and positions.dtype == torch.int32 == slot_mapping.dtype
    rc = _lib.kernels().fi_latent_prepare(
        _p(q), q.stride(0), _p(dkv), dkv.stride(0), _p(norm_w), eps, _p(positions), _p(cos_sin), cos_sin.shape[0],
        _p(slot_mapping), _p(cache), _p(q_out), q_out.shape[2], nope_off, rot_off, dim + rot, T, nh, dim, rot,
        cos_sin.shape[1], rank, _DT[q.dtype], _stream())
    _lib.check(rc, "fi_latent_prepare")
    _count()


def attend_rows(q_cat, cache, block_tables, row_lens, seq_of_row, rank: int, scale: float, window: int, sinks,
                max_len: int):
    """q_cat [R, nh, kd]; row r sees the first ``row_lens[r]`` tokens (the last ``window`` of them) of sequence
    ``seq_of_row[r]`` (None: sequence r).  sinks: fp32 [nh] or None.  Returns the sums of latents [nh, R, rank]."""
    R, nh, kd = q_cat.shape
    if not q_cat.is_cuda:
        out = torch.zeros(nh, R, rank, dtype=q_cat.dtype)
        rows = cache.view(-1, kd)
        bs = cache.shape[2]
        for r in range(R):
            n = int(row_lens[r])
            if n <= 0:
                continue
            b = r if seq_of_row is None else int(seq_of_row[r])
            pos = torch.arange(max(0, n - window) if window else 0, n)
            k = rows[block_tables[b].long()[pos // bs] * bs + pos % bs].float()
            s = (q_cat[r].float() @ k.t()) * scale
            if sinks is not None:
                s = torch.cat([s, sinks[:, None]], dim=1)
            a = torch.softmax(s, dim=-1)[:, :k.shape[0]]
            out[:, r] = (a @ k[:, :rank]).to(out.dtype)
        return out
    if _ops._BOUNDS_CHECK:
        _ops._check_index("latent_attn.row_lens", row_lens, 0, block_tables.shape[1] * cache.shape[2] + 1, "tokens per block table row")
        _ops._check_index("latent_attn.block_tables", block_tables, 0, cache.shape[0], "blocks of the cache pool")
        _ops._check_index("latent_attn.seq_of_row", seq_of_row, 0, block_tables.shape[0], "rows of the block table")
    assert q_cat.is_contiguous() and cache.is_contiguous() and cache.dtype == q_cat.dtype and block_tables.is_contiguous()
    dt, dev = _DT[q_cat.dtype], q_cat.device
    out = torch.empty(nh, R, rank, dtype=q_cat.dtype, device=dev)
    lib = _lib.kernels()
    bs = cache.shape[2]
    if q_cat.dtype != torch.float32 and kd % 8 == 0 and rank % 2 == 0 and rank <= 512 and kd <= 640 and R <= 65535:
        seen = min(int(max_len), window + 63) if window else int(max_len)
        chunks = max(1, (seen + 63) // 64)
        ctas = max(1, R * ((nh + 15) // 16))
        # up to 8 splits merge inside a thread-block cluster; long contexts of few rows take more, merged by a kernel
        splits = int(max(1, min(2 * 148 // ctas, chunks, 16 if chunks > 64 else 8)))
        ws_o = ws_ml = None
        if splits > 8:
            n_o = R * nh * splits * rank
            ws = scratch("mla_ws", (n_o + R * nh * splits * 2) * 4, dev).view(torch.float32)
            ws_o, ws_ml = ws[:n_o], ws[n_o:]
        rc = lib.fi_mla_decode(_p(q_cat), _p(cache), _p(out), out.stride(0), out.stride(1), _p(block_tables), _p(row_lens),
                               _p(seq_of_row), _p(ws_o), _p(ws_ml), R, nh, kd, rank, block_tables.shape[1], bs, splits,
                               int(window), _p(sinks), scale, dt, _stream())
        _lib.check(rc, "fi_mla_decode")
        _count(2 if splits > 8 else 1)
        return out
    rc = lib.fi_latent_rows(_p(q_cat), _p(cache), _p(out), out.stride(0), out.stride(1), _p(block_tables), _p(row_lens),
                            _p(seq_of_row), R, nh, kd, rank, block_tables.shape[1], bs, cache.shape[0] * bs, int(window),
                            _p(sinks), scale, dt, _stream())
    _lib.check(rc, "fi_latent_rows")
    _count()
    return out


class ContextPlan:
    """Which cached tokens the long portions of a step can see, laid out in blocks of a temporary pool: every sequence
    starts a new block; rows past its end have slot -1.  Built once per step and window size."""

    def __init__(self, block_tables, block_size: int, seq_lens, q_lens, window: int, device):
        n_blk, firsts, seq_of_blk, lens, table = 0, [], [], [], []
        for b, (n, q) in enumerate(zip(seq_lens, q_lens)):
            first = max(0, n - q - (window - 1)) if window else 0
            blocks = (n - first + POOL_BLOCK - 1) // POOL_BLOCK
            lens.append(n - first)
            table.append(range(n_blk, n_blk + blocks))
            seq_of_blk += [b] * blocks
            firsts += [first + i * POOL_BLOCK for i in range(blocks)]
            n_blk += blocks
        self.blocks, self.rows = n_blk, n_blk * POOL_BLOCK
        width = max(len(t) for t in table)
        B = len(lens)
        host = torch.zeros(2 * n_blk + B * (width + 2), dtype=torch.int32)
        host[:n_blk] = torch.tensor(seq_of_blk, dtype=torch.int32)
        host[n_blk:2 * n_blk] = torch.tensor(firsts, dtype=torch.int32)
        host[2 * n_blk:2 * n_blk + B] = torch.tensor(lens, dtype=torch.int32)
        host[2 * n_blk + B:2 * n_blk + 2 * B] = torch.tensor(list(seq_lens), dtype=torch.int32)
        host[2 * n_blk + 2 * B:] = torch.tensor([list(t) + [0] * (width - len(t)) for t in table], dtype=torch.int32).view(-1)
        d = host.to(device)
        self.lens = d[2 * n_blk:2 * n_blk + B]
        self.table = d[2 * n_blk + 2 * B:].view(B, width)
        seq = d[:n_blk].long()[:, None]
        pos = d[n_blk:2 * n_blk].long()[:, None] + torch.arange(POOL_BLOCK, device=device)
        end = d[2 * n_blk + B:2 * n_blk + 2 * B].long()[seq]
        inside = pos < end
        blk = block_tables.long()[seq, torch.where(inside, pos // block_size, torch.zeros_like(pos))]
        slots = torch.where(inside, blk * block_size + pos % block_size, torch.full_like(pos, -1))
        self.slots = slots.to(torch.int32).view(-1).contiguous()


def context_pool(plan: ContextPlan, cache, up_weight, nh: int, dim: int, rot: int, vdim: int, rank: int, hd: int):
    """Gathers the plan's latents, applies the stacked key | value up-projections [nh * (dim + vdim), rank] and returns
    the temporary K and V pools [blocks, nh, POOL_BLOCK, hd] (K = [key | rotary key | 0], V = [value | 0])."""
    n, dt, dev = plan.rows, cache.dtype, cache.device
    kd = rank + rot
    pitch = (rank + 7) // 8 * 8
    lib = _lib.kernels()
    c = torch.empty(n, pitch, dtype=dt, device=dev)
    num_rows = cache.shape[0] * cache.shape[2]
    rc = lib.fi_latent_gather(_p(cache), _p(plan.slots), _p(c), n, rank, kd, pitch, num_rows, _DT[dt], _stream())
    _lib.check(rc, "fi_latent_gather")
    kv = _ops.linear(c[:, :rank], up_weight)
    half = n * nh * hd * 2
    pools = scratch("latent_pool", 2 * half + 512, dev)
    k_pool = pools[:half].view(dt).view(plan.blocks, nh, POOL_BLOCK, hd)
    v_pool = pools[half:2 * half].view(dt).view(plan.blocks, nh, POOL_BLOCK, hd)
    rc = lib.fi_latent_pool(_p(cache), _p(plan.slots), _p(kv), kv.stride(0), _p(k_pool), _p(v_pool), n, nh, dim, rot, vdim,
                            rank, hd, num_rows, _DT[dt], _stream())
    _lib.check(rc, "fi_latent_pool")
    _count(2)
    return k_pool, v_pool
