"""Grouped-head attention over paged keys and values with norms on queries and keys, a constant in the softmax
denominator, an output gate, or two maps per head.

``prepare`` (one norm over the whole projection, values taken from the keys before norm and rotation) and
``prepare_heads`` (a norm per head, with or without a weight; two rotation layouts; a factor per position; two maps) turn
the merged projection of a step into cache rows and queries; ``attend_rows`` is the general form over flattened query rows
(32-bit models, head sizes outside the tensor-core kernels).  Kernels: csrc/attn/qk_prepare.cu, csrc/attn/head_prepare.cu,
csrc/attn/latent_rows.cu; the tensor-core forms are ``ops.paged_attention_decode`` and ``ops.paged_attention_prefill``.
CPU tensors run PyTorch forms.
"""
from __future__ import annotations

from dataclasses import dataclass

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


def prepare(proj, wq, wk, eps: float, positions, cos_sin, slot_mapping, k_cache, v_cache, H: int, G: int, dim: int,
            vdim: int = 0, v_cos_sin=None):
    """proj [T, >= (H + G) * dim] (q | k); caches [blocks, G, block size, hd] with hd >= dim (the rest is cleared); slots
    < 0 write no cache row.  ``vdim`` > 0: values have a projection of their own, proj [.. | v (G * vdim)], whose channels
    2 i and 2 i + 1 turn by angle i of ``v_cos_sin`` [positions, vdim] (None: as they are); otherwise the value is the key
    before norm and rotation.  Returns queries [T, H, hd] in the type of ``proj``."""
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
        v = raw.view(T, G, dim)
        if vdim:
            v = proj[:, (H + G) * dim:(H + G) * dim + G * vdim].float().reshape(T, G, vdim)
            if v_cos_sin is not None:
                vcs = v_cos_sin[positions.long()][:, None]
                v = _turn(v, vcs[..., :vdim // 2], vcs[..., vdim // 2:], vdim, True)
        at = torch.nonzero(slot_mapping >= 0).view(-1)
        slot = slot_mapping[at].long()
        for cache, rows in ((k_cache, k), (v_cache, v)):
            full = torch.zeros(at.shape[0], G, cache.shape[3], dtype=cache.dtype)
            full[..., :rows.shape[-1]] = rows[at].to(cache.dtype)
            cache[slot // bs, :, slot % bs] = full
        return q_out
    if _ops._BOUNDS_CHECK:
        _ops._check_index("qk_attn.prepare.slot_mapping", slot_mapping, -(1 << 31), k_cache.shape[0] * bs,
                          "flat slots of the cache pool; negative = skip")
        _ops._check_index("qk_attn.prepare.positions", positions, 0, cos_sin.shape[0], "rows of the cos/sin table")
    assert proj.stride(1) == 1 and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert k_cache.dtype == v_cache.dtype == proj.dtype and positions.dtype == slot_mapping.dtype == torch.int32
    assert v_cos_sin is None or v_cos_sin.shape == (cos_sin.shape[0], vdim)
    rc = _lib.kernels().fi_qk_prepare(_p(proj), proj.stride(0), _p(wq), _p(wk), eps, _p(positions), _p(cos_sin),
                                      cos_sin.shape[0], _p(slot_mapping), _p(q_out), _p(k_cache), _p(v_cache), T, H, G, dim,
                                      hd, cos_sin.shape[1], bs, (H + G) * dim if vdim else 0, vdim, v_cache.shape[3],
                                      _p(v_cos_sin), _DT[proj.dtype], _stream())
    _lib.check(rc, "fi_qk_prepare")
    _count()
    return q_out


@dataclass(frozen=True)
class HeadSpec:
    """What :func:`prepare_heads` does to a head: sizes, columns of the projection (q from 0), the RMS norm's constant and
    order, the rotation's layout (neighbours 2 i and 2 i + 1, or halves), pitches of the rows it writes."""
    H: int
    G: int
    dim: int
    vdim: int
    maps: int                      # queries (and keys) per head, each of ``dim`` channels
    eps: float
    q_pitch: int                   # channels of a query row; map m's channels start at m * q_shift
    q_shift: int = 0
    rope_dims: int = 0             # channels that turn (0: none)
    neighbours: bool = False
    weight_last: bool = False      # the norm's weight multiplies what is already rotated

    @property
    def k_off(self) -> int:
        return self.H * self.maps * self.dim

    @property
    def v_off(self) -> int:
        return (self.H + self.G) * self.maps * self.dim


def _turn(x, cos, sin, dims: int, neighbours: bool):
    """x [T, n, dim] fp32, cos / sin [T, 1, dims / 2]."""
    if not neighbours:
        return _rotate_halves(x, cos, sin)
    out = x.clone()
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out[..., 0:dims:2] = u * cos - v * sin
    out[..., 1:dims:2] = v * cos + u * sin
    return out


def prepare_heads(proj, wq, wk, spec: HeadSpec, positions, cos_sin, factor, slot_mapping, k_cache, v_cache):
    """proj [T, >= v_off + G * vdim] (q | k | v); ``wq``, ``wk`` fp32 [dim] or None; ``cos_sin`` fp32 [positions, rope_dims]
    or None; ``factor`` fp32 [positions] (multiplies queries) or None; caches [blocks, G, block size, pitch] whose rows are
    padded with zeros; slots < 0 write no cache row.  Returns queries [T, H * maps, q_pitch] in the type of ``proj``."""
    s, T, bs, kp, vp = spec, proj.shape[0], k_cache.shape[2], k_cache.shape[3], v_cache.shape[3]
    q_out = torch.empty(T, s.H * s.maps, s.q_pitch, dtype=proj.dtype, device=proj.device)
    max_pos = (cos_sin if cos_sin is not None else factor if factor is not None else k_cache).shape[0]
    if not proj.is_cuda:
        def heads(lo, n, w):
            x = proj[:, lo:lo + n * s.dim].float().view(T, n, s.dim)
            inv = torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + s.eps)
            w = 1.0 if w is None else w
            if cos_sin is None:
                return x * inv * w
            half, cs = s.rope_dims // 2, cos_sin[positions.long()][:, None]
            if s.weight_last:
                return _turn(x * inv, cs[..., :half], cs[..., half:], s.rope_dims, s.neighbours) * w
            return _turn(x * inv * w, cs[..., :half], cs[..., half:], s.rope_dims, s.neighbours)
        q = heads(0, s.H * s.maps, wq)
        if factor is not None:
            q = q * factor[positions.long()][:, None, None]
        q_out.zero_()
        for m in range(s.maps):
            q_out[:, m::s.maps, m * s.q_shift:m * s.q_shift + s.dim] = q[:, m::s.maps].to(proj.dtype)
        k = heads(s.k_off, s.G * s.maps, wk).reshape(T, s.G, s.maps * s.dim)
        v = proj[:, s.v_off:s.v_off + s.G * s.vdim].float().view(T, s.G, s.vdim)
        at = torch.nonzero(slot_mapping >= 0).view(-1)
        slot = slot_mapping[at].long()
        for cache, rows in ((k_cache, k), (v_cache, v)):
            full = torch.zeros(at.shape[0], s.G, cache.shape[3], dtype=cache.dtype)
            full[..., :rows.shape[-1]] = rows[at].to(cache.dtype)
            cache[slot // bs, :, slot % bs] = full
        return q_out
    if _ops._BOUNDS_CHECK:
        _ops._check_index("qk_attn.prepare_heads.slot_mapping", slot_mapping, -(1 << 31), k_cache.shape[0] * bs,
                          "flat slots of the cache pool; negative = skip")
        if cos_sin is not None or factor is not None:
            _ops._check_index("qk_attn.prepare_heads.positions", positions, 0, max_pos, "rows of the position tables")
    assert proj.stride(1) == 1 and k_cache.is_contiguous() and v_cache.is_contiguous()
    assert k_cache.dtype == v_cache.dtype == proj.dtype and positions.dtype == slot_mapping.dtype == torch.int32
    assert cos_sin is None or factor is None or cos_sin.shape[0] == factor.shape[0]
    rc = _lib.kernels().fi_head_prepare(
        _p(proj), proj.stride(0), s.k_off, s.v_off, _p(wq), _p(wk), s.eps, _p(positions), _p(cos_sin), s.rope_dims,
        int(s.neighbours), int(s.weight_last), _p(factor), max_pos, _p(slot_mapping), _p(q_out), s.q_shift, s.q_pitch,
        _p(k_cache), kp, _p(v_cache), vp, T, s.H, s.G, s.maps, s.dim, s.vdim, bs, _DT[proj.dtype], _stream())
    _lib.check(rc, "fi_head_prepare")
    _count()
    return q_out


def attend_rows(q, k_cache, v_cache, block_tables, row_lens, seq_of_row, scale: float, window: int, sinks, gate, dim: int,
                diff=None, sigmoid=None):
    """q [R, H, hd]; row r sees the first ``row_lens[r]`` tokens (the last ``window`` of them) of sequence
    ``seq_of_row[r]`` (None: sequence r).  Returns [R, H * dim], gated by ``sigmoid(gate)`` (a value per channel or per
    head).  ``diff = (lambda, scale, eps)``: query heads 2 j and 2 j + 1 meet the two halves of the key rows and are the
    maps of output head j, ``rms(a1 - lambda a2) * scale``; returns [R, H / 2 * dim].  ``sigmoid``
    (:class:`ops.SigmoidWeights`): no softmax."""
    R, H, hd = q.shape
    G, bs = k_cache.shape[1], k_cache.shape[2]
    if not q.is_cuda:
        if diff is not None:
            split = k_cache.shape[3] == 2 * hd           # else query rows are [q1 | 0] and [0 | q2]
            one, two = (attend_rows(q[:, m::2].float(), k_cache[..., m * hd:(m + 1) * hd] if split else k_cache, v_cache,
                                    block_tables, row_lens, seq_of_row, scale, window, None if sinks is None else sinks[m::2],
                                    None, dim) for m in range(2))
            o = (one - diff[0] * two).view(R, H // 2, dim)
            o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + diff[2]) * diff[1]
            return o.reshape(R, -1).to(q.dtype)
        out = torch.zeros(R, H, dim, dtype=q.dtype)
        for r in range(R):
            n = int(row_lens[r])
            if n <= 0:
                continue
            b = r if seq_of_row is None else int(seq_of_row[r])
            first = max(0, n - window) if window else 0
            if sigmoid is not None and sigmoid.chunk:
                first = (n - 1) // sigmoid.chunk * sigmoid.chunk
            pos = torch.arange(first, n)
            blk = block_tables[b].long()[pos // bs]
            k = k_cache[blk, :, pos % bs].float().repeat_interleave(H // G, 1)              # [n, H, hd]
            v = v_cache[blk, :, pos % bs].float().repeat_interleave(H // G, 1)
            s = torch.einsum("hd,nhd->hn", q[r].float(), k) * scale
            if sigmoid is not None:
                o = torch.einsum("hn,nhd->hd", torch.sigmoid(s + sigmoid.bias[:, None]), v)[:, :dim]
                if sigmoid.turn is not None:
                    cs = sigmoid.turn[n - 1]
                    o = _turn(o[None], cs[:dim // 2], -cs[dim // 2:], dim, True)[0]
                out[r] = o.to(out.dtype)
                continue
            if sinks is not None:
                s = torch.cat([s, sinks[:, None]], dim=1)
            a = torch.softmax(s, dim=-1)[:, :k.shape[0]]
            out[r] = torch.einsum("hn,nhd->hd", a, v)[:, :dim].to(out.dtype)
        if gate is not None:
            gate = gate.float().view(R, H, -1) if gate.shape[1] == H else gate.float().reshape(R, H, dim)
            out = (out.float() * torch.sigmoid(gate)).to(out.dtype)
        return out.reshape(R, H * dim)
    maps = 1 if diff is None else 2
    if k_cache.shape[3] != hd * maps or v_cache.shape[3] != dim:
        raise ValueError("the general row kernel reads caches without padded channels")
    if _ops._BOUNDS_CHECK:
        _ops._check_index("qk_attn.row_lens", row_lens, 0, block_tables.shape[1] * bs + 1, "tokens per block table row")
        _ops._check_index("qk_attn.block_tables", block_tables, 0, k_cache.shape[0], "blocks of the cache pool")
    assert q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous() and block_tables.is_contiguous()
    out = torch.empty(R, H // maps * dim, dtype=q.dtype, device=q.device)
    rc = _lib.kernels().fi_attn_rows(_p(q), _p(k_cache), _p(v_cache), _p(out), _p(block_tables), _p(row_lens), _p(seq_of_row),
                                     R, H, G, hd * maps, dim, block_tables.shape[1], bs, k_cache.shape[0], int(window),
                                     _ops.attn_extra(H, dim, sinks, gate, diff, sigmoid), scale, _DT[q.dtype], _stream())
    _lib.check(rc, "fi_attn_rows")
    _count()
    return out
