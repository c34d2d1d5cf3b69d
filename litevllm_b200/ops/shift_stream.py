"""32-bit residual stream whose layers read a short causal convolution of the normalised stream, and mixers that blend the
present input with the previous token's.  With ``n = x / rms(x)``, per channel:

    h1_t = sum_j a1_j n_(t - taps + 1 + j),   h2_t = sum_j a2_j n_(t - taps + 1 + j)
    blend i:  h1_t + (h1_(t-1) - h1_t) mu_i

A layer ``h + conv(h)`` of ``h = n w`` has taps ``a_j = w (conv_j + [j = taps - 1])`` (:func:`fold_taps`), so both sublayers
share one ring of the last taps + 1 values of ``n`` per request slot (position p in row p mod (taps + 1)).

:func:`layer_inputs` advances the stream by what a layer returned (:class:`Summed`, :class:`Paired`) or starts it
(:class:`Embedded`) and returns what the next layer reads; :func:`normed` does the same at the end of the model.  Kernels:
csrc/misc/shift_stream.cu; CPU tensors run the PyTorch form.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _DT, _check_index, _count, _lib, _p, _stream
from .. import ops as _ops

BLENDS = 5


@dataclass
class ShiftSpec:
    """``a1`` (and ``a2``, for layers with a second sublayer) fp32 [taps, W], ``mu`` fp32 [5, W] or None."""
    a1: torch.Tensor
    a2: torch.Tensor | None = None
    mu: torch.Tensor | None = None

    @property
    def taps(self) -> int:
        return self.a1.shape[0]

    @property
    def outputs(self) -> int:
        return 1 + (self.a2 is not None) + (BLENDS if self.mu is not None else 0)


def fold_taps(norm, conv):
    """``norm`` [W], ``conv`` [W, taps] (last column: the present token) -> taps of h + conv(h), fp32 [taps, W]."""
    a = conv.float().t().clone()
    a[-1] += 1.0
    return (a * norm.float()).contiguous()


@dataclass
class Embedded:
    """norm(table[token] + pairs[row]) * weight, row = (previous * mul_prev + token * mul_cur) mod buckets of ``pairs``
    [buckets + 1, W], its last row for a sequence's first token.  ``last_token`` int32 [slots] remembers tokens."""
    ids: torch.Tensor
    table: torch.Tensor
    pairs: torch.Tensor
    mul_prev: int
    mul_cur: int
    weight: torch.Tensor
    last_token: torch.Tensor


@dataclass
class Summed:
    """x + y + f (+ the weighted rows of chosen experts)."""
    y: torch.Tensor
    f: torch.Tensor | None = None
    routed: object = None


@dataclass
class Paired:
    """x + norm(y) * w + norm(y2) * w2 + f (+ the weighted rows of chosen experts)."""
    y: torch.Tensor
    w: torch.Tensor
    y2: torch.Tensor
    w2: torch.Tensor
    f: torch.Tensor | None = None
    routed: object = None


def tiles(batch, taps: int, width: int):
    """(running count of tiles per portion int32 [B + 1], their number, tokens per tile) of the convolution kernels on rows of
    ``width`` channels: long tiles where they still fill the device."""
    T, blocks = sum(batch.q_lens_cpu), -(-width // 512)
    t = next((n for n in (64, 32, 16) if T // n * blocks >= 888), 8 if taps <= 8 else 16)
    key = f"tiles{t}"
    if key not in batch.extras:
        n = (batch.cu_q[1:] - batch.cu_q[:-1] + t - 1) // t
        batch.extras[key] = (F.pad(torch.cumsum(n, 0), (1, 0)).to(torch.int32), sum(-(-m // t) for m in batch.q_lens_cpu), t)
    return batch.extras[key]


def sequences(batch):
    """CPU path: (slot, first row, end row, position of the first row) of the step's live sequences."""
    slots, lens = batch.extras["slot_ids"].tolist(), batch.seq_lens.tolist()
    if batch.is_decode:
        return [(s, i, i + 1, n - 1) for i, (s, n) in enumerate(zip(slots, lens)) if n > 0 and s >= 0]
    cu = batch.cu_q.tolist()
    return [(s, cu[i], cu[i + 1], lens[i] - (cu[i + 1] - cu[i])) for i, s in enumerate(slots) if cu[i + 1] > cu[i]]


def ring_before(ring, pos0: int, n: int):
    """The last ``n`` rows before position ``pos0`` (zeros before the start) of a slot's ring [rows, C]."""
    rows = [ring[p % ring.shape[0]] if p >= 0 else torch.zeros_like(ring[0]) for p in range(pos0 - n, pos0)]
    return torch.stack(rows) if rows else ring[:0]


def ring_store(ring, pos0: int, x) -> None:
    for i in range(max(0, x.shape[0] - ring.shape[0]), x.shape[0]):
        ring[(pos0 + i) % ring.shape[0]].copy_(x[i])


def _rms(x, eps: float):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def _advance(src, x, batch, eps: float):
    """CPU form: the stream's new value (fp32 [T, W])."""
    if isinstance(src, Embedded):
        rows = torch.full_like(src.ids, src.pairs.shape[0] - 1)
        for slot, lo, hi, pos0 in sequences(batch):
            prev = src.ids[lo:hi].clone()
            prev[1:], prev[0] = src.ids[lo:hi - 1], int(src.last_token[slot])
            r = (prev * src.mul_prev + src.ids[lo:hi] * src.mul_cur) % (src.pairs.shape[0] - 1)
            rows[lo:hi] = r
            if pos0 == 0:
                rows[lo] = src.pairs.shape[0] - 1
            src.last_token[slot] = int(src.ids[hi - 1])
        return _rms(src.table[src.ids].float() + src.pairs[rows].float(), eps) * src.weight
    if isinstance(src, Paired):
        v = x + _rms(src.y.float(), eps) * src.w + _rms(src.y2.float(), eps) * src.w2
    else:
        v = x + src.y.float()
    if src.f is not None:
        v = v + src.f.float()
    return v if src.routed is None else v + src.routed.combined()


def _source_args(src, x, x_out, h_dtype):
    """Leading arguments of ``fi_shift_rows`` from ``ids`` to ``x_out``."""
    if isinstance(src, Embedded):
        assert src.ids.dtype == torch.int64 and src.table.is_contiguous() and src.pairs.is_contiguous()
        assert src.table.dtype == src.pairs.dtype == h_dtype and src.last_token.dtype == torch.int32
        if _ops._BOUNDS_CHECK:
            _check_index("shift_stream.ids", src.ids, 0, src.table.shape[0], "rows of the embedding table")
        return (_p(src.ids), _p(src.table), src.table.shape[0], _p(src.pairs), src.pairs.shape[0] - 1, src.mul_prev, src.mul_cur,
                _p(src.last_token), None, None, 0, None, 0, _p(src.weight), None, None, 0, None, 0, None, None, 0.0, 0, _p(x_out))
    pair, r, f = isinstance(src, Paired), src.routed, src.f
    assert x.is_contiguous() and x.dtype == torch.float32 and src.y.stride(1) == 1 and src.y.dtype == h_dtype
    assert f is None or (f.stride(1) == 1 and f.dtype == h_dtype)
    assert not pair or (src.y2.stride(1) == 1 and src.y2.dtype == h_dtype)
    if r is not None:
        assert r.rows.dtype == h_dtype and r.rows.stride(1) == 1 and not r.pass_through
    w = r.weights if r is not None else 0.0
    one = not isinstance(w, torch.Tensor)               # a weight for all choices
    assert one or w.is_contiguous()
    return (None, None, 0, None, 0, 0, 0, None, _p(x), _p(src.y), src.y.stride(0), _p(src.y2) if pair else None,
            src.y2.stride(0) if pair else 0, _p(src.w) if pair else None, _p(src.w2) if pair else None, _p(f),
            f.stride(0) if f is not None else 0, _p(r.rows) if r else None, r.rows.stride(0) if r else 0,
            _p(r.slot_of) if r else None, None if one else _p(w), float(w) if one else 0.0,
            (r.slot_of if one else w).shape[1] if r else 0, _p(x_out))


def _mode(src) -> int:
    return 0 if isinstance(src, Embedded) else 2 if isinstance(src, Paired) else 1


def layer_inputs(src, x, spec: ShiftSpec, ring, batch, eps: float, h_dtype):
    """Advances the stream ``x`` (fp32 [T, W], in place) and returns [outputs, T, W] in ``h_dtype``: h1 (, h2) (, blends).
    ``ring`` fp32 [slots, taps + 1, W] of the next layer, updated in place."""
    T, W = x.shape
    if not x.is_cuda:
        x.copy_(_advance(src, x, batch, eps))
        n, out = _rms(x, eps), torch.zeros(spec.outputs, T, W)
        taps = spec.taps
        for slot, lo, hi, pos0 in sequences(batch):
            seq = torch.cat([ring_before(ring[slot], pos0, taps), n[lo:hi]])
            win = seq.unfold(0, taps, 1)                                     # [hi - lo + 1, W, taps], first: the token before
            h = (win * spec.a1.t()).sum(-1)
            parts = [h[1:]] + ([(win[1:] * spec.a2.t()).sum(-1)] if spec.a2 is not None else [])
            if spec.mu is not None:
                parts += [h[1:] + (h[:-1] - h[1:]) * m for m in spec.mu]
            out[:, lo:hi] = torch.stack(parts)
            ring_store(ring[slot], pos0, n[lo:hi])
        return out.to(h_dtype)
    w8 = (W + 7) // 8 * 8
    buf = torch.empty(spec.outputs, T, w8, dtype=h_dtype, device=x.device)
    out = buf[:, :, :W]
    slots, B = batch.extras["slot_ids"], batch.seq_lens.shape[0]
    assert ring.is_contiguous() and ring.dtype == torch.float32 and tuple(ring.shape[1:]) == (spec.taps + 1, W)
    lib, decode = _lib.kernels(), batch.is_decode
    inv = None if decode else torch.empty(T, dtype=torch.float32, device=x.device)
    rc = lib.fi_shift_rows(_mode(src), 2 if decode else 0, *_source_args(src, x, x, h_dtype), _p(inv), None, None, _p(spec.a1),
                           _p(spec.a2), _p(spec.mu), spec.taps, _p(ring), _p(buf), w8, T * w8, _p(slots), _p(batch.seq_lens),
                           _p(batch.cu_q), B, ring.shape[0], T, W, eps, _DT[h_dtype], _stream())
    _lib.check(rc, "fi_shift_rows")
    _count()
    if not decode:
        base, n_tiles, tile = tiles(batch, spec.taps, W)
        first = isinstance(src, Embedded)
        rc = lib.fi_shift_conv(_p(x), _p(inv), _p(spec.a1), _p(spec.a2), _p(spec.mu), spec.taps, _p(ring), _p(buf), w8, T * w8,
                               _p(src.ids) if first else None, _p(src.last_token) if first else None, _p(slots),
                               _p(batch.seq_lens), _p(batch.cu_q), _p(base), n_tiles, tile, B, ring.shape[0], W, _DT[h_dtype],
                               _stream())
        _lib.check(rc, "fi_shift_conv")
        _count()
    return out


def normed(src, x, w, batch, eps: float, h_dtype, sel=None, keep: bool = False):
    """The end of the model: norm(stream) * w of the rows ``sel`` (int64, None: all); ``keep``: ``x`` is advanced too."""
    T, W = x.shape
    if not x.is_cuda:
        v = _advance(src, x, batch, eps)
        if keep:
            x.copy_(v)
        return (_rms(v if sel is None else v.index_select(0, sel), eps) * w).to(h_dtype)
    rows = T if sel is None else sel.shape[0]
    if sel is not None and _ops._BOUNDS_CHECK:
        _check_index("shift_stream.sel", sel, 0, T, "token rows of the step")
    assert not (keep and sel is not None) and not isinstance(src, Embedded)
    w8 = (W + 7) // 8 * 8
    out = torch.empty(rows, w8, dtype=h_dtype, device=x.device)[:, :W]
    rc = _lib.kernels().fi_shift_rows(_mode(src), 1, *_source_args(src, x, x if keep else None, h_dtype), None, _p(w), _p(sel), None,
                                      None, None, 0, None, _p(out), w8, 0, None, None, None, 0, 0, rows, W, eps, _DT[h_dtype],
                                      _stream())
    _lib.check(rc, "fi_shift_rows")
    _count()
    return out
