"""32-bit residual stream with norms before and after each sublayer and a weighted average over depth, with one norm
that sublayers read side by side, or with norms on the sublayers' outputs only.

    start    X_0 = table[ids] * scale
    add      x = x + y + sum_k w_k e_k        (y: mixer, e: outputs of the chosen experts)
    step     x = x + norm(y) * w_post
    post     x = x + norm(y + sum_k w_k e_k) * w_post
    average  X_n = x + norm(y) * w_post;  x = sum_{j <= n} a_j X_j
    each returns h = norm(x) * w_pre, the input of the next sublayer (start, post: x itself without ``w_pre``)

The norm is an RMS norm over ``groups`` equal consecutive parts of the vector.  On a GPU each form is one kernel
(csrc/misc/residual_stream.cu); CPU tensors run the PyTorch form.
"""
from __future__ import annotations

import torch

from . import _DT, _check_index, _count, _lib, _p, _stream
from .. import ops as _ops


def grouped_rmsnorm(x, w, eps: float, groups: int, out_dtype=None):
    """PyTorch form (CPU path): fp32 arithmetic, weight fp32 [W]."""
    xf = x.float().view(*x.shape[:-1], groups, -1)
    y = xf / torch.sqrt(xf.pow(2).mean(-1, keepdim=True) + eps)
    return (y.reshape(x.shape) * w.float()).to(out_dtype or x.dtype)


def _padded_rows(rows: int, width: int, dtype, device):
    """[rows, width] whose rows start on multiples of 16 bytes (what the TMA operand loads ask for)."""
    w8 = (width + 7) // 8 * 8
    buf = torch.empty(rows, w8, dtype=dtype, device=device)
    return buf[:, :width] if w8 != width else buf


def start(ids, table, w_pre, eps: float, groups: int, x0, scale: float = 1.0):
    """``x0`` (fp32 [T, W]) receives the embedding output; returns h in the table's dtype."""
    T, W = x0.shape
    if not table.is_cuda:
        x0.copy_(table.index_select(0, ids.long()).float() * scale)
        return x0.to(table.dtype) if w_pre is None else grouped_rmsnorm(x0, w_pre, eps, groups, table.dtype)
    if _ops._BOUNDS_CHECK:
        _check_index("residual_stream.start.ids", ids, 0, table.shape[0], "rows of the embedding table")
    assert ids.dtype == torch.int64 and x0.dtype == torch.float32 and x0.is_contiguous() and table.is_contiguous()
    same = w_pre is None and table.dtype == torch.float32
    h = None if same else _padded_rows(T, W, table.dtype, table.device)
    rc = _lib.kernels().fi_stream_start(_p(ids), _p(table), table.shape[0], float(scale), _p(w_pre), _p(x0), _p(h),
                                        W if same else h.stride(0), T, W, groups, eps, _DT[table.dtype], _stream())
    _lib.check(rc, "fi_stream_start")
    _count()
    return x0 if same else h


def step(y, x, w_post, w_pre, eps: float, groups: int, x_out, h_dtype):
    """``x_out = x + norm(y) * w_post`` (may alias ``x``); returns ``norm(x_out) * w_pre`` (None without ``w_pre``)."""
    T, W = x.shape
    if not x.is_cuda:
        x_out.copy_(x + grouped_rmsnorm(y, w_post, eps, groups, torch.float32))
        return None if w_pre is None else grouped_rmsnorm(x_out, w_pre, eps, groups, h_dtype)
    assert x.is_contiguous() and x_out.is_contiguous() and x.dtype == x_out.dtype == torch.float32 and y.stride(1) == 1
    h = None if w_pre is None else _padded_rows(T, W, h_dtype, x.device)
    rc = _lib.kernels().fi_stream_step(_p(y), y.stride(0), _DT[y.dtype], _p(x), _p(w_post), _p(w_pre), _p(x_out), _p(h),
                                       h.stride(0) if h is not None else W, _DT[h_dtype], T, W, groups, eps, _stream())
    _lib.check(rc, "fi_stream_step")
    _count()
    return h


def post(y, x, routed, w_post, w_pre, eps: float, groups: int, x_out, h_dtype, sel=None):
    """``x_out = x + norm(y + routed) * w_post`` (``x_out`` may alias ``x``); returns ``norm(x_out) * w_pre``, without
    ``w_pre`` ``x_out`` itself in ``h_dtype``.  ``y`` or ``routed`` (:class:`ops.moe.RoutedRows`) may be None.  ``sel``
    (int64 token rows): only these rows are wanted; h has one row per entry and ``x_out`` is not written."""
    T, W = x.shape
    if not x.is_cuda:
        s = torch.zeros_like(x) if y is None else y.float()
        if routed is not None:
            s = s + routed.combined(x)
        v = x + grouped_rmsnorm(s, w_post, eps, groups, torch.float32)
        if sel is not None:
            v = v.index_select(0, sel)
        elif x_out is not None:
            x_out.copy_(v)
        return v.to(h_dtype) if w_pre is None else grouped_rmsnorm(v, w_pre, eps, groups, h_dtype)
    assert x.is_contiguous() and x.dtype == torch.float32 and (y is None or y.stride(1) == 1)
    rows = T if sel is None else sel.shape[0]
    if sel is not None:
        x_out = None
        assert sel.dtype == torch.int64
        if _ops._BOUNDS_CHECK:
            _check_index("residual_stream.post.sel", sel, 0, T, "token rows of the step")
    same = w_pre is None and x_out is not None and h_dtype == torch.float32
    h = None if same else _padded_rows(rows, W, h_dtype, x.device)
    r = routed
    if r is not None:
        assert r.rows.dtype == h_dtype and r.rows.stride(1) == 1 and r.weights.is_contiguous()
    rc = _lib.kernels().fi_stream_post(
        _p(y), y.stride(0) if y is not None else 0, _DT[h_dtype if y is None else y.dtype], _p(x), _p(r.rows) if r else None,
        r.rows.stride(0) if r else 0, _p(r.slot_of) if r else None, _p(r.weights) if r else None,
        r.weights.shape[1] if r else 0, 1 if r is not None and r.pass_through else 0, _p(w_post), _p(w_pre), _p(x_out), _p(h),
        W if same else h.stride(0), _DT[h_dtype], _p(sel), rows, W, groups, eps, _stream())
    _lib.check(rc, "fi_stream_post")
    _count()
    return x_out if same else h


def average(y, x, w_post, w_pre, eps: float, groups: int, hist, n: int, avg, x_out, h_dtype, sel=None):
    """``hist`` fp32 [>= n + 1, T, W] holds X_0 .. X_(n-1) and receives X_n; ``avg`` fp32 [n + 1]; ``x_out`` (fp32
    [T, W] or None) the average.  ``sel`` (int64 token rows): only these rows are wanted; h has one row per entry and
    neither X_n nor ``x_out`` is written."""
    T, W = x.shape
    if not x.is_cuda:
        xn = x + grouped_rmsnorm(y, w_post, eps, groups, torch.float32)
        hist[n].copy_(xn)
        v = torch.einsum("j,jtw->tw", avg, hist[:n + 1])
        if sel is not None:
            v = v.index_select(0, sel)
        elif x_out is not None:
            x_out.copy_(v)
        return None if w_pre is None else grouped_rmsnorm(v, w_pre, eps, groups, h_dtype)
    assert hist.is_contiguous() and hist.dtype == torch.float32 and avg.dtype == torch.float32 and y.stride(1) == 1
    rows = T if sel is None else sel.shape[0]
    if sel is not None:
        x_out = None
        assert sel.dtype == torch.int64
        if _ops._BOUNDS_CHECK:
            _check_index("residual_stream.average.sel", sel, 0, T, "token rows of the step")
    h = None if w_pre is None else _padded_rows(rows, W, h_dtype, x.device)
    rc = _lib.kernels().fi_stream_average(_p(y), y.stride(0), _DT[y.dtype], _p(x), _p(w_post), _p(w_pre), _p(hist),
                                          hist.stride(0), _p(avg), n, _p(x_out), _p(h),
                                          h.stride(0) if h is not None else W, _DT[h_dtype], _p(sel), rows, W, groups,
                                          eps, _stream())
    _lib.check(rc, "fi_stream_average")
    _count()
    return h


def add(y, x, routed, w_pre, eps: float, groups: int, x_out, h_dtype, sel=None):
    """``x_out = x + y + routed`` (``x_out`` may alias ``x``); returns ``norm(x_out) * w_pre`` (None without ``w_pre``).
    ``routed`` (:class:`ops.moe.RoutedRows` or None): weighted sum of expert outputs.  ``sel`` (int64 token rows): only
    these rows are wanted; h has one row per entry and ``x_out`` is not written."""
    T, W = x.shape
    if not x.is_cuda:
        v = x + y.float()
        if routed is not None:
            v = v + routed.combined()
        if sel is not None:
            v = v.index_select(0, sel)
        elif x_out is not None:
            x_out.copy_(v)
        return None if w_pre is None else grouped_rmsnorm(v, w_pre, eps, groups, h_dtype)
    assert x.is_contiguous() and x.dtype == torch.float32 and y.stride(1) == 1
    rows = T if sel is None else sel.shape[0]
    if sel is not None:
        x_out = None
        assert sel.dtype == torch.int64
        if _ops._BOUNDS_CHECK:
            _check_index("residual_stream.add.sel", sel, 0, T, "token rows of the step")
    h = None if w_pre is None else _padded_rows(rows, W, h_dtype, x.device)
    r = routed
    if r is not None:
        assert r.rows.dtype == y.dtype and r.rows.stride(1) == 1 and r.weights.is_contiguous()
    rc = _lib.kernels().fi_stream_add(
        _p(y), y.stride(0), _DT[y.dtype], _p(x), _p(r.rows) if r else None, r.rows.stride(0) if r else 0,
        _p(r.slot_of) if r else None, _p(r.weights) if r else None, r.weights.shape[1] if r else 0, _p(w_pre), _p(x_out),
        _p(h), h.stride(0) if h is not None else W, _DT[h_dtype], _p(sel), rows, W, groups, eps, _stream())
    _lib.check(rc, "fi_stream_add")
    _count()
    return h
