"""Mixture-of-experts ops: routing and the fused expert MLP.

CUDA path (csrc/moe/moe_kernels.cu + the grouped mode of csrc/gemm/awq_gemm.cu):
  route -> align (counting sort by expert + tile table, on the device, no host sync) -> gather ->
  grouped int4 gate|up GEMM with the activation in the epilogue -> grouped int4 down GEMM ->
  weighted combine.  Only the experts in ``[e_lo, e_hi)`` (this rank's shard) are computed; with
  expert parallelism the per-rank partial outputs are summed by the caller.
CPU path: a plain per-expert loop in fp32 (the oracle).
Reference: vllm/model_executor/layers/fused_moe/fused_moe.py:4-77 (softmax/topk/sort + Python loop)
and vllm/model_executor/models/gemma4/moe.py:465-623 (execution ladder).
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _ACT, _DT, _count, _lib, _p, _stream, reference, scratch, status_word
from .awq import Int4Weight

ROUTER_MODES = {"softmax": 0, "sigmoid": 1, "sqrt_softplus": 2}


class FiGrouped(ctypes.Structure):
    _fields_ = [("tile_expert", ctypes.c_void_p), ("tile_row0", ctypes.c_void_p), ("tile_rows", ctypes.c_void_p),
                ("n_tiles", ctypes.c_void_p), ("max_tiles", ctypes.c_int), ("num_experts", ctypes.c_int),
                ("expert_rows", ctypes.c_int), ("reserved", ctypes.c_int)]


def route(logits: torch.Tensor, top_k: int, mode: str = "softmax", bias: torch.Tensor | None = None,
          expert_scale: torch.Tensor | None = None, renormalize: bool = True, routed_scale: float = 1.0,
          groups: int = 1, keep_groups: int = 1, group_best: int = 2):
    """logits [T, E] float32 (any row pitch) -> (ids int32 [T, k], weights float32 [T, k]).  Selection is by score +
    ``bias``, weights come from the scores.  With ``keep_groups < groups`` the experts form ``groups`` equal groups of
    neighbours, and only the ``keep_groups`` with the largest sums of their ``group_best`` (1 or 2) best selection scores
    can be chosen."""
    T, E = logits.shape
    if not logits.is_cuda:
        lf = logits.float()
        if mode == "softmax":
            score = torch.softmax(lf, dim=-1)
        else:
            score = torch.sigmoid(lf) if mode == "sigmoid" else torch.sqrt(torch.nn.functional.softplus(lf))
        sel = score + (bias.float() if bias is not None else 0.0)
        if keep_groups < groups:
            per = sel.view(T, groups, -1)
            gs = torch.topk(per, min(group_best, per.shape[-1]), dim=-1).values.sum(-1)
            drop = torch.ones_like(gs, dtype=torch.bool).scatter_(1, torch.topk(gs, keep_groups, dim=-1).indices, False)
            sel = per.masked_fill(drop[..., None], float("-inf")).view(T, E)
        ids = torch.topk(sel, top_k, dim=-1).indices
        w = torch.gather(score, 1, ids)
        if renormalize:
            w = w / w.sum(-1, keepdim=True).clamp_min(1e-20)
        w = w * routed_scale
        if expert_scale is not None:
            w = w * expert_scale.float()[ids]
        return ids.to(torch.int32), w.float()
    ids = torch.empty(T, top_k, dtype=torch.int32, device=logits.device)
    w = torch.empty(T, top_k, dtype=torch.float32, device=logits.device)
    assert logits.dtype == torch.float32 and logits.stride(1) == 1
    rc = _lib.kernels().fi_moe_route(_p(logits), _p(bias), _p(expert_scale), logits.stride(0), _p(ids), _p(w), T, E, top_k,
                                     ROUTER_MODES[mode], 1 if renormalize else 0, float(routed_scale), groups, keep_groups,
                                     group_best, _stream())
    _lib.check(rc, "fi_moe_route")
    _count()
    return ids, w


@dataclass(frozen=True)
class Assigned:
    """Choices without a router: token t takes the experts ``table[token_ids[t]]`` (table int32 [vocab, K], ids int64 [T])."""
    table: torch.Tensor
    token_ids: torch.Tensor

    @property
    def shape(self) -> tuple[int, int]:
        return self.token_ids.shape[0], self.table.shape[1]

    def ids(self) -> torch.Tensor:
        return self.table.index_select(0, self.token_ids)


@dataclass
class RoutedRows:
    """Outputs of the chosen experts before their weighted sum: choice k of token t is row ``slot_of[t, k]`` of ``rows``
    (row t * K + k without a map), its weight ``weights[t, k]`` (a number: of every choice).  A choice whose slot is negative has no row: it adds nothing,
    or with ``pass_through`` the experts' input itself."""
    rows: torch.Tensor               # [T * K, H]
    weights: torch.Tensor | float    # fp32 [T, K]
    slot_of: torch.Tensor | None = None
    pass_through: bool = False

    def combined(self, x: torch.Tensor | None = None) -> torch.Tensor:
        """fp32 [T, H]; PyTorch form (the kernels fold the sum into the residual add).  ``x``: the experts' input."""
        w = self.weights if isinstance(self.weights, torch.Tensor) else torch.full(self.slot_of.shape, self.weights)
        T, K = w.shape
        if self.slot_of is None:
            return (self.rows.float().view(T, K, -1) * w[..., None]).sum(1)
        none = (self.slot_of < 0)[..., None]
        r = self.rows.index_select(0, self.slot_of.clamp(min=0).reshape(-1).long()).float().view(T, K, -1)
        r = torch.where(none, x.float()[:, None] if self.pass_through else torch.zeros_like(r), r)
        return (r * w[..., None]).sum(1)


_stack_tables: dict[tuple, torch.Tensor] = {}


def _stacked_tile_table(E: int, T: int, bn: int, device) -> tuple[torch.Tensor, int]:
    """(int32 table, number of tiles n): matrix [n], first row [n] and rows [n] of each tile of ``bn`` rows of E stacked matrices
    of T rows, then n itself.  The few tables of small steps are kept (captured steps hold their addresses), others are
    written by a kernel."""
    n = E * -(-T // bn)
    key = (E, T, bn, str(device))
    t = _stack_tables.get(key)
    if t is None:
        if T <= 64:
            with torch.inference_mode(False):
                t = _stack_tables[key] = torch.empty(3 * n + 1, dtype=torch.int32, device=device)
        else:
            t = scratch("stack_tiles", (3 * n + 1) * 4, device).view(torch.int32)[:3 * n + 1]
        at = t.data_ptr()
        rc = _lib.kernels().fi_stack_tiles(E, T, bn, at, at + 4 * n, at + 8 * n, at + 12 * n, _stream())
        _lib.check(rc, "fi_stack_tiles")
        _count()
    return t, n


def stacked_linear(x: torch.Tensor, w: torch.Tensor):
    """x [E, T, K] (rows of one pitch, matrices back to back), w [E, N, K] -> E matrices [T, N], by one grouped product."""
    from .. import ops
    E, T, K = x.shape
    N = w.shape[1]
    if not x.is_cuda or x.dtype == torch.float32 or K % 8 or N % 8 or x.stride(1) % 8 \
            or x.stride(0) != T * x.stride(1) or x.data_ptr() % 16 or not w.is_contiguous():
        return [ops.linear(x[e], w[e]) for e in range(E)]
    out = torch.empty(E, T, N, dtype=x.dtype, device=x.device)
    many = T >= ops._PERSISTENT_MIN_T
    bn = 128 if many else 16 if T <= 16 else 32 if T <= 32 else 64
    t, n = _stacked_tile_table(E, T, bn, x.device)
    at = t.data_ptr()
    g = FiGrouped(at, at + 4 * n, at + 8 * n, at + 12 * n, n, E, N, 0)
    if many:
        rc = _lib.kernels().fi_dense_gemm_persistent_grouped(_p(x), _p(w), _p(out), E * T, N, K, x.stride(1), N, 0, 0.0, 0, _DT[x.dtype],
                                                             ctypes.byref(g), _p(status_word(x.device)), _stream())
    else:
        rc = _lib.kernels().fi_dense_gemm_grouped(_p(x), _p(w), _p(out), E * T, N, K, x.stride(1), N, 0, 0.0, 0, _DT[x.dtype], bn,
                                                  ctypes.byref(g), _p(status_word(x.device)), _stream())
    _lib.check(rc, "stacked_linear")
    _count()
    return out


def _tile_table(ids, n: int, E: int, bn: int, dev, scratch_name: str):
    """Routes sorted by expert and the table of tiles of ``bn`` rows, built on the device.  Returns (sorted_route,
    slot_of, offsets, tile_expert, tile_row0, tile_rows, n_tiles, bound of n_tiles)."""
    bound = min(n, E + (n + bn - 1) // bn)
    ints = scratch(scratch_name, (2 * n + E + 1 + 3 * bound + 8) * 4, dev).view(torch.int32)
    out, o = [], 0
    for size in (n, n, E + 1, bound, bound, bound, 1):
        out.append(ints[o:o + size])
        o += size
    if isinstance(ids, Assigned):
        assert ids.table.dtype == torch.int32 and ids.table.is_contiguous() and ids.token_ids.dtype == torch.int64
        assert ids.token_ids.is_contiguous()
        rc = _lib.kernels().fi_moe_align_assigned(_p(ids.table), _p(ids.token_ids), *ids.table.shape, n, E, bn, *[_p(t) for t in out],
                                                  _stream())
    else:
        rc = _lib.kernels().fi_moe_align(_p(ids), n, 0, E, bn, *[_p(t) for t in out], _stream())
    _lib.check(rc, "fi_moe_align")
    _count()
    return (*out, bound)


def expert_rows(x: torch.Tensor, w_gate_up: torch.Tensor, w_down: torch.Tensor, ids: torch.Tensor | Assigned,
                weights: torch.Tensor | float, act: str = "silu", act_limit: float = 0.0, pass_through: bool = False) -> RoutedRows:
    """Unquantised experts: x [T, H], ``w_gate_up`` [E, 2 I, H] (gate | up), ``w_down`` [E, H, I], ids / weights of
    :func:`route` (or :class:`Assigned` choices of one weight); ids from E on have no row (``pass_through``: they stand for x itself).  ``act`` and ``act_limit`` as in
    :func:`ops.gated_linear`.  No host synchronisation.  16-bit weights whose rows are whole 16-byte groups run grouped tcgen05
    products (persistent tiles when an expert sees many rows), everything else the general 32-bit kernel."""
    T, H = x.shape
    E, two_i, _ = w_gate_up.shape
    inter, K = two_i // 2, ids.shape[1]
    if not x.is_cuda:
        rows = torch.zeros(T * K, H, dtype=x.dtype)
        flat = (ids.ids() if isinstance(ids, Assigned) else ids).reshape(-1).long()
        for e in flat[flat < E].unique().tolist():
            at = torch.nonzero(flat == e).view(-1)
            h = x[at // K].float() @ w_gate_up[e].float().t()
            a = reference.apply_gated(h[:, :inter], h[:, inter:], act, act_limit).to(x.dtype)
            rows[at] = (a.float() @ w_down[e].float().t()).to(x.dtype)
        slots = torch.where(flat < E, torch.arange(T * K), -1).view(T, K).to(torch.int32)
        return RoutedRows(rows, weights, slots, pass_through)
    n, dev, lib, st, dt = T * K, x.device, _lib.kernels(), _stream(), _DT[x.dtype]
    rows = torch.empty(n, (H + 7) // 8 * 8, dtype=x.dtype, device=dev)[:, :H]
    if n == 0:
        return RoutedRows(rows, weights, None, pass_through)
    mean = (n + E - 1) // E
    tensor = x.dtype != torch.float32 and H % 8 == 0 and inter % 8 == 0 and x.stride(0) % 8 == 0
    persistent = tensor and mean >= 64
    bn = 128 if persistent else 32 if not tensor else 16 if mean <= 8 else 32 if mean <= 24 else 64
    # the table lives in scratch: the sum over the choices is enqueued before the next layer's table
    order, slots, offsets, t_e, t_r0, t_n, n_tiles, bound = _tile_table(ids, n, E, bn, dev, "expert_tiles")
    slot_of = slots.view(T, K)
    acts = torch.empty(n, inter, dtype=x.dtype, device=dev)
    if not tensor:
        if act not in ("silu", "clipped_swiglu"):
            raise ValueError("the general expert kernel computes silu gates, plain or clipped")
        w1, w2 = w_gate_up.contiguous(), w_down.contiguous()
        rc = lib.fi_moe_expert_rows(_p(x), x.stride(0), _p(w1), _p(acts), inter, _p(order), _p(t_e), _p(t_r0), _p(t_n),
                                    _p(n_tiles), bound, inter, H, K, 1, _ACT[act], act_limit, dt, st)
        _lib.check(rc, "fi_moe_expert_rows(gate_up)")
        rc = lib.fi_moe_expert_rows(_p(acts), inter, _p(w2), _p(rows), rows.stride(0), None, _p(t_e), _p(t_r0), _p(t_n),
                                    _p(n_tiles), bound, H, inter, K, 0, 0, 0.0, dt, st)
        _lib.check(rc, "fi_moe_expert_rows(down)")
        _count(2)
        return RoutedRows(rows, weights, slot_of, pass_through)
    x_sorted = torch.empty(n, H, dtype=x.dtype, device=dev)
    xc = x if x.is_contiguous() else x.contiguous()
    rc = lib.fi_moe_gather(_p(xc), _p(order), _p(offsets), E, n, K, H, _p(x_sorted), dt, st)
    _lib.check(rc, "fi_moe_gather")
    g1 = FiGrouped(_p(t_e), _p(t_r0), _p(t_n), _p(n_tiles), bound, E, two_i, 0)
    g2 = FiGrouped(_p(t_e), _p(t_r0), _p(t_n), _p(n_tiles), bound, E, H, 0)
    sw = _p(status_word(dev))
    if persistent:
        rc = lib.fi_dense_gemm_persistent_grouped(_p(x_sorted), _p(w_gate_up), _p(acts), n, inter, H, H, inter, _ACT[act],
                                                  act_limit, inter, dt, ctypes.byref(g1), sw, st)
        _lib.check(rc, "fi_dense_gemm_persistent_grouped(gate_up)")
        rc = lib.fi_dense_gemm_persistent_grouped(_p(acts), _p(w_down), _p(rows), n, H, inter, inter, rows.stride(0), 0, 0.0, 0, dt,
                                                  ctypes.byref(g2), sw, st)
        _lib.check(rc, "fi_dense_gemm_persistent_grouped(down)")
    else:
        rc = lib.fi_dense_gemm_grouped(_p(x_sorted), _p(w_gate_up), _p(acts), n, inter, H, H, inter, _ACT[act], act_limit, inter, dt, bn,
                                       ctypes.byref(g1), sw, st)
        _lib.check(rc, "fi_dense_gemm_grouped(gate_up)")
        rc = lib.fi_dense_gemm_grouped(_p(acts), _p(w_down), _p(rows), n, H, inter, inter, rows.stride(0), 0, 0.0, 0, dt, bn,
                                       ctypes.byref(g2), sw, st)
        _lib.check(rc, "fi_dense_gemm_grouped(down)")
    _count(3)
    return RoutedRows(rows, weights, slot_of, pass_through)


def _reference_experts(x, w_gate_up: Int4Weight, w_down: Int4Weight, ids, weights, num_experts, e_lo, e_hi, act):
    T, H = x.shape
    inter = w_gate_up.N // (num_experts * 2)
    gu = w_gate_up.dense().view(num_experts, 2 * inter, -1)
    dn = w_down.dense().view(num_experts, H, inter)
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    xf = x.float()
    for e in range(e_lo, e_hi):
        tok, slot = torch.nonzero(ids == e, as_tuple=True)
        if tok.numel() == 0:
            continue
        h = xf[tok] @ gu[e - 0].t()
        a = reference.apply_act(h[:, :inter], act) * h[:, inter:]
        a = a.to(x.dtype).float()
        y = (a @ dn[e].t()).to(x.dtype).float()
        out.index_add_(0, tok, y * weights[tok, slot][:, None])
    return out.to(x.dtype)


def fused_experts(x: torch.Tensor, w_gate_up: Int4Weight, w_down: Int4Weight, ids: torch.Tensor,
                  weights: torch.Tensor, num_experts_local: int, e_lo: int, act: str = "gelu_tanh",
                  residual: torch.Tensor | None = None, ep_heap=None) -> torch.Tensor:
    """x [T, H]; stacked int4 experts (``w_gate_up``: [E_local * 2I, H], ``w_down``: [E_local * H, I]);
    ids/weights from :func:`route` (global expert ids).  Returns sum_k w * expert(x) [+ residual]
    over the local experts ``[e_lo, e_lo + num_experts_local)``.  With ``ep_heap`` (the symmetric
    heap of an expert-parallel group, GPU only) the result is also summed over the ranks."""
    T, H = x.shape
    K = ids.shape[1]
    e_hi = e_lo + num_experts_local
    inter = w_gate_up.N // (num_experts_local * 2)
    if not x.is_cuda:
        local = ids - e_lo
        out = _reference_experts(x, w_gate_up, w_down, local, weights, num_experts_local, 0, num_experts_local, act)
        return out if residual is None else (out.float() + residual.float()).to(x.dtype)
    if w_gate_up.qw is None or w_down.qw is None:
        raise RuntimeError("expert weights are not in the device runtime layout (were they loaded on the CPU?)")
    n = T * K
    bn = 16 if n // max(num_experts_local, 1) < 16 else 32 if n // num_experts_local < 48 else 64
    max_tiles = min(n, num_experts_local + (n + bn - 1) // bn)
    dev = x.device
    ints = scratch("moe_ints", (2 * n + num_experts_local + 1 + 3 * max_tiles + 8) * 4, dev).view(torch.int32)
    o = 0
    sorted_route = ints[o:o + n]; o += n
    slot_of = ints[o:o + n]; o += n
    offsets = ints[o:o + num_experts_local + 1]; o += num_experts_local + 1
    tile_expert = ints[o:o + max_tiles]; o += max_tiles
    tile_row0 = ints[o:o + max_tiles]; o += max_tiles
    tile_rows = ints[o:o + max_tiles]; o += max_tiles
    n_tiles = ints[o:o + 1]
    lib = _lib.kernels()
    st = _stream()
    rc = lib.fi_moe_align(_p(ids), n, e_lo, e_hi, bn, _p(sorted_route), _p(slot_of), _p(offsets), _p(tile_expert),
                          _p(tile_row0), _p(tile_rows), _p(n_tiles), st)
    _lib.check(rc, "fi_moe_align")
    esz = x.element_size()
    acts = scratch("moe_acts", n * (2 * H + inter) * esz + 1024, dev)
    x_sorted = acts[: n * H * esz].view(x.dtype).view(n, H)
    a_sorted = acts[n * H * esz: n * (H + inter) * esz].view(x.dtype).view(n, inter)
    y_sorted = acts[n * (H + inter) * esz: n * (2 * H + inter) * esz].view(x.dtype).view(n, H)
    rc = lib.fi_moe_gather(_p(x), _p(sorted_route), _p(offsets), num_experts_local, n, K, H, _p(x_sorted),
                           _DT[x.dtype], st)
    _lib.check(rc, "fi_moe_gather")
    g = FiGrouped(_p(tile_expert), _p(tile_row0), _p(tile_rows), _p(n_tiles), max_tiles, num_experts_local,
                  2 * inter, 0)
    sw = _p(status_word(dev))
    rc = lib.fi_awq_gemm_grouped(_p(x_sorted), _p(w_gate_up.qw), _p(w_gate_up.scales_t), _p(w_gate_up.zeros_t),
                                 _p(a_sorted), None, None, n, inter, H, w_gate_up.group, H, inter, _ACT[act], inter,
                                 0, _DT[x.dtype], 1, bn, sw, st, ctypes.byref(g))
    _lib.check(rc, "fi_awq_gemm_grouped(gate_up)")
    g2 = FiGrouped(_p(tile_expert), _p(tile_row0), _p(tile_rows), _p(n_tiles), max_tiles, num_experts_local, H, 0)
    rc = lib.fi_awq_gemm_grouped(_p(a_sorted), _p(w_down.qw), _p(w_down.scales_t), _p(w_down.zeros_t), _p(y_sorted),
                                 None, None, n, H, inter, w_down.group, inter, H, 0, 0, 0, _DT[x.dtype], 1, bn, sw,
                                 st, ctypes.byref(g2))
    _lib.check(rc, "fi_awq_gemm_grouped(down)")
    out = torch.empty(T, H, dtype=x.dtype, device=dev)
    if ep_heap is not None and ep_heap.fits_low_latency(T, H):
        # expert parallel: the combine also sums the ranks' partial outputs (one kernel, peer stores)
        comm = ep_heap.comm_desc(mode=1, T=T, N=H, xfer_16bit=2)
        rc = lib.fi_moe_combine_allreduce(_p(y_sorted), _p(slot_of), _p(weights), _p(residual), _p(out), T, K, H,
                                          _DT[x.dtype], sw, st, ctypes.byref(comm))
        _lib.check(rc, "fi_moe_combine_allreduce")
        _count(5)
        return out
    rc = lib.fi_moe_combine(_p(y_sorted), _p(slot_of), _p(weights), _p(residual), _p(out), T, K, H, _DT[x.dtype], st)
    _lib.check(rc, "fi_moe_combine")
    _count(5)
    if ep_heap is not None:       # too large for the low-latency slabs: library collective
        from ..parallel import state as pstate
        pstate.all_reduce(out)
    return out
