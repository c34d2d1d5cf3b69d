"""Gated delta rule (GatedDeltaNet linear attention of Qwen3.5 / Qwen3-Next).

Per value head, with state ``S [dk, dv]``, decay ``a_t = exp(g_t)`` and write strength ``beta_t``::

    S_t = a_t S_{t-1} + k_t (beta_t (v_t - a_t S_{t-1}^T k_t))^T        o_t = S_t^T q_t

* :func:`gated_delta_recurrent` - the rule as written, one token at a time (the oracle).
* :func:`gated_delta_chunked`   - the same result from chunks of 64 tokens: inside a chunk the
  token-to-token dependence is a unit lower-triangular system that is solved once
  (``(I + tril(K_beta K^T * decay, -1))^-1``), so a chunk costs a handful of matrix products and only
  the chunk-to-chunk state update is sequential.  Used for prefill.
* :func:`gated_delta_step` / :func:`conv1d_step` - one decode step for a batch of sequences on state
  pools indexed by slot (CUDA kernels in csrc/linear_attn/gated_delta.cu; PyTorch on the CPU).

* :func:`time_mix` and :func:`ssd` - linear attention with channel decays and a bonus for the current token, or with scalar
  decays, a skip and a short convolution in front (csrc/linear_attn/decay_scan.cu; PyTorch on the CPU).
* :func:`delta_portions` / :func:`delta_step` - the rule with one decay per key channel, its short convolutions, unit
  vectors, head norm and gate included (csrc/linear_attn/channel_delta.cu; PyTorch on the CPU).

Reference: vllm/model_executor/models/qwen3_5.py:127-200 (chunk-64 rule), :203-260 (recurrent rule).
"""
from __future__ import annotations

import torch
import torch.nn.functional as F

from . import _DT, _count, _lib, _p, _stream, scratch, status_word


def gated_delta_recurrent(q, k, v, g, beta, S0=None):
    """q, k: [L, H, dk]; v: [L, H, dv]; g, beta: [L, H]; S0: [H, dk, dv] or None.  fp32 in, fp32 out.
    Returns (o [L, H, dv], S [H, dk, dv])."""
    L, H, dk = q.shape
    dv = v.shape[-1]
    S = torch.zeros(H, dk, dv, dtype=torch.float32, device=q.device) if S0 is None else S0.float().clone()
    o = torch.empty(L, H, dv, dtype=torch.float32, device=q.device)
    for t in range(L):
        S = S * torch.exp(g[t])[:, None, None]
        mem = torch.einsum("hkv,hk->hv", S, k[t])
        delta = (v[t] - mem) * beta[t][:, None]
        S = S + k[t][:, :, None] * delta[:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o, S


def gated_delta_chunked(q, k, v, g, beta, S0=None, chunk: int = 64):
    """Same contract as :func:`gated_delta_recurrent`, computed chunk-wise."""
    L, H, dk = q.shape
    dv = v.shape[-1]
    dev = q.device
    pad = (-L) % chunk
    if pad:
        # padded tokens: beta = 0 (no write), g = 0 (no decay), q = k = 0: they change nothing
        zp = lambda t: F.pad(t, (0, 0) * (t.dim() - 1) + (0, pad))
        q, k, v, g, beta = zp(q), zp(k), zp(v), zp(g), zp(beta)
    N = (L + pad) // chunk
    # [H, N, C, d]
    qc = q.float().permute(1, 0, 2).reshape(H, N, chunk, dk)
    kc = k.float().permute(1, 0, 2).reshape(H, N, chunk, dk)
    vc = v.float().permute(1, 0, 2).reshape(H, N, chunk, dv)
    bc = beta.float().t().reshape(H, N, chunk)
    gc = g.float().t().reshape(H, N, chunk).cumsum(-1)                 # log decay from the chunk start (inclusive)
    v_beta = vc * bc[..., None]
    k_beta = kc * bc[..., None]
    diff = gc[..., :, None] - gc[..., None, :]                          # log decay from token j to token i
    lower = torch.tril(torch.ones(chunk, chunk, dtype=torch.bool, device=dev))
    decay = torch.where(lower, diff, torch.full_like(diff, float("-inf"))).exp()
    # token i's write sees the writes of tokens j < i of its chunk: (I + A) U = V_beta with strictly lower A
    A = torch.tril((k_beta @ kc.transpose(-1, -2)) * decay, diagonal=-1)
    eye = torch.eye(chunk, dtype=torch.float32, device=dev)
    T = torch.linalg.solve_triangular(eye + A, eye.expand_as(A).contiguous(), upper=False)
    u = T @ v_beta                                                       # writes if the incoming state were zero
    w = T @ (k_beta * gc.exp()[..., None])                               # what each write reads from the incoming state
    S = torch.zeros(H, dk, dv, dtype=torch.float32, device=dev) if S0 is None else S0.float().clone()
    o = torch.empty(H, N, chunk, dv, dtype=torch.float32, device=dev)
    strict = torch.tril(torch.ones(chunk, chunk, dtype=torch.bool, device=dev), diagonal=0)
    for i in range(N):
        qi, ki = qc[:, i], kc[:, i]
        attn = torch.where(strict, (qi @ ki.transpose(-1, -2)) * decay[:, i], torch.zeros((), device=dev))
        v_new = u[:, i] - w[:, i] @ S
        o[:, i] = (qi * gc[:, i].exp()[..., None]) @ S + attn @ v_new
        g_last = gc[:, i, -1]
        S = S * g_last.exp()[:, None, None] + (ki * (g_last[:, None] - gc[:, i]).exp()[..., None]).transpose(-1, -2) @ v_new
    o = o.reshape(H, N * chunk, dv).permute(1, 0, 2)[:L].contiguous()
    return o, S


def gated_delta_step(pool: torch.Tensor, slots: torch.Tensor, q, k, v, g, beta, out=None):
    """One token per sequence.  pool: fp32 [num_slots, H, dk, dv] (updated in place); slots: int32 [B];
    q, k: fp32 [B, H, dk]; v: fp32 [B, H, dv]; g, beta: fp32 [B, H].  Returns o fp32 [B, H, dv]."""
    B, H, dk = q.shape
    dv = v.shape[-1]
    if out is None:
        out = torch.empty(B, H, dv, dtype=torch.float32, device=q.device)
    if not q.is_cuda:
        for b in range(B):
            s = int(slots[b])
            if s < 0:
                continue
            o, S = gated_delta_recurrent(q[b:b + 1], k[b:b + 1], v[b:b + 1], g[b:b + 1], beta[b:b + 1], pool[s])
            pool[s].copy_(S)
            out[b] = o[0]
        return out
    for t in (q, k, v, g, beta):
        assert t.dtype == torch.float32 and t.is_contiguous()
    assert pool.dtype == torch.float32 and pool.is_contiguous() and slots.dtype == torch.int32
    rc = _lib.kernels().fi_gdn_step(_p(pool), _p(slots), _p(q), _p(k), _p(v), _p(g), _p(beta), _p(out), B, H, dk, dv,
                                    _stream())
    _lib.check(rc, "fi_gdn_step")
    _count()
    return out


def conv1d_step(x: torch.Tensor, pool: torch.Tensor, slots: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """Causal depthwise convolution + SiLU for one new input per sequence.  x: [B, C]; pool:
    [num_slots, C, kw - 1] (the previous inputs, updated in place); w: [C, kw].  Returns fp32 [B, C]."""
    B, C = x.shape
    kw = w.shape[1]
    if not x.is_cuda:
        y = torch.empty(B, C, dtype=torch.float32)
        for b in range(B):
            s = int(slots[b])
            if s < 0:
                y[b] = 0
                continue
            win = torch.cat([pool[s].float(), x[b].float()[:, None]], dim=1)        # [C, kw]
            y[b] = F.silu((win * w.float()).sum(-1))
            pool[s].copy_(win[:, 1:].to(pool.dtype))
        return y
    y = torch.empty(B, C, dtype=torch.float32, device=x.device)
    assert x.stride(1) == 1 and pool.is_contiguous() and w.is_contiguous() and pool.dtype == x.dtype == w.dtype
    rc = _lib.kernels().fi_conv1d_step(_p(x), x.stride(0), _p(pool), _p(slots), _p(w), _p(y), B, C, kw, _DT[x.dtype],
                                       _stream())
    _lib.check(rc, "fi_conv1d_step")
    _count()
    return y


# ---------------------------------------------------------------------------- HGRN2
def _hgrn2_gates(q, f, f_bias, lower):
    """fp32 activated query, write strength 1 - forget gate: [n, H * d] each."""
    z = f.float() + f_bias
    return F.silu(q.float()), (1.0 - lower) * torch.sigmoid(-z)


def _hgrn2_tokens(q, k, v, S):
    """q, k: fp32 [L, H, d] (activated query, write strength), v: fp32 [L, H, dv], S: fp32 [H, d, dv], updated in
    place.  Returns o fp32 [L, H, dv]."""
    o = torch.empty(q.shape[0], v.shape[1], v.shape[2], dtype=torch.float32, device=q.device)
    for t in range(q.shape[0]):
        S.mul_((1.0 - k[t])[:, :, None]).add_(k[t][:, :, None] * v[t][:, None, :])
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    return o


def hgrn2_scan(q, f, v, f_bias, lower, pool, slots, cu_q, seq_lens, H: int, d: int, dv: int):
    """Portions of sequences: ``f_t = l + (1 - l) sigmoid(z_t + b)``, ``S = diag(f) S + (1 - f) v^T``, ``o = S^T silu(q)``.

    q, f [T, H * d] and v [T, H * dv]: projection outputs (any row pitch; q and v share a dtype).  f_bias, lower: fp32
    [H * d].  pool: fp32 [num_slots, H, d, dv], updated in place; slots, seq_lens: int32 [B]; cu_q: int32 [B + 1].  A
    portion as long as its sequence starts from a zero state.  Returns o fp32 [T, H, dv]."""
    T, B = q.shape[0], slots.shape[0]
    o = torch.empty(T, H, dv, dtype=torch.float32, device=q.device)
    if not q.is_cuda:
        qa, ka = _hgrn2_gates(q, f, f_bias, lower)
        cu, lens = cu_q.tolist(), seq_lens.tolist()
        for b, s in enumerate(slots.tolist()):
            lo, hi = cu[b], cu[b + 1]
            if hi <= lo:
                continue
            S = pool[s]
            if lens[b] == hi - lo:
                S.zero_()
            o[lo:hi] = _hgrn2_tokens(qa[lo:hi].view(-1, H, d), ka[lo:hi].view(-1, H, d),
                                     v[lo:hi].float().reshape(-1, H, dv), S)
        return o
    assert q.dtype == v.dtype and q.stride(1) == f.stride(1) == v.stride(1) == 1
    assert pool.dtype == torch.float32 and pool.is_contiguous() and slots.dtype == torch.int32 == cu_q.dtype
    assert f.dtype == torch.float32, "the forget gate's projection stays 32-bit"
    rc = _lib.kernels().fi_hgrn2_scan(_p(q), q.stride(0), _p(f), f.stride(0), _p(v), v.stride(0), _p(f_bias), _p(lower),
                                      _p(pool), _p(slots), _p(cu_q), _p(seq_lens), _p(o), B, H, d, dv, pool.shape[0],
                                      _DT[q.dtype], _DT[f.dtype], _stream())
    _lib.check(rc, "fi_hgrn2_scan")
    _count()
    return o


def head_norm(o, w, eps: float, out_dtype, gate=None):
    """RMS norm of every head's row: o fp32 [T, H, dv], w fp32 [dv] -> [T, H * dv], times ``sigmoid(gate)`` if there is a
    gate [T, H * dv] (any row pitch and type)."""
    T, H, dv = o.shape
    if not o.is_cuda:
        y = (o / torch.sqrt(o.pow(2).mean(-1, keepdim=True) + eps) * w).reshape(T, H * dv)
        return (y if gate is None else y * torch.sigmoid(gate.float())).to(out_dtype)
    out = torch.empty(T, H * dv, dtype=out_dtype, device=o.device)
    assert gate is None or gate.stride(1) == 1
    rc = _lib.kernels().fi_head_norm(_p(o), _p(w), _p(gate), gate.stride(0) if gate is not None else 0,
                                     _DT[gate.dtype] if gate is not None else 0, H, _p(out), T * H, dv, eps,
                                     _DT[out_dtype], _stream())
    _lib.check(rc, "fi_head_norm")
    _count()
    return out


def hgrn2_step(q, f, v, f_bias, lower, pool, slots, seq_lens, norm_w, eps: float, H: int, d: int, dv: int, out_dtype):
    """One token per sequence, head norm included: same operands as :func:`hgrn2_scan`.  Rows with ``seq_lens`` <= 0
    are padding (zero output, no state touched).  Returns [B, H * dv]."""
    B = slots.shape[0]
    if not q.is_cuda:
        qa, ka = _hgrn2_gates(q, f, f_bias, lower)
        o = torch.zeros(B, H, dv, dtype=torch.float32)
        for b, (s, n) in enumerate(zip(slots.tolist(), seq_lens.tolist())):
            if n <= 0 or s < 0:
                continue
            if n == 1:
                pool[s].zero_()
            o[b] = _hgrn2_tokens(qa[b:b + 1].view(1, H, d), ka[b:b + 1].view(1, H, d), v[b:b + 1].float().reshape(1, H, dv),
                                 pool[s])[0]
        return head_norm(o, norm_w, eps, out_dtype)
    assert q.dtype == v.dtype and pool.dtype == torch.float32 and pool.is_contiguous()
    out = torch.empty(B, H * dv, dtype=out_dtype, device=q.device)
    rc = _lib.kernels().fi_hgrn2_step(_p(q), q.stride(0), _p(f), f.stride(0), _p(v), v.stride(0), _p(f_bias), _p(lower),
                                      _p(pool), _p(slots), _p(seq_lens), _p(norm_w), eps, _p(out), B, H, d, dv,
                                      pool.shape[0], _DT[q.dtype], _DT[f.dtype], _DT[out_dtype], _stream())
    _lib.check(rc, "fi_hgrn2_step")
    _count()
    return out


# ---------------------------------------------------------------------------- delta rule with channel decays
DELTA_CHUNK = 16


class DeltaSpec:
    """Sizes and small weights of one layer: ``H`` value heads, ``G`` query / key heads, ``d`` and ``dv`` channels, the
    convolution ``conv`` fp32 [2 G d + H dv, taps], ``rate`` fp32 [H] (exp of the stored logarithm) and ``bias`` fp32
    [H * d] of the decays."""

    def __init__(self, H: int, G: int, d: int, dv: int, conv, rate, bias):
        self.H, self.G, self.d, self.dv, self.conv, self.rate, self.bias = H, G, d, dv, conv, rate, bias
        self.taps = conv.shape[1]
        self.channels = 2 * G * d + H * dv


def _delta_operands(x, z, b, m: DeltaSpec):
    """x fp32 [taps - 1 + L, C] (with the inputs before the portion) -> q, k [L, H, d], v [L, H, dv], g [L, H, d],
    beta [L, H]."""
    L, G, H, d = z.shape[0], m.G, m.H, m.d
    y = F.silu((x.unfold(0, m.taps, 1) * m.conv).sum(-1))
    q, k = y[:, :G * d].view(L, G, d), y[:, G * d:2 * G * d].view(L, G, d)
    q = q / torch.sqrt(q.pow(2).sum(-1, keepdim=True) + 1e-6) * d ** -0.5
    k = k / torch.sqrt(k.pow(2).sum(-1, keepdim=True) + 1e-6)
    g = torch.exp(-m.rate[:, None] * F.softplus(z.float() + m.bias).view(L, H, d))
    return (q.repeat_interleave(H // G, 1), k.repeat_interleave(H // G, 1), y[:, 2 * G * d:].view(L, H, m.dv), g,
            torch.sigmoid(b.float()))


def _delta_sequence(x, z, b, m: DeltaSpec, S, ring, pos0: int):
    """One portion on the CPU; ``S`` and ``ring`` are updated in place.  Returns fp32 [L, H, dv]."""
    L, taps = x.shape[0], m.taps
    before = [ring[p % taps] if p >= 0 else torch.zeros(m.channels) for p in range(pos0 - taps + 1, pos0)]
    q, k, v, g, beta = _delta_operands(torch.cat([torch.stack(before), x.float()] if before else [x.float()]), z, b, m)
    o = torch.empty(L, m.H, m.dv)
    for t in range(L):
        S.mul_(g[t][:, :, None])
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S.add_(k[t][:, :, None] * u[:, None, :])
        o[t] = torch.einsum("hkv,hk->hv", S, q[t])
    for p in range(max(pos0, pos0 + L - taps + 1), pos0 + L):
        ring[p % taps].copy_(x[p - pos0])
    return o


def delta_chunks(cu_q):
    """Running count (int32 [B + 1]) of the chunks of each portion."""
    n = (cu_q[1:] - cu_q[:-1] + DELTA_CHUNK - 1) // DELTA_CHUNK
    return F.pad(torch.cumsum(n, 0), (1, 0)).to(torch.int32)


def delta_portions(x, z, b, m: DeltaSpec, pool, ring, slots, cu_q, seq_lens, chunk_base, n_chunks: int):
    """Portions of sequences.  x [T, C] (q | k | v projections), z [T, H * d] fp32 (decays), b [T, H] fp32 (write
    strengths), rows of any pitch.  pool fp32 [num_slots, H, d, dv] and ring fp32 [num_slots, taps, C], updated in place;
    slots, seq_lens: int32 [B]; cu_q: int32 [B + 1]; ``chunk_base`` of :func:`delta_chunks`, ``n_chunks`` its last entry.
    A portion as long as its sequence starts from a zero state.  Returns o fp32 [T, H, dv]."""
    T, B = x.shape[0], slots.shape[0]
    if not x.is_cuda:
        o = torch.empty(T, m.H, m.dv, dtype=torch.float32)
        cu, lens = cu_q.tolist(), seq_lens.tolist()
        for i, s in enumerate(slots.tolist()):
            lo, hi = cu[i], cu[i + 1]
            if hi <= lo:
                continue
            if lens[i] == hi - lo:
                pool[s].zero_()
            o[lo:hi] = _delta_sequence(x[lo:hi], z[lo:hi], b[lo:hi], m, pool[s], ring[s], lens[i] - (hi - lo))
        return o
    lib = _lib.kernels()
    per = lib.fi_delta_work_floats(m.d, m.dv)
    if per < 0:
        raise ValueError(f"no kernel for {m.d} key channels and {m.dv} value channels per head")
    assert x.stride(1) == z.stride(1) == b.stride(1) == 1 and z.dtype == b.dtype == torch.float32
    assert pool.dtype == ring.dtype == torch.float32 and pool.is_contiguous() and ring.is_contiguous()
    assert slots.dtype == cu_q.dtype == seq_lens.dtype == chunk_base.dtype == torch.int32
    work = scratch("delta_work", n_chunks * m.H * per * 4, x.device)
    o = torch.empty(T, m.H, m.dv, dtype=torch.float32, device=x.device)
    rc = lib.fi_delta_portions(_p(x), x.stride(0), _p(z), z.stride(0), _p(b), b.stride(0), _p(m.conv), _p(m.rate), _p(m.bias),
                               _p(pool), _p(ring), _p(slots), _p(cu_q), _p(seq_lens), _p(chunk_base), n_chunks, _p(work),
                               _p(o), B, m.H, m.G, m.d, m.dv, m.taps, pool.shape[0], _DT[x.dtype], _p(status_word(x.device)),
                               _stream())
    _lib.check(rc, "fi_delta_portions")
    _count(2)
    return o


def delta_step(x, z, b, m: DeltaSpec, pool, ring, slots, seq_lens, norm_w, eps: float, gate, out_dtype):
    """One token per sequence with head norm and output gate: operands as in :func:`delta_portions`, ``norm_w`` fp32
    [dv], ``gate`` [B, H * dv] or None.  Rows with ``seq_lens`` <= 0 are padding (zero output, no state touched).
    Returns [B, H * dv]."""
    B = slots.shape[0]
    if not x.is_cuda:
        o = torch.zeros(B, m.H, m.dv, dtype=torch.float32)
        for i, (s, n) in enumerate(zip(slots.tolist(), seq_lens.tolist())):
            if n <= 0 or s < 0:
                continue
            if n == 1:
                pool[s].zero_()
            o[i] = _delta_sequence(x[i:i + 1], z[i:i + 1], b[i:i + 1], m, pool[s], ring[s], n - 1)[0]
        return head_norm(o, norm_w, eps, out_dtype, gate)
    assert x.stride(1) == z.stride(1) == b.stride(1) == 1 and z.dtype == b.dtype == torch.float32
    assert pool.dtype == ring.dtype == torch.float32 and pool.is_contiguous() and ring.is_contiguous()
    assert gate is None or gate.stride(1) == 1
    out = torch.empty(B, m.H * m.dv, dtype=out_dtype, device=x.device)
    rc = _lib.kernels().fi_delta_step(
        _p(x), x.stride(0), _p(z), z.stride(0), _p(b), b.stride(0), _p(m.conv), _p(m.rate), _p(m.bias), _p(pool), _p(ring),
        _p(slots), _p(seq_lens), _p(norm_w), eps, _p(gate), gate.stride(0) if gate is not None else 0,
        _DT[gate.dtype] if gate is not None else 0, _p(out), B, m.H, m.G, m.d, m.dv, m.taps, pool.shape[0], _DT[x.dtype],
        _DT[out_dtype], _stream())
    _lib.check(rc, "fi_delta_step")
    _count()
    return out


# ---------------------------------------------------------------------------- decays with a bonus or a skip
def time_mix_tokens(r, k, v, w, u, S):
    """CPU form: r, k, w [L, H, d], v [L, H, dv], u [H, d]; ``S`` [H, d, dv] is updated in place."""
    o = torch.empty(v.shape)
    for t in range(r.shape[0]):
        kv = k[t][:, :, None] * v[t][:, None, :]
        o[t] = torch.einsum("hkv,hk->hv", S + u[:, :, None] * kv, r[t])
        S.mul_(w[t][:, :, None]).add_(kv)
    return o


def ssd_tokens(x, b, c, dt, rate, skip, S):
    """CPU form: x [L, H, dv], b, c [L, H, d], dt [L, H], rate, skip [H]; ``S`` [H, d, dv] is updated in place."""
    o = torch.empty(x.shape)
    for t in range(x.shape[0]):
        S.mul_(torch.exp(-rate * dt[t])[:, None, None]).add_((dt[t][:, None] * b[t])[:, :, None] * x[t][:, None, :])
        o[t] = torch.einsum("hkv,hk->hv", S, c[t]) + skip[:, None] * x[t]
    return o


def part_norm(o, w, parts: int, eps: float, out_dtype, gate=None, gate_first: bool = False):
    """RMS norm over ``parts`` equal parts of each row of o fp32 [T, n], times ``w`` fp32 [n]; ``silu(gate)`` (any row pitch
    and type) multiplies before the norm (``gate_first``) or after it."""
    T, n = o.shape
    if not o.is_cuda:
        g = None if gate is None else F.silu(gate.float())
        y = o * g if gate_first else o
        y = y.view(T, parts, -1)
        y = (y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)).view(T, n) * w
        return (y if g is None or gate_first else y * g).to(out_dtype)
    assert o.is_contiguous() and o.dtype == torch.float32 and (gate is None or gate.stride(1) == 1)
    out = torch.empty(T, n, dtype=out_dtype, device=o.device)
    rc = _lib.kernels().fi_part_norm(_p(o), _p(gate), gate.stride(0) if gate is not None else 0,
                                     _DT[gate.dtype] if gate is not None else 0, int(gate_first), _p(w), parts, _p(out), T,
                                     n // parts, eps, _DT[out_dtype], _stream())
    _lib.check(rc, "fi_part_norm")
    _count()
    return out


def _check_pool(pool, batch) -> None:
    assert pool.dtype == torch.float32 and pool.is_contiguous() and batch.extras["slot_ids"].dtype == batch.seq_lens.dtype == torch.int32


# segments are worth their second pass when one portion is at least this long
_SEGMENT_FROM = 512


def _segments(batch, heads: int, dv: int, length: int = 0):
    """(running count of segments per portion int32 [B + 1], tokens per segment, number of segments) for a step of few long
    portions, or None: the portions fill the device as they are.  ``length``: tokens per segment (0: chosen)."""
    T, blocks = sum(batch.q_lens_cpu), heads * -(-dv // 64)
    if length == 0:
        longest = max(batch.q_lens_cpu)
        if longest < _SEGMENT_FROM or T * blocks > 64 * longest:       # twice the work must pay for the parallelism
            return None
        length = min(512, max(64, -(-T * blocks // 592) + 15 & ~15))
    key = f"segments{length}"
    if key not in batch.extras:
        n = (batch.cu_q[1:] - batch.cu_q[:-1] + length - 1) // length
        batch.extras[key] = (F.pad(torch.cumsum(n, 0), (1, 0)).to(torch.int32), length, sum(-(-m // length) for m in batch.q_lens_cpu))
    return batch.extras[key]


def _scan(kind: int, q, k, v, z, zb, u, rate, pool, batch, G: int, segment: int = 0):
    T, (slots, H, d, dv) = v.shape[0], pool.shape
    o = torch.empty(T, H * dv, dtype=torch.float32, device=v.device)
    assert q.dtype == k.dtype == v.dtype and z.dtype == torch.float32 and q.stride(1) == k.stride(1) == v.stride(1) == z.stride(1) == 1
    _check_pool(pool, batch)
    seg, cut = (None, 0, 0, None, None), _segments(batch, H, dv, segment)
    if cut is not None:
        base, length, n = cut
        work = scratch("decay_segments", n * H * d * (dv + 1) * 4, v.device)
        seg = (_p(base), length, n, _p(work), work.data_ptr() + n * H * d * dv * 4)
    rc = _lib.kernels().fi_decay_scan(kind, _p(q), q.stride(0), _p(k), k.stride(0), _p(v), v.stride(0), _p(z), z.stride(0), _p(zb),
                                      _p(u), _p(rate), _p(pool), _p(batch.extras["slot_ids"]), _p(batch.cu_q), _p(batch.seq_lens),
                                      _p(o), *seg, batch.seq_lens.shape[0], H, G, d, dv, slots, _DT[v.dtype], _stream())
    _lib.check(rc, "fi_decay_scan")
    _count(1 if cut is None else 3)
    return o


def time_mix(r, k, v, gate, z, w0, u, pool, batch, norm_w, eps: float, out_dtype):
    """Time mixing of a step: ``o = r S + (r . (u * k)) v``, ``S[i, :] = w_i S[i, :] + k_i v`` with ``ln w = -e^(z + w0)``, then per
    head norm, ``norm_w`` and ``silu(gate)``.

    r, k, v, gate [T, H * d] (any row pitch, one type), z fp32 [T, H * d], w0 [H * d], u [H, d], norm_w [H * d] fp32; pool fp32
    [slots, H, d, d], updated in place.  A sequence whose first position is 0 starts from zero.  Returns [T, H * d]."""
    slots_n, H, d, dv = pool.shape
    T = r.shape[0]
    if not r.is_cuda:
        from .shift_stream import sequences
        o = torch.zeros(T, H * dv)
        for slot, lo, hi, pos0 in sequences(batch):
            if pos0 == 0:
                pool[slot].zero_()
            w = torch.exp(-torch.exp(z[lo:hi].float() + w0))
            h = [t.float().reshape(hi - lo, H, -1) for t in (r[lo:hi], k[lo:hi], v[lo:hi], w)]
            o[lo:hi] = time_mix_tokens(*h, u, pool[slot]).view(hi - lo, -1)
        return part_norm(o, norm_w, H, eps, out_dtype, gate)
    if not batch.is_decode:
        return part_norm(_scan(0, r, k, v, z, w0, u, None, pool, batch, H), norm_w, H, eps, out_dtype, gate)
    assert r.dtype == k.dtype == v.dtype == gate.dtype and z.dtype == torch.float32
    assert r.stride(1) == k.stride(1) == v.stride(1) == gate.stride(1) == z.stride(1) == 1
    _check_pool(pool, batch)
    out = torch.empty(T, H * dv, dtype=out_dtype, device=r.device)
    rc = _lib.kernels().fi_decay_step(_p(r), r.stride(0), _p(k), k.stride(0), _p(v), v.stride(0), _p(z), z.stride(0), _p(w0), _p(u),
                                      _p(gate), gate.stride(0), _p(norm_w), eps, _p(pool), _p(batch.extras["slot_ids"]),
                                      _p(batch.seq_lens), _p(out), T, H, d, dv, slots_n, _DT[r.dtype], _DT[out_dtype], _stream())
    _lib.check(rc, "fi_decay_step")
    _count()
    return out


def conv_silu(x, w, bias, ring, batch, out_dtype):
    """silu(causal convolution + bias) of a step's portions: x [T, C] (any row pitch), w fp32 [taps, C] (last row: the present
    token), ring fp32 [slots, taps, C], updated in place.  Returns [T, C]."""
    T, C = x.shape
    taps = w.shape[0]
    if not x.is_cuda:
        from .shift_stream import ring_before, ring_store, sequences
        y = torch.zeros(T, C)
        for slot, lo, hi, pos0 in sequences(batch):
            seq = torch.cat([ring_before(ring[slot], pos0, taps - 1), x[lo:hi].float()])
            y[lo:hi] = F.silu((seq.unfold(0, taps, 1) * w.t()).sum(-1) + bias)
            ring_store(ring[slot], pos0, x[lo:hi].float())
        return y.to(out_dtype)
    from .shift_stream import tiles
    base, n_tiles, tile = tiles(batch, taps, C)
    assert x.stride(1) == 1 and ring.is_contiguous() and w.is_contiguous() and ring.dtype == w.dtype == bias.dtype == torch.float32
    y = torch.empty(T, C, dtype=out_dtype, device=x.device)
    rc = _lib.kernels().fi_conv_silu(_p(x), x.stride(0), _p(w), _p(bias), taps, _p(ring), _p(y), _p(batch.extras["slot_ids"]),
                                     _p(batch.cu_q), _p(batch.seq_lens), _p(base), n_tiles, tile, batch.seq_lens.shape[0], C,
                                     ring.shape[0], _DT[x.dtype], _DT[out_dtype], _stream())
    _lib.check(rc, "fi_conv_silu")
    _count()
    return y


def ssd(xbc, z, dt, dt_bias, rate, skip, conv, conv_b, pool, ring, G: int, batch, norm_w, parts: int, eps: float, out_dtype):
    """State-space step: x | B | C = silu(conv(xbc) + conv_b); dt = softplus(dt + dt_bias); ``S = exp(-rate dt) S + dt B x^T``,
    ``y = S^T C + skip x``; then ``norm(y silu(z))`` over ``parts`` equal parts, times ``norm_w``.

    xbc [T, H dv + 2 G d] (x, B and C of G groups; any row pitch), z [T, H dv], dt fp32 [T, H]; conv fp32 [taps, channels]; pool
    fp32 [slots, H, d, dv] and ring fp32 [slots, taps, channels], updated in place.  Returns [T, H dv]."""
    slots_n, H, d, dv = pool.shape
    T, inner = xbc.shape[0], H * dv
    if not xbc.is_cuda:
        from .shift_stream import sequences
        u = conv_silu(xbc, conv, conv_b, ring, batch, torch.float32)
        o = torch.zeros(T, inner)
        for slot, lo, hi, pos0 in sequences(batch):
            if pos0 == 0:
                pool[slot].zero_()
            L = hi - lo
            b, c = (u[lo:hi, at:at + G * d].reshape(L, G, d).repeat_interleave(H // G, 1) for at in (inner, inner + G * d))
            o[lo:hi] = ssd_tokens(u[lo:hi, :inner].reshape(L, H, dv), b, c, F.softplus(dt[lo:hi].float() + dt_bias), rate, skip,
                                  pool[slot]).view(L, inner)
        return part_norm(o, norm_w, parts, eps, out_dtype, z, True)
    if batch.is_decode:
        _check_pool(pool, batch)
        assert xbc.stride(1) == dt.stride(1) == 1 and dt.dtype == torch.float32 and ring.is_contiguous()
        o = torch.empty(T, inner, dtype=torch.float32, device=xbc.device)
        rc = _lib.kernels().fi_decay_step_conv(_p(xbc), xbc.stride(0), _p(dt), dt.stride(0), _p(dt_bias), _p(rate), _p(skip), _p(conv),
                                               _p(conv_b), conv.shape[0], _p(ring), _p(pool), _p(batch.extras["slot_ids"]),
                                               _p(batch.seq_lens), _p(o), T, H, G, d, dv, slots_n, _DT[xbc.dtype], _stream())
        _lib.check(rc, "fi_decay_step_conv")
        _count()
    else:
        u = conv_silu(xbc, conv, conv_b, ring, batch, out_dtype)
        o = _scan(1, u[:, inner + G * d:], u[:, inner:inner + G * d], u[:, :inner], dt, dt_bias, skip, rate, pool, batch, G)
    return part_norm(o, norm_w, parts, eps, out_dtype, z, True)
