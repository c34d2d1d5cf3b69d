"""Mechanisms of the Luzerax design one by one: the op layer (CPU forms and, marked gpu, the kernels) against the plain
functions in ``luzerax_oracle.py``.  Inputs are planted so that a key, a map, a group, a bound or a choice that is missed
shows."""
import pytest
import torch

import luzerax_oracle as O
from litevllm_b200 import ops
from litevllm_b200.layers.head_attention import position_factor
from litevllm_b200.layers.rope import get_cos_sin
from litevllm_b200.ops import moe
from litevllm_b200.ops import qk_attn
from litevllm_b200.ops import residual_stream as stream

gpu = pytest.mark.gpu
DEV = ["cpu", pytest.param("cuda", marks=gpu)]
DT = {"f32": torch.float32, "bf16": torch.bfloat16, "f16": torch.float16}


def rnd(*shape, seed=0, std=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std


def close(got, want, tol):
    got, want = got.detach().double().cpu(), want.double()
    err = float((got - want).abs().max()) / max(1.0, float(want.abs().max()))
    assert err < tol, err


def i32(device, *x):
    return torch.tensor(x, dtype=torch.int32, device=device)


# ------------------------------------------------------------------ residual stream
@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("T, W, top, shared", [(1, 24, 2, True), (5, 33, 3, False), (40, 320, 0, True), (7, 1536, 8, True), (3, 4104, 1, False),
                                               (2100, 512, 4, True), (2, 8192, 6, True)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_stream_normalises_what_a_sublayer_returns(T, W, top, shared, dtype, device):
    """Shared expert, chosen experts and passed-through inputs are summed before the norm; the stream itself is what the
    next sublayer reads.  A large eps shows whether it stands inside the root."""
    dt, eps, tol = DT[dtype], 0.3, 2e-6 if dtype == "f32" else 6e-3
    d = lambda t: None if t is None else t.to(device)
    y = rnd(T, W, seed=1).to(dt) if shared else None
    x, post, scale, final = rnd(T, W, seed=2, std=3.0), rnd(W, seed=3), rnd(W, seed=7), rnd(W, seed=8)
    routed, s = None, torch.zeros(T, W) if y is None else y.float()
    if top:
        rows, a = rnd(T * top, W, seed=4).to(dt), rnd(T, top, seed=5).abs()
        order = torch.randperm(T * top, generator=torch.Generator().manual_seed(6)).to(torch.int32).view(T, top)
        order[:, top // 2] = -1                                  # this choice stands for the input
        picked = torch.where((order < 0)[..., None], x[:, None], rows.float()[order.clamp(min=0).long()])
        s = s + (picked * a[..., None]).sum(1)
        routed = moe.RoutedRows(d(rows), d(a), d(order), True)
        dropped = moe.RoutedRows(d(rows), d(a), d(order), False)
        zero = torch.where((order < 0)[..., None], torch.zeros(()), rows.float()[order.clamp(min=0).long()])
        out = torch.empty(T, W, device=device)
        stream.post(d(y), d(x), dropped, d(post), None, eps, 1, out, dt)
        close(out, O.sublayer(x, (0 if y is None else y.float()) + (zero * a[..., None]).sum(1), post, 1.0, eps), 3e-6)
    want = O.sublayer(x, s, post, scale, eps)
    out = torch.empty(T, W, device=device)
    h = stream.post(d(y), d(x), routed, d(post * scale), None, eps, 1, out, dt)
    close(out, want, 3e-6)
    assert h.dtype == dt and torch.equal(h, out.to(dt))
    same = d(x).clone()                                      # the sum may replace its input
    h = stream.post(d(y), same, routed, d(post * scale), d(final), eps, 1, same, dt)
    close(same, want, 3e-6)
    close(h.float(), O.rms_norm(want, final, eps), tol)
    sel = torch.tensor([T - 1, 0, T // 2])
    h = stream.post(d(y), d(x), routed, d(post * scale), d(final), eps, 1, None, dt, sel=d(sel))
    close(h.float(), O.rms_norm(want, final, eps)[sel], tol)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("W", [33, 640])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_stream_starts_with_the_embedding(W, dtype, device):
    table, ids = rnd(11, W, seed=1).to(DT[dtype]), torch.tensor([10, 0, 3, 3])
    x0 = torch.empty(4, W, device=device)
    h = stream.start(ids.to(device), table.to(device), None, 1e-6, 1, x0)
    assert torch.equal(x0.cpu(), table.float()[ids]) and torch.equal(h.cpu(), table[ids])


# ------------------------------------------------------------------ queries and keys
@pytest.mark.parametrize("device", DEV)
def test_factor_of_queries_changes_with_the_last_token_of_a_span(device):
    f = position_factor(40, 0.5, 8, torch.device(device))
    close(f, O.temperature(torch.arange(40), 0.5, 8), 1e-7)
    assert float(f[6]) == 1.0 and float(f[7]) > 1.3 and float(f[7]) == float(f[14]) < float(f[15])
    assert bool((position_factor(5, 0.5, 1, torch.device("cpu"))[1:] > position_factor(5, 0.5, 1, torch.device("cpu"))[:-1]).all())


def _check_rows(device, dtype, H, G, dim, vdim, maps, spec, wq, wk, cos_sin, factor, want, pos, pitch):
    """Runs the prepare op over rubbish-filled caches and compares queries and cache rows with ``want(kind, raw)``."""
    dt, T = DT[dtype], pos.shape[0]
    proj = rnd(T, spec.v_off + G * vdim + 3, seed=1)
    proj[:, :dim] *= 6.0                                      # a norm over more than one head would not undo that
    proj[:, spec.k_off + dim:spec.k_off + 2 * dim] *= 0.1
    proj = proj.to(dt)
    slots = torch.tensor([3, 40, 5, -1, 9, 31, 17, 0, 2], dtype=torch.int32)[:T]
    k_cache, v_cache = (torch.full((3, G, 16, n), 5.0, dtype=dt, device=device) for n in (max(pitch, maps * dim), max(pitch, vdim)))
    d = lambda t: None if t is None else t.to(device)
    q = qk_attn.prepare_heads(d(proj), d(wq), d(wk), spec, d(pos), cos_sin, factor, d(slots), k_cache, v_cache)
    f = proj.float()
    want_q = want("q", f[:, :spec.k_off].view(T, H, maps, dim))
    want_k = want("k", f[:, spec.k_off:spec.v_off].view(T, G, maps, dim))
    want_v = f[:, spec.v_off:spec.v_off + G * vdim].view(T, G, vdim)
    tol = 1e-5 if dtype == "f32" else 1e-2
    full = torch.zeros(T, H, maps, spec.q_pitch)
    for m in range(maps):
        full[:, :, m, m * spec.q_shift:m * spec.q_shift + dim] = want_q[:, :, m]
    close(q.float().view(T, H, maps, -1), full, tol)
    for t in range(T):
        if slots[t] >= 0:
            b, o = int(slots[t]) // 16, int(slots[t]) % 16
            for cache, rows, e in ((k_cache, want_k[t].reshape(G, -1), tol), (v_cache, want_v[t], 1e-7)):
                n = rows.shape[-1]
                close(cache[b, :, o, :n].float(), rows, e)
                assert cache.shape[3] == n or float(cache[b, :, o, n:].abs().max()) == 0.0
    untouched = [i for i in range(48) if i not in slots.tolist()]
    assert bool((k_cache.transpose(1, 2).reshape(48, -1)[untouched] == 5.0).all())


POS = torch.tensor([0, 1, 2, 50, 51, 300, 7, 8, 9], dtype=torch.int32)
HEADS = [(3, 1, 24, 40, 0), (6, 2, 20, 24, 64), (2, 2, 5, 7, 0), (16, 4, 64, 128, 128), (4, 1, 72, 200, 256), (3, 3, 16, 64, 64), (2, 1, 7, 64, 64)]


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("H, G, dim, vdim, pitch", HEADS)
def test_two_maps_per_head(H, G, dim, vdim, pitch, dtype, device):
    eps, wq, wk = 1e-3, rnd(dim, seed=2), rnd(dim, seed=3)
    spec = qk_attn.HeadSpec(H, G, dim, vdim, 2, eps, pitch or dim, dim if pitch else 0)
    factor = position_factor(512, 0.7, 6, torch.device(device))

    def want(kind, x):
        y = O.rms_norm(x, wq if kind == "q" else wk, eps)
        return y * O.temperature(POS, 0.7, 6).float()[:, None, None, None] if kind == "q" else y
    _check_rows(device, dtype, H, G, dim, vdim, 2, spec, wq, wk, None, factor, want, POS, pitch)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("neighbours, last", [(True, True), (True, False), (False, False), (False, True)])
@pytest.mark.parametrize("H, G, dim, vdim, pitch, dims", [(3, 1, 24, 40, 0, 8), (6, 2, 40, 24, 64, 40), (2, 2, 6, 7, 0, 2), (8, 2, 128, 128, 128, 64),
                                                          (4, 1, 136, 64, 256, 16), (3, 3, 16, 64, 64, 0), (2, 1, 30, 64, 64, 22)])
def test_rotated_heads(H, G, dim, vdim, pitch, dims, neighbours, last, dtype, device):
    """Both layouts of pairs, the norm's weight before and after the rotation, without a weight, partial rotation."""
    eps, base = 1e-3, 700.0
    wq, wk = (rnd(dim, seed=2), rnd(dim, seed=3)) if not (neighbours and last) else (None, None)
    spec = qk_attn.HeadSpec(H, G, dim, vdim, 1, eps, pitch or dim, 0, dims, neighbours, last)
    cs = get_cos_sin(dims, 512, base, None, torch.device(device)) if dims else None

    def turn(x):
        if neighbours or not dims:
            return O.rotate_neighbours(x, POS, dims, base)
        order = torch.arange(dim)
        order[:dims] = torch.arange(dims).view(2, -1).t().reshape(-1)     # halves interleaved are neighbours
        return O.rotate_neighbours(x[..., order], POS, dims, base)[..., torch.argsort(order)]

    def want(kind, x):
        w = wq if kind == "q" else wk
        w = 1.0 if w is None else w
        x = x[:, :, 0]
        y = O.rms(turn(x), eps) * w if last else turn(O.rms(x, eps) * w)
        return y[:, :, None]
    _check_rows(device, dtype, H, G, dim, vdim, 1, spec, wq, wk, cs, None, want, POS, pitch)


# ------------------------------------------------------------------ attention
class Paged:
    """Keys and values of several sequences in shuffled pages; unused rows hold rubbish, padding zeros."""

    def __init__(self, lens, G, kn, vn, kp, vp, bs, dtype, device, seed=0):
        self.bs = bs
        per = [(n + bs - 1) // bs for n in lens]
        order = torch.randperm(sum(per), generator=torch.Generator().manual_seed(seed)) + 1
        self.table = torch.zeros(len(lens), max(per), dtype=torch.int32)
        at = 0
        for b, n in enumerate(per):
            self.table[b, :n] = order[at:at + n].to(torch.int32)
            at += n
        self.k, self.v = (torch.full((sum(per) + 1, G, bs, p), 7.0, dtype=dtype) for p in (kp, vp))
        self.k[..., kn:] = 0
        self.v[..., vn:] = 0
        self.k, self.v = self.k.to(device), self.v.to(device)

    def fill(self, b, k, v):
        pos = torch.arange(k.shape[0])
        blk, off = self.table[b].long()[pos // self.bs], pos % self.bs
        for cache, rows in ((self.k, k), (self.v, v)):
            cache[blk.to(cache.device), :, off.to(cache.device), :rows.shape[-1]] = rows.to(cache)


class Heads:
    """Queries and keys ``[T, heads, maps, dim]`` as the kernels want them, and their plain evaluation."""

    def __init__(self, H, G, dim, vdim, maps, form, dtype):
        self.H, self.G, self.dim, self.vdim, self.maps, self.form, self.dt = H, G, dim, vdim, maps, form, DT[dtype]
        self.hd = 0 if form == "rows" else next(h for h in (64, 128, 256) if max(maps * dim, vdim) <= h)
        self.diff = (0.6, 0.7, 1e-3) if maps == 2 else None

    def pages(self, lens, device):
        return Paged(lens, self.G, self.maps * self.dim, self.vdim, self.hd or self.maps * self.dim, self.hd or self.vdim, 16, self.dt, device)

    def kernel_queries(self, q):
        out = torch.zeros(q.shape[0], self.H, self.maps, self.hd or self.dim, dtype=self.dt)
        for m in range(self.maps):
            lo = m * self.dim if self.hd else 0
            out[:, :, m, lo:lo + self.dim] = q[:, :, m]
        return out.view(q.shape[0], self.H * self.maps, -1)

    def run(self, q, pages, rows, scale, gate, device, max_len):
        """q: rows as in ``kernel_queries``; rows: (sequence, visible length) each."""
        lens, seq, table = i32(device, *[n for _, n in rows]), i32(device, *[b for b, _ in rows]), pages.table.to(device)
        q = self.kernel_queries(q).to(device)
        if self.form == "rows":
            return qk_attn.attend_rows(q, pages.k, pages.v, table, lens, seq, scale, 0, None, gate, self.vdim, self.diff)
        kw = dict(v_dim=self.vdim, gate=gate, diff=self.diff)
        args = (q.view(len(rows), -1), pages.k, pages.v, table[seq.long()], lens)
        if self.form == "decode":
            return ops.paged_attention_decode(*args, self.H * self.maps, self.G, self.hd, scale, max_kv_len=max_len, **kw)
        cu = torch.arange(len(rows) + 1, dtype=torch.int32, device=device)          # portions of one token
        return ops.paged_attention_prefill(*args, cu, 1, self.H * self.maps, self.G, self.hd, scale, **kw)

    def want(self, q, k, v, scale, gate=None):
        """q [Tq, H, maps, dim] the last positions of k [Tk, G, maps, dim], v [Tk, G, vdim] -> [Tq, H * vdim]."""
        q, k, v = q.float(), k.float(), v.float()
        a = [torch.stack([O.causal_attention(q[:, h, m], k[:, h // (self.H // self.G), m], v[:, h // (self.H // self.G)], scale)
                          for h in range(self.H)], 1) for m in range(self.maps)]
        if self.maps == 2:
            o = O.subtract_maps(a[0], a[1], self.diff[0], 1.0 - self.diff[1], self.diff[2])
        else:
            o = a[0] if gate is None else a[0] * torch.sigmoid(gate.float())[..., None]
        return o.reshape(q.shape[0], -1)


FORMS = [pytest.param("rows", "f32", "cpu"), pytest.param("rows", "f32", "cuda", marks=gpu), pytest.param("rows", "bf16", "cuda", marks=gpu),
         pytest.param("decode", "bf16", "cuda", marks=gpu), pytest.param("decode", "f16", "cuda", marks=gpu),
         pytest.param("portions", "bf16", "cuda", marks=gpu)]
SHAPES = [(3, 1, 24, 40, 2), (6, 2, 20, 24, 2), (17, 1, 32, 64, 2), (4, 4, 64, 128, 2), (8, 2, 16, 200, 2), (2, 1, 100, 32, 2),
          (3, 1, 24, 40, 1), (17, 1, 128, 64, 1), (8, 2, 136, 72, 1)]


@pytest.mark.parametrize("form, dtype, device", FORMS)
@pytest.mark.parametrize("H, G, dim, vdim, maps", SHAPES)
def test_rows_against_cached_keys(H, G, dim, vdim, maps, form, dtype, device):
    s = Heads(H, G, dim, vdim, maps, form, dtype)
    lens = [1, 16, 17, 130, 260]
    rows = [(b, n) for b, n in enumerate(lens)] + [(4, 64), (4, 65), (3, 1), (4, 129)]
    pages = s.pages(lens, device)
    ks, vs = [rnd(n, G, maps, dim, seed=b).to(s.dt) for b, n in enumerate(lens)], [rnd(n, G, vdim, seed=30 + b).to(s.dt) for b, n in enumerate(lens)]
    for b in range(len(lens)):
        pages.fill(b, ks[b].flatten(2), vs[b])
    q = rnd(len(rows), H, maps, dim, seed=9).to(s.dt)
    gate = rnd(len(rows), H + 5, seed=10, std=2.0).to(s.dt)[:, 5:] if maps == 1 else None
    scale = 1.5 * dim ** -0.5
    got = s.run(q, pages, rows, scale, None if gate is None else gate.to(device), device, max(lens))
    for i, (b, n) in enumerate(rows):
        want = s.want(q[i:i + 1], ks[b][:n], vs[b][:n], scale, None if gate is None else gate[i:i + 1])
        close(got[i].float(), want[0], 3e-5 if dtype == "f32" else 3e-2)


@pytest.mark.parametrize("form, dtype, device", FORMS)
@pytest.mark.parametrize("far", [0, 1, 15, 16, 63, 64, 127, 128, 240, 299])
def test_each_map_finds_its_own_key(far, form, dtype, device):
    """The first map's query matches the key at ``far``, the second one's the key at the mirrored place; the difference of
    their values must come out, and not the other map's."""
    s, n = Heads(2, 1, 32, 48, 2, form, dtype), 300
    k, v = rnd(n, 1, 2, 32, seed=1, std=0.05), rnd(n, 1, 48, seed=2)
    a, b, other = rnd(32, seed=3), rnd(32, seed=4), n - 1 - far
    k[far, 0, 0], k[other, 0, 1] = a, b
    k[other, 0, 0] = -a
    k, v = k.to(s.dt), v.to(s.dt)
    pages = s.pages([n], device)
    pages.fill(0, k.flatten(2), v)
    q = torch.stack([a, b]).expand(1, 2, 2, 32).contiguous().to(s.dt)
    got = s.run(q, pages, [(0, n)], 2.0, None, device, n).float().cpu().view(2, 48)
    close(got, s.want(q, k, v, 2.0).view(2, 48), 1e-5 if dtype == "f32" else 2e-2)
    o = v[far, 0].float() - 0.6 * v[other, 0].float()
    close(got[0], O.rms(o, 1e-3) * 0.7, 0.1)


@gpu
@pytest.mark.parametrize("H, G, dim, vdim, maps", [(6, 2, 20, 24, 2), (4, 1, 32, 64, 2), (4, 2, 64, 128, 2), (3, 3, 48, 72, 2), (2, 1, 72, 200, 2), (5, 1, 30, 30, 2),
                                                   (6, 2, 40, 24, 1), (8, 2, 128, 128, 1), (2, 1, 64, 40, 1)])
def test_long_portions(H, G, dim, vdim, maps):
    """Portions whose context lies partly in the cache, on the prefill kernels; the first key stands out for one query in
    every sequence, in one map only."""
    s = Heads(H, G, dim, vdim, maps, "portions", "bf16")
    spans = [(0, 64), (100, 70), (131, 300), (5, 128), (400, 65)]            # (tokens before, new tokens)
    lens = [a + n for a, n in spans]
    pages = s.pages(lens, "cuda")
    ks, vs = [rnd(n, G, maps, dim, seed=b).to(s.dt) for b, n in enumerate(lens)], [rnd(n, G, vdim, seed=30 + b).to(s.dt) for b, n in enumerate(lens)]
    T = sum(n for _, n in spans)
    q = rnd(T, H, maps, dim, seed=22).to(s.dt)
    gate = rnd(T, H + 8, seed=23).to(s.dt)[:, 8:] if maps == 1 else None
    at, scale = 0, 1.5 * dim ** -0.5
    for b, (a, n) in enumerate(spans):
        pages.fill(b, ks[b].flatten(2), vs[b])
        q[at + n // 2, :, b % maps] += 2.0 * ks[b][0, :, b % maps].repeat_interleave(H // G, 0)
        at += n
    cu = torch.tensor([0] + [n for _, n in spans]).cumsum(0).to(torch.int32).cuda()
    qk = s.kernel_queries(q).cuda().view(T, -1)
    got = ops.paged_attention_prefill(qk, pages.k, pages.v, pages.table.cuda(), i32("cuda", *lens), cu, 300, H * maps, G, s.hd, scale, v_dim=vdim,
                                      gate=None if gate is None else gate.cuda(), diff=s.diff)
    at = 0
    for b, (a, n) in enumerate(spans):
        close(got[at:at + n].float(), s.want(q[at:at + n], ks[b], vs[b], scale, None if gate is None else gate[at:at + n]), 4e-2)
        at += n
    ops.check_status(torch.device("cuda", 0))


@gpu
@pytest.mark.parametrize("n", [600, 4300, 9000])
@pytest.mark.parametrize("maps", [1, 2])
@pytest.mark.parametrize("splits", [0, 2, 5, 12, 40])
def test_few_rows_over_long_contexts(n, maps, splits):
    """One row split over many blocks, merged inside a cluster, by the last block or by the merge kernel; a far key stands
    out."""
    s = Heads(4, 2, 32, 64, maps, "decode", "bf16")
    k, v = rnd(n, 2, maps, 32, seed=1, std=0.5).bfloat16(), rnd(n, 2, 64, seed=2).bfloat16()
    pages = s.pages([n], "cuda")
    pages.fill(0, k.flatten(2), v)
    q = rnd(1, 4, maps, 32, seed=3, std=0.3).bfloat16()
    q[0, 0, maps - 1] += 3 * k[0, 0, maps - 1]
    q[0, 3, 0] += 3 * k[n // 2, 1, 0]
    gate = rnd(1, 4, seed=5).bfloat16() if maps == 1 else None
    got = ops.paged_attention_decode(s.kernel_queries(q).cuda().view(1, -1), pages.k, pages.v, pages.table.cuda(), i32("cuda", n), 4 * maps, 2, s.hd, 0.8,
                                     max_kv_len=n, splits=splits, v_dim=64, gate=None if gate is None else gate.cuda(), diff=s.diff)
    # averages over thousands of keys are small beside the difference's norm: rounding of the weights shows there
    close(got[0].float(), s.want(q, k, v, 0.8, gate)[0], 1.5e-2 if maps == 1 else 6e-2)


def test_two_maps_refuse_gates_and_odd_groups():
    with pytest.raises(ValueError, match="gate"):
        ops.attn_extra(4, 8, gate=torch.zeros(2, 4), diff=(0.5, 0.5, 1e-6))
    with pytest.raises(ValueError, match="fits neither"):
        ops.attn_extra(4, 8, gate=torch.zeros(2, 5))


# ------------------------------------------------------------------ feed-forward
@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("T, K, I", [(1, 64, 40), (7, 33, 19), (60, 256, 136), (300, 512, 264), (1100, 128, 72)])
def test_clipped_gates(T, K, I, dtype, device):
    """Bounds on both halves (the gate's from above only), reached by a good part of the channels; every product kernel."""
    dt, limit = DT[dtype], 0.7
    x, w = rnd(T, K, seed=1).to(dt), rnd(2 * I, K, seed=2, std=2.0 * K ** -0.5).to(dt)
    got = ops.gated_linear(x.to(device), w.to(device), "clipped_swiglu", act_limit=limit)
    f = {"p.gate": w[:I].float(), "p.up": w[I:].float(), "p.down": torch.eye(I)}
    close(got.float(), O.clipped_expert(x.float(), f, "p.", limit), 1e-5 if dtype == "f32" else 8e-3)
    if device == "cuda":
        ops.check_status(torch.device("cuda", 0))


@pytest.mark.parametrize("device", DEV)
def test_the_gate_is_bounded_from_above_only(device):
    x = torch.tensor([[-3.0], [-0.5], [0.4], [50.0]], device=device)
    w = torch.tensor([[1.0], [1.0]], device=device)
    got = ops.gated_linear(x, w, "clipped_swiglu", act_limit=2.0).cpu()[:, 0]
    g, u = torch.tensor([-3.0, -0.5, 0.4, 2.0]), torch.tensor([-2.0, -0.5, 0.4, 2.0])
    close(got, g * torch.sigmoid(1.702 * g) * (u + 1), 1e-6)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("E, top, groups, keep", [(12, 3, 3, 2), (6, 2, 3, 1), (9, 2, 9, 4), (64, 6, 8, 3), (160, 8, 8, 3), (5, 5, 1, 1), (1, 1, 1, 1),
                                                  (40, 4, 40, 7), (500, 32, 4, 2)])
def test_choice_of_experts(E, top, groups, keep, device):
    T = 50
    z, c = rnd(T, E + 3, seed=E, std=2.0), rnd(E, seed=E + 1, std=0.3) - 0.1      # sums of score and correction change sign
    ids, w = moe.route(z.to(device)[:, 3:], top, mode="softmax", bias=c.to(device), renormalize=True, groups=groups, keep_groups=keep,
                       group_best=1)
    for t in range(T):
        want, _ = O.choose(z[t, 3:], c, groups, keep, top)
        got = dict(zip(ids[t].tolist(), w[t].tolist()))
        assert set(got) == set(want)
        for e, a in want.items():
            assert abs(got[e] - float(a)) < 1e-5


@pytest.mark.parametrize("device", DEV)
def test_groups_are_ranked_by_their_best_and_dropped_entirely(device):
    """Group 0 holds the single best output and weak others, group 1 two good ones: group 0 wins over group 1 only when one
    score counts.  All sums are negative, so a dropped expert that counted as zero would be chosen."""
    s = torch.softmax(torch.zeros(9), -1)
    choice = torch.tensor([-0.1, -3.0, -3.0, -1.0, -1.1, -3.0, -0.2, -1.3, -1.4])
    route = lambda best: moe.route(torch.zeros(1, 9, device=device), 3, bias=(choice - s).to(device), groups=3, keep_groups=2, group_best=best)
    ids, w = route(1)
    assert sorted(ids[0].tolist()) == [0, 6, 7]
    close(w, torch.full((1, 3), 1 / 3), 1e-6)                                     # scores without the correction
    assert sorted(route(2)[0][0].tolist()) == [3, 4, 6]


@pytest.mark.parametrize("device", DEV)
def test_softmax_without_a_correction_is_unchanged(device):
    z = rnd(30, 16, seed=3)
    ids, w = moe.route(z.to(device), 4)
    p, want = torch.topk(torch.softmax(z, -1), 4, dim=-1)
    assert torch.equal(ids.cpu().long(), want)
    close(w, p / p.sum(-1, keepdim=True), 1e-6)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("T, H, I, E, identity, top", [(1, 33, 7, 5, 2, 2), (9, 64, 40, 6, 6, 3), (20, 72, 24, 4, 1, 4), (130, 256, 96, 8, 4, 2),
                                                       (40, 512, 264, 32, 8, 4), (1500, 256, 136, 16, 4, 3), (64, 40, 50, 1, 3, 1)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_expert_products_with_choices_that_pass_the_input_on(T, H, I, E, identity, top, dtype, device):
    """Every tile size of the grouped products and the general kernel; one expert gets most tokens, one none, and tokens
    may choose nothing but pass-through outputs."""
    if device == "cpu" and T > 200:
        pytest.skip("large cases run on the kernels")
    dt, limit = DT[dtype], 0.8
    x, w1, w2 = rnd(T, H, seed=1).to(dt), rnd(E, 2 * I, H, seed=2, std=2 * H ** -0.5).to(dt), rnd(E, H, I, seed=3, std=I ** -0.5).to(dt)
    z = rnd(T, E + identity, seed=4)
    z[:, 0] += 1.5
    if E > top:
        z[:, E - 1] = -50.0
    z[T // 2, E:] += 60.0
    a, ids = torch.topk(z, top, dim=1)
    ids, a = ids.to(torch.int32), torch.sigmoid(a)
    got = moe.expert_rows(x.to(device), w1.to(device), w2.to(device), ids.to(device), a.to(device), "clipped_swiglu", limit, True)
    got = moe.RoutedRows(got.rows.clone(), got.weights, None if got.slot_of is None else got.slot_of.clone(), got.pass_through)
    assert torch.equal(got.slot_of.cpu() < 0, ids >= E)
    f = x.float()
    every = torch.stack([O.clipped_expert(f, {"p.gate": w1[e, :I].float(), "p.up": w1[e, I:].float(), "p.down": w2[e].float()}, "p.", limit)
                         if e < E else f for e in range(E + identity)], dim=1)
    want = (torch.gather(every, 1, ids.long()[..., None].expand(T, top, H)) * a[..., None]).sum(1)
    close(got.combined(x.to(device)), want, 1e-5 if dtype == "f32" else 1.5e-2)
    if device == "cuda":
        ops.check_status(torch.device("cuda", 0))
