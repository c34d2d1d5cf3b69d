"""Mechanisms of the Pofadra design one by one: the op layer (CPU forms and, marked gpu, the kernels) against the plain
functions in ``pofadra_oracle.py``.  Inputs are planted so that a key, an edge, a sink, a group or a state that is missed
shows."""
import pytest
import torch

import pofadra_oracle as O
from litevllm_b200 import ops
from litevllm_b200.layers.rope import get_cos_sin
from litevllm_b200.ops import linear_attn as lin
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


# ------------------------------------------------------------------ residual stream, soft cap
@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("T, W, top", [(1, 24, 2), (5, 33, 3), (40, 320, 0), (7, 1536, 8), (3, 4104, 1), (2100, 512, 4), (2, 8192, 6)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_stream_adds_mixer_and_chosen_experts(T, W, top, dtype, device):
    dt, eps, tol = DT[dtype], 1e-5, 2e-6 if dtype == "f32" else 6e-3
    d = lambda t: t.to(device)
    y, x, w = rnd(T, W, seed=1).to(dt), rnd(T, W, seed=2, std=20.0), rnd(W, seed=3)
    routed, extra = None, torch.zeros(T, W)
    if top:
        rows, a = rnd(T * top, W, seed=4).to(dt), rnd(T, top, seed=5)
        order = torch.randperm(T * top, generator=torch.Generator().manual_seed(6)).to(torch.int32).view(T, top)
        extra = (rows.float()[order.long().view(-1)].view(T, top, W) * a[..., None]).sum(1)
        routed = moe.RoutedRows(d(rows), d(a), d(order))
    want = x + y.float() + extra
    out = torch.empty(T, W, device=device)
    h = stream.add(d(y), d(x), routed, d(w), eps, 1, out, dt)
    close(out, want, 2e-6)
    close(h.float(), O.rms_norm(want, w, eps), tol)
    same = d(x).clone()                                     # the sum may replace its input; the next norm is optional
    assert stream.add(d(y), same, routed, None, eps, 1, same, dt) is None
    close(same, want, 2e-6)
    sel = torch.tensor([T - 1, 0, T // 2])
    h = stream.add(d(y), d(x), routed, d(w), eps, 1, None, dt, sel=d(sel))
    close(h.float(), O.rms_norm(want, w, eps)[sel], tol)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("W", [33, 640])
def test_stream_start_scales_the_embedding(W, device):
    table, w = rnd(11, W, seed=1).bfloat16(), rnd(W, seed=2)
    ids = torch.tensor([10, 0, 3, 3])
    x0 = torch.empty(4, W, device=device)
    h = stream.start(ids.to(device), table.to(device), w.to(device), 0.5, 1, x0, 12.5)
    want = table.float()[ids] * 12.5
    close(x0, want, 1e-7)
    close(h.float(), O.rms_norm(want, w, 0.5), 6e-3)         # a large eps shows whether it stands inside the root


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("n", [4, 31, 1000])
def test_soft_cap(n, device):
    x = rnd(3, n + 5, seed=1, std=30.0)[:, :n]
    x[0, :4] = torch.tensor([1e-3, -1e4, 1e4, 0.0])
    for cap in (1.5, 30.0):
        buf = torch.zeros(3, n + 5, device=device)
        buf[:, :n] = x.to(device)
        ops.soft_cap(buf[:, :n], cap)
        close(buf[:, :n] / cap, O.soft_cap(x.double(), cap) / cap, 4e-7)
        assert float(buf[:, n:].abs().max()) == 0.0


# ------------------------------------------------------------------ attention
class Paged:
    """Keys and values of several sequences in shuffled pages of one pool; heads padded from dim to hd."""

    def __init__(self, lens, G, dim, hd, bs, dtype, device, seed=0):
        self.bs, self.dim = bs, dim
        per = [(n + bs - 1) // bs for n in lens]
        order = torch.randperm(sum(per), generator=torch.Generator().manual_seed(seed)) + 1
        self.table = torch.zeros(len(lens), max(per), dtype=torch.int32)
        at = 0
        for b, n in enumerate(per):
            self.table[b, :n] = order[at:at + n].to(torch.int32)
            at += n
        pool = torch.full((sum(per) + 1, G, bs, hd), 7.0, dtype=dtype)                       # unused rows hold rubbish
        pool[..., dim:] = 0
        self.k, self.v = pool.clone().to(device), pool.clone().to(device)

    def slots(self, b, pos):
        return (self.table[b].long()[pos // self.bs] * self.bs + pos % self.bs).to(torch.int32)

    def fill(self, b, k, v):
        pos = torch.arange(k.shape[0])
        blk, off = self.table[b].long()[pos // self.bs], pos % self.bs
        for cache, rows in ((self.k, k), (self.v, v)):
            cache[blk.to(cache.device), :, off.to(cache.device), :self.dim] = rows.to(cache)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("H, G, dim, hd, dims", [(3, 1, 24, 24, 8), (6, 2, 40, 64, 40), (2, 2, 5, 5, 2), (16, 4, 128, 128, 64), (4, 1, 136, 256, 16),
                                                 (3, 3, 16, 64, 0)])
def test_queries_keys_and_values(H, G, dim, hd, dims, dtype, device):
    """One head is scaled up: a norm per head instead of one over the projection would undo that."""
    dt, T, eps, base = DT[dtype], 9, 1e-4, 700.0
    proj = rnd(T, (2 * H + G) * dim, seed=1)
    proj[:, :dim] *= 6.0
    proj[:, H * dim:H * dim + dim] *= 0.2
    proj = proj.to(dt)
    wq, wk = rnd(H * dim, seed=2), rnd(G * dim, seed=3)
    pos = torch.tensor([0, 1, 2, 50, 51, 300, 7, 8, 9], dtype=torch.int32)
    slots = torch.tensor([3, 40, 5, -1, 9, 31, 17, 0, 2], dtype=torch.int32)
    k_cache, v_cache = (torch.full((3, G, 16, hd), 5.0, dtype=dt, device=device) for _ in range(2))
    d = lambda t: t.to(device)
    q = qk_attn.prepare(d(proj), d(wq), d(wk), eps, d(pos), get_cos_sin(dims, 512, base, None, torch.device(device)), d(slots),
                        k_cache, v_cache, H, G, dim)
    f = proj.float()
    want_q = O.rotate_half(O.rms_norm(f[:, :H * dim], wq, eps).view(T, H, dim), pos, dims, base)
    raw = f[:, H * dim:(H + G) * dim]
    want_k = O.rotate_half(O.rms_norm(raw, wk, eps).view(T, G, dim), pos, dims, base)
    tol = 1e-5 if dtype == "f32" else 1e-2
    close(q[..., :dim].float(), want_q, tol)
    assert hd == dim or float(q[..., dim:].abs().max()) == 0.0
    for t in range(T):
        if slots[t] >= 0:
            b, o = int(slots[t]) // 16, int(slots[t]) % 16
            close(k_cache[b, :, o, :dim].float(), want_k[t], tol)
            close(v_cache[b, :, o, :dim].float(), raw.view(T, G, dim)[t], 1e-7)
            assert hd == dim or float(k_cache[b, :, o, dim:].abs().max()) == float(v_cache[b, :, o, dim:].abs().max()) == 0.0
    untouched = [i for i in range(48) if i not in slots.tolist()]
    assert bool((k_cache.transpose(1, 2).reshape(48, -1)[untouched] == 5.0).all())


def _attend(form, q, pages, rows, scale, window, sinks, gate, dim, device, max_len):
    """Runs one of the three forms over query rows (sequence, visible length); returns [R, H * dim]."""
    lens, seq = i32(device, *[n for _, n in rows]), i32(device, *[b for b, _ in rows])
    table = pages.table.to(device)
    H, G, hd = q.shape[1], pages.k.shape[1], pages.k.shape[3]
    if form == "rows":
        return qk_attn.attend_rows(q, pages.k, pages.v, table, lens, seq, scale, window, sinks, gate, dim)
    if form == "decode":
        return ops.paged_attention_decode(q.view(len(rows), -1), pages.k, pages.v, table[seq.long()], lens, H, G, hd, scale, window,
                                          max_kv_len=max_len, sinks=sinks, v_dim=dim, gate=gate)
    cu = torch.arange(len(rows) + 1, dtype=torch.int32, device=device)          # portions of one token
    return ops.paged_attention_prefill(q.view(len(rows), -1), pages.k, pages.v, table[seq.long()], lens, cu, 1, H, G, hd, scale,
                                       window, sinks=sinks, v_dim=dim, gate=gate)


FORMS = [pytest.param("rows", "f32", "cpu"), pytest.param("rows", "f32", "cuda", marks=gpu), pytest.param("rows", "bf16", "cuda", marks=gpu),
         pytest.param("decode", "bf16", "cuda", marks=gpu), pytest.param("decode", "f16", "cuda", marks=gpu),
         pytest.param("portions", "bf16", "cuda", marks=gpu)]


@pytest.mark.parametrize("form, dtype, device", FORMS)
@pytest.mark.parametrize("H, G, dim", [(3, 1, 24), (6, 2, 40), (16, 16, 64), (17, 1, 128), (8, 2, 136)])
@pytest.mark.parametrize("window", [0, 1, 17, 64, 200])
def test_rows_against_cached_keys(H, G, dim, window, form, dtype, device):
    dt = DT[dtype]
    hd = dim if form == "rows" else next(h for h in (64, 128, 256) if dim <= h)
    lens = [1, 16, 17, 130, 260]
    rows = [(b, n) for b, n in enumerate(lens)] + [(4, 64), (4, 65), (3, 1), (4, 129)]
    pages = Paged(lens, G, dim, hd, 16, dt, device)
    ks, vs = [rnd(n, G, dim, seed=b).to(dt) for b, n in enumerate(lens)], [rnd(n, G, dim, seed=30 + b).to(dt) for b, n in enumerate(lens)]
    for b in range(len(lens)):
        pages.fill(b, ks[b], vs[b])
    q = torch.zeros(len(rows), H, hd, dtype=dt)
    q[..., :dim] = rnd(len(rows), H, dim, seed=9).to(dt)
    gate = rnd(len(rows), H * dim + 8, seed=10).to(dt)[:, 8:]
    scale = 1.5 * dim ** -0.5
    got = _attend(form, q.to(device), pages, rows, scale, window, torch.zeros(H, device=device), gate.to(device), dim, device, max(lens))
    for i, (b, n) in enumerate(rows):
        want = O.attend(q[i:i + 1, :, :dim].float(), ks[b][:n].float(), vs[b][:n].float(), scale, window).view(-1)
        close(got[i].float(), want * torch.sigmoid(gate[i].float()), 2e-5 if dtype == "f32" else 1.5e-2)


@pytest.mark.parametrize("form, dtype, device", FORMS)
@pytest.mark.parametrize("distance", [0, 15, 16, 17, 62, 63, 64, 65, 95, 96, 100, 255])
def test_one_key_stands_out_at_the_window_edge(distance, form, dtype, device):
    """The key that matches the query lies ``distance`` tokens back: its value must come out, and only if it is inside."""
    dt, dim, n, window = DT[dtype], 64, 256, 96
    k, v = rnd(n, 1, dim, seed=1, std=0.1), rnd(n, 1, dim, seed=2)
    mark = rnd(dim, seed=3)
    k[n - 1 - distance, 0] = mark
    k, v = k.to(dt), v.to(dt)
    pages = Paged([n], 1, dim, dim, 16, dt, device)
    pages.fill(0, k, v)
    q = (mark * 4).expand(1, 2, dim).contiguous().to(dt)
    got = _attend(form, q.to(device), pages, [(0, n)], 0.3, window, torch.zeros(2, device=device), None, dim, device, n).float().cpu().view(2, dim)
    close(got, O.attend(q.float(), k.float(), v.float(), 0.3, window)[0], 1e-5 if dtype == "f32" else 1.5e-2)
    there = v[n - 1 - distance, 0].float()
    assert (float((got[0] - there).norm() / there.norm()) < 0.1) == (distance < window)


@pytest.mark.parametrize("form, dtype, device", FORMS)
@pytest.mark.parametrize("score", [-40.0, -5.0, 0.0, 3.0])
def test_the_constant_in_the_denominator_counts_once(score, form, dtype, device):
    """n equal keys with one score: the output is n e^s / (1 + n e^s), however the work is split and however small e^s."""
    if dtype == "f16":
        score = max(score, -7.0)                             # what the output's type can still hold
    for n in (1, 300):
        k, v = torch.ones(n, 1, 64), torch.ones(n, 1, 64)
        pages = Paged([n], 1, 64, 64, 16, DT[dtype], device)
        pages.fill(0, k, v)
        q = torch.full((1, 3, 64), score / 16.0, dtype=DT[dtype], device=device)
        got = _attend(form, q, pages, [(0, n)], 0.25, 0, torch.zeros(3, device=device), None, 64, device, n)
        e = n * torch.exp(torch.tensor(float(q[0, 0, 0]) * 16.0))
        want = (e / (1 + e)).expand(3 * 64)
        rel = (got[0].float().cpu() - want).abs().max() / want[0]
        assert float(rel) < (1e-4 if dtype == "f32" else 1e-2)


@gpu
@pytest.mark.parametrize("H, G, dim", [(6, 2, 40), (4, 1, 64), (8, 2, 128), (3, 3, 96), (2, 1, 200)])
@pytest.mark.parametrize("window", [0, 1, 33, 128, 300])
def test_long_portions(H, G, dim, window):
    """Portions whose context lies partly in the cache, on the prefill kernels; a far key stands out for one query in
    every sequence."""
    dt = torch.bfloat16
    hd = next(h for h in (64, 128, 256) if dim <= h)
    spans = [(0, 64), (100, 70), (131, 300), (5, 128), (400, 65)]            # (tokens before, new tokens)
    lens = [a + n for a, n in spans]
    pages = Paged(lens, G, dim, hd, 16, dt, "cuda")
    ks, vs = [rnd(n, G, dim, seed=b).to(dt) for b, n in enumerate(lens)], [rnd(n, G, dim, seed=30 + b).to(dt) for b, n in enumerate(lens)]
    T = sum(n for _, n in spans)
    q = rnd(T, H, dim, seed=22).to(dt)
    gate = rnd(T, H * dim + 16, seed=23).to(dt)[:, 16:]
    at, scale = 0, 1.5 * dim ** -0.5
    for b, (a, n) in enumerate(spans):
        pages.fill(b, ks[b], vs[b])
        j = a + n // 2
        oldest = ks[b][max(0, j - max(window - 1, 0))]                       # [G, dim]
        q[at + n // 2] += 2.0 * oldest.repeat_interleave(H // G, 0)
        at += n
    qp = torch.zeros(T, H, hd, dtype=dt)
    qp[..., :dim] = q
    cu = torch.tensor([0] + [n for _, n in spans]).cumsum(0).to(torch.int32).cuda()
    got = ops.paged_attention_prefill(qp.cuda().view(T, -1), pages.k, pages.v, pages.table.cuda(), i32("cuda", *lens), cu, 300, H, G, hd,
                                      scale, window, sinks=torch.zeros(H, device="cuda"), v_dim=dim, gate=gate.cuda())
    at = 0
    for b, (a, n) in enumerate(spans):
        want = O.attend(q[at:at + n].float(), ks[b].float(), vs[b].float(), scale, window).view(n, -1)
        close(got[at:at + n].float(), want * torch.sigmoid(gate[at:at + n].float()), 2e-2)
        at += n
    ops.check_status(torch.device("cuda", 0))


@gpu
@pytest.mark.parametrize("n, window", [(600, 0), (4300, 0), (4300, 70), (9000, 4200)])
def test_few_rows_over_long_contexts(n, window):
    """One row split over many blocks, merged inside a cluster, by the last block or by the merge kernel; far keys stand
    out and the constant counts once."""
    H, G, dim = 4, 2, 64
    k, v = rnd(n, G, dim, seed=1, std=0.5).bfloat16(), rnd(n, G, dim, seed=2).bfloat16()
    pages = Paged([n], G, dim, dim, 16, torch.bfloat16, "cuda")
    pages.fill(0, k, v)
    first = max(0, n - window) if window else 0
    q = rnd(1, H, dim, seed=3, std=0.3).bfloat16()
    q[0, 0] += 2 * k[first, 0]
    q[0, 2] += 2 * k[max(0, first - 1), 1]
    got = _attend("decode", q.cuda(), pages, [(0, n)], 0.4, window, torch.zeros(H, device="cuda"), None, dim, "cuda", n)
    close(got[0].float(), O.attend(q.float(), k.float(), v.float(), 0.4, window).view(-1), 1.5e-2)


# ------------------------------------------------------------------ delta rule
class Delta:
    """Random operands of one layer and their plain evaluation, sequence by sequence."""

    def __init__(self, H, G, d, dv, taps, seed=0):
        self.H, self.G, self.d, self.dv, self.taps = H, G, d, dv, taps
        C = 2 * G * d + H * dv
        self.conv, self.A_log = rnd(C, taps, seed=seed + 1, std=0.7), rnd(H, seed=seed + 2) - 1.0
        self.bias = rnd(H * d, seed=seed + 3, std=2.5) - 3.0

    def spec(self, device):
        return lin.DeltaSpec(self.H, self.G, self.d, self.dv, self.conv.to(device), torch.exp(self.A_log).to(device), self.bias.to(device))

    def inputs(self, T, dtype, seed):
        return (rnd(T, self.conv.shape[0], seed=seed).to(dtype), rnd(T, self.H * self.d, seed=seed + 1), rnd(T, self.H, seed=seed + 2, std=2.0))

    def run(self, x, z, b):
        """Whole sequence from its start: (outputs, final state) in float64."""
        T, G, H, d, dv = x.shape[0], self.G, self.H, self.d, self.dv
        y = O.silu(O.short_conv(x.double(), self.conv.double()))
        q, k, v = y[:, :G * d].view(T, G, d), y[:, G * d:2 * G * d].view(T, G, d), y[:, 2 * G * d:].view(T, H, dv)
        g = O.decay(z.double(), self.A_log.double(), self.bias.double(), H)
        return O.delta_rule(O.unit(q) * d ** -0.5, O.unit(k), v, g, torch.sigmoid(b.double()), torch.zeros(H, d, dv).double())


HEADS = [(1, 1, 5, 7, 4), (3, 1, 12, 20, 3), (2, 2, 64, 48, 4), (4, 2, 72, 130, 2), (1, 1, 130, 66, 1), (1, 1, 300, 16, 5), (8, 8, 128, 128, 4),
         (40, 20, 32, 64, 4)]


def _portions(m, x, z, b, spec, pool, ring, slots, lens, done, device):
    d = lambda t: t.to(device)
    cu = torch.tensor([0] + lens).cumsum(0).to(torch.int32).to(device)
    return lin.delta_portions(d(x), d(z), d(b), spec, pool, ring, i32(device, *slots), cu, i32(device, *done), lin.delta_chunks(cu),
                              sum(-(-n // 16) for n in lens))


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("H, G, d, dv, taps", HEADS)
def test_portions_of_several_sequences(H, G, d, dv, taps, device):
    """Sequences of unequal length in one step, three times: the next portion starts from the state and the convolution
    inputs the one before left; portions shorter than the convolution included."""
    if device == "cpu" and H > 4:
        pytest.skip("large cases run on the kernels")
    m = Delta(H, G, d, dv, taps)
    parts = ([1, 2, 16, 33, 50], [17, 1, 2, 15, 4], [1, 3, 18, 1, 16])
    slots, n_slots = [4, 0, 6, 2, 5], 7
    pool, ring = torch.full((n_slots, H, d, dv), 3.0, device=device), torch.full((n_slots, taps, m.conv.shape[0]), 3.0, device=device)
    seqs = [m.inputs(sum(p[b] for p in parts), torch.float32, 10 * b) for b in range(5)]
    wants = [m.run(*s) for s in seqs]
    spec, done = m.spec(device), [0] * 5
    for lens in parts:
        rows = [tuple(t[done[b]:done[b] + n] for t in seqs[b]) for b, n in enumerate(lens)]
        before = list(done)
        done = [a + n for a, n in zip(done, lens)]
        o = _portions(m, *[torch.cat([r[i] for r in rows]) for i in range(3)], spec, pool, ring, slots, lens, done, device)
        at = 0
        for b, n in enumerate(lens):
            close(o[at:at + n], wants[b][0][before[b]:done[b]], 2e-5)
            at += n
    for b in range(5):
        close(pool[slots[b]], wants[b][1], 2e-5)
    for s in set(range(n_slots)) - set(slots):
        assert bool((pool[s] == 3.0).all()) and bool((ring[s] == 3.0).all())


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("H, G, d, dv, taps", HEADS)
def test_single_tokens_over_slots(H, G, d, dv, taps, dtype, device):
    """Every sequence token by token through the step form (a padded row beside them), then one more through the portion
    form: both forms leave the same state and ring."""
    if device == "cpu" and (H > 4 or dtype == "bf16"):
        pytest.skip("large cases run on the kernels")
    m, T, eps = Delta(H, G, d, dv, taps), 7, 1e-4
    slots = [3, 0, 5]
    pool, ring = torch.full((6, H, d, dv), 3.0, device=device), torch.full((6, taps, m.conv.shape[0]), 3.0, device=device)
    seqs = [m.inputs(T + 1, DT[dtype], 10 * b) for b in range(3)]
    wants = [m.run(*s) for s in seqs]
    spec, w, gate = m.spec(device), rnd(dv, seed=6), rnd(4, H * dv, seed=7)
    d_ = lambda t: t.to(device)
    for t in range(T):
        x, z, b = (torch.stack([s[i][t] for s in seqs] + [torch.full_like(seqs[0][i][0], 9.0)]) for i in range(3))
        out = lin.delta_step(d_(x), d_(z), d_(b), spec, pool, ring, i32(device, *slots, 1), i32(device, t + 1, t + 1, t + 1, 0), d_(w), eps,
                             d_(gate), torch.float32)
        for i in range(3):
            want = O.rms_norm(wants[i][0][t], w.double(), eps).reshape(-1) * torch.sigmoid(gate[i].double())
            close(out[i], want, 3e-5)
        assert float(out[3].abs().max()) == 0.0
    assert bool((pool[[1, 2, 4]] == 3.0).all()) and bool((ring[[1, 2, 4]] == 3.0).all())
    o = _portions(m, *[torch.cat([s[i][T:] for s in seqs]) for i in range(3)], spec, pool, ring, slots, [1] * 3, [T + 1] * 3, device)
    for i in range(3):
        close(o[i], wants[i][0][T], 2e-5)
        close(pool[slots[i]], wants[i][1], 2e-5)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("single", [False, True])
def test_a_far_write_survives_slow_decay(single, device):
    """One token writes a large value under its own key, hundreds of tokens with almost no decay and orthogonal keys
    follow; the last query asks for the first key."""
    T, d, dv = 600, 16, 8
    m = Delta(1, 1, d, dv, 1)
    m.conv = torch.ones_like(m.conv)
    m.A_log, m.bias = torch.tensor([-9.0]), torch.zeros(d)
    x = torch.full((T, 2 * d + dv), -20.0)                   # silu of it is nearly zero
    x[:, d + 1] = 5.0                                        # keys along channel 1 ..
    x[0, d:2 * d] = -20.0
    x[0, d] = 5.0                                            # .. the first along channel 0
    x[:, 0] = 5.0                                            # queries along channel 0
    x[:, 2 * d:] = rnd(T, dv, seed=1, std=0.1)
    x[0, 2 * d:] = 9.0
    z, b = torch.zeros(T, d), torch.full((T, 1), 8.0)
    want, S = m.run(x, z, b)
    spec = m.spec(device)
    pool, ring = torch.zeros(1, 1, d, dv, device=device), torch.zeros(1, 1, 2 * d + dv, device=device)
    if single:
        if device == "cpu":
            pytest.skip("the CPU forms share their recurrence")
        for t in range(T):
            o = lin.delta_step(x[t:t + 1].to(device), z[t:t + 1].to(device), b[t:t + 1].to(device), spec, pool, ring, i32(device, 0),
                               i32(device, t + 1), torch.ones(dv, device=device), 1e-6, None, torch.float32)
        close(o[0], O.rms_norm(want[-1], torch.ones(dv).double(), 1e-6).view(-1), 3e-5)
    else:
        o = _portions(m, x, z, b, spec, pool, ring, [0], [T], [T], device)
        close(o, want, 3e-5)
        assert float(o[-1].min()) > 0.8 * 9.0 * d ** -0.5    # nearly all of it is still there
    close(pool[0], S, 3e-5)


@pytest.mark.parametrize("device", DEV)
def test_decays_act_on_key_channels_and_may_vanish(device):
    """Channels that forget at once beside channels that never do, in one head: products of decays underflow to zero
    inside a chunk and nothing is divided by them."""
    T, d, dv = 40, 12, 6
    m = Delta(2, 1, d, dv, 2)
    m.A_log = torch.tensor([4.0, -8.0])
    m.bias = torch.where(torch.arange(2 * d) % 2 == 0, torch.tensor(60.0), torch.tensor(-60.0))
    x, z, b = m.inputs(T, torch.float32, 3)
    want, S = m.run(x, z, b)
    pool, ring = torch.zeros(1, 2, d, dv, device=device), torch.zeros(1, 2, m.conv.shape[0], device=device)
    o = _portions(m, x, z, b, m.spec(device), pool, ring, [0], [T], [T], device)
    assert bool(torch.isfinite(o).all())
    close(o, want, 2e-5)
    close(pool[0], S, 2e-5)


@gpu
@pytest.mark.parametrize("B, n", [(1, 2000), (9, 300), (24, 100)])
def test_every_column_width_of_the_scan(B, n):
    """Few and many sequences take scans with one, two or four columns per lane."""
    m = Delta(8, 4, 128, 128, 4)
    pool, ring = torch.zeros(B, 8, 128, 128, device="cuda"), torch.zeros(B, 4, m.conv.shape[0], device="cuda")
    x, z, b = m.inputs(n, torch.bfloat16, 5)
    # plain evaluation of a few heads would take minutes for all: compare with the recurrence of the CPU form
    o = _portions(m, x.repeat(B, 1), z.repeat(B, 1), b.repeat(B, 1), m.spec("cuda"), pool, ring, list(range(B)), [n] * B, [n] * B, "cuda")
    p0, r0 = torch.zeros(1, 8, 128, 128), torch.zeros(1, 4, m.conv.shape[0])
    want = _portions(m, x, z, b, m.spec("cpu"), p0, r0, [0], [n], [n], "cpu")
    for i in range(B):
        close(o[i * n:(i + 1) * n], want, 3e-5)
        close(pool[i], p0[0], 3e-5)
        close(ring[i], r0[0], 1e-7)
    ops.check_status(torch.device("cuda", 0))


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dv", [7, 64, 130, 512, 600])
@pytest.mark.parametrize("gate_type", ["f32", "bf16"])
def test_head_norm_with_gate(dv, gate_type, device):
    o, w = rnd(5, 3, dv, seed=1), rnd(dv, seed=2)
    gate = rnd(5, 3 * dv + 16, seed=3).to(DT[gate_type])[:, 16:]
    got = lin.head_norm(o.to(device), w.to(device), 1e-3, torch.float32, gate.to(device))
    close(got, O.rms_norm(o, w, 1e-3).reshape(5, 3 * dv) * torch.sigmoid(gate.float()), 2e-6)


# ------------------------------------------------------------------ experts
@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("E, top, groups, keep", [(8, 3, 4, 3), (6, 2, 3, 1), (9, 2, 3, 2), (64, 6, 8, 3), (12, 3, 12, 5), (160, 8, 8, 3), (5, 5, 1, 1),
                                                  (1, 1, 1, 1), (40, 4, 40, 7)])
def test_choice_of_experts(E, top, groups, keep, device):
    T = 50
    z, c = rnd(T, E + 3, seed=E, std=2.0), rnd(E, seed=E + 1) - 0.5          # sums of score and correction change sign
    ids, w = moe.route(z.to(device)[:, 3:], top, mode="sigmoid", bias=c.to(device), renormalize=False, routed_scale=1.7, groups=groups,
                       keep_groups=keep)
    for t in range(T):
        want, _ = O.choose(z[t, 3:], c, groups, keep, top, 1.7)
        got = dict(zip(ids[t].tolist(), w[t].tolist()))
        assert set(got) == set(want)
        for e, a in want.items():
            assert abs(got[e] - float(a)) < 1e-5


@pytest.mark.parametrize("device", DEV)
def test_groups_are_ranked_by_two_scores_and_dropped_entirely(device):
    """Group 0 holds the single best expert but a weak second one; groups 1 and 2 win.  All sums are negative, so a dropped
    expert that counted as zero would be chosen."""
    s = torch.sigmoid(torch.zeros(9))
    choice = torch.tensor([-0.1, -3.0, -3.0, -1.0, -1.1, -3.0, -1.2, -1.3, -1.4])
    ids, w = moe.route(torch.zeros(1, 9, device=device), 3, mode="sigmoid", bias=(choice - s).to(device), renormalize=False,
                       routed_scale=2.0, groups=3, keep_groups=2)
    assert sorted(ids[0].tolist()) == [3, 4, 6]
    close(w, torch.full((1, 3), 1.0), 1e-6)                                  # the score 1/2 times two: no correction in it


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("T, H, I, E, top", [(1, 33, 7, 5, 2), (9, 64, 40, 6, 3), (20, 72, 24, 4, 4), (130, 256, 96, 8, 2), (700, 128, 200, 3, 2),
                                             (40, 512, 264, 32, 4), (1500, 256, 136, 16, 1), (64, 40, 50, 1, 1)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_expert_products(T, H, I, E, top, dtype, device):
    """Every tile size of the grouped products and the general kernel; one expert gets most tokens, one gets none."""
    if device == "cpu" and T > 200:
        pytest.skip("large cases run on the kernels")
    dt = DT[dtype]
    x, w1, w2 = rnd(T, H, seed=1).to(dt), rnd(E, 2 * I, H, seed=2, std=H ** -0.5).to(dt), rnd(E, H, I, seed=3, std=I ** -0.5).to(dt)
    z = rnd(T, E, seed=4)
    z[:, 0] += 2.0
    if E > top:
        z[:, E - 1] = -50.0
    a, ids = torch.topk(z, top, dim=1)
    ids, a = ids.to(torch.int32), torch.sigmoid(a)
    got = moe.expert_rows(x.to(device), w1.to(device), w2.to(device), ids.to(device), a.to(device))
    got = moe.RoutedRows(got.rows.clone(), got.weights, None if got.slot_of is None else got.slot_of.clone()).combined()
    f = x.float()
    every = torch.stack([(O.silu(f @ w1[e, :I].float().t()) * (f @ w1[e, I:].float().t())) @ w2[e].float().t() for e in range(E)], dim=1)
    want = (torch.gather(every, 1, ids.long()[..., None].expand(T, top, H)) * a[..., None]).sum(1)
    close(got, want, 1e-5 if dtype == "f32" else 1.5e-2)
    if device == "cuda":
        ops.check_status(torch.device("cuda", 0))
