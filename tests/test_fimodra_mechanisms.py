"""Mechanisms of the Fimodra design one by one: the op layer (CPU forms and, marked gpu, the kernels) against the plain
functions in ``fimodra_oracle.py``.  Inputs are planted so that a key, an edge or a state that is missed shows."""
import pytest
import torch

import fimodra_oracle as O
from litevllm_b200 import ops
from litevllm_b200.layers.rope import get_cos_sin
from litevllm_b200.ops import latent_attn as la
from litevllm_b200.ops import linear_attn as lin
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


# ------------------------------------------------------------------ residual stream
SHAPES = [(1, 24, 3), (5, 33, 1), (3, 96, 4), (40, 320, 5), (7, 1536, 1), (2, 4104, 2), (3, 9000, 3), (2100, 512, 2),
          (2100, 1000, 1), (1100, 1600, 2), (1, 8192, 1), (3, 2049, 1)]


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("T, W, groups", SHAPES)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_stream_boundaries(T, W, groups, dtype, device):
    dt, eps, tol = DT[dtype], 1e-5, 2e-6 if dtype == "f32" else 6e-3
    y = rnd(T, W, seed=1, std=3.0).to(dt)
    x, wa, wb = rnd(T, W, seed=2), rnd(W, seed=3), rnd(W, seed=4)
    hist, avg = rnd(5, T, W, seed=5), rnd(4, seed=6)
    d = lambda t: t.to(device)
    xn = x + O.grouped_rms_norm(y.float(), wa, eps, groups)
    out = torch.empty(T, W, device=device)
    h = stream.step(d(y), d(x), d(wa), d(wb), eps, groups, out, dt)
    close(out, xn, 2e-6)
    close(h.float(), O.grouped_rms_norm(xn, wb, eps, groups), tol)
    same = d(x).clone()                                     # the sum may replace its input; the next norm is optional
    assert stream.step(d(y), same, d(wa), None, eps, groups, same, dt) is None
    close(same, xn, 2e-6)
    hd = d(hist).clone()
    h = stream.average(d(y), d(x), d(wa), d(wb), eps, groups, hd, 3, d(avg), out, dt)
    want = O.depth_average(list(hist[:3]) + [xn], avg)
    close(hd[3], xn, 2e-6)
    assert torch.equal(hd[4].cpu(), hist[4])
    close(out, want, 4e-6)
    close(h.float(), O.grouped_rms_norm(want, wb, eps, groups), tol)
    sel = torch.tensor([T - 1, 0, T // 2])
    h = stream.average(d(y), d(x), d(wa), d(wb), eps, groups, hd, 3, d(avg), None, dt, sel=d(sel))
    close(h.float(), O.grouped_rms_norm(want, wb, eps, groups)[sel], tol)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("W, groups", [(33, 3), (128, 1), (640, 5)])
def test_stream_start(W, groups, device):
    table, w = rnd(11, W, seed=1).bfloat16(), rnd(W, seed=2)
    ids = torch.tensor([10, 0, 3, 3])
    x0 = torch.empty(4, W, device=device)
    h = stream.start(ids.to(device), table.to(device), w.to(device), 1e-6, groups, x0)
    assert torch.equal(x0.cpu(), table.float()[ids])
    close(h.float(), O.grouped_rms_norm(table.float()[ids], w, 1e-6, groups), 6e-3)


def test_eps_stands_inside_the_root_and_groups_are_separate():
    x = torch.zeros(1, 8)
    x[0, :4] = 1e-3
    want = torch.tensor([[1e-3 / (1e-6 + 1e-6) ** 0.5] * 4 + [0.0] * 4])
    close(stream.grouped_rmsnorm(x, torch.ones(8), 1e-6, 2), want, 1e-6)
    close(O.grouped_rms_norm(x, torch.ones(8), 1e-6, 2), want, 1e-6)


# ------------------------------------------------------------------ products
@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("T, K, I", [(1, 64, 48), (3, 33, 21), (20, 72, 136), (70, 128, 200), (130, 320, 96), (1500, 256, 264)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_gated_product_with_biases(T, K, I, dtype, device):
    dt, tol = DT[dtype], 1e-5 if dtype == "f32" else 1.5e-2
    x, w, b = rnd(T, K, seed=1).to(dt), rnd(2 * I, K, seed=2, std=K ** -0.5).to(dt), rnd(2 * I, seed=3).to(dt)
    got = ops.gated_linear(x.to(device), w.to(device), "relu", bias=b.to(device))
    z = x.float() @ w.float().t() + b.float()
    close(got.float(), torch.relu(z[:, :I]) * z[:, I:], tol)


@gpu
@pytest.mark.parametrize("splits", [1, 2, 4])
def test_gated_product_bias_with_split_k(splits):
    x, w, b = rnd(8, 512, seed=1).bfloat16(), rnd(2 * 128, 512, seed=2, std=0.05).bfloat16(), rnd(256, seed=3).bfloat16()
    got = ops.gated_linear(x.cuda(), w.cuda(), "relu", bias=b.cuda(), splits=splits)
    z = x.float() @ w.float().t() + b.float()
    close(got.float(), torch.relu(z[:, :128]) * z[:, 128:], 1.5e-2)


@gpu
@pytest.mark.parametrize("T, N, K", [(1024, 256, 128), (1300, 136, 72), (2048, 128, 640)])
def test_32_bit_output_of_prefill_products(T, N, K):
    x, w, b = rnd(T, K, seed=1).bfloat16(), rnd(N, K, seed=2).bfloat16(), rnd(N, seed=3).bfloat16()
    got = ops.linear(x.cuda(), w.cuda(), b.cuda(), out_dtype=torch.float32)
    assert got.dtype == torch.float32
    close(got, x.float() @ w.float().t() + b.float(), 2e-6)


# ------------------------------------------------------------------ latent attention
class Paged:
    """Cache rows of several sequences in shuffled pages of one pool."""

    def __init__(self, lens, kd, bs, dtype, device, seed=0):
        self.bs, self.kd = bs, kd
        per = [(n + bs - 1) // bs for n in lens]
        order = torch.randperm(sum(per), generator=torch.Generator().manual_seed(seed)) + 1
        self.table = torch.zeros(len(lens), max(per), dtype=torch.int32)
        at = 0
        for b, n in enumerate(per):
            self.table[b, :n] = order[at:at + n].to(torch.int32)
            at += n
        self.cache = torch.full((sum(per) + 1, 1, bs, kd), 7.0, dtype=dtype, device=device)   # unused rows hold rubbish

    def slot(self, b, pos):
        return self.table[b].long()[pos // self.bs] * self.bs + pos % self.bs

    def fill(self, b, rows):
        self.cache.view(-1, self.kd)[self.slot(b, torch.arange(len(rows))).to(self.cache.device)] = rows.to(self.cache)


GEOMETRY = [(3, 24, 8, 16), (1, 9, 2, 5), (16, 64, 16, 32), (17, 136, 24, 16), (4, 512, 64, 16), (2, 520, 64, 16), (5, 40, 64, 64)]


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16", "f16"])
@pytest.mark.parametrize("nh, rank, rot, bs", GEOMETRY)
@pytest.mark.parametrize("window", [0, 1, 17, 64, 200])
def test_rows_against_cached_latents(nh, rank, rot, bs, window, dtype, device):
    if device == "cpu" and (dtype == "f16" or rank > 200):
        pytest.skip("the CPU form is one code for all types and sizes")
    dt, kd = DT[dtype], rank + rot
    lens = [1, bs, bs + 1, 130, 260]
    rows = [(b, n) for b, n in enumerate(lens)] + [(4, 64), (4, 65), (3, 1), (4, 129)]
    pages = Paged(lens, kd, bs, dt, device)
    data = [rnd(n, kd, seed=b).to(dt) for b, n in enumerate(lens)]
    for b, r in enumerate(data):
        pages.fill(b, r)
    q = rnd(len(rows), nh, kd, seed=9).to(dt)
    sink = rnd(nh, seed=10) * 2
    scale = 1.5 * kd ** -0.5
    got = la.attend_rows(q.to(device), pages.cache, pages.table.to(device),
                         torch.tensor([n for _, n in rows], dtype=torch.int32, device=device),
                         torch.tensor([b for b, _ in rows], dtype=torch.int32, device=device), rank, scale, window,
                         sink.to(device), max(lens))
    for i, (b, n) in enumerate(rows):
        k = data[b][:n].float()[:, None].expand(n, nh, kd)
        want = O.sink_attention(q[i:i + 1].float(), k, k[..., :rank], scale, window, sink)[0]
        close(got[:, i].float(), want, 2e-5 if dtype == "f32" else 1.5e-2)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("distance", [0, 15, 16, 17, 62, 63, 64, 65, 95, 96, 100, 255])
def test_one_key_stands_out_at_the_window_edge(distance, dtype, device):
    """The key that matches the query lies ``distance`` tokens back: its value must come out, and only if it is inside."""
    dt, rank, rot, n, window = DT[dtype], 32, 16, 256, 96
    kd = rank + rot
    rows = rnd(n, kd, seed=1, std=0.1)
    mark = rnd(kd, seed=2)
    rows[n - 1 - distance] = mark
    pages = Paged([n], kd, 16, dt, device)
    pages.fill(0, rows)
    q = (mark * 4).expand(1, 2, kd).contiguous().to(dt)
    sink = torch.tensor([-3.0, 2.0])
    got = la.attend_rows(q.to(device), pages.cache, pages.table.to(device), torch.tensor([n], dtype=torch.int32, device=device),
                         None, rank, 0.3, window, sink.to(device), n)[:, 0].float().cpu()
    k = rows.to(dt).float()[:, None].expand(n, 2, kd)
    close(got, O.sink_attention(q.float(), k, k[..., :rank], 0.3, window, sink)[0], 1e-5 if dtype == "f32" else 1.5e-2)
    seen = float((got[0] - mark[:rank]).norm() / mark[:rank].norm()) < 0.1
    assert seen == (distance < window)


@pytest.mark.parametrize("device", DEV)
def test_the_sink_takes_weight_and_counts_once(device):
    """One visible key with score s: its weight is exp(s) / (exp(s) + exp(sink)), however the work is split."""
    kd, rank = 24, 16
    for n in (1, 300):
        rows = torch.zeros(n, kd)
        rows[:, :rank] = 1.0                       # equal keys and values: the output is 1 minus the sink's share
        pages = Paged([n], kd, 16, torch.float32, device)
        pages.fill(0, rows)
        q = torch.full((1, 3, kd), 0.25)
        sink = torch.tensor([-100.0, 4.0, 40.0])
        got = la.attend_rows(q.to(device), pages.cache, pages.table.to(device), torch.tensor([n], dtype=torch.int32, device=device),
                             None, rank, 0.5, 0, sink.to(device), n)[:, 0, 0].cpu()
        e = n * torch.exp(torch.tensor(0.25 * rank * 0.5))
        close(got, e / (e + torch.exp(sink)), 1e-5)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("nh, dim, rot, rank, dims", [(3, 24, 8, 40, 8), (1, 3, 2, 9, 2), (5, 16, 12, 24, 6), (40, 32, 32, 512, 32)])
def test_cache_rows_and_rotated_queries(nh, dim, rot, rank, dims, dtype, device):
    dt, T, kd = DT[dtype], 9, rank + rot
    base, eps = 700.0, 1e-4
    proj = rnd(T, nh * (dim + rot) + kd, seed=1).to(dt)
    pos = torch.tensor([0, 1, 2, 50, 51, 300, 7, 8, 9], dtype=torch.int32)
    slots = torch.tensor([3, 40, 5, -1, 9, 31, 17, 0, 2], dtype=torch.int32)
    w = rnd(rank, seed=2)
    cache = torch.zeros(3, 1, 16, kd, dtype=dt, device=device)
    q, d = proj[:, :nh * (dim + rot)], proj[:, nh * (dim + rot):]
    out = torch.full((T, nh, dim + rot + 6), 5.0, dtype=dt, device=device)
    dev = lambda t: t.to(device)
    pd = dev(proj)
    la.prepare(pd[:, :nh * (dim + rot)], pd[:, nh * (dim + rot):], dev(w), eps, dev(pos), get_cos_sin(dims, 512, base, None, torch.device(device)),
               dev(slots), cache, out, nh, dim, rot, rank, 0, dim)
    tol = 1e-5 if dtype == "f32" else 1e-2
    qh = q.float().view(T, nh, dim + rot)
    turned = O.rotate_interleaved(qh[..., dim:].transpose(0, 1), pos, dims, base).transpose(0, 1)
    close(out[..., :dim].float(), qh[..., :dim], 1e-7)
    close(out[..., dim:dim + rot].float(), turned, tol)
    assert float(out[..., dim + rot:].abs().max()) == 0.0
    rows = torch.cat([O.rms_norm(d[:, :rank].float(), w, eps), O.rotate_interleaved(d[:, rank:].float(), pos, dims, base)], dim=1)
    flat = cache.view(-1, kd).float().cpu()
    for t in range(T):
        if slots[t] >= 0:
            close(flat[slots[t]], rows[t], tol)
    untouched = [i for i in range(48) if i not in slots.tolist()]
    assert float(flat[untouched].abs().max()) == 0.0


@gpu
@pytest.mark.parametrize("nh, dim, rot, vdim, rank", [(3, 24, 8, 40, 56), (2, 48, 16, 64, 128), (4, 96, 32, 128, 64), (2, 12, 4, 6, 20),
                                                      (2, 128, 64, 128, 96), (1, 200, 56, 250, 64)])
@pytest.mark.parametrize("window", [0, 1, 33, 128, 300])
def test_long_portions(nh, dim, rot, vdim, rank, window):
    """Portions whose context lies partly in the cache: gathered, up-projected and run by the prefill kernels; a far key
    stands out for one query in every sequence."""
    kd, dt = rank + rot, torch.bfloat16
    spans = [(0, 64), (100, 70), (131, 300), (5, 128), (400, 65)]            # (tokens before, new tokens)
    lens = [a + n for a, n in spans]
    pages = Paged(lens, kd, 16, dt, "cuda")
    data = [rnd(n, kd, seed=b, std=0.5).to(dt) for b, n in enumerate(lens)]
    w_uk, w_uv = rnd(nh * dim, rank, seed=20, std=rank ** -0.5).to(dt), rnd(nh * vdim, rank, seed=21, std=rank ** -0.5).to(dt)
    q = rnd(sum(n for _, n in spans), nh, dim + rot, seed=22).to(dt)
    sink, scale = rnd(nh, seed=23), 2.0 * (dim + rot) ** -0.5
    keys, values = [], []
    for r in data:
        c = r[:, :rank].float()
        keys.append(torch.cat([(c @ w_uk.float().t()).view(-1, nh, dim), r[:, None, rank:].float().expand(-1, nh, rot)], dim=-1).to(dt))
        values.append((c @ w_uv.float().t()).view(-1, nh, vdim).to(dt))
    at = 0
    for b, (a, n) in enumerate(spans):
        j = a + n // 2
        q[at + n // 2] = q[at + n // 2] + 3.0 * keys[b][max(0, j - max(window - 1, 0))]      # the oldest visible key
        at += n
        pages.fill(b, data[b])
    hd = next(h for h in (64, 128, 256) if max(dim + rot, vdim) <= h)
    plan = la.ContextPlan(pages.table.cuda(), 16, lens, [n for _, n in spans], window, torch.device("cuda"))
    k_pool, v_pool = la.context_pool(plan, pages.cache, torch.cat([w_uk, w_uv]).cuda(), nh, dim, rot, vdim, rank, hd)
    qp = torch.zeros(q.shape[0], nh, hd, dtype=dt)
    qp[..., :dim + rot] = q
    cu = torch.tensor([0] + [n for _, n in spans]).cumsum(0).to(torch.int32).cuda()
    got = ops.paged_attention_prefill(qp.cuda().view(-1, nh * hd), k_pool, v_pool, plan.table, plan.lens, cu, 300, nh, nh, hd, scale,
                                      window, sinks=sink.cuda(), v_dim=vdim).view(-1, nh, vdim)
    at = 0
    for b, (a, n) in enumerate(spans):
        want = O.sink_attention(q[at:at + n].float(), keys[b].float(), values[b].float(), scale, window, sink)
        close(got[at:at + n].float(), want, 2e-2)
        at += n
    ops.check_status(torch.device("cuda", 0))


# ------------------------------------------------------------------ HGRN2
def _hgrn2_case(H, d, dv, T, dtype, seed=0):
    g = [rnd(T, H * d, seed=seed + 1), rnd(T, H * d, seed=seed + 2), rnd(T, H * dv, seed=seed + 3)]
    q, f, v = (t.to(dtype) for t in g)
    bias, lower = rnd(H * d, seed=90, std=4.0) + 2.0, torch.rand(H * d, generator=torch.Generator().manual_seed(91)) * 0.9
    lower[::3] = 0.0
    qa = (q.float() * torch.sigmoid(q.float())).view(T, H, d)
    fa = (lower + (1 - lower) * torch.sigmoid(f.float() + bias)).view(T, H, d)
    return q, f, v, bias, lower, qa, fa, v.float().view(T, H, dv)


HEADS = [(1, 5, 7), (3, 12, 20), (2, 64, 48), (2, 72, 130), (1, 130, 66), (1, 300, 16), (16, 128, 128), (80, 32, 64)]


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("H, d, dv", HEADS)
def test_scan_over_portions(H, d, dv, device):
    """Sequences of unequal length in one step, twice: the second portion starts from the state the first one left."""
    if device == "cpu" and H > 3:
        pytest.skip("large cases run on the kernels")
    first, second = [1, 2, 16, 33, 100], [17, 1, 50, 15, 4]
    slots, n_slots = [4, 0, 6, 2, 5], 7
    pool = torch.full((n_slots, H, d, dv), 3.0, device=device)              # what an earlier request left behind
    state, done = {}, {b: 0 for b in range(5)}
    for part, lens in enumerate((first, second)):
        q, f, v, bias, lower, qa, fa, va = _hgrn2_case(H, d, dv, sum(lens), torch.float32, seed=10 * part)
        cu = torch.tensor([0] + lens).cumsum(0).to(torch.int32)
        for b, n in enumerate(lens):
            done[b] += n
        dev = lambda t: t.to(device)
        o = lin.hgrn2_scan(dev(q), dev(f), dev(v), dev(bias), dev(lower), pool, dev(torch.tensor(slots, dtype=torch.int32)),
                           dev(cu), dev(torch.tensor([done[b] for b in range(5)], dtype=torch.int32)), H, d, dv)
        for b in range(5):
            a, e = int(cu[b]), int(cu[b + 1])
            want, state[b] = O.outer_product_recurrence(qa[a:e], fa[a:e], va[a:e], state.get(b, torch.zeros(H, d, dv)))
            close(o[a:e], want, 2e-5)
            close(pool[slots[b]], state[b], 2e-5)
    for s in set(range(n_slots)) - set(slots):
        assert bool((pool[s] == 3.0).all())


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("H, d, dv", HEADS[:7])
def test_step_over_slots(H, d, dv, dtype, device):
    dt, eps = DT[dtype], 1e-4
    slots, lens = [3, 0, 5, 1, 0], [8, 1, 2, 40, 0]                        # position 0 starts fresh; the last row is padding
    pool0 = rnd(6, H, d, dv, seed=5)
    q, f, v, bias, lower, qa, fa, va = _hgrn2_case(H, d, dv, 5, torch.float32)
    w = rnd(dv, seed=6)
    pool = pool0.clone().to(device)
    dev = lambda t: t.to(device)
    out = lin.hgrn2_step(dev(q), dev(f), dev(v), dev(bias), dev(lower), pool, dev(torch.tensor(slots, dtype=torch.int32)),
                         dev(torch.tensor(lens, dtype=torch.int32)), dev(w), eps, H, d, dv, dt).float().view(5, H, dv)
    for b in range(4):
        S = torch.zeros(H, d, dv) if lens[b] == 1 else pool0[slots[b]]
        o, S = O.outer_product_recurrence(qa[b:b + 1], fa[b:b + 1], va[b:b + 1], S)
        close(out[b], O.rms_norm(o[0], w, eps), 2e-5 if dtype == "f32" else 1e-2)
        close(pool[slots[b]], S, 1e-5)
    assert float(out[4].abs().max()) == 0.0
    assert torch.equal(pool[[2, 4]].cpu(), pool0[[2, 4]])


@pytest.mark.parametrize("device", DEV)
def test_a_far_write_survives_slow_forgetting(device):
    """One token writes strongly through an open gate, hundreds of nearly closed gates follow: the value is still read."""
    H, d, dv, T = 1, 16, 8, 400
    q, f, v = torch.full((T, d), 3.0), torch.full((T, d), 12.0), rnd(T, dv, seed=1, std=0.1)
    f[0] = -12.0
    v[0] = 5.0
    zero = torch.zeros(d)
    pool = torch.zeros(1, H, d, dv, device=device)
    dev = lambda t: t.to(device)
    i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device=device)
    o = lin.hgrn2_scan(dev(q), dev(f), dev(v), dev(zero), dev(zero), pool, i32(0), i32(0, T), i32(T), H, d, dv)
    qa, fa = (q * torch.sigmoid(q)).double().view(T, H, d), torch.sigmoid(f.double()).view(T, H, d)
    want, _ = O.outer_product_recurrence(qa, fa, v.double().view(T, H, dv), torch.zeros(H, d, dv).double())
    close(o, want, 3e-5)
    assert float(o[-1].min()) > 0.9 * 5.0 * d * float(qa[0, 0, 0])


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dv", [7, 64, 130, 512, 600])
def test_head_norm(dv, device):
    o, w = rnd(5, 3, dv, seed=1), rnd(dv, seed=2)
    close(lin.head_norm(o.to(device), w.to(device), 1e-3, torch.float32), O.rms_norm(o, w, 1e-3).reshape(5, 3 * dv), 2e-6)


@gpu
@pytest.mark.parametrize("H, d, dv", [(4, 128, 128), (3, 24, 40)])
def test_scan_of_16_bit_projections(H, d, dv):
    """q and v as 16-bit columns of one product, the gate as 32-bit values of another."""
    T = 70
    q, f, v, bias, lower, qa, _, va = _hgrn2_case(H, d, dv, T, torch.bfloat16)
    f = rnd(T, H * d, seed=7)
    fa = (lower + (1 - lower) * torch.sigmoid(f + bias)).view(T, H, d)
    qv = torch.cat([q, v], dim=1).cuda()
    pool = torch.zeros(2, H, d, dv, device="cuda")
    i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device="cuda")
    o = lin.hgrn2_scan(qv[:, :H * d], f.cuda(), qv[:, H * d:], bias.cuda(), lower.cuda(), pool, i32(1), i32(0, T), i32(T), H, d, dv)
    want, S = O.outer_product_recurrence(qa, fa, va, torch.zeros(H, d, dv))
    close(o, want, 2e-5)
    close(pool[1], S, 2e-5)


@gpu
@pytest.mark.parametrize("n, window", [(600, 0), (4300, 0), (4300, 70), (9000, 4200)])
def test_few_rows_over_long_contexts(n, window):
    """One row split over many blocks, merged inside a cluster or by the merge kernel; far keys stand out."""
    nh, rank, rot = 3, 128, 16
    kd = rank + rot
    rows = rnd(n, kd, seed=1, std=0.3).bfloat16()
    pages = Paged([n], kd, 16, torch.bfloat16, "cuda")
    pages.fill(0, rows)
    first = max(0, n - window) if window else 0
    q = rnd(1, nh, kd, seed=2, std=0.3).bfloat16()
    q[0, 0] += 2 * rows[first]
    q[0, 1] += 2 * rows[max(0, first - 1)]
    sink = torch.tensor([1.0, 0.0, 3.0])
    got = la.attend_rows(q.cuda(), pages.cache, pages.table.cuda(), torch.tensor([n], dtype=torch.int32, device="cuda"), None, rank, 0.4,
                         window, sink.cuda(), n)[:, 0]
    k = rows.float()[:, None].expand(n, nh, kd)
    close(got.float(), O.sink_attention(q.float(), k, k[..., :rank], 0.4, window, sink)[0], 1.5e-2)
