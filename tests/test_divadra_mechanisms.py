"""Mechanisms of the Divadra design one by one: the op layer (CPU forms and, marked gpu, the kernels) against the plain
functions in ``divadra_oracle.py``.  Inputs are planted so that a key, an edge, a lost input or a lost state shows."""
from types import SimpleNamespace

import pytest
import torch

import divadra_oracle as O
from litevllm_b200 import ops
from litevllm_b200.layers.fused_moe.routed_experts import AssignedExperts
from litevllm_b200.layers.rope import get_cos_sin
from litevllm_b200.ops import linear_attn as lin
from litevllm_b200.ops import moe, qk_attn
from litevllm_b200.ops import shift_stream as stream

gpu = pytest.mark.gpu
DEV = ["cpu", pytest.param("cuda", marks=gpu)]
DT = {"f32": torch.float32, "bf16": torch.bfloat16, "f16": torch.float16}


def rnd(*shape, seed=0, std=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * std


def close(got, want, tol):
    got, want = got.detach().double().cpu(), want.double()
    assert got.shape == want.shape
    err = float((got - want).abs().max()) / max(1.0, float(want.abs().max()))
    assert err < tol, err


def i32(device, *x):
    return torch.tensor(x, dtype=torch.int32, device=device)


def make_batch(device, slots, lens, done, decode=False):
    """A step of ``lens[i]`` new tokens for the sequence in slot ``slots[i]``, which has ``done[i]`` tokens behind it."""
    cu = [sum(lens[:i]) for i in range(len(lens) + 1)]
    return SimpleNamespace(is_decode=decode, q_lens_cpu=list(lens), seq_lens=i32(device, *(a + b for a, b in zip(lens, done))),
                           cu_q=None if decode else i32(device, *cu), extras={"slot_ids": i32(device, *slots)})


def steps(total, sizes):
    """Portions of unequal sequences: (sequence, first, end) lists per step; single tokens are decode steps."""
    at, out, i = [0] * len(total), [], 0
    while any(a < n for a, n in zip(at, total)):
        n = sizes[i % len(sizes)]
        live = [s for s in range(len(total)) if at[s] < total[s]]
        out.append([(s, at[s], min(total[s], at[s] + n)) for s in live])
        for s in live:
            at[s] = min(total[s], at[s] + n)
        i += 1
    return out


def run_steps(device, total, sizes, slots, fn):
    """Feeds the sequences step by step; ``fn(batch, pieces)`` returns a list of [rows, ..] tensors, gathered per sequence."""
    got = [[] for _ in total]
    for pieces in steps(total, sizes):
        lens = [e - a for _, a, e in pieces]
        decode = all(n == 1 for n in lens)
        out = fn(make_batch(device, [slots[s] for s, _, _ in pieces], lens, [a for _, a, _ in pieces], decode), pieces)
        lo = 0
        for (s, _, _), n in zip(pieces, lens):
            got[s].append([t[lo:lo + n].detach().float().cpu() for t in out])
            lo += n
    return [[torch.cat(parts) for parts in zip(*g)] for g in got]


def cat_rows(device, seqs, pieces):
    return torch.cat([seqs[s][a:e] for s, a, e in pieces]).to(device)


# ------------------------------------------------------------------ stream, input convolutions, blends
SHIFT = [(24, 4, True, True), (33, 3, True, True), (160, 1, True, True), (640, 2, False, True), (1536, 4, True, False), (2052, 5, True, True),
         (3000, 8, True, True), (4104, 3, True, False), (8192, 4, True, True), (72, 9, True, True), (40, 16, True, True)]


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("W, taps, second, blends", SHIFT)
def test_inputs_of_a_layer(W, taps, second, blends, dtype, device):
    """Unequal sequences in portions of 1 to 40 tokens and single tokens; slots hold rubbish before a sequence starts."""
    dt, eps, tol = DT[dtype], 1e-2, 3e-6 if dtype == "f32" else 8e-3
    d = lambda t: t.to(device)
    total, slots = [45, 3, 70, 1], [2, 5, 0, 3]
    w1, w2, c1, c2, mu = rnd(W, seed=1), rnd(W, seed=2), rnd(W, taps, seed=3), rnd(W, taps, seed=4), rnd(5, W, seed=5)
    spec = stream.ShiftSpec(d(stream.fold_taps(w1, c1)), d(stream.fold_taps(w2, c2)) if second else None, d(mu) if blends else None)
    xs, ys, fs = ([rnd(n, W, seed=s + 10 * i, std=sd).to(t).float() for s, n in enumerate(total)]
                  for i, (sd, t) in enumerate(((20.0, torch.float32), (3.0, dt), (5.0, dt)), 1))
    ring = d(rnd(7, taps + 1, W, seed=9, std=50.0))

    def fn(batch, pieces):
        x = cat_rows(device, xs, pieces)
        out = stream.layer_inputs(stream.Summed(cat_rows(device, ys, pieces).to(dt), cat_rows(device, fs, pieces).to(dt)), x, spec, ring,
                                  batch, eps, dt)
        assert out.shape[0] == spec.outputs
        return [x, *out]
    for sizes in ([40, 1, 1, 7], [1], [2, 3]):
        got = run_steps(device, total, sizes, slots, fn)
        for s in range(len(total)):
            v = xs[s] + ys[s] + fs[s]
            close(got[s][0], v, 2e-6)
            want = [O.sublayer_input(v, w1, c1, eps)] + ([O.sublayer_input(v, w2, c2, eps)] if second else [])
            if blends:
                before = torch.cat([torch.zeros(1, W), want[0][:-1]])
                want += [want[0] + (before - want[0]) * m for m in mu]
            for a, b in zip(got[s][1:], want, strict=True):
                close(a, b, tol)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("W, top", [(24, 2), (33, 0), (320, 3), (1100, 1), (2048, 8), (4096, 2)])
def test_two_normed_outputs_and_experts_join_the_stream(W, top, dtype, device):
    dt, eps, T = DT[dtype], 0.3, 11
    d = lambda t: t.to(device)
    x, y, y2 = rnd(T, W, seed=1, std=4.0), rnd(T, W, seed=2, std=0.5).to(dt), rnd(T, W, seed=3, std=40.0).to(dt)
    w, w2, wf = rnd(W, seed=4), rnd(W, seed=5), rnd(W, seed=6)
    want = x + O.rms(y.float(), eps) * w + O.rms(y2.float(), eps) * w2
    routed = None
    if top:
        rows, a = rnd(T * top, W, seed=7).to(dt), rnd(T, top, seed=8)
        order = torch.randperm(T * top, generator=torch.Generator().manual_seed(6)).to(torch.int32).view(T, top)
        want = want + (rows.float()[order.long().view(-1)].view(T, top, W) * a[..., None]).sum(1)
        routed = moe.RoutedRows(d(rows), d(a), d(order))
        if top == 2:                                        # one weight for all choices
            want = want - (rows.float()[order.long().view(-1)].view(T, top, W) * (a[..., None] - 0.5)).sum(1)
            routed = moe.RoutedRows(d(rows), 0.5, d(order))
    src = stream.Paired(d(y), d(w), d(y2), d(w2), None, routed)
    buf, tol = d(x).clone(), 3e-6 if dtype == "f32" else 6e-3
    h = stream.normed(src, buf, d(wf), None, eps, dt, keep=True)
    close(buf, want, 3e-6)
    close(h.float(), O.rms(want, eps) * wf, tol)
    sel = torch.tensor([T - 1, 0, 4, 4])
    buf = d(x).clone()
    h = stream.normed(src, buf, d(wf), None, eps, dt, d(sel))
    close(h.float(), (O.rms(want, eps) * wf)[sel], tol)
    close(buf, x, 1e-9)                                     # rows are picked, the stream stays as it was
    spec = stream.ShiftSpec(d(rnd(3, W, seed=9)), None, d(rnd(5, W, seed=10)))
    ring = torch.zeros(T, 4, W, device=device)
    for decode in (False, True):
        buf = d(x).clone()
        stream.layer_inputs(src, buf, spec, ring, make_batch(device, list(range(T)), [1] * T, [0] * T, decode), eps, dt)
        close(buf, want, 3e-6)


@pytest.mark.parametrize("device", DEV)
def test_many_rows_and_padded_rows(device):
    """Steps of thousands of tokens take other launch shapes; padded rows of a decode bucket touch nothing."""
    W, eps = 264, 1e-5
    w1, c1 = rnd(W, seed=1), rnd(W, 4, seed=2)
    spec = stream.ShiftSpec(stream.fold_taps(w1, c1).to(device))
    ring, v = torch.zeros(3, 5, W, device=device), rnd(4500, W, seed=3)
    lens, lo = [4100, 1, 399], 0
    x = v.to(device).clone()
    zero = torch.zeros_like(x)
    out = stream.layer_inputs(stream.Summed(zero), x, spec, ring, make_batch(device, [1, 2, 0], lens, [0, 0, 0]), eps, torch.float32)
    for n in lens:
        close(out[0, lo:lo + n], O.sublayer_input(v[lo:lo + n], w1, c1, eps), 3e-6)
        lo += n
    before = ring.clone()
    b = make_batch(device, [0, 0, 0], [1, 1, 1], [399, -1, -1], True)
    out = stream.layer_inputs(stream.Summed(zero[:3]), x[:3].clone(), spec, ring, b, eps, torch.float32)
    close(out[0, :1], O.sublayer_input(torch.cat([v[-399:], v[:1]]), w1, c1, eps)[-1:], 3e-6)
    assert float(out[0, 1:].abs().max()) == 0.0
    assert torch.equal(ring[1:], before[1:]) and torch.equal(ring[0, :4], before[0, :4])       # position 399 is row 4 of 5


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("W, buckets, mul", [(24, 7, (3, 5)), (33, 1, (2, 2)), (320, 4093, (113, 19)), (1500, 50, (1 << 33, 1000003))])
def test_pairs_of_tokens_start_the_stream(W, buckets, mul, dtype, device):
    dt, eps, V = DT[dtype], 0.2, 29
    table, pairs, w = rnd(V, W, seed=1).to(dt), rnd(buckets + 1, W, seed=2).to(dt), rnd(W, seed=3)
    pairs[-1] += 3.0
    cfg = {"norm": {"eps": eps}, "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul[0], "mul_cur": mul[1]}}}
    weights = {"embed": table.float(), "bigram": pairs.float(), "embed.norm": w}
    total, slots = [30, 2, 41, 1], [3, 0, 5, 1]
    ids = [torch.randint(0, V, (n,), generator=torch.Generator().manual_seed(s)) for s, n in enumerate(total)]
    last = torch.full((6,), 11, dtype=torch.int32, device=device)
    spec = stream.ShiftSpec(rnd(2, W, seed=4).to(device))
    ring = torch.zeros(6, 3, W, device=device)

    def fn(batch, pieces):
        tok = cat_rows(device, ids, pieces)
        x = torch.empty(tok.shape[0], W, device=device)
        stream.layer_inputs(stream.Embedded(tok, table.to(device), pairs.to(device), *mul, w.to(device), last), x, spec, ring, batch, eps, dt)
        return [x]
    for sizes in ([18, 1, 2], [1], [2], [64]):
        got = run_steps(device, total, sizes, slots, fn)
        for s in range(len(total)):
            close(got[s][0], O.embed(cfg, weights, ids[s].tolist()), 3e-6)


# ------------------------------------------------------------------ queries, keys, turned values
@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("H, G, dim, vdim, hd, dims", [(3, 1, 24, 10, 0, 8), (6, 2, 40, 24, 64, 40), (2, 2, 5, 6, 0, 2), (16, 4, 128, 64, 128, 64),
                                                       (4, 1, 136, 200, 256, 16), (3, 3, 16, 48, 64, 0)])
def test_queries_keys_and_turned_values(H, G, dim, vdim, hd, dims, dtype, device):
    """One head is scaled up: a norm per head instead of one over the projection would undo that."""
    dt, T, eps, base = DT[dtype], 9, 1e-4, 700.0
    kw, vw = (hd, hd) if hd else (dim, vdim)
    nq, nk = H * dim, G * dim
    proj = rnd(T, nq + nk + G * vdim, seed=1)
    proj[:, :dim] *= 6.0
    proj[:, nq:nq + dim] *= 0.2
    proj = proj.to(dt)
    wq, wk = rnd(nq, seed=2), rnd(nk, seed=3)
    pos = torch.tensor([0, 1, 2, 50, 51, 300, 7, 8, 9], dtype=torch.int32)
    slots = torch.tensor([3, 40, 5, -1, 9, 31, 17, 0, 2], dtype=torch.int32)
    k_cache, v_cache = (torch.full((3, G, 16, n), 5.0, dtype=dt, device=device) for n in (kw, vw))
    d, dev = (lambda t: t.to(device)), torch.device(device)
    q = qk_attn.prepare(d(proj), d(wq), d(wk), eps, d(pos), get_cos_sin(dims, 512, base, None, dev), d(slots), k_cache, v_cache, H, G, dim,
                        vdim, get_cos_sin(vdim, 512, base, None, dev))
    f = proj.float()
    want_q = O.rotate_half((O.rms(f[:, :nq], eps) * wq).view(T, H, dim), pos, dims, base)
    want_k = O.rotate_half((O.rms(f[:, nq:nq + nk], eps) * wk).view(T, G, dim), pos, dims, base)
    raw = f[:, nq + nk:].reshape(T, G, vdim)                # pairs lie side by side here: half m | half m + vdim / 2 in the oracle
    want_v = O.rotate_half(raw.view(T, G, -1, 2).transpose(2, 3).reshape(T, G, vdim), pos, vdim, base)
    want_v = want_v.view(T, G, 2, -1).transpose(2, 3).reshape(T, G, vdim)
    tol = 1e-5 if dtype == "f32" else 1e-2
    close(q[..., :dim].float(), want_q, tol)
    assert kw == dim or float(q[..., dim:].abs().max()) == 0.0
    for t in range(T):
        if slots[t] >= 0:
            b, o = int(slots[t]) // 16, int(slots[t]) % 16
            for cache, want in ((k_cache, want_k), (v_cache, want_v)):
                close(cache[b, :, o, :want.shape[-1]].float(), want[t], tol)
                assert want.shape[-1] == cache.shape[-1] or float(cache[b, :, o, want.shape[-1]:].abs().max()) == 0.0
    used = {int(s) for s in slots if s >= 0}
    for s in set(range(48)) - used:
        assert float(k_cache[s // 16, :, s % 16].float().sub(5.0).abs().max()) == 0.0


# ------------------------------------------------------------------ attention without a softmax
class Pages:
    """Keys and values of several sequences in shuffled pages of one pool; rows padded to the kernels' width (0: none)."""

    def __init__(self, lens, G, dim, vdim, hd, bs, dtype, device, seed=0):
        per = [(n + bs - 1) // bs for n in lens]
        order = torch.randperm(sum(per), generator=torch.Generator().manual_seed(seed)) + 1
        self.bs, self.table, at = bs, torch.zeros(len(lens), max(per), dtype=torch.int32), 0
        for b, n in enumerate(per):
            self.table[b, :n] = order[at:at + n].to(torch.int32)
            at += n

        def pool(width, used):
            p = torch.full((sum(per) + 1, G, bs, width), 7.0, dtype=dtype)                   # unused rows hold rubbish
            p[..., used:] = 0
            return p.to(device)
        self.k, self.v = pool(hd or dim, dim), pool(hd or vdim, vdim)

    def fill(self, b, k, v):
        pos = torch.arange(k.shape[0])
        blk, off = self.table[b].long()[pos // self.bs], pos % self.bs
        for cache, rows in ((self.k, k), (self.v, v)):
            cache[blk.to(cache.device), :, off.to(cache.device), :rows.shape[-1]] = rows.to(cache)


def swap(v, back=False):
    """Channels in halves <-> pairs side by side."""
    return v.view(*v.shape[:-1], *((-1, 2) if back else (2, -1))).transpose(-1, -2).reshape(v.shape)


def padded(q, hd):
    return torch.nn.functional.pad(q, (0, hd - q.shape[-1])) if hd else q


FORMS = [("rows", "f32", "cpu"), pytest.param("rows", "f32", "cuda", marks=gpu), pytest.param("rows", "bf16", "cuda", marks=gpu),
         pytest.param("decode", "bf16", "cuda", marks=gpu), pytest.param("decode", "f16", "cuda", marks=gpu),
         pytest.param("prefill", "bf16", "cuda", marks=gpu)]


def head_size(form, dim, vdim):
    return 0 if form == "rows" else next(h for h in (64, 128, 256) if max(dim, vdim) <= h)


def one_row_each(form, q, pages, lens, scale, sig, vdim, splits=0):
    """The last position of every sequence; q [B, H, dim]."""
    B, H, device, G = q.shape[0], q.shape[1], pages.k.device, pages.k.shape[1]
    hd = pages.k.shape[3]
    q = padded(q, hd).to(device)
    table, ln = pages.table.to(device), i32(device, *lens)
    if form == "rows":
        return qk_attn.attend_rows(q, pages.k, pages.v, table, ln, None, scale, 0, None, None, vdim, sigmoid=sig)
    if form == "decode":
        return ops.paged_attention_decode(q.view(B, -1), pages.k, pages.v, table, ln, H, G, hd, scale, max_kv_len=max(lens), v_dim=vdim, sigmoid=sig,
                                          splits=splits)
    return ops.paged_attention_prefill(q.view(B, -1), pages.k, pages.v, table, ln, i32(device, *range(B + 1)), 1, H, G, hd, scale, v_dim=vdim, sigmoid=sig)


def sigmoid_weights(bias, chunk, vdim, device, rows=4096, base=500.0, turn=True):
    return ops.SigmoidWeights(bias.to(device), chunk, get_cos_sin(vdim, rows, base, None, torch.device(device)) if turn else None)


def want_rows(q, ks, vs, lens, scale, bias, chunk, vdim, base=500.0, turn=True):
    """q [B, H, dim] is each sequence's last position; values in pairs side by side, as cached."""
    out = []
    for b, n in enumerate(lens):
        o = O.attend(q[b:b + 1].float(), ks[b].float(), swap(vs[b].float(), back=True), scale, bias, chunk or 1 << 30)
        out.append(O.rotate_half(o, torch.tensor([n - 1]), vdim, base, -1.0) if turn else o)
    return swap(torch.cat(out)).reshape(len(lens), -1)


@pytest.mark.parametrize("form, dtype, device", FORMS)
@pytest.mark.parametrize("H, G, dim, vdim", [(3, 1, 24, 10), (6, 2, 40, 64), (16, 16, 64, 24), (17, 1, 128, 128), (8, 2, 136, 72)])
@pytest.mark.parametrize("chunk", [0, 1, 17, 64, 200])
def test_rows_against_cached_keys(H, G, dim, vdim, chunk, form, dtype, device):
    dt, lens, scale = DT[dtype], [1, 5, 64, 200, 201, 333], 0.3
    pages = Pages(lens, G, dim, vdim, head_size(form, dim, vdim), 16, dt, device)
    ks, vs = [rnd(n, G, dim, seed=n).to(dt) for n in lens], [rnd(n, G, vdim, seed=n + 1).to(dt) for n in lens]
    for b in range(len(lens)):
        pages.fill(b, ks[b], vs[b])
    q, bias = rnd(len(lens), H, dim, seed=5).to(dt), rnd(H, seed=6) - 1.0
    want = want_rows(q, ks, vs, lens, scale, bias, chunk, vdim)
    tol = 1e-5 if dtype == "f32" else 2e-2
    for splits in (0, 1, 3, 12) if form == "decode" else (0,):
        close(one_row_each(form, q, pages, lens, scale, sigmoid_weights(bias, chunk, vdim, device), vdim, splits).float(), want, tol)
    plain = one_row_each(form, q, pages, lens, scale, sigmoid_weights(bias, chunk, vdim, device, turn=False), vdim)
    close(plain.float(), want_rows(q, ks, vs, lens, scale, bias, chunk, vdim, turn=False), tol)


@pytest.mark.parametrize("form, dtype, device", FORMS)
@pytest.mark.parametrize("chunk", [15, 16, 50, 64, 96, 128])
def test_one_key_stands_out_at_the_edge_of_a_chunk(chunk, form, dtype, device):
    """Weights are all but zero except for one key: the first of the last position's chunk counts, the one before does not."""
    dt, H, G, dim, vdim = DT[dtype], 4, 2, 32, 48
    for n in (chunk, chunk + 1, 2 * chunk, 2 * chunk + 5, 3 * chunk + chunk // 2 + 1):
        first = (n - 1) // chunk * chunk
        for at, seen in ((first, True), (first - 1, False), (n - 1, True)):
            if at < 0:
                continue
            pages = Pages([n], G, dim, vdim, head_size(form, dim, vdim), 16, dt, device)
            k, v = torch.zeros(n, G, dim), rnd(n, G, vdim, seed=1)
            k[at, :, 0] = 8.0
            pages.fill(0, k, v)
            q = torch.zeros(1, H, dim)
            q[..., 0] = 4.0
            bias = torch.full((H,), -20.0)
            got = one_row_each(form, q.to(dt), pages, [n], 1.0, sigmoid_weights(bias, chunk, vdim, device, turn=False), vdim)
            want = v[at].repeat_interleave(H // G, 0).reshape(1, -1) if seen else torch.zeros(1, H * vdim)
            close(got.float(), want, 1e-2 if dt != torch.float32 else 1e-5)


@gpu
@pytest.mark.parametrize("H, G, dim, vdim", [(6, 2, 40, 24), (4, 1, 64, 64), (8, 2, 128, 128), (3, 3, 96, 50), (2, 1, 200, 104)])
@pytest.mark.parametrize("chunk", [0, 33, 128, 200, 300])
def test_long_portions(H, G, dim, vdim, chunk):
    """Portions over earlier tokens in one call, with tiles that cross chunks and pages of 16 and 128 tokens."""
    scale, base = 0.2, 500.0
    lens, done = [300, 70, 513, 64], [0, 250, 90, 0]
    total = [a + b for a, b in zip(lens, done)]
    for dtype, bs in (("bf16", 16), ("f16", 128)):
        dt, hd = DT[dtype], head_size("prefill", dim, vdim)
        pages = Pages(total, G, dim, vdim, hd, bs, dt, "cuda", seed=3)
        bias = rnd(H, seed=6) - 2.0
        qs, want = [], []
        for b, n in enumerate(total):
            k, v, q = rnd(n, G, dim, seed=b).to(dt), rnd(n, G, vdim, seed=b + 9).to(dt), rnd(lens[b], H, dim, seed=b + 20).to(dt)
            far = (n - 1) // (chunk or n + 1) * (chunk or n + 1)
            k[far] = q[-1, ::H // G][:, :dim] * 2                                            # a key that stands out for the last row
            pages.fill(b, k, v)
            o = O.attend(q.float(), k.float(), swap(v.float(), back=True), scale, bias, chunk or 1 << 30)
            want.append(swap(O.rotate_half(o, torch.arange(n - lens[b], n), vdim, base, -1.0)).reshape(lens[b], -1))
            qs.append(q)
        q = padded(torch.cat(qs), hd).cuda()
        cu = [sum(lens[:i]) for i in range(len(lens) + 1)]
        got = ops.paged_attention_prefill(q.view(sum(lens), -1), pages.k, pages.v, pages.table.cuda(), i32("cuda", *total), i32("cuda", *cu),
                                          max(lens), H, G, hd, scale, v_dim=vdim, sigmoid=sigmoid_weights(bias, chunk, vdim, "cuda", base=base))
        close(got.float(), torch.cat(want), 2e-2)
    ops.check_status(torch.device("cuda"))


@gpu
def test_weights_reach_from_nothing_to_one():
    """Scores of both signs and any size, in the tiled kernel too: sigmoid, not its clipped or shifted form."""
    n, dim = 128, 64
    pages = Pages([n], 1, dim, dim, 64, 16, torch.bfloat16, "cuda")
    score = torch.tensor([-200.0, -60.0, -9.0, -3.0, 0.0, 2.0, 7.0, 50.0, 200.0])
    k, v = torch.zeros(n, 1, dim), torch.zeros(n, 1, dim)
    k[:9, 0, 0] = score
    v[torch.arange(9), 0, torch.arange(9)] = 1.0
    pages.fill(0, k, v)
    q = torch.zeros(n, 1, dim, dtype=torch.bfloat16)
    q[..., 0] = 1.0
    sig = ops.SigmoidWeights(torch.full((1,), -1.0, device="cuda"))
    got = ops.paged_attention_prefill(q.view(n, -1).cuda(), pages.k, pages.v, pages.table.cuda(), i32("cuda", n), i32("cuda", 0, n), n, 1, 1, 64, 1.0,
                                      sigmoid=sig)[-1, :9].float().cpu()
    want = torch.sigmoid(score.bfloat16().float() - 1.0)
    assert float(((got - want).abs() / want.clamp(min=1e-7)).max()) < 1e-2


def test_sigmoid_weights_go_with_nothing_else():
    sig = ops.SigmoidWeights(torch.zeros(2))
    with pytest.raises(ValueError, match="without a softmax"):
        ops.attn_extra(2, 8, sinks=torch.zeros(2), sigmoid=sig)
    with pytest.raises(ValueError, match="turn"):
        ops.attn_extra(2, 8, sigmoid=ops.SigmoidWeights(torch.zeros(2), 0, torch.zeros(4, 6)))


# ------------------------------------------------------------------ recurrences
MIX = [(2, 12), (3, 5), (4, 64), (1, 130), (2, 72), (1, 300)]


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("H, d", MIX)
def test_time_mixing(H, d, dtype, device):
    """Portions and single tokens of unequal sequences; decays from a token to thousands; slots hold rubbish."""
    dt, eps, n = DT[dtype], 1e-3, H * d
    total, slots = [50, 2, 37, 1], [4, 0, 2, 1]
    proj = [[rnd(m, n, seed=s + 10 * j).to(dt) for s, m in enumerate(total)] for j in range(4)]
    zs = [rnd(m, n, seed=s + 50) for s, m in enumerate(total)]
    w0, u, norm = rnd(n, seed=1, std=3.0) - 2.0, rnd(H, d, seed=2), rnd(n, seed=3)
    pool = rnd(5, H, d, d, seed=4).to(device)
    d_ = lambda t: t.to(device)

    def fn(batch, pieces):
        r, k, v, g = (cat_rows(device, p, pieces) for p in proj)
        return [lin.time_mix(r, k, v, g, cat_rows(device, zs, pieces), d_(w0), d_(u), pool, batch, d_(norm), eps, dt)]
    for sizes in ([64], [1], [16, 1, 3]):
        got = run_steps(device, total, sizes, slots, fn)
        for s, m in enumerate(total):
            r, k, v, g = (p[s].float().view(m, H, d) for p in proj)
            o, S = O.time_mix(r, k, v, torch.exp(-torch.exp(zs[s] + w0)).view(m, H, d), u, torch.zeros(H, d, d))
            want = O.rms(o, eps).reshape(m, n) * norm * O.silu(g.reshape(m, n))
            close(got[s][0], want, 2e-5 if dtype == "f32" else 8e-3)
            close(pool[slots[s]], S, 2e-5)


SSD = [(4, 20, 12, 2, 5, 3), (3, 7, 5, 3, 1, 1), (6, 64, 64, 1, 4, 4), (2, 130, 130, 2, 2, 2), (8, 32, 128, 4, 32, 4), (2, 48, 300, 1, 3, 9)]


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
@pytest.mark.parametrize("H, dv, N, G, parts, taps", SSD)
def test_state_space(H, dv, N, G, parts, taps, dtype, device):
    """Groups shared by heads, norm parts that cross heads or divide them, convolutions of 1 to 9 taps."""
    dt, eps, inner = DT[dtype], 1e-3, H * dv
    C = inner + 2 * G * N
    total, slots = [50, 2, 37, 1], [4, 0, 2, 1]
    xbc = [rnd(m, C, seed=s).to(dt) for s, m in enumerate(total)]
    zs = [rnd(m, inner, seed=s + 20).to(dt) for s, m in enumerate(total)]
    dts = [rnd(m, H, seed=s + 40, std=2.0) for s, m in enumerate(total)]
    conv, cb, bias, rate, skip, norm = rnd(C, taps, seed=1), rnd(C, seed=2), rnd(H, seed=3) - 2, torch.exp(rnd(H, seed=4, std=2.0) - 1), rnd(H, seed=5), rnd(inner, seed=6)
    pool, ring = rnd(5, H, N, dv, seed=7).to(device), rnd(5, taps, C, seed=8, std=30.0).to(device)
    d = lambda t: t.contiguous().to(device)

    def fn(batch, pieces):
        x = torch.cat([cat_rows(device, zs, pieces), cat_rows(device, xbc, pieces)], 1)
        return [lin.ssd(x[:, inner:], x[:, :inner], cat_rows(device, dts, pieces), d(bias), d(rate), d(skip), d(conv.t()), d(cb), pool, ring, G, batch,
                        d(norm), parts, eps, dt)]
    for sizes in ([64], [1], [16, 1, 3]):
        got = run_steps(device, total, sizes, slots, fn)
        for s, m in enumerate(total):
            y = O.silu(O.causal_conv(xbc[s].float(), conv) + cb)
            x, B, Cc = torch.split(y, [inner, G * N, G * N], dim=-1)
            o, S = O.ssd(x.reshape(m, H, dv), B.reshape(m, G, N), Cc.reshape(m, G, N), O.softplus(dts[s] + bias), rate, skip, torch.zeros(H, N, dv))
            want = O.part_norm(o.reshape(m, inner) * O.silu(zs[s].float()), parts, eps) * norm
            close(got[s][0], want, 3e-5 if dtype == "f32" else 2e-2)
            close(pool[slots[s]], S, 3e-5 if dtype == "f32" else 2e-2)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("single", [False, True])
def test_a_far_write_survives_slow_decay(single, device):
    """One write, then 3000 tokens that only decay: rounding of the factors must not add up."""
    H, d, n, z = 1, 8, 3000, -9.0
    k, v, r = torch.zeros(n, d), torch.zeros(n, d), torch.zeros(n, d)
    k[0], v[0], r[-1] = 1.0, torch.arange(1.0, d + 1), 1.0
    u, w0, norm = torch.zeros(H, d), torch.full((d,), z), torch.ones(d)
    pool, xs = torch.full((1, H, d, d), 9.0, device=device), [r, k, v]
    sizes = [n - 40] + [1] * 40 if single else [n]
    run_steps(device, [n], sizes, [0], lambda b, p: [lin.time_mix(*(cat_rows(device, [x], p) for x in xs), torch.ones(p[0][2] - p[0][1], d, device=device),
                                                                  torch.zeros(p[0][2] - p[0][1], d, device=device), w0.to(device), u.to(device), pool, b,
                                                                  norm.to(device), 1e-6, torch.float32)])
    factor = torch.exp(-torch.exp(torch.tensor(z, dtype=torch.float64))) ** (n - 1)
    want = (k[0][:, None] * v[0][None]).double() * factor
    assert float((pool[0, 0].double().cpu() / want - 1).abs().max()) < 2e-4
    # the same for the scalar form: softplus(dt + bias) * rate = e^z
    taps, C = 2, 3 * d
    xbc = torch.zeros(n, C)
    conv, cb = torch.zeros(taps, C), torch.zeros(C)
    conv[-1] = 1.0
    xbc[0] = 2.0
    pool, ring = torch.full((1, H, d, d), 9.0, device=device), torch.full((1, taps, C), 9.0, device=device)
    dev = lambda t: t.to(device)
    dt0 = torch.tensor([0.5])
    run_steps(device, [n], sizes, [0], lambda b, p: [lin.ssd(cat_rows(device, [xbc], p), torch.ones(p[0][2] - p[0][1], d, device=device),
                                                             torch.zeros(p[0][2] - p[0][1], 1, device=device), dev(dt0), dev(torch.tensor([1.3e-4])),
                                                             dev(torch.ones(1)), dev(conv), dev(cb), pool, ring, 1, b, dev(torch.ones(d)), 1, 1e-6,
                                                             torch.float32)])
    step = torch.nn.functional.softplus(dt0.double())
    a = O.silu(torch.tensor(2.0, dtype=torch.float64))
    want = step * a * a * torch.exp(-1.3e-4 * step) ** (n - 1)
    assert float((pool.double().cpu() / want - 1).abs().max()) < 2e-4


@pytest.mark.parametrize("device", DEV)
def test_the_bonus_counts_for_the_current_token_only(device):
    H, d = 2, 16
    k, v, r = rnd(2, H * d, seed=1), rnd(2, H * d, seed=2), rnd(2, H * d, seed=3)
    norm, z, w0 = torch.ones(H * d), torch.zeros(2, H * d), torch.full((H * d,), 5.0)          # e^-148: the state is gone at once
    for bonus in (0.0, 3.0):
        pool, u = torch.zeros(1, H, d, d, device=device), torch.full((H, d), bonus)
        got = run_steps(device, [2], [2], [0], lambda b, p: [lin.time_mix(*(t.to(device) for t in (r, k, v, torch.ones(2, H * d), z, w0, u)), pool, b,
                                                                          norm.to(device), 1e-6, torch.float32)])[0][0]
        o = torch.zeros(2, H, d)
        R, K, V = (t.view(2, H, d) for t in (r, k, v))
        for h in range(H):
            o[0, h] = bonus * (R[0, h] @ K[0, h]) * V[0, h]
            o[1, h] = bonus * (R[1, h] @ K[1, h]) * V[1, h] + (R[1, h] @ K[0, h]) * V[0, h]
        close(got, O.rms(o, 1e-6).reshape(2, -1) * O.silu(torch.ones(1)), 1e-4)


@gpu
@pytest.mark.parametrize("B, n", [(1, 2000), (9, 300), (24, 100)])
def test_every_column_width_of_the_scans(B, n):
    """Few and many sequences take other launch shapes; results do not depend on it."""
    H, d = 8, 64
    x, z = rnd(4, n, H * d, seed=1), rnd(n, H * d, seed=2)
    w0, u = rnd(H * d, seed=3) - 2, rnd(H, d, seed=4)
    tile = lambda t: t.repeat(B, 1).cuda()
    one, many = torch.zeros(1, H, d, d, device="cuda"), torch.zeros(B, H, d, d, device="cuda")
    a = lin._scan(0, *(t.cuda() for t in x[:3]), z.cuda(), w0.cuda(), u.cuda(), None, one, make_batch("cuda", [0], [n], [0]), H)
    b = lin._scan(0, *(tile(t) for t in x[:3]), tile(z), w0.cuda(), u.cuda(), None, many, make_batch("cuda", list(range(B)), [n] * B, [0] * B), H)
    for i in range(B):
        close(b[i * n:(i + 1) * n], a.cpu(), 1e-5)
        close(many[i], one[0].cpu(), 1e-5)
    G, rate, skip = 2, torch.rand(H, generator=torch.Generator().manual_seed(1)), rnd(H, seed=5)
    args = (x[0, :, :G * d], x[1, :, :G * d], x[2], z[:, :H])
    one.zero_(), many.zero_()
    a = lin._scan(1, *(t.cuda() for t in args), w0[:H].cuda(), skip.cuda(), rate.cuda(), one, make_batch("cuda", [0], [n], [0]), G)
    b = lin._scan(1, *(tile(t) for t in args), w0[:H].cuda(), skip.cuda(), rate.cuda(), many, make_batch("cuda", list(range(B)), [n] * B, [0] * B), G)
    for i in range(B):
        close(b[i * n:(i + 1) * n], a.cpu(), 1e-5)


@gpu
@pytest.mark.parametrize("H, G, d, dv", [(4, 2, 64, 64), (2, 1, 12, 20), (2, 2, 130, 66), (3, 1, 5, 7), (1, 1, 300, 40)])
@pytest.mark.parametrize("segment", [16, 48, 100])
def test_segments_of_long_portions(H, G, d, dv, segment):
    """Portions cut into segments that run side by side: new and continued sequences, portions of any length."""
    lens, done, slots = [500, 1, 97, 48], [0, 30, 65, 0], [3, 0, 2, 1]
    n = sum(lens)
    q, k, v, z = rnd(n, H * d, seed=1), rnd(n, H * d, seed=2), rnd(n, H * dv, seed=3), rnd(n, H * d, seed=4)
    w0, u, rate, pool = rnd(H * d, seed=5, std=2.0) - 3, rnd(H * d, seed=6), torch.exp(rnd(H, seed=7)), rnd(4, H, d, dv, seed=8)
    cuda = lambda *ts: [t.cuda() for t in ts]
    for kind, args in ((0, (q, k, v, z, w0, u, rate)), (1, (q[:, :G * d], k[:, :G * d], v, z[:, :H].contiguous(), w0[:H].contiguous(), u[:H].contiguous(), rate))):
        got = []
        for cut in (segment, 10 ** 6):                      # one segment: the plain walk, up to the chain of one
            p, b = pool.cuda(), make_batch("cuda", slots, lens, done)
            got.append((lin._scan(kind, *cuda(*args), p, b, H if kind == 0 else G, cut), p))
        p, b = pool.cuda(), make_batch("cuda", slots, lens, done)
        plain = (lin._scan(kind, *cuda(*args), p, b, H if kind == 0 else G), p)
        for o, s in got:
            close(o, plain[0].cpu(), 2e-5)
            close(s, plain[1].cpu(), 2e-5)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("n, parts", [(7, 3), (64, 4), (200, 1), (512, 2), (1000, 3), (2048, 1), (4096, 2), (8192, 1), (9000, 1)])
def test_norm_of_parts_with_a_gate_on_either_side(n, parts, device):
    o, g, w = rnd(5, n * parts, seed=1, std=3.0), rnd(5, n * parts, seed=2), rnd(n * parts, seed=3)
    o[:, :n] *= 20.0
    d = lambda t: t.to(device)
    for dt, tol in ((torch.float32, 3e-6), (torch.bfloat16, 6e-3)):
        gate = torch.zeros(5, n * parts + 8, dtype=dt, device=device)[:, 8:]
        gate.copy_(g)
        f = gate.float().cpu()
        close(lin.part_norm(d(o), d(w), parts, 0.1, dt, gate, True).float(), O.part_norm(o * O.silu(f), parts, 0.1) * w, tol)
        close(lin.part_norm(d(o), d(w), parts, 0.1, dt, gate).float(), O.part_norm(o, parts, 0.1) * w * O.silu(f), tol)
        close(lin.part_norm(d(o), d(w), parts, 0.1, dt).float(), O.part_norm(o, parts, 0.1) * w, tol)


# ------------------------------------------------------------------ feed-forwards, products
@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("T, W, ff, E, top, V", [(1, 33, 7, 5, 2, 9), (9, 64, 40, 6, 3, 20), (20, 72, 24, 4, 4, 3), (130, 256, 96, 8, 1, 50), (700, 128, 200, 3, 2, 11)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_experts_assigned_by_token(T, W, ff, E, top, V, dtype, device):
    dt, gen = DT[dtype], torch.Generator().manual_seed(0)
    layer = AssignedExperts(W, ff, E, top, V, dt)
    w = {"table": torch.stack([torch.randperm(E, generator=gen)[:top] for _ in range(V)]).to(torch.int32)}
    for e in range(E):
        for n, o, k in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
            w[f"e{e}.{n}"] = (torch.randn(o, k, generator=gen) * 1.5 * k ** -0.5).to(dt).float()
    for name, where in layer.destinations("").items():
        where(w[name]) if callable(where) and not isinstance(where, torch.Tensor) else where.data.copy_(w[name])
    layer, ids, x = layer.to(device), torch.randint(0, V, (T,), generator=gen), torch.randn(T, W, generator=gen).to(dt)
    got = layer(x.to(device), ids.to(device))
    routed = moe.RoutedRows(got.rows.cpu(), got.weights, got.slot_of.cpu())
    close(routed.combined(), O.experts(x.float(), w, "", ids.tolist()), 1e-5 if dtype == "f32" else 2e-2)


def test_expert_tables_are_checked():
    layer = AssignedExperts(8, 4, 3, 2, 5, torch.float32)
    take = layer.destinations("")["table"]
    good = torch.zeros(5, 2, dtype=torch.int32)
    take(good + torch.tensor([0, 2], dtype=torch.int32))
    assert layer.table.tolist() == [[0, 2]] * 5
    for bad, match in ((good[:4], "shape"), (good + 3, "below 3"), (good - 1, "below 3"), (good.float(), "integers")):
        with pytest.raises(ValueError, match=match):
            take(bad)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("T, K, N", [(1, 64, 64), (17, 72, 200), (40, 256, 136), (300, 128, 512), (1100, 96, 128), (5, 33, 7)])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_stacked_products(T, K, N, dtype, device):
    dt = DT[dtype]
    buf = torch.zeros(5, T, (K + 7) // 8 * 8, dtype=dt, device=device)
    x = buf[:, :, :K]
    x.copy_(rnd(5, T, K, seed=1))
    w = rnd(4, N, K, seed=2, std=K ** -0.5).to(dt)
    got = moe.stacked_linear(x[:4], w.to(device))
    for e in range(4):
        close(got[e].float(), x[e].float().cpu() @ w[e].float().t(), 1e-5 if dtype == "f32" else 1e-2)


@pytest.mark.parametrize("device", DEV)
@pytest.mark.parametrize("T", [3, 100, 1100])
@pytest.mark.parametrize("dtype", ["f32", "bf16"])
def test_products_with_squared_relu_and_tanh(T, dtype, device):
    dt = DT[dtype]
    x, w = rnd(T, 320, seed=1).to(dt), rnd(136, 320, seed=2, std=0.1).to(dt)
    y = x.float() @ w.float().t()
    tol = 1e-5 if dtype == "f32" else 1e-2
    for act, want in (("relu2", torch.relu(y) ** 2), ("tanh", torch.tanh(y))):
        close(ops.linear(x.to(device), w.to(device), act=act).float(), want, tol)
