"""Kernels and throughput of the Divadra design at sizes that resemble a real model's layers, beside the like kernels of the
closest models the framework served before (HGRN2 and the delta rule for the recurrences, Pofadra's windowed attention,
layer boundary and routed experts) and beside a Pofadra model of equal width, depth, heads, experts and vocabulary.
Random weights, one GPU.

    python benchmarks/divadra_shapes.py [--kernels] [--models] [--sizes 1024 2048 4096] [--only TEXT] [--json out.json]

A kernel's roofline time is the larger of its algorithmic bytes over the measured copy bandwidth and its FLOPs over the
measured product rate (MEASURED_PEAKS.json); "x roofline" is the measured time over that.  Caches are flushed between
iterations; times are medians from CUDA events.  ``python bench.py --divadra`` prints the same as one JSON line.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path
from types import SimpleNamespace

ROOT = Path(__file__).resolve().parents[1]
if str(ROOT) not in sys.path:
    sys.path.insert(0, str(ROOT))

from benchmarks.fimodra_shapes import BATCH, CONTEXT, FP32_TFLOPS, TOKENS, Timer, _peaks, throughput_row  # noqa: E402

# width: state space (heads, vdim, state, groups, norm groups, taps), attention (heads, kv heads, dim, vdim, rotated, chunk),
# time mixing (heads, dim), dense ff, experts (count, chosen, ff)
SIZES = {1024: ((16, 64, 128, 2, 2, 4), (8, 2, 128, 128, 128, 512), (16, 64), 2816, (16, 4, 512)),
         2048: ((32, 64, 128, 4, 4, 4), (16, 4, 128, 128, 128, 1024), (32, 64), 5632, (32, 4, 768)),
         4096: ((64, 128, 128, 8, 8, 4), (32, 8, 128, 128, 128, 1024), (64, 64), 11008, (64, 6, 1024))}


def kernel_rows(width: int, iters: int = 10, only: str = "") -> list[dict]:
    import torch

    from litevllm_b200 import ops
    from litevllm_b200.layers.rope import get_cos_sin
    from litevllm_b200.ops import linear_attn as lin
    from litevllm_b200.ops import moe, qk_attn
    from litevllm_b200.ops import residual_stream as rs
    from litevllm_b200.ops import shift_stream as ss
    hbm, tensor, _ = _peaks()
    time_us = Timer(torch, iters)
    (MH, mdv, N, MG, parts, taps), (H, G, dim, vdim, rot, chunk), (RH, rd), ff, (E, top, eff) = SIZES[width]
    W, T, B, ctx = width, TOKENS, BATCH, CONTEXT
    g = torch.Generator(device="cuda").manual_seed(0)
    bf, f32 = torch.bfloat16, torch.float32

    def rnd(*s, dtype=bf, std=1.0):
        return (torch.randn(*s, generator=g, device="cuda") * std).to(dtype)

    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    rows = []

    def case(name, fn, nbytes, flops=0.0, peak=tensor, likes=()):
        if only not in name:
            return
        us = time_us(fn)
        roof = max(nbytes / (hbm * 1e3), flops / (peak * 1e6))
        r = {"width": width, "kernel": name, "us": round(us, 1), "roofline_us": round(roof, 1), "x_roofline": round(us / roof, 2)}
        if not only:
            r["likes"] = []
            for lname, lfn, lbytes, lflops, lpeak in likes:
                lus = time_us(lfn)
                lroof = max(lbytes / (hbm * 1e3), lflops / (lpeak * 1e6))
                r["likes"].append({"kernel": lname, "us": round(lus, 1), "roofline_us": round(lroof, 1), "x_roofline": round(lus / lroof, 2)})
        rows.append(r)

    def step(lens, decode=False):
        """Batch fields the recurrent kernels read."""
        B = len(lens)
        return SimpleNamespace(is_decode=decode, q_lens_cpu=[1] * B if decode else lens, seq_lens=i32([100] * B if decode else lens),
                               cu_q=None if decode else i32([sum(lens[:i]) for i in range(B + 1)]), extras={"slot_ids": i32(list(range(B)))})

    prefill, decode = step([1024] * 8), step([1] * B, True)
    # ---- layer boundary beside Pofadra's (mixer, experts, one norm) and RMSNorm with its residual add
    spec = ss.ShiftSpec(rnd(4, W, dtype=f32), rnd(4, W, dtype=f32), rnd(5, W, dtype=f32))
    short = ss.ShiftSpec(spec.a1, spec.a2)
    table, pairs, last = rnd(32000, W), rnd(4094, W), torch.zeros(64, dtype=torch.int32, device="cuda")
    for batch, n, tag in ((prefill, T, "prefill"), (decode, B, "decode")):
        ring = torch.zeros(64, 5, W, device="cuda")
        y, y2, x, w, ys = rnd(n, W), rnd(n, W), rnd(n, W, dtype=f32), rnd(W, dtype=f32), rnd(n * top, W)
        order = torch.randperm(n * top, generator=g, device="cuda").to(torch.int32).view(n, top)
        routed = moe.RoutedRows(ys, torch.rand(n, top, generator=g, device="cuda"), order)
        res, wb = rnd(n, W), rnd(W)
        rbytes = 0 if n > B else n * 4 * W * 4        # ring rows of a decoded token
        ids = torch.randint(0, 32000, (n,), device="cuda")
        # two kernels in portions: the stream is read twice
        again = n * W * 4 if n > B else 0
        likes = [(f"layer boundary (mixer + {top} experts + norm)", lambda: rs.add(y, x, routed, w, 1e-6, 1, x, bf), n * W * (12 + 2 * top), 0, tensor),
                 ("RMSNorm + residual", lambda: ops.rmsnorm(y, wb, 1e-6, residual=res), n * W * 8, 0, tensor)]
        case(f"layer boundary (two normed mixers + {top} experts .. inputs and blends), {tag}",
             lambda: ss.layer_inputs(ss.Paired(y, w, y2, w, None, routed), x, spec, ring, batch, 1e-6, bf),
             n * W * (12 + 2 * top + 14) + again + rbytes, likes=likes)
        case(f"layer boundary (mixer + dense .. two inputs), {tag}",
             lambda: ss.layer_inputs(ss.Summed(y, y2), x, short, ring, batch, 1e-6, bf), n * W * (12 + 4) + again + rbytes, likes=likes[1:])
        emb = ss.Embedded(ids, table, pairs, 31, 7, w, last)
        case(f"embedding pair .. two inputs, {tag}", lambda: ss.layer_inputs(emb, x, short, ring, batch, 1e-6, bf),
             n * W * (4 + 4 + 4) + again + rbytes,
             likes=[("embedding + norm", lambda: rs.start(ids, table, w, 1e-6, 1, x), n * W * 8, 0, tensor)])
        del ys
    # ---- recurrences beside HGRN2 (and, for decode, the delta rule, which also convolves)
    C, inner, RN = MH * mdv + 2 * MG * N, MH * mdv, RH * rd
    conv, cb, rate = rnd(taps, C, dtype=f32), rnd(C, dtype=f32), torch.rand(MH, generator=g, device="cuda")
    mb, skip, w0, u = rnd(MH, dtype=f32), rnd(MH, dtype=f32), rnd(RN, dtype=f32), rnd(RH, rd, dtype=f32)
    for lens in ([1024] * 8, [8192]):
        n, batch = sum(lens), step(lens)
        a = (batch.extras["slot_ids"], batch.cu_q, batch.seq_lens)

        def hgrn2(LH, d, dv):
            q, f, b, lo = rnd(n, LH * (d + dv)), rnd(n, LH * d, dtype=f32), rnd(LH * d, dtype=f32), torch.rand(LH * d, generator=g, device="cuda")
            pool = torch.zeros(len(lens), LH, d, dv, device="cuda")
            return (f"HGRN2 scan, {LH} heads of {d} x {dv}",
                    lambda: lin.hgrn2_scan(q[:, :LH * d], f, q[:, LH * d:], b, lo, pool, *a, LH, d, dv),
                    n * LH * (d * 6 + dv * 6), n * LH * d * dv * 5.0, FP32_TFLOPS)
        rkvg, z, pool = rnd(4, n, RN), rnd(n, RN, dtype=f32), torch.zeros(len(lens), RH, rd, rd, device="cuda")
        case(f"time mixing scan, {len(lens)} x {lens[0]}", lambda: lin._scan(0, rkvg[0], rkvg[1], rkvg[2], z, w0, u, None, pool, batch, RH),
             n * RN * 14, n * RN * rd * 5.0, FP32_TFLOPS, likes=[hgrn2(RH, rd, rd)])
        xbc, dt, spool = rnd(n, C), rnd(n, MH, dtype=f32), torch.zeros(len(lens), MH, N, mdv, device="cuda")
        case(f"state-space scan, {len(lens)} x {lens[0]}",
             lambda: lin._scan(1, xbc[:, inner + MG * N:], xbc[:, inner:inner + MG * N], xbc[:, :inner], dt, mb, skip, rate, spool, batch, MG),
             n * (C * 2 + MH * 4 + inner * 4), n * MH * N * mdv * 5.0, FP32_TFLOPS, likes=[hgrn2(MH, N, mdv)])
        if len(lens) > 1:
            ring = torch.zeros(len(lens), taps, C, device="cuda")
            yb, res, wb = rnd(n, W), rnd(n, W), rnd(W)
            case("short convolution with SiLU", lambda: lin.conv_silu(xbc, conv, cb, ring, batch, bf), n * C * 4,
                 likes=[("RMSNorm + residual", lambda: ops.rmsnorm(yb, wb, 1e-6, residual=res), n * W * 8, 0, tensor)])
            o, wn, gate = rnd(n, inner, dtype=f32), rnd(inner, dtype=f32), rnd(n, inner)
            ho, hw = rnd(n, inner // 64, 64, dtype=f32), rnd(64, dtype=f32)
            like = ("head norm with gate", lambda: lin.head_norm(ho, hw, 1e-6, bf, gate), n * inner * 8, 0, tensor)
            case(f"gate and norm of {parts} parts", lambda: lin.part_norm(o, wn, parts, 1e-6, bf, gate, True), n * inner * 8, likes=[like])
            o2, wn2, gate2 = rnd(n, RN, dtype=f32), rnd(RN, dtype=f32), rnd(n, RN)
            case("head norm, weight and gate", lambda: lin.part_norm(o2, wn2, RH, 1e-6, bf, gate2), n * RN * 8, likes=[like])
            del o, gate, ho, o2, gate2
        del rkvg, z, xbc
    pool, spool = torch.zeros(256, RH, rd, rd, device="cuda"), torch.zeros(256, MH, N, mdv, device="cuda")
    ring = torch.zeros(256, taps, C, device="cuda")
    for n in (B, 128):
        batch = step([1] * n, True)
        sl, ln = batch.extras["slot_ids"], batch.seq_lens

        def hgrn2_step(LH, d, dv):
            h, b, lo, w = rnd(n, LH * (2 * d + dv), dtype=f32), rnd(LH * d, dtype=f32), torch.rand(LH * d, generator=g, device="cuda"), rnd(dv, dtype=f32)
            p = torch.zeros(256, LH, d, dv, device="cuda")
            return (f"HGRN2 step, {LH} heads of {d} x {dv}",
                    lambda: lin.hgrn2_step(h[:, :LH * d], h[:, LH * (d + dv):], h[:, LH * d:LH * (d + dv)], b, lo, p, sl, ln, w, 1e-6, LH, d, dv, bf),
                    n * LH * d * dv * 8, 0, tensor)

        def delta(LH, d, dv):
            m = lin.DeltaSpec(LH, LH, d, dv, rnd(LH * (2 * d + dv), taps, dtype=f32), torch.rand(LH, generator=g, device="cuda"), rnd(LH * d, dtype=f32))
            x, zg, b, w = rnd(n, m.channels), rnd(n, LH * (d + dv), dtype=f32), rnd(n, LH, dtype=f32), rnd(dv, dtype=f32)
            p, r = torch.zeros(256, LH, d, dv, device="cuda"), torch.zeros(256, taps, m.channels, device="cuda")
            return (f"delta step, {LH} heads of {d} x {dv}",
                    lambda: lin.delta_step(x, zg[:, :LH * d], b, m, p, r, sl, ln, w, 1e-6, zg[:, LH * d:], bf),
                    n * LH * d * dv * 8 + n * m.channels * 4 * (taps + 1), 0, tensor)
        rkvg, z, wn = rnd(4, n, RN), rnd(n, RN, dtype=f32), rnd(RN, dtype=f32)
        case(f"time mixing step, batch {n} (decays .. gated norm)",
             lambda: lin.time_mix(*rkvg, z, w0, u, pool, batch, wn, 1e-6, bf), n * RN * rd * 8 + n * RN * 14, likes=[hgrn2_step(RH, rd, rd)])
        p, dt, wn2 = rnd(n, inner + C, dtype=f32), rnd(n, MH, dtype=f32), rnd(inner, dtype=f32)
        case(f"state-space step, batch {n} (convolution .. gated norm)",
             lambda: lin.ssd(p[:, inner:], p[:, :inner], dt, mb, rate, skip, conv, cb, spool, ring, MG, batch, wn2, parts, 1e-6, bf),
             n * MH * N * mdv * 8 + n * C * 4 * (taps + 1) + n * inner * 6, likes=[hgrn2_step(MH, N, mdv), delta(MH, N, mdv)])
    del pool, spool
    # ---- attention, prefill
    nblk = T // 16 + 1
    kc, vc = rnd(nblk, G, 16, dim, std=0.5), rnd(nblk, G, 16, vdim, std=0.5)
    table = i32([[1 + s * 64 + j for j in range(64)] for s in range(8)])
    pos, slots = i32(list(range(1024)) * 8), i32(list(range(16, T + 16)))
    cu, ln = i32([1024 * i for i in range(9)]), i32([1024] * 8)
    proj, wq, wk = rnd(T, (H + 2 * G) * dim), rnd(H * dim, dtype=f32), rnd(G * dim, dtype=f32)
    cs, vcs = (get_cos_sin(n, 4096, 1e4, None, torch.device("cuda")) for n in (rot, vdim))
    sig = ops.SigmoidWeights(rnd(H, dtype=f32), chunk, vcs)
    pre = lambda: qk_attn.prepare(proj, wq, wk, 1e-6, pos, cs, slots, kc, vc, H, G, dim, vdim, vcs)
    q = pre()
    case("queries, keys, values: norm, rotations, cache rows, prefill", pre, T * (2 * H + 4 * G) * dim * 2,
         likes=[("the same with keys as values", lambda: qk_attn.prepare(proj, wq, wk, 1e-6, pos, cs, slots, kc, vc, H, G, dim), T * (2 * H + 3 * G) * dim * 2, 0, tensor)])
    seen = 8 * sum(i % chunk + 1 for i in range(1024))
    io = T * (2 * H + 2 * G) * dim * 2
    gate, sinks = rnd(T, H * dim), torch.zeros(H, device="cuda")
    case(f"sigmoid attention, prefill 8 x 1024, chunks of {chunk}",
         lambda: ops.paged_attention_prefill(q.view(T, -1), kc, vc, table, ln, cu, 1024, H, G, dim, 0.1, v_dim=vdim, sigmoid=sig), io, 4.0 * seen * H * dim,
         likes=[(f"windowed attention with sink and gate, window {chunk}",
                 lambda: ops.paged_attention_prefill(q.view(T, -1), kc, vc, table, ln, cu, 1024, H, G, dim, 0.1, chunk, sinks=sinks, v_dim=dim, gate=gate),
                 io + T * H * dim * 2, 4.0 * 8 * sum(min(i + 1, chunk) for i in range(1024)) * H * dim, tensor),
                ("causal attention", lambda: ops.paged_attention_prefill(q.view(T, -1), kc, vc, table, ln, cu, 1024, H, G, dim, 0.1), io,
                 4.0 * 8 * (1024 * 1025 // 2) * H * dim, tensor)])
    table = i32([[1 + j for j in range(512)]])
    cu, ln = i32([0, 8192]), i32([8192])
    whole = ops.SigmoidWeights(sig.bias, 8192, get_cos_sin(vdim, 8192, 1e4, None, torch.device("cuda")))
    case("sigmoid attention, prefill 1 x 8192, one chunk",
         lambda: ops.paged_attention_prefill(q.view(T, -1), kc, vc, table, ln, cu, 8192, H, G, dim, 0.1, v_dim=vdim, sigmoid=whole), io,
         4.0 * (8192 * 8193 // 2) * H * dim,
         likes=[("causal attention", lambda: ops.paged_attention_prefill(q.view(T, -1), kc, vc, table, ln, cu, 8192, H, G, dim, 0.1), io,
                 4.0 * (8192 * 8193 // 2) * H * dim, tensor)])
    # ---- attention, decode (the last position of a chunk)
    nb = B * ctx // 16 + 1
    kc, vc = rnd(nb, G, 16, dim, std=0.5), rnd(nb, G, 16, vdim, std=0.5)
    table = i32([[1 + s * (ctx // 16) + j for j in range(ctx // 16)] for s in range(B)])
    seen = min(chunk, ctx)
    qd, ln, short_ln = rnd(B, H * dim), i32([ctx] * B), i32([seen] * B)
    case(f"sigmoid attention, decode batch {B}, {seen} keys",
         lambda: ops.paged_attention_decode(qd, kc, vc, table, ln, H, G, dim, 0.1, max_kv_len=ctx, v_dim=vdim, sigmoid=sig), B * seen * G * dim * 4,
         4.0 * B * seen * H * dim,
         likes=[("attention", lambda: ops.paged_attention_decode(qd, kc, vc, table, short_ln, H, G, dim, 0.1, max_kv_len=seen),
                 B * seen * G * dim * 4, 4.0 * B * seen * H * dim, tensor)])
    projd, posd, slotd = rnd(B, (H + 2 * G) * dim), i32([ctx - 1] * B), i32([16 + i * ctx for i in range(B)])
    case("queries, keys, values, decode", lambda: qk_attn.prepare(projd, wq, wk, 1e-6, posd, cs, slotd, kc, vc, H, G, dim, vdim, vcs),
         B * (2 * H + 4 * G) * dim * 2,
         likes=[("the same with keys as values", lambda: qk_attn.prepare(projd, wq, wk, 1e-6, posd, cs, slotd, kc, vc, H, G, dim),
                 B * (2 * H + 3 * G) * dim * 2, 0, tensor)])
    del kc, vc, proj
    # ---- products and experts
    w4, wd, wu = rnd(4, RN, W, std=0.03), rnd(4 * RN, W, std=0.03), rnd(ff, W, std=0.03)
    for n, tag in ((T, f"{T} tokens"), (B, f"decode batch {B}")):
        x4, x1 = rnd(5, n, W), rnd(n, W)
        io, fl = 4 * RN * W * 2 + 4 * n * (W + RN) * 2, 8.0 * n * RN * W
        case(f"four projections of four blends, {tag}", lambda: moe.stacked_linear(x4[:4], w4), io, fl,
             likes=[("one product of the same size", lambda: ops.linear(x1, wd), 4 * RN * W * 2 + n * (W + 4 * RN) * 2, fl, tensor)])
        case(f"product with squared ReLU, {tag}", lambda: ops.linear(x1, wu, act="relu2"), ff * W * 2 + n * (W + ff) * 2, 2.0 * n * ff * W,
             likes=[("product with SiLU", lambda: ops.linear(x1, wu, act="silu"), ff * W * 2 + n * (W + ff) * 2, 2.0 * n * ff * W, tensor)])
    w1, w2 = rnd(E, 2 * eff, W, std=0.03), rnd(E, W, eff, std=0.03)
    tab = torch.rand(32000, E, generator=g, device="cuda").topk(top, -1).indices.to(torch.int32)
    for n, tag in ((T, f"{T} tokens"), (B, f"decode batch {B}")):
        x, z, ids = rnd(n, W), rnd(n, E, dtype=f32), torch.randint(0, 32000, (n,), device="cuda")
        e = moe.Assigned(tab, ids)
        used = int(e.ids().unique().numel())
        nb, fl = used * 3 * eff * W * 2 + n * W * 2 + n * top * W * 2, 6.0 * n * top * eff * W
        re, ra = moe.route(z, top)
        case(f"assigned experts, {tag} (assignment, sort .. down product)", lambda: moe.expert_rows(x, w1, w2, e, 1.0 / top), nb, fl,
             likes=[("routed experts (sort .. down product)", lambda: moe.expert_rows(x, w1, w2, re, ra), nb, fl, tensor)])
    return rows


def _configs(width: int, layers: int) -> dict:
    """Divadra, and a Pofadra model of equal width, depth, attention heads, recurrent state, experts and vocabulary."""
    from litevllm_b200.models.presets import divadra_config, pofadra_config
    m, a, r, ff, (E, top, eff) = SIZES[width]
    pattern = ("pmsfpmpm" * layers)[:2 * layers]
    ours = divadra_config(width, 32000, pattern, m, a, r, ff, (E, top, eff))
    state_space = divadra_config(width, 32000, ("sm" * layers)[:2 * layers], m, a, r, ff, (E, top, eff))
    LH = max(1, width // 128)
    pofadra = pofadra_config(width, 32000, ("ddda" * layers)[:layers], (a[0], a[1], a[2], a[4], a[5]), (LH, LH, 128, 128, 4), (E, top, 4, 2, eff))
    return {"divadra": ours, "divadra, state space only": state_space, "pofadra": pofadra}


def run(sizes, kernels: bool = True, models: bool = True, only: str = "") -> dict:
    import torch
    torch.cuda.set_device(0)
    out = {"metric": "Divadra kernels and throughput beside the closest models", "peaks": _peaks(), "tokens": TOKENS}
    if kernels:
        with torch.inference_mode():
            out["kernels"] = [r for w in sizes for r in kernel_rows(w, only=only)]
    if models:
        out["models"] = [throughput_row(w, name, cfg, layers=8) for w in sizes for name, cfg in _configs(w, 8).items()]
    return out


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("--kernels", action="store_true")
    ap.add_argument("--models", action="store_true")
    ap.add_argument("--sizes", type=int, nargs="*", default=sorted(SIZES))
    ap.add_argument("--only", default="", help="kernel cases whose name contains this (without the like kernels)")
    ap.add_argument("--json", default=None)
    a = ap.parse_args()
    both = a.kernels == a.models
    res = run(a.sizes, a.kernels or both, a.models or both, a.only)
    for r in res.get("kernels", []):
        print(f"{r['width']:5d} {r['kernel']:78s} {r['us']:9.1f} us  {r['x_roofline']:7.2f} x roofline"
              + "".join(f"   | {k['kernel']:36s} {k['us']:9.1f} us {k['x_roofline']:7.2f} x" for k in r.get("likes", [])))
    for r in res.get("models", []):
        print(r)
    if a.json:
        Path(a.json).write_text(json.dumps(res, indent=1))


if __name__ == "__main__":
    main()
