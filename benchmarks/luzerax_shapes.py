"""Kernels and throughput of the Luzerax design at sizes that resemble a real model's layers, beside the like kernels of the
models the framework served before (grouped causal attention with head norms, routed and dense gated feed-forwards, RMSNorm
with its residual add) and beside a Pofadra model of equal width, depth, heads, experts and vocabulary whose layers are all
attention over everything.  Random weights, one GPU.

    python benchmarks/luzerax_shapes.py [--kernels] [--models] [--sizes 1024 2048 4096] [--only TEXT] [--json out.json]

A kernel's roofline time is the larger of its algorithmic bytes over the measured copy bandwidth and its FLOPs over the
measured product rate (MEASURED_PEAKS.json); "x roofline" is the measured time over that.  Caches are flushed between
iterations; times are medians from CUDA events.  ``python bench.py --luzerax`` prints the same as one JSON line.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

ROOT = Path(__file__).resolve().parents[1]
if str(ROOT) not in sys.path:
    sys.path.insert(0, str(ROOT))

from benchmarks.fimodra_shapes import BATCH, CONTEXT, TOKENS, Timer, _peaks, throughput_row  # noqa: E402

# width: heads, kv heads, experts (count, pass-through outputs, chosen, groups, kept groups, ff, ff of the shared expert);
# two maps of 64 channels or one of 128 per head, values of 128
SIZES = {1024: (8, 2, (16, 4, 4, 5, 3, 512, 512)), 2048: (16, 4, (32, 8, 4, 5, 3, 768, 1024)),
         4096: (32, 8, (64, 16, 6, 10, 5, 1024, 2048))}
DIM, VDIM, ROT = 64, 128, 64


def kernel_rows(width: int, iters: int = 10, only: str = "") -> list[dict]:
    import torch

    from litevllm_b200 import ops
    from litevllm_b200.layers.head_attention import position_factor
    from litevllm_b200.layers.rope import get_cos_sin
    from litevllm_b200.ops import moe, qk_attn
    from litevllm_b200.ops import residual_stream as rs
    hbm, tensor, _ = _peaks()
    time_us = Timer(torch, iters)
    H, G, (E, ident, top, groups, keep, ff, sff) = SIZES[width]
    W, T, B, ctx, d, dv = width, TOKENS, BATCH, CONTEXT, 2 * DIM, VDIM
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

    # ---- sublayer boundaries beside RMSNorm with its residual add and beside the boundary with experts of Pofadra
    for n, tag in ((T, "prefill"), (B, "decode")):
        y, x, w, ys = rnd(n, W), rnd(n, W, dtype=f32), rnd(W, dtype=f32), rnd(n * top, W)
        order = torch.randperm(n * top, generator=g, device="cuda").to(torch.int32).view(n, top)
        a = torch.rand(n, top, generator=g, device="cuda")
        routed, some = moe.RoutedRows(ys, a, order), order.clone()
        some[:, 0] = torch.where(torch.arange(n, device="cuda") % 2 == 0, -1, some[:, 0])
        passing = moe.RoutedRows(ys, a, some, True)
        res, wb = rnd(n, W), rnd(W)
        like = ("RMSNorm + residual", lambda: ops.rmsnorm(y, wb, 1e-6, residual=res), n * W * 8, 0, tensor)
        plus = ("layer boundary with experts (Pofadra)", lambda: rs.add(y, x, routed, w, 1e-6, 1, x, bf), n * W * (12 + 2 * top), 0, tensor)
        case(f"boundary (norm, scale, stream), {tag}", lambda: rs.post(y, x, None, w, None, 1e-6, 1, x, bf), n * W * 12, likes=[like])
        case(f"boundary with shared and {top} chosen experts, {tag}", lambda: rs.post(y, x, passing, w, None, 1e-6, 1, x, bf), n * W * (12 + 2 * top), likes=[plus])
        del ys
    # ---- queries, keys, values
    nblk = T // 16 + 1
    kc, vc = rnd(nblk, G, 16, d, std=0.5), rnd(nblk, G, 16, dv, std=0.5)
    cu, ln = i32([1024 * i for i in range(9)]), i32([1024] * 8)
    table = i32([[1 + s * 64 + j for j in range(64)] for s in range(8)])
    pos, slots = i32(list(range(1024)) * 8), i32(list(range(16, T + 16)))
    dev = torch.device("cuda")
    cs, factor = get_cos_sin(ROT, 4096, 1e4, None, dev), position_factor(4096, 0.4, 256, dev)
    proj, wq = rnd(T, (H + G) * d + G * dv + H + 8)[:, :(H + G) * d + G * dv + H], rnd(DIM, dtype=f32)
    two = qk_attn.HeadSpec(H, G, DIM, dv, 2, 1e-6, d, DIM)
    one = qk_attn.HeadSpec(H, G, d, dv, 1, 1e-6, d, 0, ROT, True, True)
    qkv, qw = rnd(T, (H + G) * d + G * dv), rnd(d)
    pre2 = lambda: qk_attn.prepare_heads(proj, wq, wq, two, pos, None, factor, slots, kc, vc)
    pre1 = lambda: qk_attn.prepare_heads(proj, None, None, one, pos, cs, None, slots, kc, vc)
    like_pre = ("rotary + head norms + cache rows", lambda: ops.rope_and_cache(qkv, pos, cs, slots, kc, vc, H, G, d, ROT, q_norm_w=qw, k_norm_w=qw, qk_norm_mode=1),
                T * (2 * H + 4 * G) * d * 2, 0, tensor)
    case("two maps: head norms, factor, query and cache rows, prefill", pre2, T * (3 * H + 4 * G) * d * 2, likes=[like_pre])
    case("gated: rotation, head norms, query and cache rows, prefill", pre1, T * (2 * H + 4 * G) * d * 2, likes=[like_pre])
    # ---- attention, prefill
    q2, q1, gate = pre2().view(T, -1), pre1().view(T, -1), proj[:, (H + G) * d + G * dv:]
    diff = (0.5, 0.6, 1e-6)
    pairs = 8 * 1024 * 1025 // 2
    io = T * (2 * H + 2 * G) * d * 2
    like_attn = lambda nq: (f"attention, prefill 8 x 1024, {nq} heads", lambda: ops.paged_attention_prefill(q2[:, :nq * d], kc, vc, table, ln, cu, 1024, nq, G, d, 0.1),
                            T * (2 * nq + 2 * G) * d * 2, 4.0 * pairs * nq * d, tensor)
    case(f"differential attention, prefill 8 x 1024, {H} heads of two maps",
         lambda: ops.paged_attention_prefill(q2, kc, vc, table, ln, cu, 1024, 2 * H, G, d, 0.1, v_dim=dv, diff=diff), io,
         2.0 * pairs * 2 * H * (DIM + dv), likes=[like_attn(2 * H)])
    case(f"gated attention, prefill 8 x 1024, {H} heads",
         lambda: ops.paged_attention_prefill(q1, kc, vc, table, ln, cu, 1024, H, G, d, 0.1, v_dim=dv, gate=gate), io, 4.0 * pairs * H * d, likes=[like_attn(H)])
    long_table, long_ln, long_cu = i32([[1 + j for j in range(T // 16)]]), i32([T]), i32([0, T])
    pairs = T * (T + 1) // 2
    like_long = lambda nq: (f"attention, prefill 1 x {T}, {nq} heads",
                            lambda: ops.paged_attention_prefill(q2[:, :nq * d], kc, vc, long_table, long_ln, long_cu, T, nq, G, d, 0.1), io, 4.0 * pairs * nq * d, tensor)
    case(f"differential attention, prefill 1 x {T}, {H} heads of two maps",
         lambda: ops.paged_attention_prefill(q2, kc, vc, long_table, long_ln, long_cu, T, 2 * H, G, d, 0.1, v_dim=dv, diff=diff), io,
         2.0 * pairs * 2 * H * (DIM + dv), likes=[like_long(2 * H)])
    # ---- attention, decode
    nb = B * ctx // 16 + 1
    kc, vc = rnd(nb, G, 16, d, std=0.5), rnd(nb, G, 16, dv, std=0.5)
    table, ln = i32([[1 + s * (ctx // 16) + j for j in range(ctx // 16)] for s in range(B)]), i32([ctx] * B)
    qd, gd = rnd(B, 2 * H * d), rnd(B, H)
    kv = B * ctx * G * (d + dv) * 2
    like_dec = lambda nq: (f"attention, decode, context {ctx}, {nq} heads", lambda: ops.paged_attention_decode(qd[:, :nq * d], kc, vc, table, ln, nq, G, d, 0.1, max_kv_len=ctx),
                           kv, 4.0 * B * ctx * nq * d, tensor)
    case(f"differential attention, decode batch {B}, context {ctx}",
         lambda: ops.paged_attention_decode(qd, kc, vc, table, ln, 2 * H, G, d, 0.1, max_kv_len=ctx, v_dim=dv, diff=diff), kv, likes=[like_dec(2 * H)])
    case(f"gated attention, decode batch {B}, context {ctx}",
         lambda: ops.paged_attention_decode(qd[:, :H * d], kc, vc, table, ln, H, G, d, 0.1, max_kv_len=ctx, v_dim=dv, gate=gd), kv, likes=[like_dec(H)])
    pos_d, slots_d = i32([ctx - 1] * B), i32([16 + s * ctx for s in range(B)])
    like_pre = ("rotary + head norms + cache rows", lambda: ops.rope_and_cache(qkv[:B], pos_d, cs, slots_d, kc, vc, H, G, d, ROT, q_norm_w=qw, k_norm_w=qw, qk_norm_mode=1),
                B * (2 * H + 4 * G) * d * 2, 0, tensor)
    case("two maps: head norms, factor, query and cache rows, decode", lambda: qk_attn.prepare_heads(proj[:B], wq, wq, two, pos_d, None, factor, slots_d, kc, vc),
         B * (3 * H + 4 * G) * d * 2, likes=[like_pre])
    case("gated: rotation, head norms, query and cache rows, decode", lambda: qk_attn.prepare_heads(proj[:B], None, None, one, pos_d, cs, None, slots_d, kc, vc),
         B * (2 * H + 4 * G) * d * 2, likes=[like_pre])
    del kc, vc, proj, qkv
    # ---- feed-forward
    w1, w2 = rnd(E, 2 * ff, W, std=0.03), rnd(E, W, ff, std=0.03)
    s1 = rnd(2 * sff, W, std=0.03)
    corr = rnd(E + ident, dtype=f32, std=0.02)
    for n, tag in ((T, f"{T} tokens"), (B, f"decode batch {B}")):
        x, z = rnd(n, W), rnd(n, E + ident, dtype=f32)
        route = lambda: moe.route(z, top, bias=corr, groups=groups, keep_groups=keep, group_best=1)
        ids, a = route()
        real = int((ids < E).sum())
        used = int(ids[ids < E].unique().numel())
        nb, fl = used * 3 * ff * W * 2 + n * W * 2 + real * W * 2, 6.0 * real * ff * W
        ids_all, a_all = moe.route(z[:, :E], top)
        nb_all, fl_all = int(ids_all.unique().numel()) * 3 * ff * W * 2 + n * W * 2 + n * top * W * 2, 6.0 * n * top * ff * W
        case(f"clipped experts, {tag} (sort .. down product)", lambda: moe.expert_rows(x, w1, w2, ids, a, "clipped_swiglu", 7.0, True), nb, fl,
             likes=[("silu experts", lambda: moe.expert_rows(x, w1, w2, ids_all, a_all), nb_all, fl_all, tensor)])
        pofadra_like = ("sigmoid choice within groups (Pofadra)", lambda: moe.route(z, top, mode="sigmoid", bias=corr, groups=groups, keep_groups=keep),
                        n * (E + ident) * 4 + n * top * 8, 0, tensor)
        case(f"choice of experts, {tag}", route, n * (E + ident) * 4 + n * top * 8,
             likes=[("softmax choice of experts", lambda: moe.route(z, top), n * (E + ident) * 4 + n * top * 8, 0, tensor), pofadra_like])
        nb = 2 * sff * W * 2 + n * (W + sff) * 2
        case(f"clipped gated product, {tag}", lambda: ops.gated_linear(x, s1, "clipped_swiglu", act_limit=7.0), nb, 4.0 * n * sff * W,
             likes=[("silu gated product", lambda: ops.gated_linear(x, s1), nb, 4.0 * n * sff * W, tensor)])
    return rows


def _configs(width: int, layers: int) -> dict:
    """Luzerax and Pofadra configurations of equal width, depth, heads, experts and vocabulary; the second Luzerax has no
    shared expert and no pass-through outputs, like Pofadra."""
    from litevllm_b200.models.presets import luzerax_config, pofadra_config
    H, G, (E, ident, top, groups, keep, ff, sff) = SIZES[width]
    attn = ((H, G, DIM, VDIM), (H, G, 2 * DIM, VDIM, ROT))
    ours = luzerax_config(width, 32000, ("dmgm" * layers)[:2 * layers], *attn, 0, (E, ident, top, groups, keep, ff, sff))
    bare = luzerax_config(width, 32000, ("dmgm" * layers)[:2 * layers], *attn, 0, (E, 0, top, 4, 2, ff, sff))
    for l in bare["layers"]:
        l["mlp"].pop("shared")
    pofadra = pofadra_config(width, 32000, "a" * layers, (H, G, 2 * DIM, ROT, 1 << 20), (2, 2, 64, 64, 2), (E, top, 4, 2, ff))
    return {"luzerax": ours, "luzerax, no shared expert": bare, "pofadra, attention only": pofadra}


def run(sizes, kernels: bool = True, models: bool = True, only: str = "") -> dict:
    import torch
    torch.cuda.set_device(0)
    out = {"metric": "Luzerax kernels and throughput beside the closest models", "peaks": _peaks(), "tokens": TOKENS}
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
        print(f"{r['width']:5d} {r['kernel']:62s} {r['us']:9.1f} us  {r['x_roofline']:7.2f} x roofline"
              + "".join(f"   | {k['kernel']:36s} {k['us']:9.1f} us {k['x_roofline']:7.2f} x" for k in r.get("likes", [])))
    for r in res.get("models", []):
        print(r)
    if a.json:
        Path(a.json).write_text(json.dumps(res, indent=1))


if __name__ == "__main__":
    main()
