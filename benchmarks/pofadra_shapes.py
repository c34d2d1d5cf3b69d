"""Kernels and throughput of the Pofadra design at sizes that resemble a real model's layers, beside the like kernels of
the closest models the framework served before (Qwen3.5-style MoE hybrids: gated delta rule, gated attention, routed
experts; HGRN2 for the recurrence) and beside a Qwen3.5-style MoE hybrid of equal width, depth, experts and vocabulary.
Random weights, one GPU.

    python benchmarks/pofadra_shapes.py [--kernels] [--models] [--sizes 1024 2048 4096] [--only TEXT] [--json out.json]

A kernel's roofline time is the larger of its algorithmic bytes over the measured copy bandwidth and its FLOPs over the
measured product rate (MEASURED_PEAKS.json); "x roofline" is the measured time over that.  Caches are flushed between
iterations; times are medians from CUDA events.  ``python bench.py --pofadra`` prints the same as one JSON line.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

ROOT = Path(__file__).resolve().parents[1]
if str(ROOT) not in sys.path:
    sys.path.insert(0, str(ROOT))

from benchmarks.fimodra_shapes import BATCH, CONTEXT, FP32_TFLOPS, TOKENS, Timer, _peaks, throughput_row  # noqa: E402

# width: attention (heads, kv heads, dim, rotated, window), delta heads (128 x 128 states, 4 taps), experts (count, chosen,
# groups, kept groups, ff)
SIZES = {1024: ((8, 2, 128, 64, 512), 8, (16, 4, 4, 2, 512)), 2048: ((16, 4, 128, 64, 1024), 16, (32, 4, 4, 2, 768)),
         4096: ((32, 8, 128, 64, 2048), 32, (64, 6, 8, 4, 1024))}


def kernel_rows(width: int, iters: int = 10, only: str = "") -> list[dict]:
    import torch

    from litevllm_b200 import ops
    from litevllm_b200.layers.fused_moe.fused_moe import fused_moe
    from litevllm_b200.layers.rope import get_cos_sin
    from litevllm_b200.ops import linear_attn as lin
    from litevllm_b200.ops import moe, qk_attn
    from litevllm_b200.ops import residual_stream as rs
    hbm, tensor, _ = _peaks()
    time_us = Timer(torch, iters)
    (H, G, dim, rot, window), LH, (E, top, groups, keep, ff) = SIZES[width]
    W, T, B, ctx, d, dv, taps = width, TOKENS, BATCH, CONTEXT, 128, 128, 4
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

    # ---- layer boundary beside RMSNorm with its residual add, and beside the weighted sum of experts on its own
    for n, tag in ((T, "prefill"), (B, "decode")):
        y, x, w, ys = rnd(n, W), rnd(n, W, dtype=f32), rnd(W, dtype=f32), rnd(n * top, W)
        order = torch.randperm(n * top, generator=g, device="cuda").to(torch.int32).view(n, top)
        routed = moe.RoutedRows(ys, torch.rand(n, top, generator=g, device="cuda"), order)
        res, wb = rnd(n, W), rnd(W)
        like = ("RMSNorm + residual", lambda: ops.rmsnorm(y, wb, 1e-6, residual=res), n * W * 8, 0, tensor)
        case(f"layer boundary (mixer + {top} experts + norm), {tag}", lambda: rs.add(y, x, routed, w, 1e-6, 1, x, bf), n * W * (12 + 2 * top), likes=[like])
        case(f"layer boundary without experts, {tag}", lambda: rs.add(y, x, None, w, 1e-6, 1, x, bf), n * W * 12, likes=[like])
        del ys
    # ---- delta rule beside the gated delta rule and HGRN2
    conv, rate, bias = rnd(LH * (2 * d + dv), taps, dtype=f32), torch.rand(LH, generator=g, device="cuda"), rnd(LH * d, dtype=f32)
    m = lin.DeltaSpec(LH, LH, d, dv, conv, rate, bias)
    for lens in ([1024] * 8, [8192]):
        n = sum(lens)
        x, z, b = rnd(n, m.channels), rnd(n, LH * d, dtype=f32), rnd(n, LH, dtype=f32)
        pool, ring = torch.zeros(len(lens), LH, d, dv, device="cuda"), torch.zeros(len(lens), taps, m.channels, device="cuda")
        cu = i32([sum(lens[:i]) for i in range(len(lens) + 1)])
        slots, ln, base = i32(list(range(len(lens)))), i32(lens), lin.delta_chunks(cu)
        nc = sum(-(-k // lin.DELTA_CHUNK) for k in lens)
        qq, kk, vv = rnd(n, LH, d, dtype=f32), rnd(n, LH, d, dtype=f32, std=0.1), rnd(n, LH, dv, dtype=f32)
        gg, bb = -rnd(n, LH, dtype=f32).abs(), torch.rand(n, LH, generator=g, device="cuda")

        def gated_delta():
            for s, k in enumerate(lens):
                r = slice(s * lens[0], s * lens[0] + k)
                lin.gated_delta_chunked(qq[r], kk[r], vv[r], gg[r], bb[r], pool[s])
        hq, hf = rnd(n, LH * (d + dv)), rnd(n, LH * d, dtype=f32)
        lower = torch.rand(LH * d, generator=g, device="cuda")
        hgrn2 = lambda: lin.hgrn2_scan(hq[:, :LH * d], hf, hq[:, LH * d:], bias, lower, pool, slots, cu, ln, LH, d, dv)
        case(f"delta rule, {len(lens)} x {lens[0]} (convolution .. state)",
             lambda: lin.delta_portions(x, z, b, m, pool, ring, slots, cu, ln, base, nc), n * LH * (d * 8 + dv * 6 + 4), n * LH * d * dv * 7.0, FP32_TFLOPS,
             likes=[("gated delta rule, chunked", gated_delta, n * LH * (d * 8 + dv * 8 + 8), n * LH * d * dv * 7.0, FP32_TFLOPS),
                    ("HGRN2 scan", hgrn2, n * LH * (d * 6 + dv * 6), n * LH * d * dv * 5.0, FP32_TFLOPS)])
        if len(lens) == 1:
            o, w, gate = rnd(n, LH, dv, dtype=f32), rnd(dv, dtype=f32), rnd(n, LH * dv)
            case("head norm with gate", lambda: lin.head_norm(o, w, 1e-6, bf, gate), n * LH * dv * 8,
                 likes=[("head norm", lambda: lin.head_norm(o, w, 1e-6, bf), n * LH * dv * 6, 0, tensor)])
            del o, gate
        del x, z, qq, kk, vv, hq, hf
    pool, ring = torch.zeros(256, LH, d, dv, device="cuda"), torch.zeros(256, taps, m.channels, device="cuda")
    for n in (B, 128):
        x, zg, b, w = rnd(n, m.channels), rnd(n, LH * (d + dv), dtype=f32), rnd(n, LH, dtype=f32), rnd(dv, dtype=f32)
        slots, ln = i32(list(range(n))), i32([100] * n)
        q3, v3, g3 = rnd(n, LH, d, dtype=f32), rnd(n, LH, dv, dtype=f32), -rnd(n, LH, dtype=f32).abs()
        h3, lower = rnd(n, LH * (2 * d + dv), dtype=f32), torch.rand(LH * d, generator=g, device="cuda")
        st = n * LH * d * dv * 8
        case(f"delta step, batch {n} (convolution .. gated norm)",
             lambda: lin.delta_step(x, zg[:, :LH * d], b, m, pool, ring, slots, ln, w, 1e-6, zg[:, LH * d:], bf), st + n * m.channels * 4 * (taps + 1),
             likes=[("gated delta rule step", lambda: lin.gated_delta_step(pool, slots, q3, q3, v3, g3, g3), st, 0, tensor),
                    ("HGRN2 step", lambda: lin.hgrn2_step(h3[:, :LH * d], h3[:, LH * (d + dv):], h3[:, LH * d:LH * (d + dv)], bias, lower, pool,
                                                          slots, ln, w, 1e-6, LH, d, dv, bf), st, 0, tensor)])
    del pool, ring
    # ---- attention, prefill
    lens = [1024] * 8
    nblk = T // 16 + 1
    kc, vc = rnd(nblk, G, 16, dim, std=0.5), rnd(nblk, G, 16, dim, std=0.5)
    table = i32([[1 + s * 64 + j for j in range(64)] for s in range(8)])
    pos, slots = i32(list(range(1024)) * 8), i32(list(range(16, T + 16)))
    cu, ln = i32([1024 * i for i in range(9)]), i32(lens)
    proj, wq, wk = rnd(T, (2 * H + G) * dim), rnd(H * dim, dtype=f32), rnd(G * dim, dtype=f32)
    sinks, cs = torch.zeros(H, device="cuda"), get_cos_sin(rot, 4096, 1e4, None, torch.device("cuda"))
    gate = proj[:, (H + G) * dim:]
    pre = lambda: qk_attn.prepare(proj, wq, wk, 1e-6, pos, cs, slots, kc, vc, H, G, dim)
    q = pre()
    qkv, qw, kw = rnd(T, (H + 2 * G) * dim), rnd(dim), rnd(dim)
    like_pre = lambda: ops.rope_and_cache(qkv, pos, cs, slots, kc, vc, H, G, dim, rot, q_norm_w=qw, k_norm_w=kw, qk_norm_mode=1)
    pairs, causal = 8 * sum(min(i + 1, window) for i in range(1024)), 8 * 1024 * 1025 // 2
    io = T * (2 * H + 2 * G) * dim * 2
    attn = lambda: ops.paged_attention_prefill(q.view(T, -1), kc, vc, table, ln, cu, 1024, H, G, dim, 0.1, window, sinks=sinks, v_dim=dim, gate=gate)
    like_attn = lambda: ops.paged_attention_prefill(q.view(T, -1), kc, vc, table, ln, cu, 1024, H, G, dim, 0.1)
    case("queries, keys, values: norm, rotation, cache rows, prefill", pre, T * (2 * H + 3 * G) * dim * 2,
         likes=[("rotary + head norms + cache rows", like_pre, T * (2 * H + 4 * G) * dim * 2, 0, tensor)])
    case(f"attention, prefill 8 x 1024, window {window}, sink and gate", attn, io + T * H * dim * 2, 4.0 * pairs * H * dim,
         likes=[("attention, prefill 8 x 1024, causal", like_attn, io, 4.0 * causal * H * dim, tensor)])
    # ---- attention, decode
    nb = B * ctx // 16 + 1
    kc, vc = rnd(nb, G, 16, dim, std=0.5), rnd(nb, G, 16, dim, std=0.5)
    table = i32([[1 + s * (ctx // 16) + j for j in range(ctx // 16)] for s in range(B)])
    qd, gd, ln = rnd(B, H * dim), rnd(B, H * dim), i32([ctx] * B)
    seen = min(window, ctx)
    short = i32([seen] * B)            # the like call has no window: a context of as many tokens
    case(f"attention, decode batch {B}, window {window}, sink and gate",
         lambda: ops.paged_attention_decode(qd, kc, vc, table, ln, H, G, dim, 0.1, window, max_kv_len=ctx, sinks=sinks, v_dim=dim, gate=gd),
         B * seen * G * dim * 4, 4.0 * B * seen * H * dim,
         likes=[(f"attention, decode, context {seen}", lambda: ops.paged_attention_decode(qd, kc, vc, table, short, H, G, dim, 0.1, max_kv_len=seen),
                 B * seen * G * dim * 4, 4.0 * B * seen * H * dim, tensor)])
    del kc, vc, proj, qkv
    # ---- routed experts
    w1, w2 = rnd(E, 2 * ff, W, std=0.03), rnd(E, W, ff, std=0.03)
    corr = rnd(E, dtype=f32, std=0.1)
    for n, tag in ((T, f"{T} tokens"), (B, f"decode batch {B}")):
        x, z = rnd(n, W), rnd(n, E, dtype=f32)
        route = lambda: moe.route(z, top, mode="sigmoid", bias=corr, renormalize=False, routed_scale=2.0, groups=groups, keep_groups=keep)
        ids, a = route()
        used = int(ids.unique().numel())
        nb, fl = used * 3 * ff * W * 2 + n * W * 2 + n * top * W * 2, 6.0 * n * top * ff * W
        case(f"routed experts, {tag} (sort .. down product)", lambda: moe.expert_rows(x, w1, w2, ids, a), nb, fl,
             likes=[("routed experts, product per expert", lambda: fused_moe(x, w1, w2, z, top), nb, fl, tensor)])
        case(f"choice of experts, {tag}", route, n * E * 4 + n * top * 8,
             likes=[("softmax choice of experts", lambda: moe.route(z, top), n * E * 4 + n * top * 8, 0, tensor)])
    return rows


def _configs(width: int, layers: int) -> dict:
    """Pofadra and Qwen3.5-style MoE configurations of equal width, depth, experts and vocabulary."""
    from litevllm_b200.models.presets import pofadra_config
    a, LH, (E, top, groups, keep, ff) = SIZES[width]
    ours = pofadra_config(width, 32000, ("ddda" * layers)[:layers], a, (LH, LH, 128, 128, 4), (E, top, groups, keep, ff))
    qwen = {"architectures": ["Qwen3_5MoeForCausalLM"], "model_type": "qwen3_5", "hidden_size": width, "num_hidden_layers": layers,
            "num_attention_heads": a[0], "num_key_value_heads": a[1], "head_dim": a[2], "intermediate_size": ff, "vocab_size": 32000,
            "rms_norm_eps": 1e-6, "rope_theta": 10000.0, "max_position_embeddings": 4096, "partial_rotary_factor": a[3] / a[2],
            "layer_types": ["full_attention" if i % 4 == 3 else "linear_attention" for i in range(layers)], "linear_num_key_heads": LH,
            "linear_num_value_heads": LH, "linear_key_head_dim": 128, "linear_value_head_dim": 128, "linear_conv_kernel_dim": 4,
            "attn_output_gate": True, "num_experts": E, "num_experts_per_tok": top, "moe_intermediate_size": ff,
            "shared_expert_intermediate_size": 0, "norm_topk_prob": True, "eos_token_id": 1}
    return {"pofadra": ours, "qwen3.5-style MoE hybrid": qwen}


def run(sizes, kernels: bool = True, models: bool = True, only: str = "") -> dict:
    import torch
    torch.cuda.set_device(0)
    out = {"metric": "Pofadra kernels and throughput beside the closest models", "peaks": _peaks(), "tokens": TOKENS}
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
