"""Kernels and throughput of the Fimodra design at sizes that resemble a real model's layers, beside the like kernels of
the models the framework served before (DeepSeek-style latent attention, the gated delta rule, RMSNorm) and beside a
Qwen3.5-style hybrid decoder of equal width, depth, feed-forward and vocabulary.  Random weights, one GPU.

    python benchmarks/fimodra_shapes.py [--kernels] [--models] [--sizes 1024 2048 4096] [--only TEXT] [--json out.json]

A kernel's roofline time is the larger of its algorithmic bytes over the measured copy bandwidth and its FLOPs over the
measured product rate (MEASURED_PEAKS.json); "x roofline" is the measured time over that.  Caches are flushed between
iterations; times are medians from CUDA events.  ``python bench.py --fimodra`` prints the same as one JSON line.
"""
from __future__ import annotations

import argparse
import gc
import json
import statistics
import sys
from pathlib import Path

ROOT = Path(__file__).resolve().parents[1]
if str(ROOT) not in sys.path:
    sys.path.insert(0, str(ROOT))

# width: heads, dim, rot, vdim, rank, window, linear heads (128 x 128 states), feed-forward
SIZES = {1024: (8, 48, 16, 64, 256, 512, 8, 2816), 2048: (16, 96, 32, 128, 512, 1024, 16, 5632),
         4096: (32, 96, 32, 128, 512, 2048, 32, 11264)}
TOKENS, BATCH, CONTEXT = 8192, 32, 2048
FP32_TFLOPS = 73.0      # 148 SMs x 128 lanes x 2 x 1.93 GHz: what 32-bit recurrences run against


def _peaks():
    p = ROOT / "MEASURED_PEAKS.json"
    d = json.loads(p.read_text()) if p.exists() else {}
    return float(d.get("hbm_gbs", 6650.0)), float(d.get("bf16_tflops", 1590.0)), "measured" if p.exists() else "fallback"


class Timer:
    def __init__(self, torch, iters: int):
        self.torch, self.iters = torch, iters
        self.flush = torch.empty(192 << 20, dtype=torch.uint8, device="cuda")

    def __call__(self, fn) -> float:
        """Median microseconds of one call."""
        t = self.torch
        for _ in range(3):
            fn()
        out = []
        for _ in range(self.iters):
            self.flush.zero_()
            a, b = t.cuda.Event(enable_timing=True), t.cuda.Event(enable_timing=True)
            a.record()
            fn()
            b.record()
            t.cuda.synchronize()
            out.append(a.elapsed_time(b) * 1e3)
        return statistics.median(out)


def kernel_rows(width: int, iters: int = 10, only: str = "") -> list[dict]:
    import torch

    from litevllm_b200 import ops
    from litevllm_b200.layers.rope import get_cos_sin
    from litevllm_b200.ops import _lib, _p, _stream
    from litevllm_b200.ops import latent_attn as la
    from litevllm_b200.ops import linear_attn as lin
    from litevllm_b200.ops import residual_stream as rs
    hbm, tensor, _ = _peaks()
    time_us = Timer(torch, iters)
    H, dim, rot, vdim, rank, window, LH, _ = SIZES[width]
    W, T, B, ctx, d, dv = width, TOKENS, BATCH, CONTEXT, 128, 128
    kd, hd = rank + rot, next(h for h in (64, 128, 256) if max(dim + rot, vdim) <= h)
    g = torch.Generator(device="cuda").manual_seed(0)
    bf, f32 = torch.bfloat16, torch.float32

    def rnd(*s, dtype=bf, std=1.0):
        return (torch.randn(*s, generator=g, device="cuda") * std).to(dtype)

    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    rows = []

    def case(name, fn, nbytes, flops=0.0, peak=tensor, like=None):
        if only not in name:
            return
        us = time_us(fn)
        roof = max(nbytes / (hbm * 1e3), flops / (peak * 1e6))
        r = {"width": width, "kernel": name, "us": round(us, 1), "roofline_us": round(roof, 1), "x_roofline": round(us / roof, 2)}
        if like is not None and not only:
            lname, lfn, lbytes, lflops, lpeak = like
            lus = time_us(lfn)
            lroof = max(lbytes / (hbm * 1e3), lflops / (lpeak * 1e6))
            r.update(like=lname, like_us=round(lus, 1), like_roofline_us=round(lroof, 1), like_x_roofline=round(lus / lroof, 2))
        rows.append(r)

    # ---- stream boundaries (prefill and decode) beside RMSNorm with its residual add
    for n, tag in ((T, "prefill"), (B, "decode")):
        y, x, w = rnd(n, W), rnd(n, W, dtype=f32), rnd(W, dtype=f32)
        out, res, wb = torch.empty_like(x), rnd(n, W), rnd(W)
        hist, avg = rnd(9, n, W, dtype=f32), rnd(9, dtype=f32)
        like = ("RMSNorm + residual", lambda: ops.rmsnorm(y, wb, 1e-6, residual=res), n * W * 8, 0, tensor)
        case(f"stream step, {tag}", lambda: rs.step(y, x, w, w, 1e-6, 2, out, bf), n * W * 12, like=like)
        case(f"stream average of 9, {tag}", lambda: rs.average(y, x, w, w, 1e-6, 2, hist, 8, avg, out, bf), n * W * (16 + 32), like=like)
        del hist
    # ---- HGRN2 beside the gated delta rule
    for lens in ([1024] * 8, [8192]):
        n = sum(lens)
        qv, f = rnd(n, LH * (d + dv)), rnd(n, LH * d, dtype=f32)
        bias, lower = rnd(LH * d, dtype=f32), torch.rand(LH * d, generator=g, device="cuda")
        pool = torch.zeros(len(lens), LH, d, dv, device="cuda")
        cu = i32([sum(lens[:i]) for i in range(len(lens) + 1)])
        slots, ln = i32(list(range(len(lens)))), i32(lens)
        scan = lambda: lin.hgrn2_scan(qv[:, :LH * d], f, qv[:, LH * d:], bias, lower, pool, slots, cu, ln, LH, d, dv)
        qq, kk, vv = rnd(n, LH, d, dtype=f32), rnd(n, LH, d, dtype=f32, std=0.1), rnd(n, LH, dv, dtype=f32)
        gg, bb = -rnd(n, LH, dtype=f32).abs(), torch.rand(n, LH, generator=g, device="cuda")

        def delta():
            for b, m in enumerate(lens):
                s = slice(b * lens[0], b * lens[0] + m)
                lin.gated_delta_chunked(qq[s], kk[s], vv[s], gg[s], bb[s], pool[b])
        nb = n * LH * (d * 6 + dv * 6)
        case(f"HGRN2 scan, {len(lens)} x {lens[0]}", scan, nb, n * LH * d * dv * 5.0, FP32_TFLOPS,
             like=("gated delta rule, chunked", delta, n * LH * (d * 8 + dv * 8 + 8), n * LH * d * dv * 7.0, FP32_TFLOPS))
        o = scan()
        w = rnd(dv, dtype=f32)
        if len(lens) == 1:
            case("head norm", lambda: lin.head_norm(o, w, 1e-6, bf), n * LH * dv * 6)
        del qv, f, qq, kk, vv, o
    pool = torch.zeros(256, LH, d, dv, device="cuda")
    for b in (B, 128):
        p, w = rnd(b, LH * (2 * d + dv), dtype=f32), rnd(dv, dtype=f32)
        slots, ln = i32(list(range(b))), i32([100] * b)
        q3, v3 = rnd(b, LH, d, dtype=f32), rnd(b, LH, dv, dtype=f32)
        g3 = -rnd(b, LH, dtype=f32).abs()
        st = b * LH * d * dv * 8
        case(f"HGRN2 step, batch {b}",
             lambda: lin.hgrn2_step(p[:, :LH * d], p[:, LH * (d + dv):], p[:, LH * d:LH * (d + dv)], bias, lower, pool, slots, ln, w, 1e-6, LH, d, dv, bf),
             st, like=("gated delta rule step", lambda: lin.gated_delta_step(pool, slots, q3, q3, v3, g3, g3), st, 0, tensor))
    del pool
    # ---- latent attention, prefill: everything between the q|dkv product and the output projection
    lens = [1024] * 8
    nblk = T // 16 + 1
    cache, cache576 = rnd(nblk, 1, 16, kd, std=0.5), rnd(nblk, 1, 16, 576, std=0.5)
    table = i32([[1 + b * 64 + j for j in range(64)] for b in range(8)])
    pos, slots = i32(list(range(1024)) * 8), i32(list(range(16, T + 16)))
    cu, ln = i32([1024 * i for i in range(9)]), i32(lens)
    proj, up = rnd(T, H * (dim + rot) + kd), rnd(H * (dim + vdim), rank, std=0.05)
    nw, sinks = rnd(rank, dtype=f32), rnd(H, dtype=f32)
    cs = get_cos_sin(rot, 4096, 1e4, None, torch.device("cuda"))
    qp = torch.empty(T, H, hd, dtype=bf, device="cuda")
    plan = la.ContextPlan(table, 16, lens, lens, window, torch.device("cuda"))
    pre = lambda: la.prepare(proj[:, :H * (dim + rot)], proj[:, H * (dim + rot):], nw, 1e-6, pos, cs, slots, cache, qp, H, dim, rot, rank, 0, dim)
    pre()
    pools = la.context_pool(plan, cache, up, H, dim, rot, vdim, rank, hd)

    def attn():
        return ops.paged_attention_prefill(qp.view(T, -1), *pools, plan.table, plan.lens, cu, 1024, H, H, hd, 0.1, window, sinks=sinks, v_dim=vdim)

    def whole():
        pre()
        la.context_pool(plan, cache, up, H, dim, rot, vdim, rank, hd)
        attn()
    pairs = 8 * sum(min(i + 1, window) for i in range(1024))
    up_fl = 2.0 * T * rank * H * (dim + vdim)
    at_fl = 2.0 * pairs * H * (dim + rot + vdim)
    io = T * (H * (dim + rot) + kd + H * vdim) * 2
    # the DeepSeek form at the same heads: 512 + 64 latent rows, per-head tiles padded to 256 channels
    qpad, kvb = rnd(T, H * 256), rnd(H * 256, 512, std=0.05)
    tmp = [torch.empty(T // 16, H, 16, 256, dtype=bf, device="cuda").normal_(0, 0.5) for _ in range(2)]
    tbt = i32([[b * 64 + j for j in range(64)] for b in range(8)])
    ctx_rows = cache576.view(-1, 576)[16:16 + T]
    tslots = i32(list(range(T)))

    def like_whole():
        kv = ops.linear(ctx_rows[:, :512].contiguous(), kvb)
        _lib.check(_lib.kernels().fi_mla_ctx_to_pool(_p(ctx_rows), _p(kv), _p(tslots), _p(tmp[0]), _p(tmp[1]), T, H, 128, 128, 256, 16, 0, _stream()), "pool")
        ops.paged_attention_prefill(qpad, tmp[0], tmp[1], tbt, ln, cu, 1024, H, H, 256, 0.1)
    causal = 8 * 1024 * 1025 // 2
    lfl = 2.0 * T * 512 * H * 256 + 2.0 * causal * H * (192 + 128)
    case("latent attention, prefill 8 x 1024 (prepare .. attention)", whole, io, up_fl + at_fl,
         like=("DeepSeek MLA prefill", like_whole, T * (H * 192 + 576 + H * 128) * 2, lfl, tensor))
    like_attn = lambda: ops.paged_attention_prefill(qpad, tmp[0], tmp[1], tbt, ln, cu, 1024, H, H, 256, 0.1)
    case("  of which the attention kernel", attn, T * H * hd * 8, at_fl,
         like=("DeepSeek MLA prefill attention kernel", like_attn, T * H * 256 * 8, 2.0 * causal * H * 320, tensor))
    case("  of which prepare", pre, T * (2 * H * (dim + rot) + 2 * kd) * 2)
    case("  of which gather + up-projection + tiles", lambda: la.context_pool(plan, cache, up, H, dim, rot, vdim, rank, hd),
         T * (kd + H * (dim + rot + vdim)) * 2, up_fl)
    del tmp, qpad, pools
    # ---- latent attention, decode rows
    nb = B * ctx // 16 + 1
    cache, cache576 = rnd(nb, 1, 16, kd, std=0.5), rnd(nb, 1, 16, 576, std=0.5)
    table = i32([[1 + b * (ctx // 16) + j for j in range(ctx // 16)] for b in range(B)])
    qc, q5, ln = rnd(B, H, kd), rnd(B, H, 576), i32([ctx] * B)
    seen = min(window, ctx)
    short = i32([seen] * B)            # the like kernel has no window: a context of as many tokens
    case(f"latent attention rows, decode batch {B}, window {window}",
         lambda: la.attend_rows(qc, cache, table, ln, None, rank, 0.1, window, sinks, ctx), B * seen * kd * 2, 2.0 * B * seen * H * (kd + rank),
         like=(f"DeepSeek MLA decode, context {seen}", lambda: la.attend_rows(q5, cache576, table, short, None, 512, 0.1, 0, None, seen),
               B * seen * 576 * 2, 2.0 * B * seen * H * (576 + 512), tensor))
    return rows


def _configs(width: int, layers: int) -> dict:
    """Fimodra and Qwen3.5-style configurations of equal width, depth, feed-forward and vocabulary."""
    from litevllm_b200.models.presets import fimodra_config
    H, dim, rot, vdim, rank, window, LH, ff = SIZES[width]
    ours = fimodra_config(width, 32000, ff, ("aaha" * layers)[:layers], H, dim, rot, vdim, rank, window, LH, 128, 128, groups=2)
    qwen = {"architectures": ["Qwen3_5ForCausalLM"], "model_type": "qwen3_5", "hidden_size": width, "num_hidden_layers": layers,
            "num_attention_heads": width // 128, "num_key_value_heads": max(1, width // 512), "head_dim": 128, "intermediate_size": ff,
            "vocab_size": 32000, "rms_norm_eps": 1e-6, "rope_theta": 10000.0, "max_position_embeddings": 4096, "partial_rotary_factor": 0.5,
            "layer_types": ["linear_attention" if i % 4 == 2 else "full_attention" for i in range(layers)], "linear_num_key_heads": LH,
            "linear_num_value_heads": LH, "linear_key_head_dim": 128, "linear_value_head_dim": 128, "linear_conv_kernel_dim": 4,
            "attn_output_gate": True, "eos_token_id": 1}
    return {"fimodra": ours, "qwen3.5-style hybrid": qwen}


def throughput_row(width: int, name: str, cfg: dict, layers: int = 8, batch: int = 32, prompt: int = 1024, steps: int = 64) -> dict:
    """Prefill tokens/s of ``8 x prompt`` token steps and decode tokens/s at ``batch`` through the engine."""
    import torch

    from litevllm_b200 import LLM, SamplingParams
    from litevllm_b200.models.presets import PRESETS
    PRESETS["shape-comparison"] = cfg
    llm = LLM("synthetic:shape-comparison", dtype="bfloat16", max_num_seqs=batch, max_model_len=prompt + steps + 64,
              max_num_batched_tokens=8192, fastinference_config={"profile": "throughput", "tuning_keyvals": {
                  "FASTINFERENCE_KV_MAX_ACTIVE_REQUESTS": str(batch), "FASTINFERENCE_LITE_PREFILL_MICROBATCH": "8",
                  "FASTINFERENCE_GPU_GREEDY_SAMPLING": "0", "FASTINFERENCE_PREFIX_CACHE_MAX_ENTRIES": "0"}})
    eng = llm.engine
    g = torch.Generator().manual_seed(1)
    ids = torch.randint(0, 32000, (batch, prompt), generator=g).tolist()
    times = []
    for rep in range(3):
        sp = SamplingParams(temperature=0.0, max_tokens=1, ignore_eos=True)
        for i in range(batch):
            eng.add_request(f"p{rep}-{i}", ids[i], sp)
        torch.cuda.synchronize()
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        while eng.has_unfinished_requests():
            eng.step()
        b.record()
        torch.cuda.synchronize()
        times.append(a.elapsed_time(b))
    prefill = batch * prompt / (min(times[1:]) / 1e3)
    sp = SamplingParams(temperature=0.0, max_tokens=steps + 32, ignore_eos=True)
    for i in range(batch):
        eng.add_request(f"d-{i}", ids[i], sp)
    while any(st.is_prefill for st in eng.scheduler.requests.values()):
        eng.step()
    for _ in range(8):
        eng.step()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    n = 0
    a.record()
    for _ in range(steps):
        n += len(eng.step())
    b.record()
    torch.cuda.synchronize()
    ms = a.elapsed_time(b)
    row = {"width": width, "layers": layers, "model": name, "prefill_tok_s": round(prefill), "decode_tok_s": round(n / (ms / 1e3)),
           "decode_ms_per_step": round(ms / steps, 3), "batch": batch, "prompt": prompt,
           "params_m": round(sum(p.numel() for p in eng.model.parameters()) / 1e6),
           "kernels_per_decode_step": eng.decode_executor.launches_per_graph.get(eng.builder.bucket_for(batch))}
    while eng.has_unfinished_requests():
        eng.step()
    llm.shutdown()
    del llm, eng
    PRESETS.pop("shape-comparison")
    gc.collect()
    torch.cuda.empty_cache()
    return row


def model_rows(width: int, layers: int = 8) -> list[dict]:
    return [throughput_row(width, name, cfg, layers) for name, cfg in _configs(width, layers).items()]


def run(sizes, kernels: bool = True, models: bool = True, only: str = "") -> dict:
    import torch
    torch.cuda.set_device(0)
    out = {"metric": "Fimodra kernels and throughput beside the closest models", "peaks": _peaks(), "tokens": TOKENS}
    if kernels:
        with torch.inference_mode():
            out["kernels"] = [r for w in sizes for r in kernel_rows(w, only=only)]
    if models:
        out["models"] = [r for w in sizes for r in model_rows(w)]
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
        print(f"{r['width']:5d} {r['kernel']:58s} {r['us']:9.1f} us  {r['x_roofline']:7.2f} x roofline"
              + (f"   | {r['like']:38s} {r['like_us']:9.1f} us {r['like_x_roofline']:7.2f} x" if "like" in r else ""))
    for r in res.get("models", []):
        print(r)
    if a.json:
        Path(a.json).write_text(json.dumps(res, indent=1))


if __name__ == "__main__":
    main()
