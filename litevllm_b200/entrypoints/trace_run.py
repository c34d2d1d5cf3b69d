"""Replays a trace of token ids through a model, step by step, and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Steps arrive on standard input, one JSON object a line::

    {"step": 7, "entries": [{"id": "q1", "tokens": [12, 9], "want": [1]}, {"id": "q2", "tokens": [4], "want": []}], "end": ["q1"]}

All entries of a step run as one batch of the engine, portions of prompts beside single tokens, through the executors,
the paged cache and the state slots that generation uses; nothing is sampled.  A step that wants logits leaves
``<step>.f32`` in ``--out`` (fp32 [wanted, vocab], in the order of the entries and of ``want``).  After every step a
line ``done <step>`` is printed.  The cache pool holds ``--max-tokens`` tokens, shared by at most four live requests.
Needs a GPU; kernels that are not built yet are compiled first.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

MAX_LIVE = 4


def _ensure_kernels(model: str) -> None:
    """Build what the model's family needs, unless the full library is there."""
    from .._C import build
    if build.full_library_is_current():
        return
    from ..models.arch import arch_from_hf_config
    from ..ops import _lib
    family = arch_from_hf_config(json.loads((Path(model) / "config.json").read_text())).family
    if family in build.KERNEL_SETS:
        _lib.use_kernel_library(build.build_set(family, verbose=False))
    else:
        build.build_all(verbose=False)


def make_engine(model: str, dtype: str, max_tokens: int, device: str = "auto"):
    from ..config.config_builder import build_vllm_config
    from ..engine.lite_engine import LiteEngine
    tokens = max(64, (max_tokens + 63) // 64 * 64)
    cfg = build_vllm_config(model, dtype=dtype, max_model_len=tokens, max_num_seqs=MAX_LIVE, max_num_batched_tokens=tokens,
                            device=device, fastinference_config={"tuning_keyvals": {
                                "FASTINFERENCE_KV_POOL_TOKENS": str(tokens),
                                "FASTINFERENCE_KV_MAX_ACTIVE_REQUESTS": str(MAX_LIVE)}})
    return LiteEngine(cfg)


def replay(engine, lines, out_dir: Path, emit) -> None:
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(str(e["id"]), [int(t) for t in e["tokens"]], [int(w) for w in e.get("want", [])])
                   for e in step["entries"]]
        logits = engine.replay_step(entries, [str(i) for i in step.get("end", [])])
        if logits is not None:
            (out_dir / f"{int(step['step'])}.f32").write_bytes(logits.cpu().numpy().astype("<f4").tobytes())
        emit(f"done {int(step['step'])}")


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay token ids through a model and write logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most at any time")
    args = ap.parse_args(argv)
    import torch
    if not torch.cuda.is_available():
        print("trace_run needs a CUDA device", file=sys.stderr)
        return 2
    _ensure_kernels(args.model)
    from .. import ops
    engine = make_engine(args.model, args.dtype, args.max_tokens)
    out = Path(args.out)
    out.mkdir(parents=True, exist_ok=True)

    def emit(text: str) -> None:
        print(text, flush=True)
    replay(engine, sys.stdin, out, emit)
    ops.check_status(engine.device)
    engine.shutdown()
    return 0


if __name__ == "__main__":
    sys.exit(main())
