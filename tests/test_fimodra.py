"""Fimodra through the framework: engine, cache and state slots, scheduler, loader and command line, on the CPU path
and (marked gpu) on the kernels, against the plain restatement in ``fimodra_oracle.py``."""
import io
import json
import random
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import fimodra_oracle as O
from litevllm_b200 import LLM, SamplingParams
from litevllm_b200.config.config_builder import build_vllm_config
from litevllm_b200.engine.lite_engine import LiteEngine
from litevllm_b200.entrypoints import trace_run
from litevllm_b200.models.arch import arch_from_hf_config
from litevllm_b200.models.registry import ModelRegistry

gpu = pytest.mark.gpu
DEVICES = [pytest.param("cpu", "float32", id="cpu"), pytest.param("cuda", "float32", id="cuda-fp32", marks=gpu),
           pytest.param("cuda", "bfloat16", id="cuda-bf16", marks=gpu)]

CONFIGS = {
    # both mixers, with and without a feed-forward, several windows, all sizes unequal
    "mixed": O.config(72, 97, 3, [
        O.layer("latent_attention", 88, heads=3, dim=24, rot_dim=8, vdim=40, kv_rank=56, window=20, base=500.0),
        O.layer("hgrn2", None, heads=5, dim=12, vdim=20),
        O.layer("latent_attention", None, heads=2, dim=40, rot_dim=24, vdim=16, kv_rank=24, window=7),
        O.layer("hgrn2", 40, heads=1, dim=72, vdim=8)]),
    # sizes that fit no vector load: odd widths, ranks and head sizes
    "odd": O.config(33, 31, 1, [
        O.layer("hgrn2", 19, heads=3, dim=5, vdim=7),
        O.layer("latent_attention", 21, heads=1, dim=3, rot_dim=2, vdim=5, kv_rank=9, window=5, scale=0.9)], eps=1e-3),
    # a window of one token, one longer than everything, a head as wide as a tile, norm parts of four channels
    "edges": O.config(32, 40, 8, [
        O.layer("latent_attention", 32, heads=4, dim=8, rot_dim=4, vdim=8, kv_rank=16, window=1),
        O.layer("latent_attention", 24, heads=16, dim=48, rot_dim=16, vdim=64, kv_rank=64, window=4096),
        O.layer("hgrn2", 16, heads=2, dim=16, vdim=16)]),
    # keys and values wider than 128: the widest prefill tile; more than 16 heads
    "wide": O.config(64, 50, 2, [
        O.layer("latent_attention", 48, heads=17, dim=128, rot_dim=32, vdim=136, kv_rank=136, window=50),
        O.layer("hgrn2", 48, heads=2, dim=130, vdim=66)]),
    "no_attention": O.config(40, 30, 5, [O.layer("hgrn2", 24, heads=2, dim=20, vdim=12)]),
    "only_attention": O.config(40, 30, 1, [
        O.layer("latent_attention", None, heads=2, dim=16, rot_dim=8, vdim=24, kv_rank=32, window=33)]),
}


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            cfg = CONFIGS[name]
            w = O.weights(cfg, seed=len(name))
            made[name] = (cfg, w, O.save(tmp_path_factory.mktemp("fimodra") / name, cfg, w))
        return made[name]
    return get


def make(path, device, dtype, tokens=256, **kw):
    return trace_run.make_engine(path, dtype, tokens, device=device, **kw)


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def run_portions(eng, rid, ids, sizes):
    """Logits of all positions of one sequence fed in portions."""
    out, at = [], 0
    for n in sizes:
        out.append(eng.replay_step([(rid, ids[at:at + n], list(range(n)))], [rid] if at + n == len(ids) else []).cpu())
        at += n
    assert at == len(ids)
    return torch.cat(out)


def cut(n, sizes):
    out, i = [], 0
    while n > 0:
        s = min(n, sizes[i % len(sizes)])
        out.append(s)
        n, i = n - s, i + 1
    return out


# ------------------------------------------------------------------ registry, configuration, loading
def test_configuration_selects_the_model():
    arch = arch_from_hf_config(CONFIGS["mixed"])
    assert arch.family == "fimodra" and arch.num_layers == 4 and arch.extra["norm_groups"] == 3
    assert ModelRegistry.resolve_model_cls(arch.architecture, arch.family).__name__ == "FimodraForCausalLM"
    assert "Fimodra" in ModelRegistry.supported_architectures()


@pytest.mark.parametrize("change, match", [
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("heads"), "heads"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=7), "rotate"),
    (lambda c: c["norm"].update(groups=5), "equal parts"),
    (lambda c: c.update(layers=[]), "no layers")])
def test_bad_configurations_are_refused(change, match):
    cfg = json.loads(json.dumps(CONFIGS["mixed"]))
    change(cfg)
    with pytest.raises(ValueError, match=match):
        arch_from_hf_config(cfg)


def test_checkpoint_must_match_the_configuration(tmp_path):
    cfg = CONFIGS["odd"]
    w = O.weights(cfg)
    for name, edit in {"missing": lambda d: d.pop("l0.mix.lower"), "extra": lambda d: d.update(other=torch.zeros(2)),
                       "shape": lambda d: d.update({"l1.mix.sink": torch.zeros(3)})}.items():
        d = dict(w)
        edit(d)
        with pytest.raises((KeyError, ValueError), match={"missing": "lacks", "extra": "no destination", "shape": "shape"}[name]):
            LiteEngine(build_vllm_config(O.save(tmp_path / name, cfg, d), dtype="float32", device="cpu", max_model_len=64))


# ------------------------------------------------------------------ whole prompts, portions, decoding
@pytest.mark.parametrize("device, dtype", DEVICES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt(model, name, device, dtype):
    cfg, w, path = model(name)
    ids = tokens(cfg, 150)
    got = run_portions(make(path, device, dtype), "a", ids, [len(ids)])
    assert O.fits(got, O.forward(cfg, w, ids), dtype)


@pytest.mark.parametrize("device, dtype", DEVICES)
@pytest.mark.parametrize("sizes", [[1], [2], [3, 2], [16], [17, 1, 1, 5], [64, 2, 65, 1], [70, 3]], ids=str)
def test_portions(model, sizes, device, dtype):
    cfg, w, path = model("mixed")
    ids = tokens(cfg, 140, seed=3)
    got = run_portions(make(path, device, dtype), "a", ids, cut(len(ids), sizes))
    assert O.fits(got, O.forward(cfg, w, ids), dtype)


@pytest.mark.parametrize("device, dtype", DEVICES)
@pytest.mark.parametrize("name", ["odd", "edges", "wide"])
def test_prompt_then_single_tokens(model, name, device, dtype):
    cfg, w, path = model(name)
    ids = tokens(cfg, 130, seed=5)
    got = run_portions(make(path, device, dtype), "a", ids, [90] + [1] * 40)
    assert O.fits(got, O.forward(cfg, w, ids), dtype)


@pytest.mark.parametrize("device, dtype", DEVICES)
def test_first_tokens_of_a_sequence(model, device, dtype):
    cfg, w, path = model("edges")
    eng = make(path, device, dtype)
    ids = tokens(cfg, 12, seed=7)
    want = O.forward(cfg, w, ids)
    for first in (1, 2, 3, 9):
        got = run_portions(eng, f"r{first}", ids, [first] + [1] * (len(ids) - first))
        assert O.fits(got, want, dtype)


@pytest.mark.parametrize("device, dtype", DEVICES)
def test_long_decoding(model, device, dtype):
    cfg, w, path = model("mixed")
    ids = tokens(cfg, 300, seed=9)
    got = run_portions(make(path, device, dtype, 320), "a", ids, [3] + [1] * 297)
    assert O.fits(got, O.forward(cfg, w, ids), dtype)


# ------------------------------------------------------------------ batches, slots and pages used again
@pytest.mark.parametrize("device, dtype", DEVICES)
def test_unequal_requests_share_steps(model, device, dtype):
    """Random portions of up to four live requests side by side, requests left out of steps, slots and pages reused;
    the pool holds what four requests need and no more."""
    cfg, w, path = model("mixed")
    rng = random.Random(1)
    lens = [5, 100, 33, 64, 2, 130, 1, 77, 48, 16]
    eng = make(path, device, dtype, 448)
    seqs = {f"q{i}": tokens(cfg, n, seed=20 + i) for i, n in enumerate(lens)}
    want = {r: O.forward(cfg, w, ids) for r, ids in seqs.items()}
    waiting, live, at, slots = list(seqs), [], {}, set()
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        step, rows, end = [], [], []
        for r in rng.sample(live, rng.randint(1, len(live))):
            lo = at.get(r, 0)
            n = min(len(seqs[r]) - lo, rng.choice([1, 1, 2, 3, 16, 40, 70]))
            step.append((r, seqs[r][lo:lo + n], list(range(n))))
            rows += [(r, lo + k) for k in range(n)]
            at[r] = lo + n
            if lo + n == len(seqs[r]):
                end.append(r)
                live.remove(r)
        got = eng.replay_step(step, end).cpu()
        slots |= {eng.scheduler.requests[r].slot_idx for r in live if r in eng.scheduler.requests}
        assert O.fits(got, torch.stack([want[r][p] for r, p in rows]), dtype)
    st = eng.stats()["backend"]["kv"]
    assert st["used_blocks"] == 0 and len(slots) <= 4 and sorted(eng.scheduler.free_slots) == [0, 1, 2, 3]


@pytest.mark.parametrize("device, dtype", DEVICES)
def test_a_used_slot_leaves_nothing_behind(model, device, dtype):
    cfg, w, path = model("no_attention")
    eng = make(path, device, dtype, 128)
    ids = tokens(cfg, 20, seed=1)
    want = O.forward(cfg, w, ids)
    for i in range(6):                     # every slot comes round again, once after a single token, once after many
        other = tokens(cfg, 1 if i % 2 else 60, seed=50 + i)
        eng.replay_step([(f"o{i}", other, [])], [f"o{i}"])
        got = run_portions(eng, f"a{i}", ids, [1, 2] + [1] * 17)
        assert O.fits(got, want, dtype)


def test_replay_rejects_bad_input(model):
    cfg, _, path = model("odd")
    eng = make(path, "cpu", "float32", 64)
    with pytest.raises(Exception, match="out of range"):
        eng.replay_step([("a", [cfg["vocab"]], [0])])
    with pytest.raises(Exception, match="out of range"):
        eng.replay_step([("b", [1], [1])])


def test_pool_and_slots_follow_the_asked_size(model):
    _, _, path = model("mixed")
    eng = make(path, "cpu", "float32", 200)          # rounded up to 256
    assert eng.plan.num_total_blocks == 1 + 256 // eng.plan.block_size and eng.plan.max_active_requests == 4
    states = [s for s in eng.kv_cache.states if s is not None]
    assert [tuple(s.shape) for s in states] == [(4, 5, 12, 20), (4, 1, 72, 8)]
    assert all(s.dtype == torch.float32 for s in states) and eng.memory.kv_cache_bytes >= eng.kv_cache.state_bytes > 0


# ------------------------------------------------------------------ generation through the public entry points
def _llm(path, device, dtype, **kw):
    cfg = {"tuning_keyvals": {"FASTINFERENCE_LITE_PREFILL_CHUNK": "24", "FASTINFERENCE_MIN_PREFILL_CHUNK": "8",
                              **kw.pop("keys", {})}}
    return LLM(path, dtype=dtype, device=device, max_model_len=256, fastinference_config=cfg, **kw)


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=gpu)])
@pytest.mark.parametrize("name", ["mixed", "edges"])
def test_greedy_generation(model, name, device):
    """Chunked prompts of unequal length beside decoding requests; every request equals its own continuation alone."""
    cfg, w, path = model(name)
    prompts = [tokens(cfg, n, seed=70 + n) for n in (3, 61, 30, 1, 45, 9)]
    llm = _llm(path, device, "float32", max_num_seqs=3, max_num_batched_tokens=40)
    outs = llm.generate(prompts, [SamplingParams(temperature=0.0, max_tokens=m, ignore_eos=True) for m in (14, 6, 9, 20, 5, 11)])
    for p, o, m in zip(prompts, outs, (14, 6, 9, 20, 5, 11)):
        want, margin = O.greedy(cfg, w, p, m)
        assert margin < 1e-4 or list(o.outputs[0].token_ids) == want
    st = llm.stats()["backend"]
    assert st["mixed_steps"] > 0 and st["kv"]["used_blocks"] == 0
    llm.shutdown()


@gpu
def test_generation_in_16_bit_is_independent_of_the_batch(model):
    cfg, _, path = model("mixed")
    prompts = [tokens(cfg, n, seed=n) for n in (100, 7, 40)]
    sp = SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True)
    llm = _llm(path, "cuda", "bfloat16", max_num_seqs=4)
    together = [list(o.outputs[0].token_ids) for o in llm.generate(prompts, sp)]
    alone = [list(llm.generate([p], sp)[0].outputs[0].token_ids) for p in prompts]
    # nearly flat random logits: the common prefix must be long, a tie may split the tails
    for a, b in zip(together, alone):
        assert sum(x == y for x, y in zip(a, b)) >= 18
    assert llm.stats()["backend"]["graph_replays"] > 0
    llm.shutdown()


def test_sampled_generation_reproduces_with_a_seed(model):
    cfg, _, path = model("mixed")
    llm = _llm(path, "cpu", "float32", max_num_seqs=2)
    sp = SamplingParams(temperature=0.8, top_k=20, seed=11, max_tokens=12, ignore_eos=True)
    a, b = (list(llm.generate([tokens(cfg, 8)], sp)[0].outputs[0].token_ids) for _ in range(2))
    assert a == b and len(a) == 12
    llm.shutdown()


def test_requests_wait_for_a_shared_pool(model):
    """A pool of 96 tokens serves requests that would need 200 together: admission waits instead of running dry."""
    cfg, w, path = model("mixed")
    llm = LLM(path, dtype="float32", device="cpu", max_model_len=96, max_num_seqs=4, fastinference_config={
        "tuning_keyvals": {"FASTINFERENCE_KV_POOL_TOKENS": "96"}})
    assert llm.engine.plan.shared_pool and llm.engine.plan.num_total_blocks == 1 + 96 // 16
    prompts = [tokens(cfg, n, seed=n) for n in (40, 30, 50, 20)]
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=10, ignore_eos=True))
    for p, o in zip(prompts, outs):
        want, margin = O.greedy(cfg, w, p, 10)
        assert margin < 1e-4 or list(o.outputs[0].token_ids) == want
    llm.shutdown()


def test_prefix_cache_stays_off_for_recurrent_state(model):
    cfg, _, path = model("mixed")
    llm = _llm(path, "cpu", "float32", keys={"FASTINFERENCE_PREFIX_CACHE_MAX_ENTRIES": "8"})
    assert not llm.engine.prefix_cache.enabled
    llm.shutdown()


def test_synthetic_preset_generates():
    llm = LLM("synthetic:tiny-fimodra-test", dtype="float32", device="cpu", max_num_seqs=2, max_model_len=64)
    out = llm.generate([[1, 2, 3]], SamplingParams(temperature=0.0, max_tokens=4, ignore_eos=True))
    assert len(out[0].outputs[0].token_ids) == 4
    llm.shutdown()


# ------------------------------------------------------------------ the trace runner
def _trace(cfg):
    a, b = tokens(cfg, 40, seed=1), tokens(cfg, 25, seed=2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:3], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[3:4], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[4:], "want": [20]}, {"id": "a", "tokens": a[30:31], "want": [0]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": a[31:], "want": [8, 1]}], "end": ["a"]}]
    return steps, {0: [(a, 0), (a, 29)], 2: [(b, 24), (a, 30)], 3: [(a, 39), (a, 32)]}


def _check_trace(cfg, w, out, wanted, dtype):
    assert sorted(p.name for p in out.glob("*.f32")) == sorted(f"{s}.f32" for s in wanted)
    for s, rows in wanted.items():
        got = torch.frombuffer(bytearray((out / f"{s}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert O.fits(got, torch.stack([O.forward(cfg, w, ids)[p] for ids, p in rows]), dtype)


def test_trace_lines_in_logits_out(model, tmp_path):
    cfg, w, path = model("mixed")
    steps, wanted = _trace(cfg)
    said = []
    trace_run.replay(make(path, "cpu", "float32", 128), io.StringIO("\n".join(json.dumps(s) for s in steps)), tmp_path, said.append)
    assert said == [f"done {i}" for i in range(4)]
    _check_trace(cfg, w, tmp_path, wanted, "float32")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_program(model, tmp_path, dtype):
    cfg, w, path = model("mixed")
    steps, wanted = _trace(cfg)
    exe = Path(__file__).resolve().parents[1] / "bin" / "trace_run"
    res = subprocess.run([sys.executable, str(exe), "--model", path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "128"],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    _check_trace(cfg, w, tmp_path, wanted, dtype)
