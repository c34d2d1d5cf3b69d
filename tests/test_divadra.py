"""Divadra through the framework: engine, cache, state slots and rings, scheduler, loader and command line, on the CPU
path and (marked gpu) on the kernels, against the plain restatement in ``divadra_oracle.py``."""
import io
import json
import random
import subprocess
import sys
from pathlib import Path

import pytest
import torch

import divadra_oracle as O
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
    # both mixers, every feed-forward, several chunks, all sizes unequal, grouped heads and groups
    "mixed": O.config(72, 97, [
        O.mamba(4, 20, 12, 2, 5, 3, O.ff(60)),
        O.pair((6, 2, 24, 20), 20, (3, 24), O.moe(6, 2, 40), dims=8, base=500.0),
        O.mamba(3, 8, 24, 1, 4, 5),
        O.pair((2, 2, 40, 16), 7, (4, 12), O.ff(88), dims=24, scale=-0.2)], taps=3),
    # sizes that fit no vector load: odd widths, ranks, head, state and expert sizes
    "odd": O.config(33, 31, [
        O.pair((3, 1, 5, 6), 5, (3, 7), O.moe(5, 3, 19), dims=2, scale=0.9, rank=3),
        O.mamba(3, 7, 5, 3, 1, 2, O.ff(21)),
        O.pair((3, 3, 7, 2), 9, (1, 9), dims=6, rank=1)], taps=5, bigram=(11, 5, 1), eps=1e-3),
    # a chunk of one token, one longer than everything, one key head for many, convolutions of one tap, one expert, one bucket
    "edges": O.config(64, 40, [
        O.pair((4, 4, 16, 16), 1, (2, 16), O.moe(1, 1, 32), dims=0),
        O.mamba(2, 16, 16, 1, 2, 1, O.moe(8, 8, 24)),
        O.pair((17, 1, 64, 32), 4096, (1, 64), O.moe(8, 1, 16), dims=32)], taps=1, bigram=(1, 2, 3)),
    # heads wider than 128, values wider than keys and the other way round, wide states, long convolutions
    "wide": O.config(96, 50, [
        O.pair((2, 1, 136, 40), 50, (1, 130), O.ff(48), dims=64, rank=40),
        O.mamba(1, 66, 130, 1, 3, 9, O.moe(16, 4, 16)),
        O.pair((2, 2, 24, 150), 33, (2, 40), rank=8)], taps=9),
    # widths, heads and chunks that the tensor-core kernels take without padding
    "aligned": O.config(128, 64, [
        O.pair((4, 2, 64, 64), 48, (2, 64), O.moe(4, 2, 64)), O.mamba(4, 32, 64, 2, 2, 4, O.ff(192)),
        O.pair((2, 1, 128, 64), 96, (4, 32), O.ff(128), rank=16)]),
    "no_attention": O.config(40, 30, [O.mamba(2, 12, 20, 2, 3, 4, O.moe(4, 2, 24)), O.mamba(4, 6, 8, 4, 2, 3, O.ff(16))], taps=2),
    "only_attention": O.config(40, 30, [O.pair((4, 2, 16, 8), 33, (2, 20), O.ff(24), dims=8)]),
}


class Model:
    def __init__(self, cfg, path_of, name):
        self.cfg, self.w = cfg, O.weights(cfg, seed=len(name))
        self.path = O.save(path_of / name, cfg, self.w)
        self._memo = {}

    def want(self, ids):
        key = tuple(ids)
        if key not in self._memo:
            self._memo[key] = O.forward(self.cfg, self.w, ids)
        return self._memo[key]

    def agrees(self, got, ids, dtype):
        return O.fits(got, self.want(ids), dtype)


@pytest.fixture(scope="module")
def model(tmp_path_factory):
    made = {}

    def get(name):
        if name not in made:
            made[name] = Model(CONFIGS[name], tmp_path_factory.mktemp("divadra"), name)
        return made[name]
    return get


def make(path, device, dtype, tokens=256):
    return trace_run.make_engine(path, dtype, tokens, device=device)


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
    assert arch.family == "divadra" and arch.num_layers == 4 and arch.extra["canon_taps"] == 3
    assert arch.layer_types == ["linear", "sliding", "linear", "sliding"]
    assert ModelRegistry.resolve_model_cls(arch.architecture, arch.family).__name__ == "DivadraForCausalLM"
    assert "Divadra" in ModelRegistry.supported_architectures()


@pytest.mark.parametrize("change, match", [
    (lambda c: c["layers"][0].update(type="other"), "unknown mixer"),
    (lambda c: c["layers"][0]["mixer"].pop("conv"), "conv"),
    (lambda c: c["layers"][0]["mixer"].update(conv=17), "taps"),
    (lambda c: c["layers"][0]["mixer"].update(groups=3), "groups"),
    (lambda c: c["layers"][0]["mixer"].update(norm_groups=3), "norm parts"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(vdim=9), "values"),
    (lambda c: c["layers"][1]["mixer"]["left"]["rot"].update(dims=7), "rotate"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "evenly"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"]["right"].pop("dim"), "dim"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "feed-forward"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=7), "choose"),
    (lambda c: c["canon"].update(taps=0), "taps"),
    (lambda c: c["embedding"]["bigram"].pop("mul_cur"), "mul_cur"),
    (lambda c: c.update(layers=[]), "no layers")])
def test_bad_configurations_are_refused(change, match):
    cfg = json.loads(json.dumps(CONFIGS["mixed"]))
    change(cfg)
    with pytest.raises(ValueError, match=match):
        arch_from_hf_config(cfg)


def test_checkpoint_must_match_the_configuration(tmp_path):
    cfg = CONFIGS["odd"]
    w = O.weights(cfg)
    edits = {"missing": (lambda d: d.pop("l1.mix.A_log"), "lacks"), "extra": (lambda d: d.update(other=torch.zeros(2)), "no destination"),
             "shape": (lambda d: d.update({"l0.mlp.e2.up": torch.zeros(3, 3)}), "shape"),
             "table": (lambda d: d.update({"l0.mlp.table": torch.full((31, 3), 5, dtype=torch.int32)}), "below 5"),
             "rank": (lambda d: d.update({"l0.mix.right.w1": torch.zeros(4, 33)}), "do not fit")}
    for name, (edit, match) in edits.items():
        d = dict(w)
        edit(d)
        with pytest.raises((KeyError, ValueError), match=match):
            LiteEngine(build_vllm_config(O.save(tmp_path / name, cfg, d), dtype="float32", device="cpu", max_model_len=64))


def test_norms_without_a_feed_forward_may_be_in_the_checkpoint(tmp_path):
    cfg = CONFIGS["odd"]
    w = O.weights(cfg)
    extra = {**w, "l2.norm2": torch.ones(33), "l2.canon2": torch.ones(33, 5)}
    ids = tokens(cfg, 12)
    eng = make(O.save(tmp_path / "extra", cfg, extra), "cpu", "float32")
    assert O.fits(run_portions(eng, "a", ids, [12]), O.forward(cfg, w, ids), "float32")


# ------------------------------------------------------------------ whole prompts, portions, decoding
@pytest.mark.parametrize("device, dtype", DEVICES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompt(model, name, device, dtype):
    m = model(name)
    ids = tokens(m.cfg, 150)
    assert m.agrees(run_portions(make(m.path, device, dtype), "a", ids, [len(ids)]), ids, dtype)


@pytest.mark.parametrize("device, dtype", DEVICES)
def test_stream_after_every_layer(model, device, dtype):
    m = model("mixed")
    ids, got, want = tokens(m.cfg, 30, seed=2), [], []
    eng = make(m.path, device, dtype)
    forward = eng.model.forward
    eng.model.forward = lambda batch, kv, inputs_embeds=None: forward(batch, kv, inputs_embeds, collect=got)
    run_portions(eng, "a", ids, [30])
    O.forward(m.cfg, m.w, ids, collect=want)
    assert len(got) == len(want) == 4
    tol = 2e-4 if dtype == "float32" else 0.05
    for a, b in zip(got, want):
        e = (a.cpu() - b).pow(2).mean(-1).sqrt() / b.pow(2).mean().sqrt()
        assert float(torch.quantile(e, 0.9)) < tol and float(e.max()) < 4 * tol


@pytest.mark.parametrize("device, dtype", DEVICES)
@pytest.mark.parametrize("name", ["mixed", "aligned"])
@pytest.mark.parametrize("sizes", [[1], [2], [3, 2], [16], [17, 1, 1, 5], [64, 2, 65, 1], [70, 3]], ids=str)
def test_portions(model, name, sizes, device, dtype):
    m = model(name)
    ids = tokens(m.cfg, 140, seed=3)
    assert m.agrees(run_portions(make(m.path, device, dtype), "a", ids, cut(len(ids), sizes)), ids, dtype)


@pytest.mark.parametrize("device, dtype", DEVICES)
@pytest.mark.parametrize("name", ["odd", "edges", "wide"])
def test_prompt_then_single_tokens(model, name, device, dtype):
    m = model(name)
    ids = tokens(m.cfg, 130, seed=5)
    assert m.agrees(run_portions(make(m.path, device, dtype), "a", ids, [90] + [1] * 40), ids, dtype)


@pytest.mark.parametrize("device, dtype", DEVICES)
def test_first_tokens_of_a_sequence(model, device, dtype):
    """The first pair of tokens, a chunk of one token, convolutions longer than what there is, the first write into a
    zero state."""
    for name in ("edges", "mixed", "wide"):
        m = model(name)
        eng = make(m.path, device, dtype)
        ids = tokens(m.cfg, 12, seed=7)
        for first in (1, 2, 3, 9):
            assert m.agrees(run_portions(eng, f"r{first}", ids, [first] + [1] * (len(ids) - first)), ids, dtype)


@pytest.mark.parametrize("device, dtype", DEVICES)
def test_long_decoding(model, device, dtype):
    m = model("mixed")
    ids = tokens(m.cfg, 300, seed=9)
    assert m.agrees(run_portions(make(m.path, device, dtype, 320), "a", ids, [3] + [1] * 297), ids, dtype)


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_prompts_take_the_kernels_for_many_tokens(model, dtype):
    """More than 4096 tokens in a step: wide tiles, split projections, persistent products."""
    m = model("aligned")
    ids = tokens(m.cfg, 4200, seed=4)
    want = m.want(ids)
    eng = make(m.path, "cuda", dtype, 4224)
    ask = [0, 1, 47, 48, 95, 96, 97, 1000, 4095, 4096, 4198]
    got = eng.replay_step([("a", ids[:4199], ask)], [])
    last = eng.replay_step([("a", ids[4199:], [0])], ["a"])
    assert O.fits(torch.cat([got, last]).cpu(), want[ask + [4199]], dtype)


# ------------------------------------------------------------------ batches, slots and pages used again
@pytest.mark.parametrize("device, dtype", DEVICES)
@pytest.mark.parametrize("name", ["mixed", "aligned"])
def test_unequal_requests_share_steps(model, name, device, dtype):
    """Random portions of up to four live requests side by side, requests left out of steps, slots and pages reused;
    the pool holds what four requests need and no more."""
    m = model(name)
    rng = random.Random(1)
    lens = [5, 100, 33, 64, 2, 130, 1, 77, 48, 16]
    eng = make(m.path, device, dtype, 448)
    seqs = {f"q{i}": tokens(m.cfg, n, seed=20 + i) for i, n in enumerate(lens)}
    waiting, live, at, slots = list(seqs), [], {}, set()
    got = {r: [] for r in seqs}
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        step, end = [], []
        for r in rng.sample(live, rng.randint(1, len(live))):
            lo = at.get(r, 0)
            n = min(len(seqs[r]) - lo, rng.choice([1, 1, 2, 3, 16, 40, 70]))
            step.append((r, seqs[r][lo:lo + n], list(range(n))))
            at[r] = lo + n
            if lo + n == len(seqs[r]):
                end.append(r)
                live.remove(r)
        y = eng.replay_step(step, end).cpu()
        for r, part, _ in step:
            got[r].append(y[:len(part)])
            y = y[len(part):]
        slots |= {eng.scheduler.requests[r].slot_idx for r in live if r in eng.scheduler.requests}
    for r, ids in seqs.items():
        assert m.agrees(torch.cat(got[r]), ids, dtype), r
    st = eng.stats()["backend"]["kv"]
    assert st["used_blocks"] == 0 and len(slots) <= 4 and sorted(eng.scheduler.free_slots) == [0, 1, 2, 3]


@pytest.mark.parametrize("device, dtype", DEVICES)
def test_a_used_slot_leaves_nothing_behind(model, device, dtype):
    for name in ("no_attention", "only_attention"):
        m = model(name)
        eng = make(m.path, device, dtype, 128)
        ids = tokens(m.cfg, 20, seed=1)
        for i in range(6):                     # every slot comes round again, once after a single token, once after many
            other = tokens(m.cfg, 1 if i % 2 else 60, seed=50 + i)
            eng.replay_step([(f"o{i}", other, [])], [f"o{i}"])
            assert m.agrees(run_portions(eng, f"a{i}", ids, [1, 2] + [1] * 17), ids, dtype)


def test_pool_slots_and_rings_follow_the_asked_size(model):
    m = model("mixed")
    eng = make(m.path, "cpu", "float32", 200)          # rounded up to 256
    assert eng.plan.num_total_blocks == 1 + 256 // eng.plan.block_size and eng.plan.max_active_requests == 4
    kv = eng.kv_cache
    assert [tuple(s.shape) for s in kv.states] == [(4, 4, 12, 20), (4, 3, 24, 24), (4, 3, 24, 8), (4, 4, 12, 12)]
    assert [tuple(s.shape) for s in kv.rings if s is not None] == [(4, 3, 128), (4, 5, 72)]
    assert [tuple(s.shape) for s in kv.inputs] == [(4, 4, 72)] * 4
    assert kv.last_tokens.dtype == torch.int32 and kv.last_tokens.shape == (4,)
    assert [(tuple(k.shape[1:]), tuple(v.shape[1:])) for k, v in kv.layers if k.numel()] == [((2, 16, 24), (2, 16, 20)), ((2, 16, 40), (2, 16, 16))]
    assert eng.memory.kv_cache_bytes >= kv.state_bytes == sum(t.numel() * 4 for t in kv.slot_tensors()) > 0


# ------------------------------------------------------------------ generation through the public entry points
def _llm(path, device, dtype, **kw):
    cfg = {"tuning_keyvals": {"FASTINFERENCE_LITE_PREFILL_CHUNK": "24", "FASTINFERENCE_MIN_PREFILL_CHUNK": "8",
                              **kw.pop("keys", {})}}
    return LLM(path, dtype=dtype, device=device, max_model_len=256, fastinference_config=cfg, **kw)


@pytest.mark.parametrize("device", ["cpu", pytest.param("cuda", marks=gpu)])
@pytest.mark.parametrize("name", ["mixed", "edges"])
def test_greedy_generation(model, name, device):
    """Chunked prompts of unequal length beside decoding requests; every request equals its own continuation alone."""
    m = model(name)
    prompts = [tokens(m.cfg, n, seed=70 + n) for n in (3, 41, 30, 1, 25, 9)]
    lens = (10, 6, 9, 12, 5, 8)
    llm = _llm(m.path, device, "float32", max_num_seqs=3, max_num_batched_tokens=40)
    outs = llm.generate(prompts, [SamplingParams(temperature=0.0, max_tokens=n, ignore_eos=True) for n in lens])
    for p, o, n in zip(prompts, outs, lens):
        want, margin = O.greedy(m.cfg, m.w, p, n)
        assert margin < 1e-4 or list(o.outputs[0].token_ids) == want
    st = llm.stats()["backend"]
    assert st["mixed_steps"] > 0 and st["kv"]["used_blocks"] == 0
    llm.shutdown()


@gpu
def test_generation_in_16_bit_is_independent_of_the_batch(model):
    m = model("mixed")
    prompts = [tokens(m.cfg, n, seed=n) for n in (100, 7, 40)]
    sp = SamplingParams(temperature=0.0, max_tokens=24, ignore_eos=True)
    llm = _llm(m.path, "cuda", "bfloat16", max_num_seqs=4)
    together = [list(o.outputs[0].token_ids) for o in llm.generate(prompts, sp)]
    alone = [list(llm.generate([p], sp)[0].outputs[0].token_ids) for p in prompts]
    # random logits: only an all but tied choice may split two runs
    for p, a, b in zip(prompts, together, alone):
        i = next((i for i, (x, y) in enumerate(zip(a, b)) if x != y), None)
        if i is not None:
            logits = m.want(p + a[:i])[-1]
            assert abs(float(logits[a[i]] - logits[b[i]])) < 0.1 * float(logits.std()), i
    assert llm.stats()["backend"]["graph_replays"] > 0
    llm.shutdown()


def test_sampled_generation_reproduces_with_a_seed(model):
    m = model("mixed")
    llm = _llm(m.path, "cpu", "float32", max_num_seqs=2)
    sp = SamplingParams(temperature=0.8, top_k=20, seed=11, max_tokens=12, ignore_eos=True)
    a, b = (list(llm.generate([tokens(m.cfg, 8)], sp)[0].outputs[0].token_ids) for _ in range(2))
    assert a == b and len(a) == 12
    llm.shutdown()


def test_requests_wait_for_a_shared_pool(model):
    """A pool of 96 tokens serves requests that would need 200 together: admission waits instead of running dry."""
    m = model("only_attention")
    llm = LLM(m.path, dtype="float32", device="cpu", max_model_len=96, max_num_seqs=4, fastinference_config={
        "tuning_keyvals": {"FASTINFERENCE_KV_POOL_TOKENS": "96"}})
    assert llm.engine.plan.shared_pool and llm.engine.plan.num_total_blocks == 1 + 96 // 16
    prompts = [tokens(m.cfg, n, seed=n) for n in (40, 30, 50, 20)]
    outs = llm.generate(prompts, SamplingParams(temperature=0.0, max_tokens=10, ignore_eos=True))
    for p, o in zip(prompts, outs):
        want, margin = O.greedy(m.cfg, m.w, p, 10)
        assert margin < 1e-4 or list(o.outputs[0].token_ids) == want
    llm.shutdown()


def test_prefix_cache_stays_off_for_recurrent_state(model):
    llm = _llm(model("mixed").path, "cpu", "float32", keys={"FASTINFERENCE_PREFIX_CACHE_MAX_ENTRIES": "8"})
    assert not llm.engine.prefix_cache.enabled
    llm.shutdown()


def test_synthetic_preset_generates():
    llm = LLM("synthetic:tiny-divadra-test", dtype="float32", device="cpu", max_num_seqs=2, max_model_len=64)
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


def _check_trace(m, out, wanted, dtype):
    assert sorted(p.name for p in out.glob("*.f32")) == sorted(f"{s}.f32" for s in wanted)
    for s, rows in wanted.items():
        got = torch.frombuffer(bytearray((out / f"{s}.f32").read_bytes()), dtype=torch.float32).view(-1, m.cfg["vocab"])
        assert O.fits(got, torch.stack([m.want(ids)[p] for ids, p in rows]), dtype)


def test_trace_lines_in_logits_out(model, tmp_path):
    m = model("mixed")
    steps, wanted = _trace(m.cfg)
    said = []
    trace_run.replay(make(m.path, "cpu", "float32", 128), io.StringIO("\n".join(json.dumps(s) for s in steps)), tmp_path, said.append)
    assert said == [f"done {i}" for i in range(4)]
    _check_trace(m, tmp_path, wanted, "float32")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_program(model, tmp_path, dtype):
    m = model("mixed")
    steps, wanted = _trace(m.cfg)
    exe = Path(__file__).resolve().parents[1] / "bin" / "trace_run"
    res = subprocess.run([sys.executable, str(exe), "--model", m.path, "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "128"],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=300)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [x for x in res.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    _check_trace(m, tmp_path, wanted, dtype)
