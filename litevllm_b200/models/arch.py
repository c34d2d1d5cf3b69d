"""Normalised architecture description read from a HuggingFace ``config.json`` dict (or a GGUF
header).  Model classes and the runtime planner only look at this record, never at raw HF keys.
Reference counterpart: vllm/model_executor/models/lite_config.py:11-158.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any


@dataclass
class QuantSpec:
    method: str = "none"          # none | awq | compressed-tensors | gguf
    bits: int = 16
    group_size: int = 128
    zero_point: bool = True
    symmetric: bool = False


@dataclass
class MoESpec:
    num_experts: int = 0
    top_k: int = 0
    expert_intermediate: int = 0
    shared_intermediate: int = 0     # dense/shared branch width (0 = none)
    n_shared_experts: int = 0
    router: str = "softmax"          # softmax | sigmoid | sqrt_softplus
    renormalize: bool = True
    routed_scaling: float = 1.0
    first_dense_layers: int = 0      # leading layers with a dense MLP instead of experts


@dataclass
class MLASpec:
    q_lora_rank: int = 0
    kv_lora_rank: int = 0
    qk_rope_dim: int = 0
    qk_nope_dim: int = 0
    v_head_dim: int = 0


@dataclass
class ModelArch:
    family: str                      # llama | qwen2 | qwen3_5 | gemma4 | deepseek_mla | qwen2_vl | fimodra | pofadra
    architecture: str
    hidden_size: int
    num_layers: int
    num_heads: int
    num_kv_heads: int
    head_dim: int
    intermediate_size: int
    vocab_size: int
    rms_eps: float = 1e-5
    rope_theta: float = 10000.0
    rope_scaling: dict[str, Any] | None = None
    rotary_dim: int | None = None
    max_position: int = 4096
    tie_embeddings: bool = False
    act: str = "silu"
    attn_bias: bool = False
    mlp_bias: bool = False
    sliding_window: int = 0
    layer_types: list[str] = field(default_factory=list)   # per layer: "full" | "sliding" | "linear"
    attn_softcap: float = 0.0
    final_softcap: float = 0.0
    qk_norm: bool = False
    norm_plus_one: bool = False      # RMSNorm multiplies by (1 + w)
    embed_scale: float = 1.0
    global_head_dim: int | None = None       # Gemma4: global layers may use another head_dim
    global_kv_heads: int | None = None
    global_rope_theta: float | None = None
    partial_rotary_factor: float = 1.0
    eos_token_ids: list[int] = field(default_factory=list)
    bos_token_id: int | None = None
    quant: QuantSpec = field(default_factory=QuantSpec)
    moe: MoESpec = field(default_factory=MoESpec)
    mla: MLASpec = field(default_factory=MLASpec)
    vision: dict[str, Any] | None = None
    extra: dict[str, Any] = field(default_factory=dict)

    def layer_type(self, i: int) -> str:
        if self.layer_types:
            return self.layer_types[i]
        return "full"

    def kv_shape(self, i: int) -> tuple[int, int]:
        """(kv heads, head_dim) of layer i."""
        if self.family == "gemma4" and self.layer_type(i) == "full":
            return (self.global_kv_heads or self.num_kv_heads, self.global_head_dim or self.head_dim)
        return (self.num_kv_heads, self.head_dim)


def _eos_list(cfg: dict) -> list[int]:
    eos = cfg.get("eos_token_id")
    if eos is None:
        return []
    if isinstance(eos, (list, tuple)):
        return [int(e) for e in eos]
    return [int(eos)]


def _quant_from_hf(cfg: dict) -> QuantSpec:
    q = cfg.get("quantization_config") or {}
    if not q:
        return QuantSpec()
    method = str(q.get("quant_method", "")).lower()
    if "awq" in method:
        return QuantSpec("awq", int(q.get("bits", q.get("w_bit", 4))),
                         int(q.get("group_size", q.get("q_group_size", 128))),
                         bool(q.get("zero_point", True)), not bool(q.get("zero_point", True)))
    if method == "compressed-tensors" or q.get("format") == "pack-quantized":
        bits, group, sym = 4, 32, True
        for grp in (q.get("config_groups") or {}).values():
            w = (grp or {}).get("weights") or {}
            bits = int(w.get("num_bits", bits))
            group = int(w.get("group_size", group) or group)
            sym = bool(w.get("symmetric", sym))
            break
        return QuantSpec("compressed-tensors", bits, group, not sym, sym)
    if "gguf" in method:
        return QuantSpec("gguf", 8, 32, False, True)
    return QuantSpec()


def _sizes(entry: dict, names: tuple, where: str) -> None:
    for n in names:
        if not isinstance(entry.get(n), int) or entry[n] <= 0:
            raise ValueError(f"{where}: {n!r} must be a positive integer, got {entry.get(n)!r}")


def arch_from_fimodra_config(cfg: dict) -> ModelArch:
    """Fimodra configurations list their layers one by one (mixer type and sizes, feed-forward or null)."""
    layers = cfg["layers"]
    if not layers:
        raise ValueError("the configuration lists no layers")
    for i, l in enumerate(layers):
        m, where = l["mixer"], f"layers[{i}]"
        if l["type"] == "latent_attention":
            _sizes(m, ("heads", "dim", "rot_dim", "vdim", "kv_rank"), where)
            dims = (m.get("rot") or {}).get("dims", m["rot_dim"])
            if dims % 2 or dims > m["rot_dim"]:
                raise ValueError(f"{where}: cannot rotate {dims} of {m['rot_dim']} dimensions")
        elif l["type"] == "hgrn2":
            _sizes(m, ("heads", "dim", "vdim"), where)
        else:
            raise ValueError(f"{where}: unknown mixer {l['type']!r}")
        if l.get("mlp"):
            _sizes(l["mlp"], ("ff",), where)
    width, groups = int(cfg["width"]), int(cfg["norm"].get("groups", 1))
    if width % groups:
        raise ValueError(f"a width of {width} does not split into {groups} equal parts")
    heads = max(l["mixer"]["heads"] for l in layers)
    arch = ModelArch(
        family="fimodra", architecture="Fimodra", hidden_size=width, num_layers=len(layers), num_heads=heads,
        num_kv_heads=1, head_dim=max(l["mixer"]["dim"] for l in layers),
        intermediate_size=max((l["mlp"]["ff"] for l in layers if l.get("mlp")), default=0),
        vocab_size=int(cfg["vocab"]), rms_eps=float(cfg["norm"]["eps"]), act="relu",
        max_position=int(cfg.get("max_position_embeddings", 1 << 20)), eos_token_ids=_eos_list(cfg),
        bos_token_id=cfg.get("bos_token_id"))
    arch.layer_types = ["linear" if l["type"] == "hgrn2" else "sliding" for l in layers]
    arch.extra.update(layers=layers, norm_groups=groups)
    return arch


def arch_from_pofadra_config(cfg: dict) -> ModelArch:
    """Pofadra configurations list their layers one by one (mixer type and sizes, routed experts or null)."""
    layers = cfg["layers"]
    if not layers:
        raise ValueError("the configuration lists no layers")
    for i, l in enumerate(layers):
        m, where = l["mixer"], f"layers[{i}]"
        if l["type"] == "attention":
            _sizes(m, ("heads", "kv_heads", "dim", "vdim"), where)
            if m["vdim"] != m["dim"]:
                raise ValueError(f"{where}: keys are the values, so 'vdim' must equal 'dim'")
            dims = m["rot"]["dims"]
            if dims % 2 or dims > m["dim"] or dims < 0:
                raise ValueError(f"{where}: cannot rotate {dims} of {m['dim']} dimensions")
            _sizes(m["mask"], ("size",), where)
        elif l["type"] == "channel_delta":
            _sizes(m, ("heads", "kv_heads", "dim", "vdim", "conv"), where)
        else:
            raise ValueError(f"{where}: unknown mixer {l['type']!r}")
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{where}: {m['heads']} heads do not share {m['kv_heads']} key heads evenly")
        if l.get("mlp"):
            if l["mlp"].get("kind") != "moe":
                raise ValueError(f"{where}: unknown feed-forward {l['mlp'].get('kind')!r}")
            r = l["mlp"]["router"]
            _sizes(l["mlp"]["expert"], ("ff",), where)
            _sizes(r, ("experts", "top"), where)
            g = r.get("groups") or {"count": 1, "keep": 1}
            _sizes(g, ("count", "keep"), where)
            if r["experts"] % g["count"] or g["keep"] > g["count"] or r["top"] > g["keep"] * (r["experts"] // g["count"]):
                raise ValueError(f"{where}: cannot choose {r['top']} of {r['experts']} experts from {g['keep']} of {g['count']} groups")
    moes = [l["mlp"] for l in layers if l.get("mlp")]
    attn = [l["mixer"] for l in layers if l["type"] == "attention"]
    arch = ModelArch(
        family="pofadra", architecture="Pofadra", hidden_size=int(cfg["width"]), num_layers=len(layers),
        num_heads=max(l["mixer"]["heads"] for l in layers), num_kv_heads=max((m["kv_heads"] for m in attn), default=1),
        head_dim=max(l["mixer"]["dim"] for l in layers), intermediate_size=max((m["expert"]["ff"] for m in moes), default=0),
        vocab_size=int(cfg["vocab"]), rms_eps=float(cfg["norm"]["eps"]), act="silu",
        embed_scale=float((cfg.get("embedding") or {}).get("scale", 1.0)), final_softcap=float(cfg.get("logit_softcap") or 0.0),
        max_position=int(cfg.get("max_position_embeddings", 1 << 20)), eos_token_ids=_eos_list(cfg),
        bos_token_id=cfg.get("bos_token_id"))
    arch.layer_types = ["linear" if l["type"] == "channel_delta" else "sliding" for l in layers]
    arch.extra.update(layers=layers)
    return arch


def arch_from_luzerax_config(cfg: dict) -> ModelArch:
    """Luzerax configurations list their layers one by one (mixer type and sizes; dense, routed or no feed-forward)."""
    layers = cfg["layers"]
    if not layers:
        raise ValueError("the configuration lists no layers")

    def positive(entry: dict, name: str, where: str) -> None:
        if not isinstance(entry.get(name), (int, float)) or not entry[name] > 0:
            raise ValueError(f"{where}: {name!r} must be a positive number, got {entry.get(name)!r}")

    for i, l in enumerate(layers):
        m, where = l["mixer"], f"layers[{i}]"
        if l["type"] not in ("attention", "attention_2"):
            raise ValueError(f"{where}: unknown mixer {l['type']!r}")
        _sizes(m, ("heads", "kv_heads", "dim", "vdim"), where)
        positive(m, "scale", where)
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{where}: {m['heads']} heads do not share {m['kv_heads']} key heads evenly")
        if l["type"] == "attention":
            if not isinstance(m.get("diff"), (int, float)):
                raise ValueError(f"{where}: 'diff' must be a number, got {m.get('diff')!r}")
            if m.get("q_temp"):
                positive(m["q_temp"], "every", where)
        else:
            dims = m["rot"]["dims"]
            if dims % 2 or dims > m["dim"] or dims < 0:
                raise ValueError(f"{where}: cannot rotate {dims} of {m['dim']} dimensions")
        mlp = l.get("mlp")
        if not mlp:
            continue
        if mlp.get("kind") == "dense":
            _sizes(mlp, ("ff",), where)
        elif mlp.get("kind") == "moe":
            r = mlp["router"]
            for part in (mlp["expert"], *([mlp["shared"]] if mlp.get("shared") else [])):
                _sizes(part, ("ff",), where)
                positive(part, "limit", where)
            _sizes(r, ("experts", "top"), where)
            g, n = r.get("groups") or {"count": 1, "keep": 1}, r["experts"] + r.get("identity", 0)
            _sizes(g, ("count", "keep"), where)
            if n % g["count"] or g["keep"] > g["count"] or r["top"] > g["keep"] * (n // g["count"]):
                raise ValueError(f"{where}: cannot choose {r['top']} of {n} router outputs from {g['keep']} of {g['count']} groups")
        else:
            raise ValueError(f"{where}: unknown feed-forward {mlp.get('kind')!r}")
    mixers, mlps = [l["mixer"] for l in layers], [l["mlp"] for l in layers if l.get("mlp")]
    arch = ModelArch(
        family="luzerax", architecture="Luzerax", hidden_size=int(cfg["width"]), num_layers=len(layers),
        num_heads=max(m["heads"] for m in mixers), num_kv_heads=max(m["kv_heads"] for m in mixers),
        head_dim=max(m["dim"] for m in mixers),
        intermediate_size=max((m["ff"] if m["kind"] == "dense" else m["expert"]["ff"] for m in mlps), default=0),
        vocab_size=int(cfg["vocab"]), rms_eps=float(cfg["norm"]["eps"]), act="silu",
        max_position=int(cfg.get("max_position_embeddings", 1 << 20)), eos_token_ids=_eos_list(cfg),
        bos_token_id=cfg.get("bos_token_id"))
    arch.layer_types = ["full"] * len(layers)
    arch.extra.update(layers=layers)
    return arch


def arch_from_divadra_config(cfg: dict) -> ModelArch:
    """Divadra configurations list their layers one by one (mixer type and sizes; dense, assigned or no feed-forward)."""
    layers, taps, bigram = cfg["layers"], cfg["canon"].get("taps"), cfg["embedding"]["bigram"]
    if not layers:
        raise ValueError("the configuration lists no layers")
    _sizes(cfg["canon"], ("taps",), "canon")
    _sizes(bigram, ("buckets",), "embedding.bigram")
    for n in ("mul_prev", "mul_cur"):
        if not isinstance(bigram.get(n), int):
            raise ValueError(f"embedding.bigram: {n!r} must be an integer, got {bigram.get(n)!r}")

    def short(n: int, where: str) -> None:
        if n > 16:
            raise ValueError(f"{where}: convolutions of at most 16 taps, got {n}")

    short(taps, "canon")
    for i, l in enumerate(layers):
        m, where = l["mixer"], f"layers[{i}]"
        if l["type"] == "mamba2":
            _sizes(m, ("heads", "vdim", "state", "groups", "norm_groups", "conv"), where)
            short(m["conv"], where)
            if m["heads"] % m["groups"]:
                raise ValueError(f"{where}: {m['heads']} heads do not share {m['groups']} groups evenly")
            if m["heads"] * m["vdim"] % m["norm_groups"]:
                raise ValueError(f"{where}: {m['heads'] * m['vdim']} channels do not make {m['norm_groups']} equal norm parts")
        elif l["type"] == "parallel":
            a, r = m["left"], m["right"]
            _sizes(a, ("heads", "kv_heads", "dim", "vdim"), where)
            _sizes(a["mask"], ("size",), where)
            _sizes(r, ("heads", "dim"), where)
            if not isinstance(a.get("scale"), (int, float)):
                raise ValueError(f"{where}: 'scale' must be a number, got {a.get('scale')!r}")
            if a["heads"] % a["kv_heads"]:
                raise ValueError(f"{where}: {a['heads']} heads do not share {a['kv_heads']} key heads evenly")
            dims = a["rot"]["dims"]
            if dims % 2 or dims > a["dim"] or dims < 0:
                raise ValueError(f"{where}: cannot rotate {dims} of {a['dim']} dimensions")
            if a["vdim"] % 2:
                raise ValueError(f"{where}: cannot rotate values of {a['vdim']} dimensions")
        else:
            raise ValueError(f"{where}: unknown mixer {l['type']!r}")
        mlp = l.get("mlp")
        if not mlp:
            continue
        if mlp.get("kind") == "dense":
            _sizes(mlp, ("ff",), where)
        elif mlp.get("kind") == "moe":
            _sizes(mlp["expert"], ("ff",), where)
            _sizes(mlp["router"], ("experts", "top"), where)
            if mlp["router"]["top"] > mlp["router"]["experts"]:
                raise ValueError(f"{where}: cannot choose {mlp['router']['top']} of {mlp['router']['experts']} experts")
        else:
            raise ValueError(f"{where}: unknown feed-forward {mlp.get('kind')!r}")
    attn = [l["mixer"]["left"] for l in layers if l["type"] == "parallel"]
    mlps = [l["mlp"] for l in layers if l.get("mlp")]
    arch = ModelArch(
        family="divadra", architecture="Divadra", hidden_size=int(cfg["width"]), num_layers=len(layers),
        num_heads=max((a["heads"] for a in attn), default=1), num_kv_heads=max((a["kv_heads"] for a in attn), default=1),
        head_dim=max((a["dim"] for a in attn), default=64),
        intermediate_size=max((m["ff"] if m["kind"] == "dense" else m["expert"]["ff"] for m in mlps), default=0),
        vocab_size=int(cfg["vocab"]), rms_eps=float(cfg["norm"]["eps"]), act="relu2",
        max_position=int(cfg.get("max_position_embeddings", 1 << 20)), eos_token_ids=_eos_list(cfg),
        bos_token_id=cfg.get("bos_token_id"))
    arch.layer_types = ["linear" if l["type"] == "mamba2" else "sliding" for l in layers]
    arch.extra.update(layers=layers, canon_taps=taps, bigram=bigram)
    return arch


def arch_from_hf_config(cfg: dict) -> ModelArch:
    """Build a :class:`ModelArch` from a HF config dict (text sub-config is unwrapped)."""
    if str(cfg.get("architecture", "")).lower() == "divadra":
        return arch_from_divadra_config(cfg)
    if str(cfg.get("architecture", "")).lower() == "luzerax":
        return arch_from_luzerax_config(cfg)
    if str(cfg.get("architecture", "")).lower() == "pofadra":
        return arch_from_pofadra_config(cfg)
    if str(cfg.get("architecture", "")).lower() == "fimodra":
        return arch_from_fimodra_config(cfg)
    archs = cfg.get("architectures") or ["LlamaForCausalLM"]
    architecture = archs[0]
    text = cfg.get("text_config") or cfg
    name = architecture.lower()
    model_type = str(text.get("model_type", cfg.get("model_type", ""))).lower()
    if "gemma4" in name or "gemma4" in model_type or "gemma3n" in name:
        family = "gemma4"
    elif "deepseekv4" in name.replace("_", "") or "deepseek_v4" in model_type:
        family = "deepseek_v4_flash"
    elif "deepseek" in name or "deepseek" in model_type:
        family = "deepseek_mla"
    elif "qwen3_5" in model_type or "qwen3_5" in name or "qwen3next" in name or "qwen3_next" in model_type:
        family = "qwen3_5"
    elif "qwen2vl" in name.replace("_", "") or model_type == "qwen2_vl":
        family = "qwen2_vl"
    elif "qwen2" in name or "qwen3" in name:
        family = "qwen2"
    else:
        family = "llama"
    hidden = int(text["hidden_size"])
    heads = int(text["num_attention_heads"])
    kv_heads = int(text.get("num_key_value_heads", heads) or heads)
    head_dim = int(text.get("head_dim") or hidden // heads)
    arch = ModelArch(
        family=family, architecture=architecture, hidden_size=hidden,
        num_layers=int(text["num_hidden_layers"]), num_heads=heads, num_kv_heads=kv_heads,
        head_dim=head_dim, intermediate_size=int(text.get("intermediate_size", 4 * hidden)),
        vocab_size=int(text["vocab_size"]), rms_eps=float(text.get("rms_norm_eps", 1e-5)),
        rope_theta=float(text.get("rope_theta", (text.get("rope_parameters") or {}).get("rope_theta", 10000.0))),
        rope_scaling=text.get("rope_scaling"),
        max_position=int(text.get("max_position_embeddings", 4096)),
        tie_embeddings=bool(text.get("tie_word_embeddings", cfg.get("tie_word_embeddings", False))),
        act=str(text.get("hidden_act", text.get("hidden_activation", "silu"))),
        attn_bias=bool(text.get("attention_bias", family == "qwen2" and "qwen3" not in name)),
        mlp_bias=bool(text.get("mlp_bias", False)),
        sliding_window=int(text.get("sliding_window") or 0),
        eos_token_ids=_eos_list(text) or _eos_list(cfg),
        bos_token_id=text.get("bos_token_id", cfg.get("bos_token_id")),
        quant=_quant_from_hf(cfg),
        vision=cfg.get("vision_config"),
    )
    arch.partial_rotary_factor = float(text.get("partial_rotary_factor", 1.0))
    arch.rotary_dim = int(head_dim * arch.partial_rotary_factor)
    if family == "qwen2" and "qwen3" in name:
        arch.qk_norm = True
    if family == "gemma4":
        lt = text.get("layer_types") or []
        arch.layer_types = ["sliding" if "sliding" in t else "full" for t in lt]
        if not arch.layer_types:
            pat = int(text.get("sliding_window_pattern", 6))
            arch.layer_types = ["full" if (i + 1) % pat == 0 else "sliding" for i in range(arch.num_layers)]
        arch.attn_softcap = float(text.get("attn_logit_softcapping") or 0.0)
        arch.final_softcap = float(text.get("final_logit_softcapping") or 0.0)
        arch.qk_norm = True
        arch.embed_scale = float(hidden) ** 0.5
        arch.global_head_dim = text.get("global_head_dim")
        arch.global_kv_heads = text.get("num_global_key_value_heads")
        arch.global_rope_theta = text.get("rope_global_base_freq", text.get("global_rope_theta"))
        arch.rope_theta = float(text.get("rope_local_base_freq", arch.rope_theta))
        arch.act = "gelu_tanh"
        n_exp = int(text.get("num_experts", 0) or 0)
        if n_exp:
            arch.moe = MoESpec(num_experts=n_exp, top_k=int(text.get("top_k_experts", text.get("num_experts_per_tok", 8))),
                               expert_intermediate=int(text.get("moe_intermediate_size", text.get("expert_intermediate_size", 704))),
                               shared_intermediate=arch.intermediate_size, router="softmax", renormalize=True)
        arch.extra["attention_k_eq_v"] = bool(text.get("attention_k_eq_v", False))
    if family == "deepseek_mla":
        arch.mla = MLASpec(int(text.get("q_lora_rank") or 0), int(text.get("kv_lora_rank", 512)),
                           int(text.get("qk_rope_head_dim", 64)), int(text.get("qk_nope_head_dim", 128)),
                           int(text.get("v_head_dim", 128)))
        arch.head_dim = arch.mla.qk_nope_dim + arch.mla.qk_rope_dim
        arch.moe = MoESpec(num_experts=int(text.get("n_routed_experts", 0) or 0),
                           top_k=int(text.get("num_experts_per_tok", 6)),
                           expert_intermediate=int(text.get("moe_intermediate_size", 2048)),
                           n_shared_experts=int(text.get("n_shared_experts", 1)),
                           shared_intermediate=int(text.get("moe_intermediate_size", 2048)) * int(text.get("n_shared_experts", 1)),
                           router=str(text.get("scoring_func", "sigmoid")),
                           renormalize=bool(text.get("norm_topk_prob", True)),
                           routed_scaling=float(text.get("routed_scaling_factor", 1.0)),
                           first_dense_layers=int(text.get("first_k_dense_replace", 0)))
        if text.get("expert_staging_gb"):       # e.g. hf_overrides={"expert_staging_gb": 40}
            arch.extra["expert_staging_gb"] = float(text["expert_staging_gb"])
    if family == "deepseek_v4_flash":
        arch.extra["v4_rows"] = {k: text[k] for k in ("num_hidden_layers", "head_dim", "sliding_window",
                                                      "compress_ratio_coarse", "layer_compress_ratios")
                                 if text.get(k) is not None}
    if family == "qwen3_5":
        lt = text.get("layer_types") or []
        interval = int(text.get("full_attention_interval", 4))
        arch.layer_types = (["linear" if "linear" in t else "full" for t in lt] if lt else
                            ["full" if (i + 1) % interval == 0 else "linear" for i in range(arch.num_layers)])
        arch.qk_norm = True
        arch.norm_plus_one = True
        arch.extra.update({k: text.get(k) for k in (
            "linear_num_key_heads", "linear_num_value_heads", "linear_key_head_dim",
            "linear_value_head_dim", "linear_conv_kernel_dim", "mrope_section", "attn_output_gate")
            if text.get(k) is not None})
        n_exp = int(text.get("num_experts", 0) or 0)
        if n_exp:
            arch.moe = MoESpec(num_experts=n_exp, top_k=int(text.get("num_experts_per_tok", 8)),
                               expert_intermediate=int(text.get("moe_intermediate_size", 512)),
                               shared_intermediate=int(text.get("shared_expert_intermediate_size", 0)),
                               router="softmax", renormalize=bool(text.get("norm_topk_prob", True)))
    if family == "qwen2_vl":
        rs = text.get("rope_scaling") or cfg.get("rope_scaling") or {}
        if rs.get("mrope_section"):
            arch.extra["mrope_section"] = list(rs["mrope_section"])
    return arch
