"""HF-style config dicts for the architectures the benchmarks name.  ``synthetic:<name>`` as a model
path builds one of these with random-init weights (no checkpoint files needed)."""
from __future__ import annotations

import copy

PRESETS: dict[str, dict] = {
    # TinyLlama-1.1B: 22 layers, hidden 2048, 32 q / 4 kv heads, head_dim 64, FFN 5632, vocab 32000
    "tinyllama-1.1b": {
        "architectures": ["LlamaForCausalLM"], "model_type": "llama", "hidden_size": 2048,
        "num_hidden_layers": 22, "num_attention_heads": 32, "num_key_value_heads": 4,
        "intermediate_size": 5632, "vocab_size": 32000, "rms_norm_eps": 1e-5, "rope_theta": 10000.0,
        "max_position_embeddings": 4096, "hidden_act": "silu", "tie_word_embeddings": False,
        "eos_token_id": 2, "bos_token_id": 1,
    },
    # 9B dense GQA decoder with zero-point AWQ int4 (group 128)
    "dense-9b-awq": {
        "architectures": ["LlamaForCausalLM"], "model_type": "llama", "hidden_size": 4096,
        "num_hidden_layers": 36, "num_attention_heads": 32, "num_key_value_heads": 8, "head_dim": 128,
        "intermediate_size": 12288, "vocab_size": 151936, "rms_norm_eps": 1e-6, "rope_theta": 1000000.0,
        "max_position_embeddings": 4096, "hidden_act": "silu", "tie_word_embeddings": False,
        "eos_token_id": 151645,
        "quantization_config": {"quant_method": "awq", "bits": 4, "group_size": 128, "zero_point": True},
    },
    # Gemma4-26B-A4B-shaped MoE
    "gemma4-26b-a4b": {
        "architectures": ["Gemma4ForConditionalGeneration"], "model_type": "gemma4",
        "text_config": {
            "model_type": "gemma4_text", "hidden_size": 2816, "num_hidden_layers": 30,
            "num_attention_heads": 16, "num_key_value_heads": 8, "head_dim": 256,
            "intermediate_size": 2112, "vocab_size": 262144, "rms_norm_eps": 1e-6,
            "sliding_window": 1024, "sliding_window_pattern": 6, "attn_logit_softcapping": 50.0,
            "final_logit_softcapping": 30.0, "rope_local_base_freq": 10000.0,
            "rope_global_base_freq": 1000000.0, "max_position_embeddings": 4096,
            "num_experts": 128, "top_k_experts": 8, "moe_intermediate_size": 704,
            "hidden_activation": "gelu_pytorch_tanh", "tie_word_embeddings": True, "eos_token_id": 1,
        },
        "quantization_config": {"quant_method": "compressed-tensors", "format": "pack-quantized",
                                "config_groups": {"group_0": {"weights": {"num_bits": 4, "group_size": 32,
                                                                           "symmetric": True}}}},
    },
    # DeepSeek-V3-style MLA + MoE (GGUF-quantised in the named config)
    "deepseek-mla-moe": {
        "architectures": ["DeepseekV3ForCausalLM"], "model_type": "deepseek_v3", "hidden_size": 4096,
        "num_hidden_layers": 43, "num_attention_heads": 64, "num_key_value_heads": 64,
        "q_lora_rank": 1024, "kv_lora_rank": 512, "qk_rope_head_dim": 64, "qk_nope_head_dim": 128,
        "v_head_dim": 128, "intermediate_size": 2048, "moe_intermediate_size": 2048,
        "n_routed_experts": 256, "num_experts_per_tok": 6, "n_shared_experts": 1,
        "scoring_func": "sigmoid", "norm_topk_prob": True, "routed_scaling_factor": 1.0,
        "first_k_dense_replace": 0, "vocab_size": 129280, "rms_norm_eps": 1e-6, "rope_theta": 10000.0,
        "max_position_embeddings": 4096, "eos_token_id": 1,
        "quantization_config": {"quant_method": "gguf"},
    },
}

# Small variants for tests (same code paths, seconds on a CPU).
PRESETS["tiny-llama-test"] = dict(PRESETS["tinyllama-1.1b"], hidden_size=256, num_hidden_layers=2,
                                  num_attention_heads=4, num_key_value_heads=2, intermediate_size=256,
                                  vocab_size=512, max_position_embeddings=512)
PRESETS["tiny-llama-awq-test"] = dict(PRESETS["tiny-llama-test"], quantization_config={
    "quant_method": "awq", "bits": 4, "group_size": 128, "zero_point": True})
PRESETS["tiny-llama-ct-test"] = dict(PRESETS["tiny-llama-test"], quantization_config={
    "quant_method": "compressed-tensors", "format": "pack-quantized",
    "config_groups": {"group_0": {"weights": {"num_bits": 4, "group_size": 32, "symmetric": True}}}})
PRESETS["tiny-gemma4-moe-test"] = {
    "architectures": ["Gemma4ForConditionalGeneration"], "model_type": "gemma4",
    "text_config": {"model_type": "gemma4_text", "hidden_size": 256, "num_hidden_layers": 3,
                    "num_attention_heads": 4, "num_key_value_heads": 2, "head_dim": 64, "intermediate_size": 192,
                    "vocab_size": 512, "rms_norm_eps": 1e-6, "sliding_window": 32, "sliding_window_pattern": 3,
                    "attn_logit_softcapping": 50.0, "final_logit_softcapping": 30.0, "rope_local_base_freq": 10000.0,
                    "rope_global_base_freq": 1000000.0, "max_position_embeddings": 512, "num_experts": 8,
                    "top_k_experts": 2, "moe_intermediate_size": 128, "tie_word_embeddings": True, "eos_token_id": 1},
    "quantization_config": {"quant_method": "compressed-tensors", "format": "pack-quantized",
                            "config_groups": {"group_0": {"weights": {"num_bits": 4, "group_size": 32,
                                                                       "symmetric": True}}}},
}
PRESETS["tiny-deepseek-test"] = dict(PRESETS["deepseek-mla-moe"], hidden_size=256, num_hidden_layers=2,
                                     num_attention_heads=4, num_key_value_heads=4, q_lora_rank=64, kv_lora_rank=64,
                                     qk_rope_head_dim=64, qk_nope_head_dim=64, v_head_dim=64, intermediate_size=256,
                                     moe_intermediate_size=256, n_routed_experts=8, num_experts_per_tok=2,
                                     vocab_size=512, max_position_embeddings=512)
# the latent geometry of the full-size model (512 + 64) with 20 heads: exercises the absorbed attention kernel
PRESETS["tiny-deepseek-mla512-test"] = dict(PRESETS["tiny-deepseek-test"], num_attention_heads=20, num_key_value_heads=20,
                                            kv_lora_rank=512, qk_nope_head_dim=128, v_head_dim=128)
# DeepSeek-V4-Flash geometry in miniature: 512-wide shared latent rows, a window shorter than the test prompts,
# two window-only layers, then a fine (ratio 4, indexer top-k smaller than the emitted rows) and a coarse
# (ratio 8, all rows) compressed layer
PRESETS["tiny-deepseek-v4-flash-test"] = {
    "architectures": ["DeepseekV4FlashForCausalLM"], "model_type": "deepseek_v4_flash", "hidden_size": 256,
    "num_hidden_layers": 4, "num_attention_heads": 4, "num_key_value_heads": 1, "head_dim": 512,
    "qk_rope_head_dim": 64, "q_lora_rank": 64, "sliding_window": 8, "compress_ratio_coarse": 8, "index_n_heads": 2,
    "index_topk": 3, "hc_mult": 4, "o_groups": 2, "o_lora_rank": 32, "n_routed_experts": 8,
    "num_experts_per_tok": 2, "moe_intermediate_size": 256, "num_hash_layers": 1, "routed_scaling_factor": 1.5,
    "vocab_size": 512, "rms_norm_eps": 1e-6, "rope_theta": 10000.0, "max_position_embeddings": 512,
    "intermediate_size": 256, "eos_token_id": 1,
}
# the same with random weights in the checkpoint's block formats (IQ2_XXS / Q2_K routed experts, Q8_0 projections)
PRESETS["tiny-deepseek-v4-flash-blocks-test"] = dict(PRESETS["tiny-deepseek-v4-flash-test"], synthetic_block_weights=True)
# the full-size geometry of the DeepSeek-V4-Flash checkpoint family; as a synthetic model its weights are random
# blocks in the checkpoint's formats (IQ2_XXS / Q2_K experts, Q8_0 projections: about 90 GB)
PRESETS["deepseek-v4-flash"] = {
    "architectures": ["DeepseekV4FlashForCausalLM"], "model_type": "deepseek_v4_flash", "hidden_size": 4096,
    "num_hidden_layers": 43, "num_attention_heads": 64, "num_key_value_heads": 1, "head_dim": 512,
    "qk_rope_head_dim": 64, "q_lora_rank": 1024, "sliding_window": 128, "index_n_heads": 64, "index_topk": 512,
    "hc_mult": 4, "o_groups": 8, "o_lora_rank": 1024, "n_routed_experts": 256, "num_experts_per_tok": 6,
    "moe_intermediate_size": 2048, "num_hash_layers": 3, "routed_scaling_factor": 1.5, "swiglu_limit": 10.0,
    "vocab_size": 129280, "rms_norm_eps": 1e-6, "rope_theta": 10000.0, "max_position_embeddings": 65536,
    "intermediate_size": 2048, "eos_token_id": 1, "synthetic_block_weights": True,
}
PRESETS["tiny-qwen35-test"] = {
    "architectures": ["Qwen3_5ForCausalLM"], "model_type": "qwen3_5", "hidden_size": 256, "num_hidden_layers": 4,
    "num_attention_heads": 4, "num_key_value_heads": 2, "head_dim": 64, "intermediate_size": 256, "vocab_size": 512,
    "rms_norm_eps": 1e-6, "rope_theta": 10000.0, "max_position_embeddings": 512, "partial_rotary_factor": 0.25,
    "full_attention_interval": 4, "linear_num_key_heads": 2, "linear_num_value_heads": 4, "linear_key_head_dim": 32,
    "linear_value_head_dim": 32, "linear_conv_kernel_dim": 4, "attn_output_gate": True, "eos_token_id": 1,
}
PRESETS["tiny-qwen35-moe-test"] = dict(PRESETS["tiny-qwen35-test"], architectures=["Qwen3_5MoeForCausalLM"],
                                      num_experts=8, num_experts_per_tok=2, moe_intermediate_size=128,
                                      shared_expert_intermediate_size=128, norm_topk_prob=True)
PRESETS["tiny-qwen3-test"] = dict(PRESETS["tiny-llama-test"], architectures=["Qwen3ForCausalLM"], model_type="qwen3",
                                  head_dim=64)
PRESETS["tiny-qwen2vl-test"] = dict(PRESETS["tiny-llama-test"], architectures=["Qwen2VLForConditionalGeneration"],
                                    model_type="qwen2_vl", attention_bias=True,
                                    vision_config={"patch_size": 14, "embed_dim": 64, "depth": 2, "num_heads": 2,
                                                   "spatial_merge_size": 2, "temporal_patch_size": 2, "mlp_ratio": 2,
                                                   "min_pixels": 28 * 28, "max_pixels": 28 * 28 * 16},
                                    rope_scaling={"type": "mrope", "mrope_section": [16, 8, 8]})


def fimodra_config(width: int, vocab: int, ff: int, pattern: str, heads: int, dim: int, rot_dim: int, vdim: int,
                   kv_rank: int, window: int, lin_heads: int, lin_dim: int, lin_vdim: int, groups: int = 4,
                   rot_base: float = 10000.0) -> dict:
    """Fimodra configuration from a layer pattern: "a" latent attention, "h" HGRN2, upper case without a feed-forward."""
    attn = {"dim": dim, "heads": heads, "kv_rank": kv_rank, "mask": {"size": window},
            "rot": {"base": rot_base, "dims": rot_dim}, "rot_dim": rot_dim, "scale": (dim + rot_dim) ** -0.5, "vdim": vdim}
    lin = {"dim": lin_dim, "heads": lin_heads, "vdim": lin_vdim}
    layers = [{"type": "latent_attention" if c in "aA" else "hgrn2", "mixer": copy.deepcopy(attn if c in "aA" else lin),
               "mlp": {"kind": "dense", "ff": ff} if c.islower() else None} for c in pattern]
    return {"architecture": "Fimodra", "width": width, "vocab": vocab, "norm": {"eps": 1e-6, "groups": groups},
            "layers": layers}


PRESETS["tiny-fimodra-test"] = fimodra_config(256, 512, 192, "ahHaA", 3, 24, 8, 40, 80, 20, 5, 32, 24)
# layers of the width and head geometry of a 1B-class decoder
PRESETS["fimodra-1b"] = fimodra_config(2048, 32000, 5632, "aaha" * 5, 16, 96, 32, 128, 512, 1024, 16, 128, 128, groups=2)


def pofadra_config(width: int, vocab: int, pattern: str, attn: tuple, delta: tuple, moe: tuple, rot_base: float = 10000.0,
                   softcap: float = 30.0, embed_scale: float = 1.0) -> dict:
    """Pofadra configuration from a layer pattern: "a" attention, "d" delta rule, upper case without a feed-forward.
    ``attn``: heads, kv heads, dim, rotated dims, window; ``delta``: heads, kv heads, dim, vdim, taps; ``moe``: experts,
    top, groups, kept groups, ff."""
    a = dict(zip(("heads", "kv_heads", "dim"), attn[:3]), vdim=attn[2], rot={"base": rot_base, "dims": attn[3]},
             mask={"size": attn[4]}, scale=attn[2] ** -0.5)
    d = dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), delta))
    ff = {"kind": "moe", "expert": {"ff": moe[4]}, "router": {"experts": moe[0], "top": moe[1], "scale": 1.0,
                                                               "groups": {"count": moe[2], "keep": moe[3]}}}
    layers = [{"type": "attention" if c in "aA" else "channel_delta", "mixer": copy.deepcopy(a if c in "aA" else d),
               "mlp": copy.deepcopy(ff) if c.islower() else None} for c in pattern]
    return {"architecture": "Pofadra", "width": width, "vocab": vocab, "norm": {"eps": 1e-6}, "layers": layers,
            "embedding": {"scale": embed_scale}, "logit_softcap": softcap}


PRESETS["tiny-pofadra-test"] = pofadra_config(160, 512, "ddaDA", (6, 2, 40, 24, 24), (4, 2, 24, 40, 3), (12, 2, 3, 2, 72))
# layers of the width and head geometry of a 1B-class decoder
PRESETS["pofadra-1b"] = pofadra_config(2048, 32000, "ddad" * 3, (16, 4, 128, 64, 1024), (16, 16, 128, 128, 4), (32, 4, 4, 2, 768))


def luzerax_config(width: int, vocab: int, pattern: str, diff: tuple, gated: tuple, ff: int, moe: tuple, rot_base: float = 1e5,
                   temp: tuple = (0.4, 4096), diff_init: float = 0.4, eps: float = 1e-6) -> dict:
    """Luzerax configuration from a layer pattern: per layer a mixer ("d" differential, "g" gated) and a feed-forward ("f"
    dense, "m" routed, "-" none).  ``diff``: heads, kv heads, dim of a map, vdim; ``gated``: heads, kv heads, dim, vdim,
    rotated dims; ``moe``: experts, pass-through outputs, top, groups, kept groups, ff, ff of the shared expert; ``temp``:
    coefficient and span of the queries' factor."""
    d = dict(zip(("heads", "kv_heads", "dim", "vdim"), diff), scale=diff[2] ** -0.5, diff=diff_init,
             q_temp=dict(zip(("coef", "every"), temp)))
    g = dict(zip(("heads", "kv_heads", "dim", "vdim"), gated[:4]), scale=gated[2] ** -0.5 * 8,
             rot={"base": rot_base, "dims": gated[4]})
    routed = {"kind": "moe", "expert": {"ff": moe[5], "limit": 7.0}, "shared": {"ff": moe[6], "limit": 5.0},
              "router": {"experts": moe[0], "identity": moe[1], "top": moe[2], "groups": {"count": moe[3], "keep": moe[4]}}}
    mlps = {"f": {"kind": "dense", "ff": ff}, "m": routed, "-": None}
    layers = [{"type": "attention" if pattern[i] == "d" else "attention_2", "mixer": copy.deepcopy(d if pattern[i] == "d" else g),
               "mlp": copy.deepcopy(mlps[pattern[i + 1]])} for i in range(0, len(pattern), 2)]
    return {"architecture": "Luzerax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": layers}


PRESETS["tiny-luzerax-test"] = luzerax_config(160, 512, "dfgmd-gf", (6, 2, 24, 40), (4, 2, 40, 24, 16), 176, (9, 3, 3, 4, 2, 48, 80),
                                              temp=(0.7, 20))
# layers of the width and head geometry of a 1B-class decoder
PRESETS["luzerax-1b"] = luzerax_config(2048, 32000, "df" + "gmdmgm" * 3, (16, 4, 64, 128), (16, 4, 128, 128, 64), 5632,
                                       (32, 8, 4, 4, 2, 768, 1536))


def divadra_config(width: int, vocab: int, pattern: str, mamba: tuple, left: tuple, right: tuple, ff: int, moe: tuple,
                   bigram: tuple = (4093, 31, 7), taps: int = 4, rot_base: float = 1e4, eps: float = 1e-6) -> dict:
    """Divadra configuration from a layer pattern: per layer a mixer ("s" state space, "p" parallel) and a feed-forward ("f"
    dense, "m" assigned experts, "-" none).  ``mamba``: heads, vdim, state, groups, norm groups, taps; ``left``: heads, kv
    heads, dim, vdim, rotated dims, chunk; ``right``: heads, dim; ``moe``: experts, top, ff; ``bigram``: buckets, multipliers."""
    s = dict(zip(("heads", "vdim", "state", "groups", "norm_groups", "conv"), mamba))
    p = {"left": dict(zip(("heads", "kv_heads", "dim", "vdim"), left[:4]), scale=left[2] ** -0.5, mask={"size": left[5]},
                      rot={"base": rot_base, "dims": left[4]}),
         "right": dict(zip(("heads", "dim"), right))}
    mlps = {"f": {"kind": "dense", "ff": ff}, "-": None,
            "m": {"kind": "moe", "expert": {"ff": moe[2]}, "router": {"experts": moe[0], "top": moe[1]}}}
    layers = [{"type": "mamba2" if pattern[i] == "s" else "parallel", "mixer": copy.deepcopy(s if pattern[i] == "s" else p),
               "mlp": copy.deepcopy(mlps[pattern[i + 1]])} for i in range(0, len(pattern), 2)]
    return {"architecture": "Divadra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers}


PRESETS["tiny-divadra-test"] = divadra_config(160, 512, "sfpmp-pf", (4, 40, 24, 2, 5, 3), (6, 2, 40, 24, 16, 20), (4, 40), 176, (9, 3, 48),
                                              bigram=(251, 31, 7), taps=3)
# layers of the width and head geometry of a 1B-class decoder
PRESETS["divadra-1b"] = divadra_config(2048, 32000, "sf" + "pmpfpm" * 3, (32, 128, 128, 4, 4, 4), (16, 4, 128, 128, 128, 1024), (32, 64), 5632,
                                       (32, 4, 768))


def get_preset(name: str) -> dict:
    key = name.lower()
    if key not in PRESETS:
        raise KeyError(f"unknown synthetic preset {name!r}; known: {sorted(PRESETS)}")
    return copy.deepcopy(PRESETS[key])
