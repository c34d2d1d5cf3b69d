"""Luzerax: a small decoder of differential and gated attention layers with dense or routed feed-forwards.

Sublayers read the 32-bit residual stream itself; what they return is normalised and scaled channel by channel:

    x <- x + rmsnorm(mixer(x)) * norm1 * ls1;   x <- x + rmsnorm(ff(x)) * norm2 * ls2

Layers are listed one by one in the configuration: a mixer with its sizes ("attention": two maps per head, weighted head
norms, queries scaled by position; "attention_2": rotary, unweighted head norms, a gate value per head) and a feed-forward
(dense, or routed experts with pass-through choices and a shared expert) or none.  The mixers are
``layers/head_attention.py``, the experts ``layers/fused_moe/routed_experts.py``.  Per sublayer boundary one kernel sums the
shared expert, the chosen experts and passed-through inputs, applies norm and scale (folded into one weight) and adds the
result to the stream; at the end it also computes the final norm of the wanted rows.
"""
from __future__ import annotations

import torch
from torch import nn

from ..layers.fused_moe.routed_experts import RoutedExperts
from ..layers.head_attention import HeadAttention
from ..layers.linear import LiteLinear
from ..ops import residual_stream as stream
from ..parallel import state as pstate
from ..utils.profiling import stage
from .arch import ModelArch


def _fp32(n: int) -> nn.Parameter:
    return nn.Parameter(torch.ones(n, dtype=torch.float32), requires_grad=False)


class GatedFeedForward(nn.Module):
    """``W_down (act(W_gate x) * (W_up x))``, or the clipped form of ``ops.gated_linear``."""

    def __init__(self, hidden: int, inter: int, dtype, act: str = "silu", act_limit: float = 0.0):
        super().__init__()
        self.gate_up_proj = LiteLinear(hidden, 2 * inter, dtype=dtype, gated_act=act, out_splits=[inter, inter], act_limit=act_limit)
        self.down_proj = LiteLinear(inter, hidden, dtype=dtype)

    def forward(self, x):
        return self.down_proj(self.gate_up_proj(x))

    def destinations(self, prefix: str) -> dict:
        return {prefix + "gate": (self.gate_up_proj, 0, "weight"), prefix + "up": (self.gate_up_proj, 1, "weight"),
                prefix + "down": (self.down_proj, 0, "weight")}


def _mixer(kind: str, m: dict, hidden: int, eps: float, dtype, max_pos: int) -> HeadAttention:
    common = (hidden, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], eps, dtype)
    if kind == "attention":
        t = m.get("q_temp")
        return HeadAttention(*common, temperature=(t["coef"], t["every"]) if t else None, diff_init=m["diff"], max_pos=max_pos)
    if kind == "attention_2":
        return HeadAttention(*common, norm_weights=False, rope_dims=m["rot"]["dims"], rope_base=m["rot"]["base"],
                             neighbours=True, norm_last=True, head_gate=True, max_pos=max_pos)
    raise ValueError(f"unknown mixer {kind!r}")


class LuzeraxLayer(nn.Module):
    def __init__(self, arch: ModelArch, i: int, dtype, max_pos: int):
        super().__init__()
        spec, W, eps = arch.extra["layers"][i], arch.hidden_size, arch.rms_eps
        self.index, self.eps, self.kind = i, eps, spec["type"]
        self.mixer = _mixer(self.kind, spec["mixer"], W, eps, dtype, max_pos)
        self.norm1, self.ls1 = _fp32(W), _fp32(W)
        self.dense = self.experts = self.shared = None
        mlp = spec.get("mlp")
        self.has_mlp = bool(mlp)
        if mlp:
            self.norm2, self.ls2 = _fp32(W), _fp32(W)
            if mlp["kind"] == "dense":
                self.dense = GatedFeedForward(W, mlp["ff"], dtype, arch.act)
            else:
                r, e, s = mlp["router"], mlp["expert"], mlp.get("shared")
                g = r.get("groups") or {"count": 1, "keep": 1}
                self.experts = RoutedExperts(W, e["ff"], r["experts"], r["top"], dtype, act="clipped_swiglu", act_limit=e["limit"],
                                             score="softmax", groups=g["count"], keep=g["keep"], group_best=1,
                                             renormalize=True, identity=r.get("identity", 0))
                self.router = LiteLinear(W, self.experts.outputs, dtype=dtype)
                if s:
                    self.shared = GatedFeedForward(W, s["ff"], dtype, "clipped_swiglu", s["limit"])

    def finish_loading(self) -> None:
        self.mixer.finish_loading()
        self.post1 = self.norm1 * self.ls1
        if self.has_mlp:
            self.post2 = self.norm2 * self.ls2

    def forward(self, h, x, batch, kv, last_norm, keep_stream: bool, sel=None):
        """h: the stream in the model's type; x: the stream (fp32), advanced in place up to the last boundary, there only
        when ``keep_stream``.  Returns the next layer's input, with ``last_norm`` the normalised rows ``sel``."""
        with stage("layer.mixer"):
            y, routed, post = self.mixer(h, batch, kv), None, self.post1
        if self.has_mlp:
            with stage("layer.mlp"):
                h = stream.post(y, x, None, post, None, self.eps, 1, x, h.dtype)
                post = self.post2
                if self.dense is not None:
                    y = self.dense(h)
                else:
                    routed = self.experts(h, self.router(h, out_dtype=torch.float32))
                    y = self.shared(h) if self.shared is not None else None
        return stream.post(y, x, routed, post, last_norm, self.eps, 1, x if keep_stream else None, h.dtype, sel)


class LuzeraxForCausalLM(nn.Module):
    supports_lora = False
    supports_multimodal = False
    supports_cuda_graph = True
    supports_mixed_batch = True        # portions of prompts and decoded tokens may share one forward pass

    def __init__(self, vllm_config):
        super().__init__()
        mc = vllm_config.model_config
        arch: ModelArch = mc.arch
        assert pstate.tp_size() == 1, "this model runs on a single GPU (or as data-parallel replicas)"
        self.arch, self.dtype, self.eps = arch, mc.dtype, arch.rms_eps
        W = arch.hidden_size
        self.embed_tokens = nn.Parameter(torch.empty(arch.vocab_size, W, dtype=mc.dtype), requires_grad=False)
        max_pos = max(mc.max_model_len, 16)
        self.layers = nn.ModuleList([LuzeraxLayer(arch, i, mc.dtype, max_pos) for i in range(arch.num_layers)])
        self.final_norm = _fp32(W)
        self.lm_head = LiteLinear(W, arch.vocab_size, dtype=mc.dtype, prefix="lm_head")

    def kv_cache_specs(self):
        from ..engine.kv_cache import KVLayerSpec
        return [KVLayerSpec(*l.mixer.cache_shape()) for l in self.layers]

    def forward(self, batch, kv_caches, inputs_embeds=None, collect=None):
        """Logits of the batch's wanted rows.  ``collect`` (a list) receives the stream after every layer (fp32)."""
        L, W = len(self.layers), self.arch.hidden_size
        x = torch.empty(batch.input_ids.shape[0], W, dtype=torch.float32, device=self.embed_tokens.device)
        h = stream.start(batch.input_ids, self.embed_tokens, None, self.eps, 1, x)
        for i, layer in enumerate(self.layers):
            last = i + 1 == L
            keep = not last or collect is not None
            h = layer(h, x, batch, kv_caches[i], self.final_norm if last else None, keep, None if keep else batch.logits_indices)
            if collect is not None:
                collect.append(x.clone())
        if collect is not None and batch.logits_indices is not None:
            h = h.index_select(0, batch.logits_indices)
        return self.lm_head(h, out_dtype=torch.float32)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights):
        """Checkpoint names: ``embed``, ``l<i>.norm1``, ``l<i>.ls1`` .., ``l<i>.mix.<name>``, ``l<i>.mlp.<name>``,
        ``l<i>.mlp.e<k>.<name>``, ``l<i>.mlp.shared.<name>``, ``final.norm``, ``head``.  Every destination must be filled
        exactly once."""
        from ..loaders.weight_utils import load_exact
        dest: dict = {"embed": self.embed_tokens, "final.norm": self.final_norm, "head": (self.lm_head, 0, "weight")}
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L.mixer
            mix, mlp = p + "mix.", p + "mlp."
            dest.update({p + "norm1": L.norm1, p + "ls1": L.ls1, mix + "o": (m.o_proj, 0, "weight")})
            dest.update({mix + n: (m.in_proj, j, "weight") for j, n in enumerate("qkvg" if m.gated else "qkv")})
            if m.q_norm is not None:
                dest.update({mix + "q.norm": m.q_norm, mix + "k.norm": m.k_norm})
            if m.diff_init is not None:
                dest.update({mix + n: getattr(m, n) for n in ("lq1", "lk1", "lq2", "lk2")})
            if L.has_mlp:
                dest.update({p + "norm2": L.norm2, p + "ls2": L.ls2})
            if L.dense is not None:
                dest.update(L.dense.destinations(mlp))
            if L.experts is not None:
                dest[mlp + "router"] = (L.router, 0, "weight")
                dest.update(L.experts.destinations(mlp))
            if L.shared is not None:
                dest.update(L.shared.destinations(mlp + "shared."))
        seen = load_exact(dest, weights)
        for L in self.layers:
            L.finish_loading()
        return seen
