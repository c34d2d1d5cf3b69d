"""Divadra: a small hybrid decoder whose layers add a mixer and a feed-forward that read the stream side by side.

    x <- x + mixer(c1(norm1(x))) + ff(c2(norm2(x))),   c(h) = h + causal convolution of h, channel by channel

The residual stream is 32-bit; it starts as the norm of a token embedding plus a row chosen by the previous and the present
token.  Layers are listed one by one in the configuration: a mixer ("mamba2", or "parallel": sigmoid attention in chunks and
time mixing side by side, whose normalised outputs are averaged) with its sizes, and a feed-forward (dense with squared
ReLU, experts assigned to token ids by a table, or none).  The mixers are ``layers/mamba2.py``, ``layers/sigmoid_attention.py``
and ``layers/time_mix.py``, the experts ``layers/fused_moe/routed_experts.py``.

``ops/shift_stream.py`` is the boundary between layers: the sum of what a layer returned, the norms of its two outputs, the
next layer's norm, both input convolutions and the blends of time mixing, in one kernel per decoded token and two per portion.
Key / value pages, recurrent states, convolution inputs and the previous token live in the cache manager.
"""
from __future__ import annotations

import torch
from torch import nn

from ..layers.fused_moe.routed_experts import AssignedExperts
from ..layers.linear import LiteLinear
from ..layers.mamba2 import Mamba2
from ..layers.sigmoid_attention import SigmoidAttention
from ..layers.time_mix import TimeMix
from ..ops import linear as _linear
from ..ops import shift_stream as stream
from ..parallel import state as pstate
from ..utils.profiling import stage
from .arch import ModelArch


def _fp32(*shape: int) -> nn.Parameter:
    return nn.Parameter(torch.ones(*shape, dtype=torch.float32), requires_grad=False)


class SquaredReluFeedForward(nn.Module):
    """``W_down relu(W_up x)^2``."""

    def __init__(self, hidden: int, inter: int, dtype):
        super().__init__()
        self.up_proj = LiteLinear(hidden, inter, dtype=dtype)
        self.down_proj = LiteLinear(inter, hidden, dtype=dtype)

    def forward(self, x):
        return self.down_proj(_linear(x, self.up_proj.weight, act="relu2"))

    def destinations(self, prefix: str) -> dict:
        return {prefix + "up": (self.up_proj, 0, "weight"), prefix + "down": (self.down_proj, 0, "weight")}


class DivadraLayer(nn.Module):
    def __init__(self, arch: ModelArch, i: int, dtype, max_pos: int):
        super().__init__()
        spec, W, eps, taps = arch.extra["layers"][i], arch.hidden_size, arch.rms_eps, arch.extra["canon_taps"]
        self.index, self.kind, m = i, spec["type"], spec["mixer"]
        self.mamba = self.left = self.right = None
        if self.kind == "mamba2":
            self.mamba = Mamba2(W, m["heads"], m["vdim"], m["state"], m["groups"], m["norm_groups"], m["conv"], eps, dtype)
        elif self.kind == "parallel":
            a, r = m["left"], m["right"]
            self.left = SigmoidAttention(W, a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["scale"], eps, dtype, a["mask"]["size"],
                                         a["rot"]["base"], a["rot"]["dims"], max_pos)
            self.right = TimeMix(W, r["heads"], r["dim"], eps, dtype)
            self.left_out, self.right_out = _fp32(W), _fp32(W)
        else:
            raise ValueError(f"layer {i}: unknown mixer {self.kind!r}")
        self.norm1, self.canon1 = _fp32(W), _fp32(W, taps)
        mlp = spec.get("mlp")
        self.has_mlp = bool(mlp)
        self.dense = self.experts = None
        if mlp:
            self.norm2, self.canon2 = _fp32(W), _fp32(W, taps)
            if mlp["kind"] == "dense":
                self.dense = SquaredReluFeedForward(W, mlp["ff"], dtype)
            else:
                r = mlp["router"]
                self.experts = AssignedExperts(W, mlp["expert"]["ff"], r["experts"], r["top"], arch.vocab_size, dtype)
        self.shift = None

    def cache_spec(self, width: int):
        from ..engine.kv_cache import KVLayerSpec
        common = dict(input_shape=(self.canon1.shape[1] + 1, width), last_token=self.index == 0)
        if self.mamba is not None:
            return KVLayerSpec(0, 0, 0, state_shape=self.mamba.state_shape(), ring_shape=self.mamba.ring_shape(), **common)
        return KVLayerSpec(*self.left.cache_shape(), state_shape=self.right.state_shape(), **common)

    def finish_loading(self) -> None:
        for m in (self.mamba, self.left, self.right):
            if m is not None:
                m.finish_loading()
        self.shift = stream.ShiftSpec(stream.fold_taps(self.norm1.data, self.canon1.data),
                                      stream.fold_taps(self.norm2.data, self.canon2.data) if self.has_mlp else None,
                                      None if self.right is None else self.right.mu.data)
        if self.right is not None:
            self.post = (self.left_out.data * 0.5, self.right_out.data * 0.5)     # the average of the two outputs

    def forward(self, inputs, batch, kv_caches):
        """inputs [outputs, T, W] of ``stream.layer_inputs``; returns what the layer adds to the stream."""
        i = self.index
        with stage("layer.mixer"):
            if self.mamba is not None:
                ys = (self.mamba(inputs[0], batch, kv_caches.states[i], kv_caches.rings[i]),)
            else:
                ys = (self.left(inputs[0], batch, kv_caches[i]), self.right(inputs[-stream.BLENDS:], batch, kv_caches.states[i]))
        f = routed = None
        if self.has_mlp:
            with stage("layer.mlp"):
                if self.dense is not None:
                    f = self.dense(inputs[1])
                else:
                    routed = self.experts(inputs[1], batch.input_ids)
        if self.mamba is not None:
            return stream.Summed(ys[0], f, routed)
        return stream.Paired(ys[0], self.post[0], ys[1], self.post[1], f, routed)


class DivadraForCausalLM(nn.Module):
    supports_lora = False
    supports_multimodal = False
    supports_cuda_graph = True
    supports_mixed_batch = True        # portions of prompts and decoded tokens may share one forward pass

    def __init__(self, vllm_config):
        super().__init__()
        mc = vllm_config.model_config
        arch: ModelArch = mc.arch
        assert pstate.tp_size() == 1, "this hybrid model runs on a single GPU (or as data-parallel replicas)"
        self.arch, self.dtype, self.eps = arch, mc.dtype, arch.rms_eps
        W, self.bigram = arch.hidden_size, arch.extra["bigram"]
        self.embed_tokens = nn.Parameter(torch.empty(arch.vocab_size, W, dtype=mc.dtype), requires_grad=False)
        self.embed_pairs = nn.Parameter(torch.empty(self.bigram["buckets"] + 1, W, dtype=mc.dtype), requires_grad=False)
        self.embed_norm, self.final_norm = _fp32(W), _fp32(W)
        max_pos = max(mc.max_model_len, 16)
        self.layers = nn.ModuleList([DivadraLayer(arch, i, mc.dtype, max_pos) for i in range(arch.num_layers)])
        self.lm_head = LiteLinear(W, arch.vocab_size, dtype=mc.dtype, prefix="lm_head")

    def kv_cache_specs(self):
        return [l.cache_spec(self.arch.hidden_size) for l in self.layers]

    def forward(self, batch, kv_caches, inputs_embeds=None, collect=None):
        """Logits of the batch's wanted rows.  ``collect`` (a list) receives the stream after every layer (fp32)."""
        x = torch.empty(batch.input_ids.shape[0], self.arch.hidden_size, dtype=torch.float32, device=self.embed_tokens.device)
        src = stream.Embedded(batch.input_ids, self.embed_tokens, self.embed_pairs, self.bigram["mul_prev"], self.bigram["mul_cur"],
                              self.embed_norm, kv_caches.last_tokens)
        for i, layer in enumerate(self.layers):
            h = stream.layer_inputs(src, x, layer.shift, kv_caches.inputs[i], batch, self.eps, self.dtype)
            if collect is not None and i:
                collect.append(x.clone())
            src = layer(h, batch, kv_caches)
        if collect is None:
            h = stream.normed(src, x, self.final_norm, batch, self.eps, self.dtype, batch.logits_indices)
        else:
            h = stream.normed(src, x, self.final_norm, batch, self.eps, self.dtype, keep=True)
            collect.append(x.clone())
            if batch.logits_indices is not None:
                h = h.index_select(0, batch.logits_indices)
        return self.lm_head(h, out_dtype=torch.float32)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights):
        """Checkpoint names: ``embed``, ``bigram``, ``embed.norm``, ``l<i>.norm1``, ``l<i>.canon1`` .., ``l<i>.mix.<name>``,
        ``l<i>.mix.left.<name>``, ``l<i>.mix.right.<name>``, ``l<i>.mlp.<name>``, ``l<i>.mlp.e<k>.<name>``, ``final.norm``,
        ``head``.  Every destination must be filled exactly once; norms in front of a feed-forward that a layer does not have
        are skipped."""
        from ..loaders.weight_utils import load_exact
        dest: dict = {"embed": self.embed_tokens, "bigram": self.embed_pairs, "embed.norm": self.embed_norm,
                      "final.norm": self.final_norm, "head": (self.lm_head, 0, "weight")}
        unused = set()
        for i, L in enumerate(self.layers):
            p = f"l{i}."
            mix, mlp = p + "mix.", p + "mlp."
            dest.update({p + "norm1": L.norm1, p + "canon1": L.canon1})
            if L.mamba is not None:
                dest.update(L.mamba.destinations(mix))
            else:
                m = L.left
                dest.update({mix + "left." + n: (m.qkv_proj, j, "weight") for j, n in enumerate("qkv")})
                dest.update({mix + "left.q.norm": m.q_norm, mix + "left.k.norm": m.k_norm, mix + "left.pb": m.bias,
                             mix + "left.o": (m.o_proj, 0, "weight"), mix + "left.out": L.left_out, mix + "right.out": L.right_out})
                dest.update(L.right.destinations(mix + "right."))
            if L.has_mlp:
                dest.update({p + "norm2": L.norm2, p + "canon2": L.canon2})
                dest.update((L.dense if L.dense is not None else L.experts).destinations(mlp))
            else:
                unused |= {p + "norm2", p + "canon2"}
        seen = load_exact(dest, ((n, t) for n, t in weights if n not in unused))
        for L in self.layers:
            L.finish_loading()
        return seen
