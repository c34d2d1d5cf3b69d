"""Pofadra: a small hybrid decoder of windowed attention and delta-rule layers with routed experts side by side.

A layer has one norm, and its mixer and its experts both read it; the residual stream is 32-bit:

    h = rmsnorm(x) * w;   x <- x + mixer(h) + experts(h)

Layers are listed one by one in the configuration: a mixer ("attention" or "channel_delta") with its sizes and routed
experts, or none.  The mixers are ``layers/windowed_attention.py`` and ``layers/channel_delta.py``, the experts
``layers/fused_moe/routed_experts.py``.  Per layer boundary one kernel adds the mixer's output and the weighted outputs of
the chosen experts to the stream and computes the next norm.  Projections that stay 32-bit (router, write strength of the
delta rule) share one product.  Key / value pages, recurrent states and convolution inputs live in the cache manager.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..layers.channel_delta import ChannelDelta
from ..layers.fused_moe.routed_experts import RoutedExperts
from ..layers.linear import LiteLinear
from ..layers.windowed_attention import WindowedAttention
from ..ops import residual_stream as stream
from ..parallel import state as pstate
from ..utils.profiling import stage
from .arch import ModelArch


def _fp32(n: int) -> nn.Parameter:
    return nn.Parameter(torch.ones(n, dtype=torch.float32), requires_grad=False)


class PofadraLayer(nn.Module):
    def __init__(self, arch: ModelArch, i: int, dtype, max_pos: int):
        super().__init__()
        spec, W, eps = arch.extra["layers"][i], arch.hidden_size, arch.rms_eps
        self.kind, m = spec["type"], spec["mixer"]
        if self.kind == "attention":
            self.mixer = WindowedAttention(W, m["heads"], m["kv_heads"], m["dim"], m["scale"], eps, dtype,
                                           window=m["mask"]["size"], rope_base=m["rot"]["base"], rope_dims=m["rot"]["dims"],
                                           sink=0.0, gated=True, max_pos=max_pos)
        elif self.kind == "channel_delta":
            self.mixer = ChannelDelta(W, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], eps, dtype)
        else:
            raise ValueError(f"layer {i}: unknown mixer {self.kind!r}")
        self.norm1 = _fp32(W)
        self.experts = None
        if spec.get("mlp"):
            r = spec["mlp"]["router"]
            g = r.get("groups") or {"count": 1, "keep": 1}
            self.experts = RoutedExperts(W, spec["mlp"]["expert"]["ff"], r["experts"], r["top"], dtype, act=arch.act,
                                         groups=g["count"], keep=g["keep"], scale=r.get("scale", 1.0))
        # 32-bit projections: router logits | write strengths
        side = [self.experts.E if self.experts else 0, m["heads"] if self.kind == "channel_delta" else 0]
        self.n_router = side[0]
        self.side_proj = LiteLinear(W, sum(side), dtype=dtype, out_splits=side) if sum(side) else None
        self.index, self.eps = i, eps

    def forward(self, h, x, batch, kv_caches, next_norm, keep_stream: bool, sel=None):
        """h: this layer's normalised input; x: the stream (fp32), advanced in place when ``keep_stream``.  Returns the
        next layer's input (rows ``sel`` only)."""
        i = self.index
        side = self.side_proj(h, out_dtype=torch.float32) if self.side_proj is not None else None
        with stage("layer.mixer"):
            if self.kind == "attention":
                y = self.mixer(h, batch, kv_caches[i])
            else:
                y = self.mixer(h, side[:, self.n_router:], batch, kv_caches.states[i], kv_caches.rings[i])
        routed = None
        if self.experts is not None:
            with stage("layer.mlp"):
                routed = self.experts(h, side[:, :self.n_router])
        return stream.add(y, x, routed, next_norm, self.eps, 1, x if keep_stream else None, h.dtype, sel)


class PofadraForCausalLM(nn.Module):
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
        W = arch.hidden_size
        self.embed_tokens = nn.Parameter(torch.empty(arch.vocab_size, W, dtype=mc.dtype), requires_grad=False)
        max_pos = max(mc.max_model_len, 16)
        self.layers = nn.ModuleList([PofadraLayer(arch, i, mc.dtype, max_pos) for i in range(arch.num_layers)])
        self.final_norm = _fp32(W)
        self.lm_head = LiteLinear(W, arch.vocab_size, dtype=mc.dtype, prefix="lm_head")

    def kv_cache_specs(self):
        from ..engine.kv_cache import KVLayerSpec
        return [KVLayerSpec(*l.mixer.cache_shape()) if l.kind == "attention" else
                KVLayerSpec(0, 0, 0, state_shape=l.mixer.state_shape(), ring_shape=l.mixer.ring_shape())
                for l in self.layers]

    def forward(self, batch, kv_caches, inputs_embeds=None, collect=None):
        """Logits of the batch's wanted rows.  ``collect`` (a list) receives the stream after every layer (fp32)."""
        L, W = len(self.layers), self.arch.hidden_size
        x = torch.empty(batch.input_ids.shape[0], W, dtype=torch.float32, device=self.embed_tokens.device)
        h = stream.start(batch.input_ids, self.embed_tokens, self.layers[0].norm1, self.eps, 1, x, self.arch.embed_scale)
        for i, layer in enumerate(self.layers):
            last = i + 1 == L
            keep = not last or collect is not None
            sel = None if keep else batch.logits_indices
            h = layer(h, x, batch, kv_caches, self.final_norm if last else self.layers[i + 1].norm1, keep, sel)
            if collect is not None:
                collect.append(x.clone())
        if collect is not None and batch.logits_indices is not None:
            h = h.index_select(0, batch.logits_indices)
        logits = self.lm_head(h, out_dtype=torch.float32)
        return ops.soft_cap(logits, self.arch.final_softcap) if self.arch.final_softcap > 0 else logits

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights):
        """Checkpoint names: ``embed``, ``l<i>.norm1``, ``l<i>.mix.<name>``, ``l<i>.mlp.e<k>.<name>``,
        ``l<i>.mlp.router``, ``l<i>.mlp.correction``, ``final.norm``, ``head``.  Every destination must be filled exactly
        once."""
        from ..loaders.weight_utils import load_exact
        dest: dict = {"embed": self.embed_tokens, "final.norm": self.final_norm, "head": (self.lm_head, 0, "weight")}
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L.mixer
            mix = p + "mix."
            dest.update({p + "norm1": L.norm1, mix + "o": (m.o_proj, 0, "weight")})
            if L.kind == "attention":
                dest.update({mix + "q": (m.qkg_proj, 0, "weight"), mix + "k": (m.qkg_proj, 1, "weight"),
                             mix + "g": (m.qkg_proj, 2, "weight"), mix + "q.norm": m.q_norm, mix + "k.norm": m.k_norm})
            else:
                for j, n in enumerate("qkv"):
                    dest[mix + n], dest[mix + n + ".conv"] = (m.in_proj, j, "weight"), m.conv_rows(n)
                dest.update({mix + "b": (L.side_proj, 1, "weight"), mix + "A_log": m.A_log, mix + "dt_bias": m.dt_bias,
                             mix + "norm": m.head_norm})
                dest.update({mix + n: m.low_rank(n) for n in ("a1", "a2", "g1", "g2")})
            if L.experts is not None:
                dest[p + "mlp.router"] = (L.side_proj, 0, "weight")
                dest.update(L.experts.destinations(p + "mlp."))
        seen = load_exact(dest, weights)
        for L in self.layers:
            if L.kind == "channel_delta":
                L.mixer.finish_loading()
        return seen
