"""Fimodra: a small hybrid decoder of windowed latent attention and HGRN2 layers.

Every sublayer is normalised before and after (RMS norm in groups), the residual stream is 32-bit, and what a layer
hands on is a learned average over the embedding output and the results of all layers up to it:

    x <- x + norm1b(mixer(norm1(x)));  x <- x + norm2b(mlp(norm2(x)));  X_(i+1) = x;  x <- sum_{j <= i+1} a_ij X_j

Layers are listed one by one in the configuration: a mixer ("latent_attention" or "hgrn2") with its sizes and a dense
gated feed-forward with biases, or none.  The mixers are ``layers/latent_attention.py`` and ``layers/hgrn2.py``, the
stream ``ops/residual_stream.py``: per sublayer boundary one kernel does post-norm, residual add, depth average and the
next pre-norm.  Latent rows are paged in the KV pool; recurrent states live in its per-slot pools.
"""
from __future__ import annotations

import torch
from torch import nn

from .. import ops
from ..layers.hgrn2 import Hgrn2
from ..layers.latent_attention import LatentAttention
from ..layers.linear import LiteLinear
from ..ops import residual_stream as stream
from ..parallel import state as pstate
from ..utils.profiling import stage
from .arch import ModelArch


def _fp32(n: int) -> nn.Parameter:
    return nn.Parameter(torch.ones(n, dtype=torch.float32), requires_grad=False)


class DenseMLP(nn.Module):
    """``W_down (act(W_gate x + b_g) * (W_up x + b_u)) + b_d``."""

    def __init__(self, hidden: int, inter: int, dtype, act: str):
        super().__init__()
        self.gate_up_proj = LiteLinear(hidden, 2 * inter, bias=True, dtype=dtype, gated_act=act, out_splits=[inter, inter])
        self.down_proj = LiteLinear(inter, hidden, bias=True, dtype=dtype)

    def forward(self, x):
        return self.down_proj(self.gate_up_proj(x))


class FimodraLayer(nn.Module):
    def __init__(self, arch: ModelArch, i: int, dtype, max_pos: int):
        super().__init__()
        spec, W, eps = arch.extra["layers"][i], arch.hidden_size, arch.rms_eps
        self.kind, m = spec["type"], spec["mixer"]
        if self.kind == "latent_attention":
            rot = m.get("rot") or {}
            self.mixer = LatentAttention(W, m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["scale"], eps,
                                         dtype, window=(m.get("mask") or {}).get("size", 0),
                                         rope_base=rot.get("base", 10000.0), rope_dims=rot.get("dims"), sinks=True,
                                         max_pos=max_pos)
        elif self.kind == "hgrn2":
            self.mixer = Hgrn2(W, m["heads"], m["dim"], m["vdim"], eps, dtype)
        else:
            raise ValueError(f"layer {i}: unknown mixer {self.kind!r}")
        self.norm1, self.norm1b = _fp32(W), _fp32(W)
        self.mlp = None
        if spec.get("mlp"):
            if spec["mlp"]["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {spec['mlp']['kind']!r}")
            self.mlp = DenseMLP(W, spec["mlp"]["ff"], dtype, arch.act)
            self.norm2, self.norm2b = _fp32(W), _fp32(W)
        self.depth_weights = nn.Parameter(torch.zeros(i + 2, dtype=torch.float32), requires_grad=False)
        self.index, self.eps, self.groups = i, eps, int(arch.extra["norm_groups"])

    def forward(self, h, src, x, hist, batch, kv_caches, next_norm, sel=None):
        """h: this layer's normalised input; src: the stream before it (fp32); x: buffer that receives what the layer
        hands on; hist: results X_0 .. X_i, X_(i+1) is added.  Returns the next sublayer's input (rows ``sel`` only)."""
        i = self.index
        with stage("layer.mixer"):
            y = self.mixer(h, batch, kv_caches[i][0] if self.kind == "latent_attention" else kv_caches.states[i])
        post = self.norm1b
        if self.mlp is not None:
            with stage("layer.mlp"):
                h = stream.step(y, src, post, self.norm2, self.eps, self.groups, x, h.dtype)
                y = self.mlp(h)
            src, post = x, self.norm2b
        return stream.average(y, src, post, next_norm, self.eps, self.groups, hist, i + 1, self.depth_weights, x, h.dtype, sel)


class FimodraForCausalLM(nn.Module):
    supports_lora = False
    supports_multimodal = False
    supports_cuda_graph = True
    supports_mixed_batch = True        # portions of prompts and decoded tokens may share one forward pass

    def __init__(self, vllm_config):
        super().__init__()
        mc = vllm_config.model_config
        arch: ModelArch = mc.arch
        assert pstate.tp_size() == 1, "this hybrid model runs on a single GPU (or as data-parallel replicas)"
        self.arch, self.dtype = arch, mc.dtype
        self.eps, self.groups = arch.rms_eps, int(arch.extra["norm_groups"])
        W = arch.hidden_size
        self.embed_tokens = nn.Parameter(torch.empty(arch.vocab_size, W, dtype=mc.dtype), requires_grad=False)
        max_pos = max(mc.max_model_len, 16)
        self.layers = nn.ModuleList([FimodraLayer(arch, i, mc.dtype, max_pos) for i in range(arch.num_layers)])
        self.final_norm = _fp32(W)
        self.lm_head = LiteLinear(W, arch.vocab_size, dtype=mc.dtype, prefix="lm_head")

    def kv_cache_specs(self):
        from ..engine.kv_cache import KVLayerSpec
        return [KVLayerSpec(1, l.mixer.cache_width(), 0) if l.kind == "latent_attention" else
                KVLayerSpec(0, 0, 0, state_shape=l.mixer.state_shape()) for l in self.layers]

    def forward(self, batch, kv_caches, inputs_embeds=None, collect=None):
        """Logits of the batch's wanted rows.  ``collect`` (a list) receives what every layer hands on (fp32)."""
        L, W = len(self.layers), self.arch.hidden_size
        T, dev = batch.input_ids.shape[0], self.embed_tokens.device
        hist = torch.empty(L + 1, T, W, dtype=torch.float32, device=dev)
        x = torch.empty(T, W, dtype=torch.float32, device=dev)
        h = stream.start(batch.input_ids, self.embed_tokens, self.layers[0].norm1, self.eps, self.groups, hist[0])
        src = hist[0]
        for i, layer in enumerate(self.layers):
            last = i + 1 == L
            nxt = self.final_norm if last else self.layers[i + 1].norm1
            sel = batch.logits_indices if last and collect is None else None
            h = layer(h, src, x, hist, batch, kv_caches, nxt, sel)
            src = x
            if collect is not None:
                collect.append(x.clone())
        if collect is not None and batch.logits_indices is not None:
            h = h.index_select(0, batch.logits_indices)
        return self.lm_head(h, out_dtype=torch.float32)

    # ------------------------------------------------------------------ loading
    def load_weights(self, weights):
        """Checkpoint names: ``embed``, ``l<i>.norm1`` .., ``l<i>.mix.<name>``, ``l<i>.mlp.<name>[.b]``, ``l<i>.dwa``,
        ``final.norm``, ``head``.  Every destination must be filled exactly once."""
        from ..loaders.weight_utils import load_exact
        dest: dict = {"embed": self.embed_tokens, "final.norm": self.final_norm, "head": (self.lm_head, 0, "weight")}
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L.mixer
            dest[p + "norm1"], dest[p + "norm1b"], dest[p + "dwa"] = L.norm1, L.norm1b, L.depth_weights
            if L.kind == "latent_attention":
                dest.update({p + "mix.q": (m.qkv_proj, 0, "weight"), p + "mix.dkv": (m.qkv_proj, 1, "weight"),
                             p + "mix.dkv.norm": m.latent_norm, p + "mix.uk": (m.up_proj, 0, "weight"),
                             p + "mix.uv": (m.up_proj, 1, "weight"), p + "mix.sink": m.sinks,
                             p + "mix.o": (m.o_proj, 0, "weight")})
            else:
                dest.update({p + "mix.q": (m.in_proj, 0, "weight"), p + "mix.v": (m.in_proj, 1, "weight"),
                             p + "mix.f": (m.in_proj, 2, "weight"), p + "mix.f.b": m.f_bias, p + "mix.lower": m.lower,
                             p + "mix.norm": m.head_norm, p + "mix.o": (m.o_proj, 0, "weight")})
            if L.mlp is not None:
                dest[p + "norm2"], dest[p + "norm2b"] = L.norm2, L.norm2b
                for name, lin, piece in (("gate", L.mlp.gate_up_proj, 0), ("up", L.mlp.gate_up_proj, 1),
                                         ("down", L.mlp.down_proj, 0)):
                    dest[p + f"mlp.{name}"] = (lin, piece, "weight")
                    dest[p + f"mlp.{name}.b"] = (lin, piece, "bias")
        return load_exact(dest, weights)
