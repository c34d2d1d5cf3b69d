"""Plain restatement of the Pofadra design for the tests: one function per mechanism, written token by token from the
equations and sharing nothing with the package under test.

Tensors are ``[tokens, ...]`` of one sequence; everything is computed in the dtype of the weights handed in (float32 or
float64).  Weights are a plain ``name -> tensor`` mapping with the checkpoint's tensor names.
"""
from __future__ import annotations

import json
import math

import torch


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


# ------------------------------------------------------------------ attention
def rotate_half(x, positions, dims, base):
    """``x [T, H, d]``: channels i and i + dims / 2 turn together (i < dims / 2), channels from ``dims`` on pass."""
    out = x.clone()
    half = dims // 2
    for i in range(half):
        angle = positions.double() * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def visible(n_q, n_k, window):
    """Queries are the last ``n_q`` of ``n_k`` positions; True where the key is seen."""
    d = torch.arange(n_k - n_q, n_k)[:, None] - torch.arange(n_k)[None, :]
    return (d >= 0) & (d < window) if window else d >= 0


def softmax_plus_one(s, keep):
    """exp(s_j) / (1 + sum exp(s_j)) over the kept places."""
    s = s.masked_fill(~keep, -math.inf)
    m = s.max(-1, keepdim=True).values.clamp(min=0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(-1, keepdim=True))


def attend(q, k, v, scale, window):
    """``q [Tq, H, d]``, ``k, v [Tk, G, d]``; query head h reads key / value head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    keep = visible(q.shape[0], k.shape[0], window)
    out = torch.empty(q.shape[0], H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        out[:, h] = softmax_plus_one((q[:, h] @ k[:, g].t()) * scale, keep) @ v[:, g]
    return out


def queries_keys_values(h, w, p, m, eps, positions):
    """Norms run over the whole projection; the value is the key before norm and rotation."""
    T, H, G, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q, k = h @ w[p + "q"].t(), h @ w[p + "k"].t()
    v = k.view(T, G, dim)
    rot = m["rot"]
    q = rotate_half(rms_norm(q, w[p + "q.norm"], eps).view(T, H, dim), positions, rot["dims"], rot["base"])
    k = rotate_half(rms_norm(k, w[p + "k.norm"], eps).view(T, G, dim), positions, rot["dims"], rot["base"])
    return q, k, v


def attention(h, w, p, m, eps):
    T = h.shape[0]
    q, k, v = queries_keys_values(h, w, p, m, eps, torch.arange(T))
    o = attend(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, -1)
    return (o * torch.sigmoid(h @ w[p + "g"].t())) @ w[p + "o"].t()


# ------------------------------------------------------------------ delta rule with a decay per key channel
def short_conv(x, taps):
    """``x [T, C]``, ``taps [C, n]``: last column multiplies the current token, zeros stand before the first."""
    n = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            if t - (n - 1 - j) >= 0:
                y[t] += taps[:, j] * x[t - (n - 1 - j)]
    return y


def delta_rule(q, k, v, g, beta, S):
    """``q, k [T, G, d]``, ``v [T, H, dv]``, ``g [T, H, d]`` (decay factors), ``beta [T, H]``, ``S [H, d, dv]``."""
    T, H, G = v.shape[0], v.shape[1], k.shape[1]
    S, out = S.clone(), torch.empty_like(v)
    for t in range(T):
        for h in range(H):
            kh, qh = k[t, h // (H // G)], q[t, h // (H // G)]
            Sh = g[t, h][:, None] * S[h]
            u = beta[t, h] * (v[t, h] - Sh.t() @ kh)
            S[h] = Sh + torch.outer(kh, u)
            out[t, h] = S[h].t() @ qh
    return out, S


def decay(z, A_log, dt_bias, heads):
    """``z [T, H * d]`` -> factors ``[T, H, d]``."""
    return torch.exp(-torch.exp(A_log)[:, None] * softplus(z + dt_bias).view(z.shape[0], heads, -1))


def delta_operands(h, w, p, m):
    T, H, G, dim, vdim = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_conv(h @ w[p + n].t(), w[p + n + ".conv"])) for n in "qkv")
    q, k = unit(q.view(T, G, dim)) * dim ** -0.5, unit(k.view(T, G, dim))
    beta = torch.sigmoid(h @ w[p + "b"].t())
    g = decay((h @ w[p + "a1"].t()) @ w[p + "a2"].t(), w[p + "A_log"], w[p + "dt_bias"], H)
    return q, k, v.view(T, H, vdim), g, beta


def channel_delta(h, w, p, m, eps):
    T, H = h.shape[0], m["heads"]
    q, k, v, g, beta = delta_operands(h, w, p, m)
    o, _ = delta_rule(q, k, v, g, beta, torch.zeros(H, m["dim"], m["vdim"], dtype=h.dtype))
    o = rms_norm(o, w[p + "norm"], eps).reshape(T, -1)
    return (o * torch.sigmoid((h @ w[p + "g1"].t()) @ w[p + "g2"].t())) @ w[p + "o"].t()


# ------------------------------------------------------------------ experts
def choose(z, correction, groups, keep, top, scale):
    """``z [E]``: router logits of one token -> {expert: weight}, and how far the closest call was from going the other
    way."""
    s = torch.sigmoid(z)
    choice = s + correction
    n = z.shape[0] // groups
    score = [sum(sorted(choice[g * n:(g + 1) * n].tolist(), reverse=True)[:2]) for g in range(groups)]
    order = sorted(range(groups), key=lambda g: -score[g])
    allowed = [e for g in order[:keep] for e in range(g * n, (g + 1) * n)]
    rank = sorted(allowed, key=lambda e: -float(choice[e]))
    margin = score[order[keep - 1]] - score[order[keep]] if keep < groups else math.inf
    if top < len(rank):
        margin = min(margin, float(choice[rank[top - 1]] - choice[rank[top]]))
    return {e: s[e] * scale for e in rank[:top]}, margin


def experts(h, w, p, r, margins=None):
    out = torch.zeros_like(h)
    gr = r["groups"]
    for t in range(h.shape[0]):
        z = w[p + "router"] @ h[t]
        chosen, margin = choose(z, w[p + "correction"], gr["count"], gr["keep"], r["top"], r["scale"])
        if margins is not None:
            margins[t] = min(margins[t], margin)
        for e, a in chosen.items():
            x = f"{p}e{e}."
            out[t] += a * (w[x + "down"] @ (silu(w[x + "gate"] @ h[t]) * (w[x + "up"] @ h[t])))
    return out


# ------------------------------------------------------------------ the model
def forward(cfg, w, tokens, collect=None, margins=None):
    """Logits of every position of one sequence, computed from scratch.  ``margins`` (a list with inf per token) receives
    each token's closest call of a router."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms_norm(x, w[p + "norm1"], eps)
        y = {"attention": attention, "channel_delta": channel_delta}[layer["type"]](h, w, p + "mix.", m, eps)
        if layer.get("mlp"):
            y = y + experts(h, w, p + "mlp.", layer["mlp"]["router"], margins)
        x = x + y
        if collect is not None:
            collect.append(x)
    return soft_cap(rms_norm(x, w["final.norm"], eps) @ w["head"].t(), cfg["logit_softcap"])


# ------------------------------------------------------------------ small random models
def attn(heads, kv_heads, dim, window, dims=None, base=10000.0, scale=None, moe=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": window},
         "rot": {"base": base, "dims": dim if dims is None else dims}, "scale": dim ** -0.5 if scale is None else scale}
    return {"type": "attention", "mixer": m, "mlp": moe}


def delta(heads, kv_heads, dim, vdim, conv, moe=None, ranks=(5, 11)):
    """``ranks``: of the decay's and the gate's low-rank factors (sizes that only the tensors know)."""
    return {"type": "channel_delta", "mlp": moe, "ranks": ranks,
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def moe(experts, top, ff, count=1, keep=1, scale=1.0):
    return {"kind": "moe", "expert": {"ff": ff},
            "router": {"experts": experts, "top": top, "scale": scale, "groups": {"count": count, "keep": keep}}}


def config(width, vocab, layers, eps=1e-6, embed=1.0, cap=20.0):
    return {"architecture": "Pofadra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "logit_softcap": cap, "layers": layers}


def weights(cfg, seed=0, sharp=2.0):
    """bf16-representable fp32 weights.  ``sharp`` widens attention scores so that single keys matter; decays reach from
    one token to thousands; corrections are as large as the scores they compete with, partly negative sums."""
    g = torch.Generator().manual_seed(seed)
    W, w = cfg["width"], {}

    def put(name, *shape, std=1.0, base=0.0):
        w[name] = (base + std * torch.randn(*shape, generator=g)).bfloat16().float()

    def lin(name, out_f, in_f, gain=1.0):
        put(name, out_f, in_f, std=gain * in_f ** -0.5)

    put("embed", cfg["vocab"], W, std=1.0 / cfg["embedding"]["scale"])
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        put(p + "norm1", W, std=0.2, base=1.0)
        if l["type"] == "attention":
            lin(p + "mix.q", H * d, W)
            lin(p + "mix.k", G * d, W)
            put(p + "mix.q.norm", H * d, std=0.4, base=sharp)
            put(p + "mix.k.norm", G * d, std=0.3, base=1.0)
            lin(p + "mix.g", H * d, W, 2.0)
        else:
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * dv)):
                lin(p + "mix." + n, rows, W, 2.0)
                put(p + "mix." + n + ".conv", rows, m["conv"], std=0.7)
            lin(p + "mix.b", H, W, 2.0)
            put(p + "mix.A_log", H, std=1.0, base=-1.0)
            put(p + "mix.norm", dv, std=0.2, base=1.0)
            ra, rg = l["ranks"]
            lin(p + "mix.a1", ra, W)
            lin(p + "mix.a2", H * d, ra)
            put(p + "mix.dt_bias", H * d, std=2.5, base=-3.0)
            lin(p + "mix.g1", rg, W)
            lin(p + "mix.g2", H * dv, rg, 2.0)
        lin(p + "mix.o", W, H * dv)
        if l["mlp"]:
            ff, E = l["mlp"]["expert"]["ff"], l["mlp"]["router"]["experts"]
            for e in range(E):
                for n, o, k in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
                    lin(f"{p}mlp.e{e}.{n}", o, k)
            lin(p + "mlp.router", E, W, 2.0)
            put(p + "mlp.correction", E, std=0.6, base=-0.4)
    put("final.norm", W, std=0.2, base=1.0)
    lin("head", cfg["vocab"], W, 3.0)
    return w


def save(folder, cfg, w):
    from safetensors.torch import save_file
    folder.mkdir(parents=True, exist_ok=True)
    plain = json.loads(json.dumps(cfg))
    for l in plain["layers"]:
        l.pop("ranks", None)
    (folder / "config.json").write_text(json.dumps(plain))
    save_file({k: v.bfloat16().contiguous() for k, v in w.items()}, str(folder / "model.safetensors"))
    return str(folder)


def greedy(cfg, w, prompt, n):
    """Greedy continuation from scratch, and the smallest margin between the best two logits on the way."""
    ids, margin = list(prompt), math.inf
    for _ in range(n):
        top = torch.topk(forward(cfg, w, ids)[-1], 2)
        margin = min(margin, float(top.values[0] - top.values[1]))
        ids.append(int(top.indices[0]))
    return ids[len(prompt):], margin


def errors(got, want):
    """Per position: root mean square over the vocabulary of the difference (mean taken off), relative to the spread of
    the logits."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    s = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / s.pow(2).mean().sqrt()


def fits(got, want, dtype, margins=None):
    """32-bit runs agree everywhere; 16-bit ones up to rounding.  Positions where a router all but tied may go either way
    in 16 bits and are left out (a position that such a token feeds moves a little)."""
    e = errors(got, want)
    if dtype == "float32":
        return float(e.max()) < 2e-4
    if margins is not None:
        e = e[torch.tensor([m > 0.02 for m in margins])]
    return e.numel() == 0 or (float(torch.quantile(e, 0.9)) < 0.08 and float(e.max()) < 0.5)
