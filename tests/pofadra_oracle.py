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
    """``z [E]``: router logits of one token -> {expert: weight}."""
    s = torch.sigmoid(z)
    choice = s + correction
    n = z.shape[0] // groups
    score = [sum(sorted(choice[g * n:(g + 1) * n].tolist(), reverse=True)[:2]) for g in range(groups)]
    best = sorted(range(groups), key=lambda g: -score[g])[:keep]
    allowed = [e for g in best for e in range(g * n, (g + 1) * n)]
    chosen = sorted(allowed, key=lambda e: -float(choice[e]))[:top]
    return {e: s[e] * scale for e in chosen}


def experts(h, w, p, r):
    out = torch.zeros_like(h)
    gr = r["groups"]
    for t in range(h.shape[0]):
        z = w[p + "router"] @ h[t]
        for e, a in choose(z, w[p + "correction"], gr["count"], gr["keep"], r["top"], r["scale"]).items():
            x = f"{p}e{e}."
            out[t] += a * (w[x + "down"] @ (silu(w[x + "gate"] @ h[t]) * (w[x + "up"] @ h[t])))
    return out


# ------------------------------------------------------------------ the model
def forward(cfg, w, tokens, collect=None):
    """Logits of every position of one sequence, computed from scratch."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rms_norm(x, w[p + "norm1"], eps)
        y = {"attention": attention, "channel_delta": channel_delta}[layer["type"]](h, w, p + "mix.", m, eps)
        if layer.get("mlp"):
            y = y + experts(h, w, p + "mlp.", layer["mlp"]["router"])
        x = x + y
        if collect is not None:
            collect.append(x)
    return soft_cap(rms_norm(x, w["final.norm"], eps) @ w["head"].t(), cfg["logit_softcap"])
