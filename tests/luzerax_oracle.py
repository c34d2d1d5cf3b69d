"""Plain restatement of the Luzerax design for the tests: one function per mechanism, written token by token from the
equations and sharing nothing with the package under test.

Tensors are ``[tokens, ...]`` of one sequence; everything is computed in the dtype of the weights handed in (float32 or
float64).  Weights are a plain ``name -> tensor`` mapping with the checkpoint's tensor names.
"""
from __future__ import annotations

import json
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------ attention
def causal_attention(q, k, v, scale):
    """One head: ``q [Tq, d]`` are the last Tq of the positions of ``k [Tk, d]``, ``v [Tk, dv]``."""
    n_q, n_k = q.shape[0], k.shape[0]
    future = torch.arange(n_k)[None, :] > torch.arange(n_k - n_q, n_k)[:, None]
    return torch.softmax(((q @ k.t()) * scale).masked_fill(future, -math.inf), dim=-1) @ v


def temperature(positions, coef, every):
    """What queries are multiplied by: 1 + coef ln(1 + the number of whole spans of ``every`` tokens up to and with p)."""
    return 1.0 + coef * torch.log(torch.floor((positions.double() + 1) / every) + 1.0)


def lam(lq1, lk1, lq2, lk2, diff):
    return torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff


def subtract_maps(a1, a2, lam_, diff, eps):
    """``a1, a2 [T, H, dv]``."""
    return rms(a1 - lam_ * a2, eps) * (1.0 - diff)


def differential_queries_keys(h, w, p, m, eps, positions):
    """``[T, heads, 2, dim]``: two maps per head."""
    q = rms_norm((h @ w[p + "q"].t()).view(-1, m["heads"], 2, m["dim"]), w[p + "q.norm"], eps)
    k = rms_norm((h @ w[p + "k"].t()).view(-1, m["kv_heads"], 2, m["dim"]), w[p + "k.norm"], eps)
    if m.get("q_temp"):
        q = q * temperature(positions, m["q_temp"]["coef"], m["q_temp"]["every"]).to(q.dtype)[:, None, None, None]
    return q, k


def differential_attention(h, w, p, m, eps):
    T, H, G, dv = h.shape[0], m["heads"], m["kv_heads"], m["vdim"]
    q, k = differential_queries_keys(h, w, p, m, eps, torch.arange(T))
    v = (h @ w[p + "v"].t()).view(T, G, dv)
    a = [torch.stack([causal_attention(q[:, j, i], k[:, j // (H // G), i], v[:, j // (H // G)], m["scale"])
                      for j in range(H)], 1) for i in range(2)]
    one = lam(w[p + "lq1"], w[p + "lk1"], w[p + "lq2"], w[p + "lk2"], m["diff"])
    return subtract_maps(a[0], a[1], one, m["diff"], eps).reshape(T, -1) @ w[p + "o"].t()


def rotate_neighbours(x, positions, dims, base):
    """``x [T, H, d]``: channels 2 i and 2 i + 1 turn together (i < dims / 2), channels from ``dims`` on pass."""
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.double() * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def rotated_queries_keys(h, w, p, m, eps, positions):
    def heads(name, n):
        x = (h @ w[p + name].t()).view(-1, n, m["dim"])
        return rms(rotate_neighbours(x, positions, m["rot"]["dims"], m["rot"]["base"]), eps)
    return heads("q", m["heads"]), heads("k", m["kv_heads"])


def gated_attention(h, w, p, m, eps):
    T, H, G, dv = h.shape[0], m["heads"], m["kv_heads"], m["vdim"]
    q, k = rotated_queries_keys(h, w, p, m, eps, torch.arange(T))
    v = (h @ w[p + "v"].t()).view(T, G, dv)
    gate = torch.sigmoid(h @ w[p + "g"].t())
    o = torch.stack([causal_attention(q[:, j], k[:, j // (H // G)], v[:, j // (H // G)], m["scale"]) * gate[:, j:j + 1]
                     for j in range(H)], 1)
    return o.reshape(T, -1) @ w[p + "o"].t()


# ------------------------------------------------------------------ feed-forward
def dense(h, w, p):
    return (silu(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def clipped_expert(h, w, p, limit):
    g = torch.clamp(h @ w[p + "gate"].t(), max=limit)
    u = torch.clamp(h @ w[p + "up"].t(), min=-limit, max=limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)) @ w[p + "down"].t()


def choose(z, correction, groups, keep, top):
    """``z [n]``: router logits of one token -> {output: weight}, and how far the closest call was from going the other
    way."""
    s = torch.softmax(z, -1)
    choice = s + correction
    n = z.shape[0] // groups
    score = [max(choice[g * n:(g + 1) * n].tolist()) for g in range(groups)]
    order = sorted(range(groups), key=lambda g: -score[g])
    allowed = [e for g in order[:keep] for e in range(g * n, (g + 1) * n)]
    rank = sorted(allowed, key=lambda e: -float(choice[e]))
    margin = score[order[keep - 1]] - score[order[keep]] if keep < groups else math.inf
    if top < len(rank):
        margin = min(margin, float(choice[rank[top - 1]] - choice[rank[top]]))
    total = sum(s[e] for e in rank[:top]) + 1e-20
    return {e: s[e] / total for e in rank[:top]}, margin


def experts(h, w, p, mlp, margins=None):
    """Outputs from ``experts`` on are the input itself; a shared expert runs for every token."""
    r, out = mlp["router"], torch.zeros_like(h)
    gr = r.get("groups") or {"count": 1, "keep": 1}
    for t in range(h.shape[0]):
        chosen, margin = choose(w[p + "router"] @ h[t], w[p + "correction"], gr["count"], gr["keep"], r["top"])
        if margins is not None:
            margins[t] = min(margins[t], margin)
        for e, a in chosen.items():
            out[t] += a * (h[t] if e >= r["experts"] else clipped_expert(h[t], w, f"{p}e{e}.", mlp["expert"]["limit"]))
    if mlp.get("shared"):
        out = out + clipped_expert(h, w, p + "shared.", mlp["shared"]["limit"])
    return out


# ------------------------------------------------------------------ the model
def sublayer(x, y, norm, scale, eps):
    return x + rms_norm(y, norm, eps) * scale


def forward(cfg, w, tokens, collect=None, margins=None):
    """Logits of every position of one sequence, computed from scratch.  ``margins`` (a list with inf per token) receives
    each token's closest call of a router."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        mix = {"attention": differential_attention, "attention_2": gated_attention}[layer["type"]]
        x = sublayer(x, mix(x, w, p + "mix.", m, eps), w[p + "norm1"], w[p + "ls1"], eps)
        if mlp:
            y = dense(x, w, p + "mlp.") if mlp["kind"] == "dense" else experts(x, w, p + "mlp.", mlp, margins)
            x = sublayer(x, y, w[p + "norm2"], w[p + "ls2"], eps)
        if collect is not None:
            collect.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["head"].t()
