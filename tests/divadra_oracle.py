"""Plain restatement of the Divadra design for the tests: one function per mechanism, written token by token from the
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


def silu(z):
    return z * torch.sigmoid(z)


def softplus(z):
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


# ------------------------------------------------------------------ embedding, input convolution
def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    return [buckets if t == 0 else (tokens[t - 1] * mul_prev + tokens[t] * mul_cur) % buckets for t in range(len(tokens))]


def embed(cfg, w, tokens):
    b = cfg["embedding"]["bigram"]
    x = w["embed"][torch.as_tensor(tokens)] + w["bigram"][torch.as_tensor(bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return rms(x, cfg["norm"]["eps"]) * w["embed.norm"]


def causal_conv(x, taps):
    """``x [T, C]``, ``taps [C, n]``: last column multiplies the current token, zeros stand before the first."""
    n = taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(n):
            if t - (n - 1 - j) >= 0:
                y[t] += taps[:, j] * x[t - (n - 1 - j)]
    return y


def sublayer_input(x, norm, taps, eps):
    h = rms(x, eps) * norm
    return h + causal_conv(h, taps)


# ------------------------------------------------------------------ state-space mixer
def ssd(x, B, C, dt, rate, D, S):
    """``x [T, H, dv]``, ``B, C [T, G, N]``, ``dt [T, H]``, ``rate, D [H]``, ``S [H, N, dv]`` -> outputs and the state."""
    H, G = x.shape[1], B.shape[1]
    S, y = S.clone(), torch.empty_like(x)
    for t in range(x.shape[0]):
        for h in range(H):
            g = h // (H // G)
            S[h] = torch.exp(-rate[h] * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = S[h].t() @ C[t, g] + D[h] * x[t, h]
    return y, S


def part_norm(x, parts, eps):
    """Each of ``parts`` equal consecutive parts by its own root mean square."""
    return rms(x.view(x.shape[0], parts, -1), eps).reshape(x.shape)


def mamba2(h, w, p, m, eps):
    T, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    z, xbc, dt = torch.split(h @ w[p + "in"].t(), [inner, inner + 2 * G * N, H], dim=-1)
    x, B, C = torch.split(silu(causal_conv(xbc, w[p + "conv"]) + w[p + "conv.b"]), [inner, G * N, G * N], dim=-1)
    y, _ = ssd(x.reshape(T, H, dv), B.reshape(T, G, N), C.reshape(T, G, N), softplus(dt + w[p + "dt_bias"]),
               torch.exp(w[p + "A_log"]), w[p + "D"], torch.zeros(H, N, dv, dtype=h.dtype))
    y = y.reshape(T, inner) * silu(z)
    return (part_norm(y, m["norm_groups"], eps) * w[p + "norm"]) @ w[p + "o"].t()


# ------------------------------------------------------------------ sigmoid attention in chunks
def rotate_half(x, positions, dims, base, sign=1.0):
    """``x [T, H, d]``: channels i and i + dims / 2 turn together (i < dims / 2), channels from ``dims`` on pass."""
    out = x.clone()
    half = dims // 2
    for i in range(half):
        angle = positions.double() * float(base) ** (-2.0 * i / dims) * sign
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def same_chunk(n_q, n_k, size):
    """Queries are the last ``n_q`` of ``n_k`` positions; True where the key is seen."""
    i, j = torch.arange(n_k - n_q, n_k)[:, None], torch.arange(n_k)[None, :]
    return (j <= i) & (i // size == j // size)


def attend(q, k, v, scale, bias, size):
    """``q [Tq, H, d]``, ``k [Tk, G, d]``, ``v [Tk, G, dv]``; query head h reads key / value head h // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    keep = same_chunk(q.shape[0], k.shape[0], size)
    out = torch.empty(q.shape[0], H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        a = torch.sigmoid((q[:, h] @ k[:, g].t()) * scale + bias[h])
        out[:, h] = torch.where(keep, a, torch.zeros_like(a)) @ v[:, g]
    return out


def left(h, w, p, m, eps):
    T, H, G, dim, dv, rot = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["rot"]
    pos = torch.arange(T)
    q = (rms(h @ w[p + "q"].t(), eps) * w[p + "q.norm"]).view(T, H, dim)
    k = (rms(h @ w[p + "k"].t(), eps) * w[p + "k.norm"]).view(T, G, dim)
    q, k = rotate_half(q, pos, rot["dims"], rot["base"]), rotate_half(k, pos, rot["dims"], rot["base"])
    v = rotate_half((h @ w[p + "v"].t()).view(T, G, dv), pos, dv, rot["base"])
    o = attend(q, k, v, m["scale"], w[p + "pb"], m["mask"]["size"])
    return rotate_half(o, pos, dv, rot["base"], -1.0).reshape(T, -1) @ w[p + "o"].t()


# ------------------------------------------------------------------ time mixing with a bonus for the current token
def time_mix(r, k, v, decay, u, S):
    """``r, k, v, decay [T, H, d]``, ``u [H, d]``, ``S [H, d, d]`` -> outputs and the state."""
    S, o = S.clone(), torch.empty_like(v)
    for t in range(r.shape[0]):
        for h in range(r.shape[1]):
            kv = torch.outer(k[t, h], v[t, h])
            o[t, h] = (S[h] + u[h][:, None] * kv).t() @ r[t, h]
            S[h] = decay[t, h][:, None] * S[h] + kv
    return o, S


def right(h, w, p, m, eps):
    T, H, d = h.shape[0], m["heads"], m["dim"]
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    mix = {n: h + (before - h) * w[p + "mu." + n] for n in "rkvgw"}
    r, k, v = ((mix[n] @ w[p + n].t()).view(T, H, d) for n in "rkv")
    gate = silu(mix["g"] @ w[p + "g"].t())
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w[p + "w1"].t()) @ w[p + "w2"].t() + w[p + "w0"])).view(T, H, d)
    o, _ = time_mix(r, k, v, decay, w[p + "u"], torch.zeros(H, d, d, dtype=h.dtype))
    return (rms(o, eps).reshape(T, -1) * w[p + "norm"] * gate) @ w[p + "o"].t()


def parallel(h, w, p, m, eps):
    a, b = left(h, w, p + "left.", m["left"], eps), right(h, w, p + "right.", m["right"], eps)
    return 0.5 * (rms(a, eps) * w[p + "left.out"] + rms(b, eps) * w[p + "right.out"])


# ------------------------------------------------------------------ feed-forwards
def dense(h, w, p):
    return torch.relu(h @ w[p + "up"].t()) ** 2 @ w[p + "down"].t()


def experts(h, w, p, tokens):
    out = torch.zeros_like(h)
    for t, token in enumerate(tokens):
        chosen = [int(e) for e in w[p + "table"][token]]
        for e in chosen:
            x = f"{p}e{e}."
            out[t] += (w[x + "down"] @ (silu(w[x + "gate"] @ h[t]) * (w[x + "up"] @ h[t]))) / len(chosen)
    return out


# ------------------------------------------------------------------ the model
def forward(cfg, w, tokens, collect=None):
    """Logits of every position of one sequence, computed from scratch."""
    eps, tokens = cfg["norm"]["eps"], [int(t) for t in tokens]
    x = embed(cfg, w, tokens)
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y = {"mamba2": mamba2, "parallel": parallel}[layer["type"]](
            sublayer_input(x, w[p + "norm1"], w[p + "canon1"], eps), w, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp"):
            h = sublayer_input(x, w[p + "norm2"], w[p + "canon2"], eps)
            y = y + (dense(h, w, p + "mlp.") if layer["mlp"]["kind"] == "dense" else experts(h, w, p + "mlp.", tokens))
        x = x + y
        if collect is not None:
            collect.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].t()


# ------------------------------------------------------------------ small random models
def mamba(heads, vdim, state, groups, norm_groups, conv, mlp=None):
    return {"type": "mamba2", "mlp": mlp, "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups,
                                                     "norm_groups": norm_groups, "conv": conv}}


def pair(attn, chunk, mix, mlp=None, dims=None, base=10000.0, scale=None, rank=5):
    """``attn``: heads, kv heads, dim, vdim; ``mix``: heads, dim.  ``rank``: of the decay's factors (a size that only the
    tensors know)."""
    H, G, dim, vdim = attn
    return {"type": "parallel", "mlp": mlp, "rank": rank, "mixer": {
        "left": {"heads": H, "kv_heads": G, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
                 "rot": {"base": base, "dims": dim if dims is None else dims}, "scale": dim ** -0.5 if scale is None else scale},
        "right": {"heads": mix[0], "dim": mix[1]}}}


def ff(n):
    return {"kind": "dense", "ff": n}


def moe(n, top, inner):
    return {"kind": "moe", "expert": {"ff": inner}, "router": {"experts": n, "top": top}}


def config(width, vocab, layers, taps=4, bigram=(53, 7, 3), eps=1e-6):
    return {"architecture": "Divadra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "canon": {"taps": taps},
            "embedding": {"bigram": dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))}, "layers": layers}


def weights(cfg, seed=0, sharp=2.0):
    """bf16-representable fp32 weights (tables int32).  ``sharp`` widens attention scores and the biases keep the weights of
    most keys small, so that single keys matter; decays reach from one token to thousands."""
    gen = torch.Generator().manual_seed(seed)
    W, w = cfg["width"], {}

    def put(name, *shape, std=1.0, base=0.0):
        w[name] = (base + std * torch.randn(*shape, generator=gen)).bfloat16().float()

    def lin(name, out_f, in_f, gain=1.0):
        put(name, out_f, in_f, std=gain * in_f ** -0.5)

    put("embed", cfg["vocab"], W)
    put("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, W, std=0.7)
    put("embed.norm", W, std=0.2, base=1.0)
    for i, l in enumerate(cfg["layers"]):
        p, m, x, mlp = f"l{i}.", l["mixer"], f"l{i}.mix.", l.get("mlp")
        for n in "12" if mlp else "1":
            put(p + "norm" + n, W, std=0.2, base=1.0)
            put(p + "canon" + n, W, cfg["canon"]["taps"], std=0.4)
        if l["type"] == "mamba2":
            H, dv, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
            C = H * dv + 2 * G * N
            lin(x + "in", H * dv + C + H, W, 1.5)
            put(x + "conv", C, m["conv"], std=0.6)
            put(x + "conv.b", C, std=0.3)
            put(x + "dt_bias", H, std=1.5, base=-1.0)
            put(x + "A_log", H, std=1.5, base=-1.0)
            put(x + "D", H, std=0.5, base=1.0)
            put(x + "norm", H * dv, std=0.2, base=1.0)
            lin(x + "o", W, H * dv)
        else:
            a, r = m["left"], m["right"]
            H, G, dim, dv = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            lin(x + "left.q", H * dim, W)
            lin(x + "left.k", G * dim, W)
            lin(x + "left.v", G * dv, W)
            put(x + "left.q.norm", H * dim, std=0.4, base=sharp)
            put(x + "left.k.norm", G * dim, std=0.3, base=1.0)
            put(x + "left.pb", H, std=0.7, base=-2.0)
            lin(x + "left.o", W, H * dv)
            n = r["heads"] * r["dim"]
            for c in "rkvgw":
                put(x + "right.mu." + c, W, std=0.3, base=0.5)
            for c in "rkvg":
                lin(x + "right." + c, n, W)
            # a first token's output is its bonus, sum(r u k), times v, and a norm follows: keep that sum away from zero
            w[x + "right.k"] = (0.8 * w[x + "right.r"] + 0.6 * w[x + "right.k"]).bfloat16().float()
            lin(x + "right.w1", l["rank"], W)
            lin(x + "right.w2", n, l["rank"])
            put(x + "right.w0", n, std=2.0, base=-2.5)
            put(x + "right.u", r["heads"], r["dim"], std=0.4, base=0.8)
            put(x + "right.norm", n, std=0.2, base=1.0)
            lin(x + "right.o", W, n)
            for c in ("left.out", "right.out"):
                put(x + c, W, std=0.2, base=1.0)
        if mlp and mlp["kind"] == "dense":
            lin(p + "mlp.up", mlp["ff"], W)
            lin(p + "mlp.down", W, mlp["ff"])
        elif mlp:
            E, top, inner = mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"]
            for e in range(E):
                for n, o, k in (("gate", inner, W), ("up", inner, W), ("down", W, inner)):
                    lin(f"{p}mlp.e{e}.{n}", o, k, 1.5)
            w[p + "mlp.table"] = torch.stack([torch.randperm(E, generator=gen)[:top] for _ in range(cfg["vocab"])]).to(torch.int32)
    put("final.norm", W, std=0.2, base=1.0)
    lin("head", cfg["vocab"], W, 3.0)
    return w


def save(folder, cfg, w):
    from safetensors.torch import save_file
    folder.mkdir(parents=True, exist_ok=True)
    plain = json.loads(json.dumps(cfg))
    for l in plain["layers"]:
        l.pop("rank", None)
    (folder / "config.json").write_text(json.dumps(plain))
    save_file({k: (v if v.dtype == torch.int32 else v.bfloat16()).contiguous() for k, v in w.items()}, str(folder / "model.safetensors"))
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


def fits(got, want, dtype):
    """32-bit runs agree everywhere; 16-bit ones up to rounding."""
    e = errors(got, want)
    if dtype == "float32":
        return float(e.max()) < 2e-4
    return float(torch.quantile(e, 0.9)) < 0.06 and float(e.max()) < 0.2
