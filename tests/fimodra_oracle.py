"""Plain restatement of the Fimodra design for the tests: one function per mechanism, written token by token
from the equations and sharing nothing with the package under test.

Tensors are ``[tokens, ...]`` of one sequence; everything is computed in the dtype of the weights handed in
(float32 or float64).  ``Weights`` is a plain ``name -> tensor`` mapping with the checkpoint's tensor names.
"""
from __future__ import annotations

import math

import torch


def grouped_rms_norm(x, w, eps, groups):
    n = x.shape[-1] // groups
    parts = []
    for g in range(groups):
        part = x[..., g * n:(g + 1) * n]
        parts.append(part / torch.sqrt((part * part).mean(-1, keepdim=True) + eps))
    return torch.cat(parts, dim=-1) * w


def rms_norm(x, w, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w


def rotate_interleaved(x, positions, dims, base):
    """``x [..., T, d]``: the first ``dims`` channels turn in neighbouring pairs, the rest pass."""
    out = x.clone()
    for i in range(dims // 2):
        angle = positions.double() * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(angle).to(x.dtype), torch.sin(angle).to(x.dtype)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_mask(n_q, n_k, window):
    """Queries are the last ``n_q`` of ``n_k`` positions; True where the key is visible."""
    i = torch.arange(n_k - n_q, n_k)[:, None]
    j = torch.arange(n_k)[None, :]
    d = i - j
    return (d >= 0) & (d < window) if window else d >= 0


def sink_attention(q, k, v, scale, window, sink):
    """``q [Tq, H, d]``, ``k [Tk, H, d]``, ``v [Tk, H, dv]``; one extra exp(sink) per head in the denominator."""
    Tq, H, _ = q.shape
    keep = window_mask(Tq, k.shape[0], window)
    out = torch.empty(Tq, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h].t()) * scale
        s = s.masked_fill(~keep, -math.inf)
        m = torch.maximum(s.max(-1).values, sink[h])
        e = torch.exp(s - m[:, None])
        out[:, h] = (e @ v[:, h]) / (e.sum(-1) + torch.exp(sink[h] - m))[:, None]
    return out


def latent_attention(h, w, p, m, eps, window):
    """``p``: tensor-name prefix of the mixer, ``m``: the mixer's entry of the configuration."""
    T = h.shape[0]
    H, dim, rot, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].t()).view(T, H, dim + rot)
    d = h @ w[p + "dkv"].t()
    c = rms_norm(d[:, :rank], w[p + "dkv.norm"], eps)
    base = m["rot"]["base"]
    kr = rotate_interleaved(d[:, rank:], pos, rot, base)
    qr = rotate_interleaved(q[..., dim:].transpose(0, 1), pos, rot, base).transpose(0, 1)
    k = torch.cat([(c @ w[p + "uk"].t()).view(T, H, dim), kr[:, None, :].expand(T, H, rot)], dim=-1)
    v = (c @ w[p + "uv"].t()).view(T, H, vdim)
    o = sink_attention(torch.cat([q[..., :dim], qr], dim=-1), k, v, m["scale"], window, w[p + "sink"])
    return o.reshape(T, H * vdim) @ w[p + "o"].t()


def outer_product_recurrence(q, f, v, S):
    """``q, f [T, H, d]``, ``v [T, H, dv]``, ``S [H, d, dv]``: forget by f, write (1 - f) v^T, read with q."""
    T, H, _ = q.shape
    out = torch.empty(T, H, v.shape[-1], dtype=q.dtype)
    S = S.clone()
    for t in range(T):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out, S


def hgrn2(h, w, p, m, eps):
    T = h.shape[0]
    H, dim, vdim = m["heads"], m["dim"], m["vdim"]
    zq = h @ w[p + "q"].t()
    q = (zq * torch.sigmoid(zq)).view(T, H, dim)
    lower = w[p + "lower"]
    f = (lower + (1 - lower) * torch.sigmoid(h @ w[p + "f"].t() + w[p + "f.b"])).view(T, H, dim)
    v = (h @ w[p + "v"].t()).view(T, H, vdim)
    o, _ = outer_product_recurrence(q, f, v, torch.zeros(H, dim, vdim, dtype=h.dtype))
    o = rms_norm(o, w[p + "norm"], eps)
    return o.reshape(T, H * vdim) @ w[p + "o"].t()


def dense_mlp(h, w, p):
    g = torch.relu(h @ w[p + "gate"].t() + w[p + "gate.b"])
    u = h @ w[p + "up"].t() + w[p + "up.b"]
    return (g * u) @ w[p + "down"].t() + w[p + "down.b"]


def depth_average(history, weights):
    out = torch.zeros_like(history[0])
    for a, x in zip(weights, history):
        out = out + a * x
    return out


def forward(cfg, w, tokens, collect=None):
    """Logits of every position of one sequence, computed from scratch."""
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][torch.as_tensor(tokens)]
    history = [x]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = grouped_rms_norm(x, w[p + "norm1"], eps, groups)
        if layer["type"] == "latent_attention":
            y = latent_attention(h, w, p + "mix.", m, eps, m["mask"]["size"])
        elif layer["type"] == "hgrn2":
            y = hgrn2(h, w, p + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + grouped_rms_norm(y, w[p + "norm1b"], eps, groups)
        if layer.get("mlp"):
            y = dense_mlp(grouped_rms_norm(x, w[p + "norm2"], eps, groups), w, p + "mlp.")
            x = x + grouped_rms_norm(y, w[p + "norm2b"], eps, groups)
        history.append(x)
        x = depth_average(history, w[p + "dwa"])
        if collect is not None:
            collect.append(x)
    return grouped_rms_norm(x, w["final.norm"], eps, groups) @ w["head"].t()


# ------------------------------------------------------------------ small random models
def layer(kind, mlp=None, **mixer):
    if kind == "latent_attention":
        mixer = dict(mixer)
        mixer["mask"] = {"size": mixer.pop("window")}
        mixer["rot"] = {"base": mixer.pop("base", 10000.0), "dims": mixer["rot_dim"]}
        mixer.setdefault("scale", (mixer["dim"] + mixer["rot_dim"]) ** -0.5)
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": mlp} if mlp else None}


def config(width, vocab, groups, layers, eps=1e-6):
    return {"architecture": "Fimodra", "width": width, "vocab": vocab, "norm": {"eps": eps, "groups": groups}, "layers": layers}


def weights(cfg, seed=0, sharp=2.0):
    """bf16-representable fp32 weights.  ``sharp`` widens the attention scores so that single keys matter."""
    g = torch.Generator().manual_seed(seed)
    W, w = cfg["width"], {}

    def put(name, *shape, std=1.0, base=0.0):
        w[name] = (base + std * torch.randn(*shape, generator=g)).bfloat16().float()

    def lin(name, out_f, in_f, gain=1.0):
        put(name, out_f, in_f, std=gain * in_f ** -0.5)

    put("embed", cfg["vocab"], W)
    for i, l in enumerate(cfg["layers"]):
        p, m = f"l{i}.", l["mixer"]
        H = m["heads"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if l["mlp"] else ()):
            put(p + n, W, std=0.2, base=1.0)
        if l["type"] == "latent_attention":
            lin(p + "mix.q", H * (m["dim"] + m["rot_dim"]), W, sharp)
            lin(p + "mix.dkv", m["kv_rank"] + m["rot_dim"], W)
            put(p + "mix.dkv.norm", m["kv_rank"], std=0.2, base=1.0)
            lin(p + "mix.uk", H * m["dim"], m["kv_rank"])
            lin(p + "mix.uv", H * m["vdim"], m["kv_rank"])
            put(p + "mix.sink", H, std=1.0, base=1.0)
            lin(p + "mix.o", W, H * m["vdim"])
        else:
            lin(p + "mix.q", H * m["dim"], W)
            lin(p + "mix.f", H * m["dim"], W)
            put(p + "mix.f.b", H * m["dim"], std=3.0, base=2.0)
            w[p + "mix.lower"] = (torch.rand(H * m["dim"], generator=g) * 0.9 * (torch.rand(H * m["dim"], generator=g) > 0.3)).bfloat16().float()
            lin(p + "mix.v", H * m["vdim"], W)
            put(p + "mix.norm", m["vdim"], std=0.2, base=1.0)
            lin(p + "mix.o", W, H * m["vdim"])
        if l["mlp"]:
            ff = l["mlp"]["ff"]
            for n, o, k in (("gate", ff, W), ("up", ff, W), ("down", W, ff)):
                lin(p + "mlp." + n, o, k)
                put(p + "mlp." + n + ".b", o, std=0.3)
        put(p + "dwa", i + 2, std=0.5)
        w[p + "dwa"][-1] += 1.0
        w[p + "dwa"] = w[p + "dwa"].bfloat16().float()
    put("final.norm", W, std=0.2, base=1.0)
    lin("head", cfg["vocab"], W)
    return w


def save(folder, cfg, w):
    import json

    from safetensors.torch import save_file
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
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


def fits(got, want, dtype):
    """32-bit runs agree everywhere; 16-bit ones up to rounding, which a norm over a few small channels can enlarge at
    a position here and there."""
    e = errors(got, want)
    if dtype == "float32":
        return float(e.max()) < 2e-4
    return float(torch.quantile(e, 0.95)) < 0.08 and float(e.max()) < 0.4
