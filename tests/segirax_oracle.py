"""Plain, slow restatement of the Segirax decoder, one function per mechanism, on PyTorch CPU tensors.

Shares no code with the package: it reads the raw ``config.json`` dictionary and the checkpoint's tensor names itself,
keeps no cache (every token attends to the tensors of the whole prefix, every recurrence is a loop over tokens) and works
in whatever dtype the caller's tensors have (the tests use float64).
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """Divides the last dimension by its root mean square."""
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()


def dynamic_tanh(x, alpha, w, b):
    return torch.tanh(alpha * x) * w + b


def residual_gate(h, w, b):
    return torch.sigmoid(h @ w.T + b)


def poly_norm(z, coef, eps):
    a, b, c, e = coef
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def rotate_half(x, positions, dims, base):
    """x ``[T, ..., n]``: the first ``dims`` of the last dimension are rotated, pair (i, i + dims / 2)."""
    half = dims // 2
    freq = torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * freq
    ang = ang.reshape([x.shape[0]] + [1] * (x.dim() - 2) + [half])
    cos, sin = ang.cos().to(x.dtype), ang.sin().to(x.dtype)
    u, v, rest = x[..., :half], x[..., half:dims], x[..., dims:]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, rest], -1)


def latent_attention(h, m, t, eps):
    """h ``[T, width]`` of one sequence from position 0; ``m``: the layer's mixer sizes; ``t(name)``: its tensors."""
    T, H = h.shape[0], m["heads"]
    d, r, vd, R = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ t("q").T).view(T, H, d + r)
    q_plain, q_rot = q[..., :d], rotate_half(q[..., d:], pos, m["rot"]["dims"], m["rot"]["base"])
    down = h @ t("dkv").T
    c = rms(down[:, :R], eps) * t("dkv.norm")
    k_rot = rotate_half(down[:, R:], pos, m["rot"]["dims"], m["rot"]["base"])
    k_plain = (c @ t("uk").T).view(T, H, d)
    v = (c @ t("uv").T).view(T, H, vd)
    gate = torch.sigmoid(h @ t("g").T)
    out = torch.zeros(T, H, vd, dtype=h.dtype)
    for i in range(T):
        s = (torch.einsum("hd,jhd->hj", q_plain[i], k_plain[:i + 1]) + torch.einsum("hd,jd->hj", q_rot[i], k_rot[:i + 1])) * m["scale"]
        out[i] = torch.einsum("hj,jhd->hd", s.softmax(-1), v[:i + 1])
    return (out * gate[..., None]).reshape(T, H * vd) @ t("o").T


def silu(x):
    return x * torch.sigmoid(x)


def decayed_recurrence(q, k, v, decay):
    """q, k ``[T, H, d]``, v ``[T, H, e]``, decay ``[H]`` -> o ``[T, H, e]`` and the last state ``[H, d, e]``."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    dec = torch.as_tensor(decay, dtype=q.dtype)
    out = []
    for i in range(T):
        S = dec[:, None, None] * S + k[i, :, :, None] * v[i, :, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[i]))
    return torch.stack(out), S


def lightning(h, m, t, eps):
    T, H = h.shape[0], m["heads"]
    q = silu(h @ t("q").T).view(T, H, m["dim"])
    k = silu(h @ t("k").T).view(T, H, m["dim"])
    v = silu(h @ t("v").T).view(T, H, m["vdim"])
    o, _ = decayed_recurrence(q, k, v, m["decay"])
    y = rms(o.reshape(T, -1), eps) * t("norm") * torch.sigmoid(h @ t("g").T)
    return y @ t("o").T


MIXERS = {"latent_attention": latent_attention, "lightning": lightning}


def forward(config, tensors, ids, dtype=torch.float64, layer_outputs=None):
    """Logits ``[T, vocab]`` of one sequence; ``layer_outputs``: a list that receives the residual after every layer."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]

    def norm(x, name):
        return dynamic_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])

    x = w["embed"][torch.as_tensor(ids)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        h = norm(x, p + ".norm1")
        y = MIXERS[layer["type"]](h, layer["mixer"], lambda n: w[f"{p}.mix.{n}"], eps)
        x = x + y * residual_gate(h, w[p + ".rg1"], w[p + ".rg1.b"])
        if layer["mlp"] is not None:
            h = norm(x, p + ".norm2")
            y = poly_norm(h @ w[p + ".mlp.up"].T, w[p + ".mlp.act"], eps) @ w[p + ".mlp.down"].T
            x = x + y * residual_gate(h, w[p + ".rg2"], w[p + ".rg2.b"])
        if layer_outputs is not None:
            layer_outputs.append(x)
    return norm(x, "final.norm") @ w["embed"].T * config["logit_scale"]


def random_tensors(config, seed, scale=None):
    """Random bf16 tensors under the checkpoint's names, sized so that every term matters."""
    g = torch.Generator().manual_seed(seed)
    W = config["width"]

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / math.sqrt(i)).bfloat16()

    def vec(n, mean=0.0, std=0.3):
        return (mean + std * torch.randn(n, generator=g)).bfloat16()

    t = {"embed": torch.randn(config["vocab"], W, generator=g).bfloat16()}

    def norm(name):
        t[name], t[name + ".b"] = vec(W, 1.0), vec(W, 0.0, 0.1)
        t[name + ".alpha"] = torch.tensor(0.5 + 0.5 * torch.rand(1, generator=g).item()).bfloat16()

    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}", layer["mixer"]
        norm(p + ".norm1")
        H = m["heads"]
        if layer["type"] == "latent_attention":
            d, r, vd, R = m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            t[p + ".mix.q"], t[p + ".mix.dkv"] = lin(H * (d + r), W, 1.5), lin(R + r, W, 1.5)
            t[p + ".mix.dkv.norm"] = vec(R, 1.0)
            t[p + ".mix.uk"], t[p + ".mix.uv"] = lin(H * d, R), lin(H * vd, R)
            t[p + ".mix.g"], t[p + ".mix.o"] = lin(H, W), lin(W, H * vd, 2.0)
        else:
            d, vd = m["dim"], m["vdim"]
            t[p + ".mix.q"], t[p + ".mix.k"], t[p + ".mix.v"] = lin(H * d, W), lin(H * d, W), lin(H * vd, W)
            t[p + ".mix.g"], t[p + ".mix.o"] = lin(H * vd, W), lin(W, H * vd, 2.0)
            t[p + ".mix.norm"] = vec(H * vd, 1.0)
        t[p + ".rg1"], t[p + ".rg1.b"] = lin(W, W), vec(W)
        if layer["mlp"] is not None:
            norm(p + ".norm2")
            ff = layer["mlp"]["ff"]
            t[p + ".mlp.up"], t[p + ".mlp.down"] = lin(ff, W), lin(W, ff)
            t[p + ".mlp.act"] = torch.tensor([0.6, 0.5, 0.3, 0.1]).bfloat16()
            t[p + ".rg2"], t[p + ".rg2.b"] = lin(W, W), vec(W)
    norm("final.norm")
    return t
