"""Plain, slow restatement of the Dofevik decoder, one function per mechanism, on PyTorch CPU tensors.

Shares no code with the package: it reads the raw ``config.json`` dictionary and the checkpoint's tensor names itself, keeps no
cache (every token attends to the tensors of the whole prefix, every pooled block is averaged anew) and works in whatever dtype
the caller's tensors have (the tests use float64).
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """Divides the last dimension by its root mean square."""
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()


def frequencies(rot):
    """Turns per position (in radians) of every pair; a linear scaling divides all of them."""
    f = rot["base"] ** (-2 * torch.arange(rot["dims"] // 2, dtype=torch.float64) / rot["dims"])
    return f / rot["scaling"]["factor"] if rot.get("scaling") else f


def rotate(x, freq, neighbours):
    """x ``[T, heads, d]`` by its positions 0 .. T - 1. Pairs of the first 2 n dimensions, n = len(freq): (2 i, 2 i + 1) with
    ``neighbours``, (i, i + n) without."""
    n = len(freq)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freq
    c, s = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
    first, second = (slice(0, 2 * n, 2), slice(1, 2 * n, 2)) if neighbours else (slice(0, n), slice(n, 2 * n))
    y = x.clone()
    y[..., first] = x[..., first] * c - x[..., second] * s
    y[..., second] = x[..., second] * c + x[..., first] * s
    return y


def in_window(T, size):
    """``[T, T]``: query i sees token j."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < size)


def block_means(x, pool):
    """x ``[T, G, d]`` -> ``[T // pool, G, d]``."""
    n = x.shape[0] // pool
    return x[:n * pool].view(n, pool, *x.shape[1:]).mean(1)


def blocks_behind_window(T, size, pool):
    """``[T, T // pool]``: query i sees block b, whose last token lies before the window."""
    i, b = torch.arange(T)[:, None], torch.arange(T // pool)[None, :]
    return (b + 1) * pool - 1 <= i - size


def softmax_with_sink(s, seen, sink):
    """Scores ``[T, n]`` of one head -> weights; the sink (a number, or None) takes part in the sum only."""
    s = s.masked_fill(~seen, -math.inf)
    top = s.max(-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink)
    e = torch.exp(s - top)
    total = e.sum(-1, keepdim=True)
    return e / (total + torch.exp(sink - top) if sink is not None else total)


def sigmoid_weights(s, seen, bias):
    """Scores ``[T, n]`` of one head -> weights that are not normalised."""
    return torch.sigmoid(s + bias) * seen


def attention(h, m, t, eps):
    """Rotated, normed grouped-query attention over a window, with a sink per head."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = ((h @ t(n).T + t(n + ".b")).view(T, -1, w) for n, w in (("q", d), ("k", d), ("v", e)))
    if m.get("rot"):
        f = frequencies(m["rot"])
        q, k = rotate(q, f, True), rotate(k, f, True)
    q, k = rms(q, eps), rms(k, eps)
    seen = in_window(T, m["mask"]["size"])
    out = torch.zeros(T, H, e, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = softmax_with_sink(q[:, a] @ k[:, g].T * m["scale"], seen, t("sink")[a]) @ v[:, g]
    return out.reshape(T, H * e) @ t("o").T


def pooled_attention(h, m, t, eps):
    """Attention with sigmoid weights over a window and over the means of the blocks behind it; values are the projected keys."""
    T, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    size, pool = m["mask"]["size"], m["mask"].get("pool")
    q, v = ((h @ t(n).T).view(T, -1, d) for n in "qk")
    q, k = rms(q, eps) * t("q.norm"), rms(v, eps) * t("k.norm")
    seen = in_window(T, size)
    if pool:
        k, v = torch.cat([k, block_means(k, pool)]), torch.cat([v, block_means(v, pool)])
        seen = torch.cat([seen, blocks_behind_window(T, size, pool)], 1)
    out = torch.zeros(T, H, d, dtype=h.dtype)
    for a in range(H):
        g = a // (H // G)
        out[:, a] = sigmoid_weights(q[:, a] @ k[:, g].T * m["scale"], seen, t("pb")[a]) @ v[:, g]
    return out.reshape(T, H * d) @ t("o").T


def latent_attention(h, m, t, eps):
    """Attention whose queries, keys and values come from normed latents, over a window; gated element by element."""
    T, H, d, r, e, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms(h @ t("dq").T, eps) * t("dq.norm") @ t("uq").T).view(T, H, d + r)
    kv = h @ t("dkv").T
    c = rms(kv[:, :R], eps) * t("dkv.norm")
    f = frequencies(m["rot"])
    qr, kr = rotate(q[..., d:], f, False), rotate(kv[:, None, R:], f, False)[:, 0]
    k, v = (c @ t("uk").T).view(T, H, d), (c @ t("uv").T).view(T, H, e)
    seen = in_window(T, m["mask"]["size"])
    out = torch.zeros(T, H, e, dtype=h.dtype)
    for a in range(H):
        out[:, a] = softmax_with_sink((q[:, a, :d] @ k[:, a].T + qr[:, a] @ kr.T) * m["scale"], seen, None) @ v[:, a]
    return (out.reshape(T, H * e) * torch.sigmoid(h @ t("g").T)) @ t("o").T


def squared_relu(h, t):
    return (h @ t("up").T).clamp(min=0) ** 2 @ t("down").T


def routing(z, top, margins=None):
    """Logits ``[T, n]`` -> weights ``[T, n]``, zero where an expert is not chosen. ``margins``: a list that receives how far every
    token's last choice was from the first expert it left out."""
    order = z.sort(-1, descending=True)
    if margins is not None and top < z.shape[-1]:
        margins.append(order.values[:, top - 1] - order.values[:, top])
    return torch.zeros_like(z).scatter(-1, order.indices[:, :top], order.values[:, :top].softmax(-1))


def experts(h, m, t, margins=None):
    r = m["router"]
    w = routing(h @ t("router").T + t("router.b"), r["top"], margins)
    y = squared_relu(h, lambda n: t("shared." + n)) if m.get("shared") else torch.zeros_like(h)
    for x in range(r["experts"]):
        y = y + w[:, x:x + 1] * squared_relu(h, lambda n: t(f"e{x}.{n}"))
    return y


MIXERS = {"attention": attention, "attention_2": pooled_attention, "latent_attention": latent_attention}


def forward(config, tensors, ids, dtype=torch.float64, layer_outputs=None, margins=None):
    """Logits ``[T, vocab]`` of one sequence; ``layer_outputs``: a list that receives the residual after every layer; ``margins``:
    see :func:`routing`."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(ids)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        x = x + MIXERS[layer["type"]](rms(x, eps) * w[p + ".norm1"], layer["mixer"], lambda n: w[f"{p}.mix.{n}"], eps)
        if layer["mlp"] is not None:
            x = x + experts(rms(x, eps) * w[p + ".norm2"], layer["mlp"], lambda n: w[f"{p}.mlp.{n}"], margins)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["head"].T


def random_tensors(config, seed):
    """Random bf16 tensors under the checkpoint's names, sized so that every term matters."""
    g = torch.Generator().manual_seed(seed)
    W, V = config["width"], config["vocab"]

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / math.sqrt(i)).bfloat16()

    def vec(n, mean=1.0, std=0.3):
        return (mean + std * torch.randn(n, generator=g)).bfloat16()

    t = {"embed": torch.randn(V, W, generator=g).bfloat16(), "head": lin(V, W), "final.norm": vec(())}
    for i, layer in enumerate(config["layers"]):
        m, mlp, q = layer["mixer"], layer["mlp"], f"l{i}.mix."
        H, d = m["heads"], m["dim"]
        t[f"l{i}.norm1"] = vec(())
        if layer["type"] == "attention":
            for n, r in (("q", H * d), ("k", m["kv_heads"] * d), ("v", m["kv_heads"] * m["vdim"])):
                t[q + n], t[f"{q}{n}.b"] = lin(r, W, 1.2), vec(r, 0.0)
            t[q + "sink"], t[q + "o"] = vec(H, 2.0, 1.0), lin(W, H * m["vdim"])
        elif layer["type"] == "attention_2":
            t[q + "q"], t[q + "k"] = lin(H * d, W), lin(m["kv_heads"] * d, W)
            t[q + "q.norm"], t[q + "k.norm"], t[q + "pb"] = vec(d), vec(d), vec(H, -2.5, 1.0)
            t[q + "o"] = lin(W, H * d, 0.5)
        else:
            R, r, e, Q = m["kv_rank"], m["rot_dim"], m["vdim"], m["q_rank"]
            t[q + "dq"], t[q + "dq.norm"], t[q + "uq"] = lin(Q, W), vec(Q), lin(H * (d + r), Q, 1.5)
            t[q + "dkv"], t[q + "dkv.norm"] = lin(R + r, W), vec(R)
            t[q + "uk"], t[q + "uv"] = lin(H * d, R, 1.5), lin(H * e, R)
            t[q + "g"], t[q + "o"] = lin(H * e, W), lin(W, H * e, 1.5)
        if mlp:
            p, n = f"l{i}.mlp.", mlp["router"]["experts"]
            t[f"l{i}.norm2"] = vec(())
            t[p + "router"], t[p + "router.b"] = lin(n, W), vec(n, 0.0, 0.5)
            for name, ff in [(f"e{x}.", mlp["expert"]["ff"]) for x in range(n)] + ([("shared.", mlp["shared"]["ff"])] if mlp.get("shared") else []):
                t[p + name + "up"], t[p + name + "down"] = lin(ff, W), lin(W, ff)
    return t
