"""Plain, slow restatement of the Saninex decoder, one function per mechanism, on PyTorch CPU tensors.

Shares no code with the package: it reads the raw ``config.json`` dictionary and the checkpoint's tensor names itself,
keeps no cache (every token attends to the tensors of the whole prefix, every recurrence and convolution is a loop over
tokens from the first) and works in whatever dtype the caller's tensors have (the tests use float64).
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """Divides the last dimension by its root mean square."""
    return x / (x.pow(2).mean(-1, keepdim=True) + eps).sqrt()


def centred_norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (1 + w)


def silu(x):
    return x * torch.sigmoid(x)


def unit(x):
    return x / (x.pow(2).sum(-1, keepdim=True) + 1e-6).sqrt()


def short_convolution(x, w):
    """x ``[T, channels]``, w ``[channels, taps]``: y_t = sum_j w[:, taps - 1 - j] x_{t - j}, nothing before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(min(taps, t + 1)):
            y[t] += w[:, taps - 1 - j] * x[t - j]
    return y


def delta_recurrence(q, k, v, beta, g):
    """q, k ``[T, H, d]``, v ``[T, H, e]``, beta and g ``[T, H]`` -> o ``[T, H, e]`` and the last state ``[H, d, e]``. The
    state decays, loses what it holds under the key and gains the value in its place, and is then read."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        held = torch.einsum("hde,hd->he", S, k[t])
        write = beta[t][:, None] * (v[t] - held)
        S = S + k[t][:, :, None] * write[:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


def gated_heads(o, w, gate, eps):
    """o ``[T, H, e]``: every head over its root mean square times w ``[e]``, then times silu of gate ``[T, H * e]``."""
    return (rms(o, eps) * w).reshape(o.shape[0], -1) * silu(gate)


def delta(h, m, t, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(short_convolution(h @ t(n).T, t(n + ".conv"))) for n in "qkv")
    of = torch.arange(H) // (H // G)
    q = (unit(q.view(T, G, d)) * d ** -0.5)[:, of]
    k = unit(k.view(T, G, d))[:, of]
    beta = torch.sigmoid(h @ t("b").T)
    step = h @ t("a").T + t("dt_bias")
    soft = torch.where(step > 0, step, torch.zeros_like(step)) + torch.log1p(torch.exp(-step.abs()))
    g = torch.exp(-torch.exp(t("A_log")) * soft)
    o, _ = delta_recurrence(q, k, v.view(T, H, e), beta, g)
    return gated_heads(o, t("norm"), h @ t("g").T, eps) @ t("o").T


def capped_attention(q, k, v, scale, cap):
    """q ``[T, H, d]``, k ``[T, G, d]``, v ``[T, G, e]``: causal softmax attention whose scores saturate at +-cap."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        kh, vh = k[:, h // (H // G)], v[:, h // (H // G)]
        for i in range(T):
            s = cap * torch.tanh((kh[:i + 1] @ q[i, h]) * scale / cap)
            out[i, h] = s.softmax(-1) @ vh[:i + 1]
    return out


def attention(h, m, t, eps):
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ t(n).T + t(n + ".b") for n in "qkv")
    q = rms(q.view(T, H, d), eps) * t("q.norm")
    k = rms(k.view(T, G, d), eps) * t("k.norm")
    o = capped_attention(q, k, v.view(T, G, e), m["scale"], m["softcap"])
    gate = torch.sigmoid(h @ t("g").T)
    return (o * gate[..., None]).reshape(T, H * e) @ t("o").T + t("o.b")


def channel_recurrence(q, k, v, alpha):
    """q, k, alpha ``[T, H, d]``, v ``[T, H, e]``: every key channel of the state has a decay of its own."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=q.dtype)
    out = []
    for t in range(T):
        S = alpha[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hde,hd->he", S, q[t]))
    return torch.stack(out), S


def gated_linear(h, m, t, eps):
    T, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ t("q").T).view(T, H, d) * d ** -0.5
    k, v = (h @ t("k").T).view(T, H, d), (h @ t("v").T).view(T, H, e)
    z = (h @ t("a1").T) @ t("a2").T + t("a2.b")
    alpha = torch.sigmoid(z).view(T, H, d) ** (1 / m["tau"])
    o, _ = channel_recurrence(q, k, v, alpha)
    return gated_heads(o, t("norm"), h @ t("g").T, eps) @ t("o").T


def parallel(h, m, t, eps):
    left = rms(attention(h, m["left"], lambda n: t("left." + n), eps), eps) * t("left.out")
    right = rms(gated_linear(h, m["right"], lambda n: t("right." + n), eps), eps) * t("right.out")
    return 0.5 * (left + right)


MIXERS = {"delta": delta, "parallel": parallel}


def clamped_glu(g, u, limit):
    g, u = torch.minimum(g, torch.full_like(g, limit)), u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def feed_forward(h, m, t):
    return clamped_glu(h @ t("gate").T, h @ t("up").T, m["limit"]) @ t("down").T


def forward(config, tensors, ids, dtype=torch.float64, layer_outputs=None):
    """Logits ``[T, vocab]`` of one sequence; ``layer_outputs``: a list that receives the residual after every layer."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(ids)]
    for i, layer in enumerate(config["layers"]):
        p = f"l{i}"
        y = MIXERS[layer["type"]](x, layer["mixer"], lambda n: w[f"{p}.mix.{n}"], eps)
        x = x + centred_norm(y, w[p + ".norm1"], eps)
        if layer["mlp"] is not None:
            y = feed_forward(x, layer["mlp"], lambda n: w[f"{p}.mlp.{n}"])
            x = x + centred_norm(y, w[p + ".norm2"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return centred_norm(x, w["final.norm"], eps) @ w["embed"].T


def random_tensors(config, seed, rank=12):
    """Random bf16 tensors under the checkpoint's names, sized so that every term matters; ``rank``: of the decay map.
    Recurrent queries resemble their keys: a first token reads (q . k) v, which is normed, so that its sign would be a matter of
    rounding where q and k happen to be orthogonal."""
    g = torch.Generator().manual_seed(seed)
    W = config["width"]

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / math.sqrt(i)).bfloat16()

    def vec(n, mean=0.0, std=0.3):
        return (mean + std * torch.randn(n, generator=g)).bfloat16()

    def alike(w):
        return (0.8 * w.float() + 0.6 * torch.randn(w.shape, generator=g) * w.float().std()).bfloat16()

    t = {"embed": torch.randn(config["vocab"], W, generator=g).bfloat16()}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}", layer["mixer"]
        t[p + ".norm1"] = vec(W, -0.4)
        if layer["type"] == "delta":
            H, G, d, e, c = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
            q = p + ".mix."
            for n, rows in (("q", G * d), ("k", G * d), ("v", H * e)):
                t[q + n], t[q + n + ".conv"] = lin(rows, W), lin(rows, c, 1.2)
            t[q + "k"], t[q + "k.conv"] = alike(t[q + "q"]), alike(t[q + "q.conv"])
            t[q + "b"], t[q + "a"], t[q + "g"], t[q + "o"] = lin(H, W), lin(H, W), lin(H * e, W), lin(W, H * e)
            t[q + "A_log"], t[q + "dt_bias"], t[q + "norm"] = vec(H, -1.0, 1.5), vec(H, -1.0, 1.0), vec(e, 1.0)
        else:
            l, q = m["left"], p + ".mix.left."
            H, G, d, e = l["heads"], l["kv_heads"], l["dim"], l["vdim"]
            for n, rows in (("q", H * d), ("k", G * d), ("v", G * e), ("o", None)):
                t[q + n] = lin(W, H * e) if n == "o" else lin(rows, W)
                t[q + n + ".b"] = vec(rows or W)
            t[q + "q.norm"], t[q + "k.norm"], t[q + "g"] = vec(d, 1.3), vec(d, 1.3), lin(H, W)
            r, q = m["right"], p + ".mix.right."
            H, d, e = r["heads"], r["dim"], r["vdim"]
            t[q + "q"], t[q + "v"] = lin(H * d, W), lin(H * e, W)
            t[q + "k"] = alike(t[q + "q"])
            t[q + "g"], t[q + "o"], t[q + "norm"] = lin(H * e, W), lin(W, H * e), vec(e, 1.0)
            t[q + "a1"], t[q + "a2"], t[q + "a2.b"] = lin(rank, W), lin(H * d, rank, 1.5), vec(H * d, 1.0, 1.5)
            t[p + ".mix.left.out"], t[p + ".mix.right.out"] = vec(W, 1.0), vec(W, 1.0)
        if layer["mlp"] is not None:
            t[p + ".norm2"] = vec(W, -0.4)
            ff = layer["mlp"]["ff"]
            t[p + ".mlp.gate"], t[p + ".mlp.up"], t[p + ".mlp.down"] = lin(ff, W), lin(ff, W), lin(W, ff)
    t["final.norm"] = vec(W)
    return t
