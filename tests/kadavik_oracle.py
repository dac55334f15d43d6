"""Plain, slow restatement of the Kadavik decoder, one function per mechanism, on PyTorch CPU tensors.

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


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z):
    return z * torch.sigmoid(z)


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def log_sigmoid(z):
    return -(torch.log1p(torch.exp(-z.abs())) + (-z).clamp(min=0))


def short_convolution(x, w):
    """x ``[T, channels]``, w ``[channels, taps]``: y_t = sum_j w[:, taps - 1 - j] x_{t - j}, nothing before the start."""
    T, taps = x.shape[0], w.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(min(taps, t + 1)):
            y[t] += w[:, taps - 1 - j] * x[t - j]
    return y


def rotary_frequencies(dims, base, scaling=None):
    """Turns per position of every pair; ``scaling`` stretches the long wavelengths and blends into the short ones."""
    out = []
    for i in range(dims // 2):
        f = base ** (-2 * i / dims)
        if scaling:
            wave = 2 * math.pi / f
            if wave > scaling["original"] / scaling["low"]:
                f = f / scaling["factor"]
            elif wave >= scaling["original"] / scaling["high"]:
                s = (scaling["original"] / wave - scaling["low"]) / (scaling["high"] - scaling["low"])
                f = (1 - s) * f / scaling["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate(x, freq):
    """x ``[T, heads, d]`` by its positions 0 .. T - 1: pairs (i, i + n) of the first 2 n dimensions, n = len(freq)."""
    n = len(freq)
    a = torch.arange(x.shape[0], dtype=torch.float64)[:, None] * freq
    c, s = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
    u, v = x[..., :n], x[..., n:2 * n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * n:]], -1)


def windowed_attention(q, k, v, scale, size, keep_first):
    """q ``[T, H, d]``, k ``[T, G, d]``, v ``[T, G, e]``: causal softmax over the last ``size`` tokens and the first
    ``keep_first`` ones."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = (j <= i) & ((i - j < size) | (j < keep_first))
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        s = (q[:, h] @ k[:, h // (H // G)].T) * scale
        out[:, h] = s.masked_fill(~seen, -math.inf).softmax(-1) @ v[:, h // (H // G)]
    return out


def attention(h, m, t, eps, shared):
    """``shared``: (keys, values) of the layer that has the projections, None for a layer with its own. Returns the output
    and the keys and values."""
    T, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def projected(n, heads, width):
        u = h @ t(n).T
        return (short_convolution(u, t(n + ".conv")) if m.get("conv") else u).view(T, heads, width)

    freq = rotary_frequencies(m["rot"]["dims"], m["rot"]["base"], m["rot"].get("scaling"))
    q = rotate(projected("q", H, d), freq)
    k, v = shared or (rotate(projected("k", G, d), freq), projected("v", G, e))
    mask = m.get("mask") or {"size": T + 1, "keep_first": 0}
    o = windowed_attention(q, k, v, m["scale"], mask["size"], mask.get("keep_first", 0)).reshape(T, H * e)
    return (o * torch.sigmoid(h @ t("g").T)) @ t("o").T, (k, v)


def stabilised_memory(q, k, v, i, f):
    """q, k ``[T, H, d]``, v ``[T, H, e]``, log gates i and f ``[T, H]`` -> o ``[T, H, e]`` and the last (S, n, m)."""
    T, H, d = q.shape
    S, n, m = (torch.zeros(*s, dtype=q.dtype) for s in ((H, d, v.shape[-1]), (H, d), (H,)))
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        m = new
        size = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hde,hd->he", S, q[t]) / size[:, None])
    return torch.stack(out), (S, n, m)


def mlstm(h, m, t, eps):
    T, H, d, e, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q, k, v = ((h @ t(n).T).view(T, H, w) for n, w in (("q", d), ("k", d), ("v", e)))
    i = soft_cap(h @ t("i").T + t("i.b"), cap)
    f = log_sigmoid(soft_cap(h @ t("f").T + t("f.b"), cap))
    o, _ = stabilised_memory(q * d ** -0.5, k, v, i, f)
    return (rms(o, eps).reshape(T, -1) * t("norm") * torch.sigmoid(h @ t("g").T)) @ t("o").T


def dense(h, t, act):
    return (act(h @ t("gate").T) * (h @ t("up").T)) @ t("down").T


def routing(z, correction, top, scale, margins=None):
    """Logits ``[T, n]`` -> weights ``[T, n]``, zero where an expert is not chosen. ``margins``: a list that receives how far
    every token's last choice was from the first expert it left out."""
    s = z.softmax(-1)
    order = (s + correction).sort(-1, descending=True)
    if margins is not None and top < z.shape[-1]:
        margins.append(order.values[:, top - 1] - order.values[:, top])
    chosen = order.indices[:, :top]
    w = s.gather(-1, chosen)
    return torch.zeros_like(s).scatter(-1, chosen, w / (w.sum(-1, keepdim=True) + 1e-20) * scale)


def experts(h, m, t, margins=None):
    r = m["router"]
    w = routing(h @ t("router").T, t("correction"), r["top"], r["scale"], margins)
    y = torch.zeros_like(h)
    for e in range(r["experts"]):
        y = y + w[:, e:e + 1] * dense(h, lambda n: t(f"e{e}.{n}"), silu)
    for e in range(r["experts"], r["experts"] + (r.get("identity") or 0)):
        y = y + w[:, e:e + 1] * h
    if m.get("shared"):
        y = y + torch.sigmoid(h @ t("shared.sg").T) * dense(h, lambda n: t("shared." + n), silu)
    return y


def feed_forward(h, m, t, margins=None):
    return dense(h, t, gelu_tanh) if m["kind"] == "dense" else experts(h, m, t, margins)


def token_side(x, e, t, eps):
    return rms((gelu_tanh(x @ t("gate").T) * e) @ t("proj").T, eps) * t("norm")


def forward(config, tensors, ids, dtype=torch.float64, layer_outputs=None, margins=None):
    """Logits ``[T, vocab]`` of one sequence; ``layer_outputs``: a list that receives the residual after every layer;
    ``margins``: see :func:`routing`."""
    w = {k: v.to(dtype) for k, v in tensors.items()}
    eps, ids = config["norm"]["eps"], torch.as_tensor(ids)
    x = w["embed"][ids] * config["embedding"]["scale"]
    kv = {}
    for i, layer in enumerate(config["layers"]):
        p, m = f"l{i}", layer["mixer"]

        def mix(n):
            return w[f"{p}.mix.{n}"]

        h = rms(x, eps) * w[p + ".norm1"]
        if layer["type"] == "mlstm":
            y = mlstm(h, m, mix, eps)
        else:
            y, kv[i] = attention(h, m, mix, eps, kv[m["kv_from"]] if m.get("kv_from") is not None else None)
        x = x + rms(y, eps) * w[p + ".norm1b"]
        if layer["mlp"] is not None:
            y = feed_forward(rms(x, eps) * w[p + ".norm2"], layer["mlp"], lambda n: w[f"{p}.mlp.{n}"], margins)
            x = x + rms(y, eps) * w[p + ".norm2b"]
        if config.get("token_side"):
            n = config["token_side"]["dim"]
            x = x + token_side(x, w["side.embed"][ids][:, i * n:(i + 1) * n], lambda a: w[f"{p}.side.{a}"], eps)
        if layer_outputs is not None:
            layer_outputs.append(x)
    return (rms(x, eps) * w["final.norm"]) @ w["embed"].T * config["logit_scale"]


def random_tensors(config, seed):
    """Random bf16 tensors under the checkpoint's names, sized so that every term matters. Memories' queries resemble their keys:
    a first token reads (q . k) v, which is normed, so that its sign would be a matter of rounding where q and k happen to be
    orthogonal."""
    g = torch.Generator().manual_seed(seed)
    W, V = config["width"], config["vocab"]

    def lin(o, i, gain=1.0):
        return (torch.randn(o, i, generator=g) * gain / math.sqrt(i)).bfloat16()

    def vec(n, mean=1.0, std=0.3):
        return (mean + std * torch.randn(n, generator=g)).bfloat16()

    def alike(w):
        return (0.8 * w.float() + 0.6 * torch.randn(w.shape, generator=g) * w.float().std()).bfloat16()

    def gated(p, ff):
        t[p + "gate"], t[p + "up"], t[p + "down"] = lin(ff, W), lin(ff, W), lin(W, ff)

    t = {"embed": (torch.randn(V, W, generator=g) / config["embedding"]["scale"]).bfloat16()}
    for i, layer in enumerate(config["layers"]):
        m, mlp, q = layer["mixer"], layer["mlp"], f"l{i}.mix."
        names = ["norm1", "norm1b"] + (["norm2", "norm2b"] if mlp else [])
        for n in names:
            t[f"l{i}.{n}"] = vec(W, 0.6 if n.endswith("b") else 1.0)
        H, d, e = m["heads"], m["dim"], m["vdim"]
        if layer["type"] == "mlstm":
            t[q + "q"], t[q + "v"], t[q + "g"], t[q + "o"] = lin(H * d, W), lin(H * e, W), lin(H * e, W), lin(W, H * e)
            t[q + "k"], t[q + "norm"] = alike(t[q + "q"]), vec(H * e)
            t[q + "i"], t[q + "i.b"], t[q + "f"], t[q + "f.b"] = lin(H, W, 2.0), vec(H, -0.5, 1.5), lin(H, W, 2.0), vec(H, 2.5, 2.0)
        else:
            rows = {"q": H * d}
            if m.get("kv_from") is None:
                rows.update(k=m["kv_heads"] * d, v=m["kv_heads"] * e)
            for n, r in rows.items():
                t[q + n] = lin(r, W, 1.2)
                if m.get("conv"):
                    t[q + n + ".conv"] = lin(r, m["conv"], 1.2)
            t[q + "g"], t[q + "o"] = lin(H * e, W), lin(W, H * e)
        p = f"l{i}.mlp."
        if mlp and mlp["kind"] == "dense":
            gated(p, mlp["ff"])
        elif mlp:
            r = mlp["router"]
            n = r["experts"] + (r.get("identity") or 0)
            t[p + "router"], t[p + "correction"] = lin(n, W), vec(n, 0.0, 0.1)
            for x in range(r["experts"]):
                gated(f"{p}e{x}.", mlp["expert"]["ff"])
            if mlp.get("shared"):
                gated(p + "shared.", mlp["shared"]["ff"])
                t[p + "shared.sg"] = lin(1, W)
        if config.get("token_side"):
            n = config["token_side"]["dim"]
            t[f"l{i}.side.gate"], t[f"l{i}.side.proj"], t[f"l{i}.side.norm"] = lin(n, W), lin(W, n), vec(W, 0.5)
    if config.get("token_side"):
        t["side.embed"] = torch.randn(V, len(config["layers"]) * config["token_side"]["dim"], generator=g).bfloat16()
    t["final.norm"] = vec(W)
    return t
