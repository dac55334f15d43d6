"""Small Dofevik configurations shared by the Dofevik tests."""
from __future__ import annotations

import torch

import dofevik_oracle as oracle
from segirax_cases import error, prompt, write_checkpoint  # noqa: F401  (the helpers fit any layered decoder)


def attention(heads, kv_heads, dim, vdim, size, *, rot=None, base=1e4, factor=0.0, scale=None):
    """rot: rotated dimensions (all of them by default)."""
    r = {"dims": dim if rot is None else rot, "base": base, **({"scaling": {"factor": factor}} if factor else {})}
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": r, "mask": {"size": size},
                                           "scale": scale or dim ** -0.5}}


def pooled(heads, kv_heads, dim, size, pool, scale=None):
    return {"type": "attention_2", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "mask": {"size": size, "pool": pool},
                                             "scale": scale or dim ** -0.5}}


def latent(heads, dim, rot, vdim, q_rank, kv_rank, size, *, base=1e4, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "mask": {"size": size},
                      "rot": {"dims": rot, "base": base}, "scale": scale or (dim + rot) ** -0.5}}


def moe(experts, top, ff, shared=0):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, **({"shared": {"ff": shared}} if shared else {})}


def model(width, vocab, layers, eps=1e-5):
    return {"architecture": "Dofevik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": [{**l, "mlp": mlp} for l, mlp in layers]}


CASES = {
    # every mixer and FFN form; heads wider than their values and the other way round, blocks that straddle pages
    "mixed": model(96, 211, [(attention(6, 2, 24, 40, 37, rot=16, factor=3.0), moe(5, 2, 40, 56)), (pooled(4, 2, 40, 50, 7), None),
                             (latent(3, 24, 8, 40, 56, 72, 45), moe(3, 1, 24)), (pooled(6, 1, 24, 23, 20), moe(4, 4, 32, 16))]),
    # nothing is a multiple of eight: the plain kernels and padded pitches
    "odd": model(52, 131, [(latent(3, 10, 6, 13, 21, 30, 29), moe(4, 2, 11, 7)), (pooled(3, 3, 10, 19, 3), moe(6, 3, 20)),
                           (attention(3, 1, 10, 13, 41, rot=6), None)], eps=1e-3),
    # wide heads and latents: the largest instances of the tensor-core kernels
    "wide": model(160, 300, [(pooled(8, 2, 128, 64, 16), moe(9, 3, 72, 40)), (attention(8, 1, 128, 128, 100, rot=64, base=5e5), moe(2, 2, 200, 136)),
                             (latent(2, 128, 64, 128, 96, 512, 70), None), (attention(2, 2, 160, 72, 64, rot=160, factor=8.0), None)]),
    # beyond them: groups of uneven size, windows of one token and longer than any prompt, blocks of one token and longer than a page
    "tall": model(128, 257, [(attention(17, 1, 16, 24, 1), moe(1, 1, 48, 32)), (pooled(5, 1, 72, 9, 1), None), (latent(18, 40, 24, 32, 72, 136, 1000), None),
                             (pooled(2, 1, 200, 30, 70), moe(7, 5, 24, 8)), (attention(5, 5, 200, 24, 130, rot=20), None)]),
    # small windows everywhere, edges shared by pages, windows and blocks
    "edges": model(64, 90, [(pooled(2, 2, 32, 16, 8), moe(4, 2, 16)), (attention(4, 2, 64, 64, 64), None), (pooled(4, 4, 64, 64, 32), None),
                            (latent(4, 32, 16, 32, 48, 64, 64), moe(4, 2, 32, 24))]),
}


def tensors(name, seed=0):
    return oracle.random_tensors(CASES[name], seed)


_clear: dict = {}


def clear_prompt(name, n, seed, margin=0.04):
    """A prompt and its logits, whose tokens choose their experts by a margin (of router logits) that rounding to 16 bits does not
    bridge."""
    key = (name, n, seed)
    if key not in _clear:
        c, t = CASES[name], tensors(name)
        g = torch.Generator().manual_seed(seed)
        ids = torch.randint(0, c["vocab"], (n,), generator=g)
        for _ in range(200):
            margins: list = []
            logits = oracle.forward(c, t, ids, margins=margins)
            close = torch.stack(margins).min(0).values < margin if margins else torch.zeros(n, dtype=torch.bool)
            if not close.any():
                break
            first = int(close.nonzero()[0])                  # a changed token moves the margins behind it
            close[first + max(8, n // 6):] = False
            ids = torch.where(close, torch.randint(0, c["vocab"], (n,), generator=g), ids)
        else:
            raise AssertionError(f"no clear prompt for {key}")
        _clear[key] = (ids.tolist(), logits)
    return _clear[key]


MARK = 7


def marked_model(kind, size, pool=0):
    """A model of one mixer whose queries look for one marked token, and a routed FFN behind it. The embedding has a constant first
    column and a last column that only the marked token has; unmarked keys point another way. Returns configuration and
    tensors."""
    if kind == "attention":
        c = model(64, 90, [(attention(4, 2, 24, 32, size, rot=8, factor=2.0, scale=0.5), moe(3, 2, 24))])
    elif kind == "pooled":
        c = model(64, 90, [(pooled(4, 2, 24, size, pool, scale=8.0 * pool / 24), moe(3, 2, 24))])
    else:
        c = model(64, 90, [(latent(4, 24, 8, 32, 40, 48, size, scale=1.0), moe(3, 2, 24))])
    t = oracle.random_tensors(c, 7)
    t["embed"] *= 0.5
    t["embed"][:, 0], t["embed"][:, -1] = 2.0, 0.0
    t["embed"][MARK, -1] = 4.0
    for n in ("norm1", "norm2"):
        t["l0." + n] = torch.tensor(1.0).bfloat16()
    t["l0.mlp.router"] *= 0.1                                # the same experts for every token
    t["l0.mlp.router.b"] = torch.tensor([2.0, -2.0, 1.0]).bfloat16()
    p = "l0.mix."
    if kind == "latent":
        R, H, d, r = 48, 4, 24, 8
        g = torch.Generator().manual_seed(3)
        for n, quiet in (("dq", 0.05), ("dkv", 0.05)):
            t[p + n] *= quiet
        t[p + "dq"][:, 0] = torch.randn(40, generator=g).bfloat16()
        t[p + "uq"].view(H, d + r, 40)[:, d:] *= 0.05            # positions hardly matter
        t[p + "dkv.norm"] = torch.ones(R).bfloat16()
        q = oracle.rms(t[p + "dq"][:, 0].double(), 1e-5) * t[p + "dq.norm"].double() @ t[p + "uq"].double().T
        look = torch.einsum("hdr,hd->r", t[p + "uk"].double().view(H, d, R), q.view(H, d + r)[:, :d])
        look = look / look.norm() * R ** 0.5
        away = torch.randn(R, generator=g, dtype=torch.float64)
        away = away - look * (away @ look) / (look @ look)
        t[p + "dkv"][:R, 0], t[p + "dkv"][:R, -1] = 0.5 * away.bfloat16(), look.bfloat16()
    else:
        d, G, H = 24, 2, 4
        t[p + "q"] *= 0.05
        t[p + "k"] *= 0.05
        t[p + "q"].view(H, d, 64)[:, 10, 0] = 3.0                # an unrotated dimension
        t[p + "k"].view(G, d, 64)[:, 12, 0] = 1.0
        t[p + "k"].view(G, d, 64)[:, 10, -1] = 4.0
        if kind == "attention":
            t[p + "q.b"] *= 0.1
            t[p + "k.b"] *= 0.1
            t[p + "sink"] = torch.tensor([1.0, 2.0, 3.0, 4.0]).bfloat16()
            t[p + "v"][:, -1] = 1.0
        else:
            t[p + "q.norm"], t[p + "k.norm"], t[p + "pb"] = torch.ones(d).bfloat16(), torch.ones(d).bfloat16(), torch.tensor([-4.0, -4.5, -5.0, -3.5]).bfloat16()
            t[p + "o"] *= 0.5
    return c, t
