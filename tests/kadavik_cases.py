"""Small Kadavik configurations shared by the Kadavik tests."""
from __future__ import annotations

import torch

import kadavik_oracle as oracle
from segirax_cases import error, prompt, write_checkpoint  # noqa: F401  (the helpers fit any layered decoder)


def memory(heads, dim, vdim, cap=15.0):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def attention(heads, kv_heads, dim, vdim, *, rot=None, scaling=None, base=1e4, conv=3, window=0, keep=0, kv_from=None, scale=None):
    """rot: rotated dimensions (all of them by default); scaling: (factor, low, high, original)."""
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
         "rot": {"dims": dim if rot is None else rot, "base": base}}
    if scaling:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if conv:
        m["conv"] = conv
    if window:
        m["mask"] = {"size": window, "keep_first": keep}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, identity=0, shared=0, scale=1.5):
    router = {"experts": experts, "top": top, "scale": scale, **({"identity": identity} if identity else {})}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router, **({"shared": {"ff": shared}} if shared else {})}


def model(width, vocab, layers, side=0, eps=1e-5, embed=4.0, logits=0.8):
    return {"architecture": "Kadavik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed}, "logit_scale": logits,
            **({"token_side": {"dim": side}} if side else {}), "layers": [{**l, "mlp": mlp} for l, mlp in layers]}


CASES = {
    # both mixers in both orders, shared keys with a window of their own, every kind of FFN and none
    "mixed": model(96, 211, [(attention(6, 2, 24, 40, rot=16, scaling=(4.0, 1.0, 4.0, 64), conv=4, window=40, keep=5), moe(5, 2, 40, 2, 56)),
                             (memory(3, 24, 40, 8.0), None), (attention(6, 2, 24, 40, rot=16, scaling=(4.0, 1.0, 4.0, 64), conv=2, window=70, kv_from=0),
                                                              dense(136)),
                             (memory(2, 48, 16), moe(3, 3, 24, 3, 16))], side=16),
    # nothing is a multiple of eight: the plain kernels and padded pitches
    "odd": model(52, 131, [(memory(3, 9, 5, 3.0), dense(37)), (attention(3, 1, 10, 13, rot=6, conv=3, window=33, keep=17), moe(4, 2, 11, 1, 7)),
                           (attention(3, 1, 10, 13, rot=6, conv=5, kv_from=1, scale=0.5), None), (memory(1, 21, 30), moe(6, 1, 20, 0, 0, 0.7))],
                 side=10, eps=1e-3, embed=1.0, logits=1.3),
    # wide heads: the tensor-core kernels' largest instances; first tokens that reach across tiles
    "wide": model(160, 300, [(memory(2, 128, 128, 4.0), moe(9, 3, 72, 0, 0)), (attention(8, 2, 128, 128, rot=64, conv=4, window=64, keep=70), moe(2, 2, 200, 1, 136)),
                             (attention(4, 1, 160, 72, conv=2, window=48), dense(96)), (memory(1, 64, 128), None)], side=40),
    # beyond them: memories whose columns or keys span several CTAs, groups of uneven size, one tap, a window of one token
    "tall": model(128, 257, [(memory(2, 256, 72), None), (attention(17, 1, 16, 24, conv=1, window=1, keep=3), dense(64)), (memory(1, 264, 136), None),
                             (attention(5, 1, 200, 72, rot=100, conv=3, window=100, keep=1), None), (memory(1, 72, 264, 30.0), moe(1, 1, 48, 3, 32))]),
    # no windows, no convolutions, no token side, everything shared from one layer
    "plain": model(64, 90, [(attention(2, 2, 32, 32, conv=0, base=100.0), dense(72)), (attention(2, 2, 32, 32, conv=0, base=100.0, kv_from=0), moe(4, 4, 16)),
                            (attention(2, 2, 32, 32, conv=0, base=100.0, kv_from=0, window=25, keep=2), dense(40))], embed=7.0),
    # memories only
    "recurrent": model(64, 97, [(memory(4, 32, 32), dense(96)), (memory(2, 64, 64, 1.0), None), (memory(1, 8, 16), moe(4, 2, 32, 2, 24))], side=8),
}


def tensors(name, seed=0):
    return oracle.random_tensors(CASES[name], seed)


_clear: dict = {}


def _shaken(t, seed):
    """The maps off by about as much as rounding to 16 bits, the routers left alone."""
    g = torch.Generator().manual_seed(seed)
    return {k: v.double() * (1 + 2.0 ** -10 * torch.randn(v.shape, generator=g, dtype=torch.float64)) if v.dim() == 2 and "router" not in k else v.double()
            for k, v in t.items()}


def clear_prompt(name, n, seed, margin=0.015):
    """A prompt and its logits, whose tokens choose their experts by a margin that rounding to 16 bits does not bridge and read
    nothing from a memory that cancels to a small part of itself (the norm behind it would blow rounding up)."""
    key = (name, n, seed)
    if key not in _clear:
        c, t = CASES[name], tensors(name)
        shaken = [_shaken(t, s) for s in range(4)] if margin > 1e-3 else []
        g = torch.Generator().manual_seed(seed)
        ids = torch.randint(0, c["vocab"], (n,), generator=g)
        for _ in range(100):
            margins: list = []
            logits = oracle.forward(c, t, ids, margins=margins)
            close = torch.stack(margins).min(0).values < margin if margins else torch.zeros(n, dtype=torch.bool)
            if not close.any():
                close = torch.stack([error(oracle.forward(c, s, ids), logits) for s in shaken]).max(0).values > 0.03 if shaken else close
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


def marked_model(window, keep, kv_from=False):
    """A model whose attention looks for one marked token: the embedding has a constant first column from which the queries
    are made, and a last column that only the marked token has. Returns configuration and tensors."""
    att = attention(4, 2, 24, 32, rot=8, conv=3, window=window, keep=keep)
    layers = [(att, dense(64))]
    if kv_from:
        layers.append((attention(4, 2, 24, 32, rot=8, conv=2, window=window + 9, keep=0, kv_from=0), None))
    c = model(64, 90, layers + [(memory(2, 16, 16), None)], side=8)
    t = oracle.random_tensors(c, 7)
    t["embed"] *= 0.5
    t["embed"][:, 0], t["embed"][:, -1] = 0.5, 0.0
    t["embed"][MARK, -1] = 1.5
    for i in range(len(layers)):
        p = f"l{i}.mix."
        t[p + "q"] *= 0.05
        t[p + "q"][:, 0] = 0
        t[p + "q"].view(4, 24, 64)[:, 8:, 0] = 1.2           # the unrotated part
        t[p + "q.conv"] *= 0.05
        t[p + "q.conv"][:, -1] = 1.0
        t[p + "g"] *= 0.1
        t[f"l{i}.norm1b"] *= 2
    t["l0.mix.k"] *= 0.1
    t["l0.mix.k"].view(2, 24, 64)[:, 8:, -1] = 1.5
    t["l0.mix.k.conv"] *= 0.05
    t["l0.mix.k.conv"][:, -1] = 1.0
    t["l0.mix.v.conv"][:, -1] = 1.5
    return c, t
