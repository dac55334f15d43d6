"""Small Saninex configurations shared by the Saninex tests."""
from __future__ import annotations

import torch

import saninex_oracle as oracle
from segirax_cases import error, prompt, write_checkpoint  # noqa: F401  (the helpers fit any layered decoder)


def delta(heads, kv_heads, dim, vdim, conv):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def parallel(left, right, scale=None, softcap=20.0, tau=8.0):
    """left: (heads, kv_heads, dim, vdim), right: (heads, dim, vdim)."""
    h, g, d, e = left
    return {"type": "parallel", "mixer": {
        "left": {"heads": h, "kv_heads": g, "dim": d, "vdim": e, "scale": scale or d ** -0.5, "softcap": softcap},
        "right": {"heads": right[0], "dim": right[1], "vdim": right[2], "tau": tau}}}


def model(width, vocab, layers, eps=1e-5):
    return {"architecture": "Saninex", "width": width, "vocab": vocab, "norm": {"eps": eps},
            "layers": [{**l, "mlp": None if ff is None else {"kind": "dense", "ff": ff[0], "limit": ff[1]}} for l, ff in layers]}


CASES = {
    # both mixers in both orders, layers with and without FFN, shared and unshared heads
    "mixed": model(96, 211, [(parallel((6, 2, 24, 40), (3, 16, 24)), (136, 0.9)), (delta(6, 3, 24, 40, 4), None),
                             (delta(2, 2, 48, 16, 3), (72, 7.0)), (parallel((3, 3, 40, 16), (2, 48, 32), softcap=4.0, tau=16.0), None)]),
    # nothing is a multiple of eight: the plain kernels and padded pitches
    "odd": model(52, 131, [(delta(3, 1, 20, 7, 2), (37, 1.2)), (parallel((3, 1, 10, 13), (3, 9, 5), scale=0.4, tau=1.0), (45, 0.5)),
                           (parallel((1, 1, 5, 3), (1, 17, 11), softcap=2.0, tau=3.0), None)], eps=1e-3),
    # wide heads: the tensor-core kernels' largest instances
    "wide": model(160, 300, [(delta(4, 2, 128, 128, 4), (256, 2.0)), (parallel((8, 2, 128, 128), (2, 128, 128), tau=16.0), (96, 1.5)),
                             (parallel((4, 1, 160, 72), (1, 64, 128), softcap=50.0), None)]),
    # beyond them: states too large for registers, groups of uneven size, long convolutions
    "tall": model(128, 257, [(delta(2, 1, 256, 256, 6), None), (parallel((5, 1, 200, 72), (1, 200, 136)), (64, 1.0)),
                             (delta(3, 3, 72, 136, 5), None), (parallel((17, 1, 16, 24), (1, 264, 8)), None)]),
    # recurrence only; a convolution of one tap
    "recurrent": model(64, 97, [(delta(4, 2, 32, 32, 1), (96, 1.0)), (delta(2, 1, 64, 64, 4), None), (delta(1, 1, 8, 16, 3), None)]),
}
RANKS = {"odd": 5, "wide": 16, "tall": 24}


def tensors(name, seed=0):
    return oracle.random_tensors(CASES[name], seed, RANKS.get(name, 12))


def far_key_model():
    """A parallel layer whose queries all look for the key of token 7; returns configuration and tensors."""
    c = model(64, 90, [(parallel((4, 2, 24, 32), (2, 16, 16), softcap=50.0), (64, 1.5)), (delta(2, 1, 16, 16, 4), None)])
    t = oracle.random_tensors(c, 7)
    x = t["embed"].double()
    p = "l0.mix.left."
    key = (oracle.rms((x[7] @ t[p + "k"].double().T + t[p + "k.b"].double()).view(2, 24), 1e-5) * t[p + "k.norm"].double())
    # the query is the bias: the wanted key, the same for every token; the cap leaves a margin of tens
    t[p + "q"] *= 0.05
    t[p + "q.b"] = (key[:, None] * t[p + "k.norm"].double().sign()).expand(2, 2, 24).reshape(-1).bfloat16()
    t[p + "q.norm"] = (4.0 * t[p + "k.norm"].double().sign()).bfloat16()
    t["l0.mix.left.g"] *= 0.1
    t["l0.mix.left.out"] *= 2
    return c, t
