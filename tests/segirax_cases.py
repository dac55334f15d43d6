"""Small Segirax configurations, checkpoints of random weights and comparison helpers shared by the Segirax tests."""
from __future__ import annotations

import json

import torch

import segirax_oracle as oracle


def latent(heads, dim, rot, vdim, rank, dims=None, base=1e4, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale or (dim + rot) ** -0.5,
                      "rot": {"dims": rot if dims is None else dims, "base": base}}}


def lightning(heads, dim, vdim, decay):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}}


def model(width, vocab, layers, eps=1e-5, logit_scale=0.7):
    return {"architecture": "Segirax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale,
            "layers": [{**l, "mlp": None if ff is None else {"kind": "dense", "ff": ff}} for l, ff in layers]}


CASES = {
    # both mixers in both orders, a layer without FFN, several widths
    "mixed": model(96, 211, [(latent(3, 24, 16, 40, 56), 136), (lightning(2, 48, 24, [0.5, 0.98]), 72),
                             (lightning(3, 16, 48, [0.9, 0.999, 0.3]), None), (latent(5, 40, 8, 16, 88, base=5e5), 200)]),
    # nothing is a multiple of eight: the plain kernels and padded pitches
    "odd": model(52, 131, [(lightning(3, 20, 7, [0.7, 0.95, 0.2]), 37), (latent(3, 10, 6, 13, 30, dims=4), 45),
                           (latent(1, 5, 2, 3, 17), None)], eps=1e-3, logit_scale=1.3),
    # wide heads and latents (the largest kernel instances), one head
    "wide": model(160, 300, [(latent(2, 128, 64, 128, 512), 256), (lightning(1, 200, 136, [0.97]), 96), (lightning(1, 128, 64, [1.0]), 64)]),
    # more heads than one decode tile, a middle-sized latent, no recurrence anywhere
    "heads": model(128, 257, [(latent(17, 16, 32, 24, 200), 128), (latent(18, 72, 48, 72, 136, scale=0.05), 64)]),
    # recurrence only
    "recurrent": model(64, 97, [(lightning(4, 32, 32, [0.0, 0.6, 0.99, 1.0]), 96), (lightning(1, 8, 16, [0.9]), None)]),
}


def tensors(name, seed=0):
    return oracle.random_tensors(CASES[name], seed)


def write_checkpoint(path, config, t):
    from safetensors.torch import save_file

    path.mkdir(parents=True, exist_ok=True)
    (path / "config.json").write_text(json.dumps(config))
    save_file({k: v.contiguous() for k, v in t.items()}, str(path / "model.safetensors"))
    return str(path)


def prompt(config, n, seed):
    return torch.randint(0, config["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def error(got, want):
    """Root mean square of the difference over the vocabulary (its mean taken off) in units of the logits' spread, per row."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / want.std()
