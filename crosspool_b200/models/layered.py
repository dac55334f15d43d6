"""Attention-side weights of layered decoders in the layout the kernels want.

Every layer's linear maps of the same input become one matrix: the mixer's input projections (those of both sides of a
parallel pair) and the residual gate (``[projections | gate | residual gate]``), each section padded to eight rows so that its
columns in the product start on a 16-byte boundary. Latent attention keeps its up-projections twice: per head for the absorbed form (decode), and with the
shared rotary key folded in as identity rows for the expanded form (prefill), so that one product writes complete per-head
keys; where queries come from a latent of their own, its norm's weight is part of the map behind it. Norm parameters, gates' biases,
sinks and decays are fp32.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Callable

import torch

from ..ops.mixers import DeltaWeights, NormParams, decay_powers, expanded_shape
from .config import (DeltaMixer, GatedLinearMixer, GroupedMixer, LatentMixer, LayerSpec, LinearMixer, MemoryMixer, ModelConfig,
                     ParallelMixer, RotarySpec, ceil8)

# get(name, shape): the checkpoint tensor (or a random one) of that name; a size of 0 is whatever the checkpoint has
Getter = Callable[[str, tuple[int, ...]], torch.Tensor]


def pad_pitch(w: torch.Tensor) -> torch.Tensor:
    """``[..., n, k]`` with a row pitch of whole 16-byte units (zeros behind the k columns)."""
    *lead, k = w.shape
    if k % 8 == 0:
        return w.contiguous()
    out = torch.zeros(*lead, ceil8(k), dtype=w.dtype, device=w.device)
    out[..., :k] = w
    return out[..., :k]


@dataclass
class LayeredLayerWeights:
    spec: LayerSpec
    norm1: NormParams                       # in front of the mixer, or behind it (ModelConfig.output_norm)
    proj: torch.Tensor                      # every linear map of the mixer's input
    proj_bias: torch.Tensor | None          # fp32
    offs: dict[str, int]                    # first column of each section of the product
    o: torch.Tensor                         # [hidden, mixer outputs] (left side of a parallel pair)
    mix: dict = field(default_factory=dict)
    o_bias: torch.Tensor | None = None
    o_right: torch.Tensor | None = None     # right side of a parallel pair
    branch_norms: tuple[NormParams, ...] = ()   # of both sides' outputs
    norm2: NormParams | None = None
    rg2: torch.Tensor | None = None         # residual gate of the FFN
    rg2_bias: torch.Tensor | None = None
    silu_cols: int = 0                      # leading columns of the product that are stored through silu
    norm1b: NormParams | None = None        # behind the mixer, where norm1 stands in front of it (ModelConfig.input_norm)
    norm2b: NormParams | None = None        # ... behind the FFN
    fp32_from: int = 0                      # columns of the product from here on are wanted in fp32 (0: none are)
    side_gate: torch.Tensor | None = None   # token side: [dim, hidden], [hidden, dim], its norm
    side_proj: torch.Tensor | None = None
    side_norm: NormParams | None = None


def _fuse(sections: list[tuple[str, torch.Tensor]]) -> tuple[torch.Tensor, dict[str, int]]:
    rows, offs, at = [], {}, 0
    for name, w in sections:
        offs[name] = at
        rows.append(w)
        pad = ceil8(w.shape[0]) - w.shape[0]
        if pad:
            rows.append(torch.zeros(pad, w.shape[1], dtype=w.dtype, device=w.device))
        at += w.shape[0] + pad
    offs["end"] = at
    return pad_pitch(torch.cat(rows, 0)), offs


def _norm(get: Getter, name: str, cfg: ModelConfig) -> NormParams:
    h = cfg.hidden_size
    return NormParams("dyt", get(name, (h,)).float().contiguous(), get(name + ".b", (h,)).float().contiguous(),
                      get(name + ".alpha", ()).float().reshape(1).contiguous(), cfg.rms_norm_eps)


def rotary_frequencies(dims: int, base: float) -> torch.Tensor:
    return float(base) ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)


def scaled_frequencies(rot: RotarySpec) -> torch.Tensor:
    """Turns per position (radians) of every pair, double."""
    f, sc = rotary_frequencies(rot.dims, rot.base), rot.scaling
    if sc is None:
        return f
    if not sc.original:
        return f / sc.factor
    turns = sc.original * f / (2 * torch.pi)                 # of the original context: original / wavelength
    blend = ((turns - sc.low) / (sc.high - sc.low)).clamp(0, 1) if sc.high > sc.low else (turns >= sc.low).double()
    return f * (blend + (1 - blend) / sc.factor)


def rotary_table(rot: RotarySpec, positions: int, device) -> torch.Tensor:
    """cos and sin of every position's angles, fp32 ``[positions, dims / 2, 2]`` rounded from double."""
    a = torch.arange(positions, dtype=torch.float64, device=device)[:, None] * scaled_frequencies(rot).to(device)
    return torch.stack([a.cos(), a.sin()], -1).float().contiguous()


def _latent(m: LatentMixer, get: Getter, p: str, hidden: int, dtype: torch.dtype, device) -> tuple[list, dict]:
    H, R, d, r, vd = m.heads, m.kv_rank, m.dim, m.rot_dim, m.vdim
    dkv, g = get(p + "dkv", (R + r, hidden)), get(p + "g", (m.gate_features, hidden))
    mix = {}
    if m.q_rank:
        # the latent's norm weight is folded into the map behind it, its division follows the product (a number per row)
        q, uq = get(p + "dq", (m.q_rank, hidden)), get(p + "uq", (H * (d + r), m.q_rank))
        mix["uq"] = pad_pitch((uq.float() * get(p + "dq.norm", (m.q_rank,)).float()).to(dtype))
    else:
        q = get(p + "q", (H * (d + r), hidden))
    uk, uv = get(p + "uk", (H * d, R)), get(p + "uv", (H * vd, R))
    mix |= {"norm": get(p + "dkv.norm", (R,)).float().contiguous(), "freq": scaled_frequencies(m.rot).to(device),
           "uk_t": pad_pitch(uk.view(H, d, R).transpose(1, 2).reshape(H * R, d)), "uv": pad_pitch(uv)}
    shape = expanded_shape(d, r, vd) if dtype == torch.bfloat16 else None
    if shape is not None:
        dq, dv = shape
        ek = torch.zeros(H, dq, R + r, dtype=uk.dtype, device=uk.device)
        ek[:, :d, :R] = uk.view(H, d, R)
        ek[:, torch.arange(d, d + r), torch.arange(R, R + r)] = 1
        ev = torch.zeros(H, dv, R, dtype=uv.dtype, device=uv.device)
        ev[:, :vd] = uv.view(H, vd, R)
        mix["exp_k"], mix["exp_v"] = pad_pitch(ek.view(H * dq, R + r)), pad_pitch(ev.view(H * dv, R))
    return [("q", q), ("kv", dkv), ("g", g)], mix


def _linear(m: LinearMixer, get: Getter, p: str, hidden: int, device) -> tuple[list, dict]:
    H, d, vd = m.heads, m.dim, m.vdim
    sections = [(n, get(p + n, (H * w, hidden))) for n, w in (("q", d), ("k", d), ("v", vd), ("g", vd))]
    return sections, {"norm": get(p + "norm", (H * vd,)).float().contiguous(),
                      "decay": torch.tensor(m.decay, dtype=torch.float32, device=device),
                      "decay_pow": decay_powers(m.decay).to(device)}


def _grouped(m: GroupedMixer, get: Getter, p: str, hidden: int) -> tuple[list, dict, dict]:
    """Projection sections, their biases, and what else the mixer has."""
    rows = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim}
    sections = [(n, get(p + n, (r, hidden))) for n, r in rows.items()] + [("hg", get(p + "g", (m.heads, hidden)))]
    biases = {n: get(f"{p}{n}.b", (r,)).float() for n, r in rows.items()}
    return sections, biases, {n: get(f"{p}{n[0]}.norm", (m.dim,)).float().contiguous() for n in ("q_norm", "k_norm")}


def _gated_linear(m: GatedLinearMixer, get: Getter, p: str, hidden: int) -> tuple[list, dict]:
    H, d, vd = m.heads, m.dim, m.vdim
    sections = [("lin_" + n, get(p + n, (H * w, hidden))) for n, w in (("q", d), ("k", d), ("v", vd), ("g", vd))]
    a1 = get(p + "a1", (m.rank, hidden))
    return sections + [("lin_a", a1)], {"norm": get(p + "norm", (vd,)).float().contiguous(), "a2": pad_pitch(get(p + "a2", (H * d, a1.shape[0]))),
                                     "a2_bias": get(p + "a2.b", (H * d,)).float().contiguous()}


def _delta(m: DeltaMixer, get: Getter, p: str, hidden: int) -> tuple[list, dict]:
    H, G, d, vd = m.heads, m.kv_heads, m.dim, m.vdim
    rows = {"q": G * d, "k": G * d, "v": H * vd, "g": H * vd, "b": H, "a": H}
    conv = torch.cat([get(f"{p}{n}.conv", (rows[n], m.conv)).float() for n in "qkv"], 0)
    w = DeltaWeights(conv.contiguous(), -get(p + "A_log", (H,)).float().exp(), get(p + "dt_bias", (H,)).float().contiguous(),
                     get(p + "norm", (vd,)).float().contiguous())
    return [(n, get(p + n, (r, hidden))) for n, r in rows.items()], {"delta": w}


def _windowed(m: GroupedMixer, get: Getter, p: str, hidden: int) -> tuple[list, dict]:
    """Grouped-query attention without head norms; a layer that reads another layer's keys and values has queries only."""
    rows = {"q": m.heads * m.dim}
    if m.kv_from is None:
        rows.update(k=m.kv_heads * m.dim, v=m.kv_heads * m.vdim)
    mix = {"conv": torch.cat([get(f"{p}{n}.conv", (r, m.conv)).float() for n, r in rows.items()], 0).t().contiguous() if m.conv else None}
    return [(n, get(p + n, (r, hidden))) for n, r in {**rows, "g": m.out_features}.items()], mix


def _scored(m: GroupedMixer, get: Getter, p: str, hidden: int) -> tuple[list, dict, dict]:
    """Grouped-query attention whose scores come from normed queries and keys, with a number per head beside them."""
    rows = {"q": m.heads * m.dim, "k": m.kv_heads * m.dim}
    if not m.tied:
        rows["v"] = m.kv_heads * m.vdim
    mix = {n: get(p + name, (m.heads,)).float().contiguous() for n, name, on in (("sink", "sink", m.sink), ("bias", "pb", m.sigmoid)) if on}
    if m.norm == "weight":
        mix |= {n: get(f"{p}{n[0]}.norm", (m.dim,)).float().contiguous() for n in ("q_norm", "k_norm")}
    return [(n, get(p + n, (r, hidden))) for n, r in rows.items()], {n: get(f"{p}{n}.b", (r,)).float() for n, r in rows.items() if m.biases}, mix


def _memory(m: MemoryMixer, get: Getter, p: str, hidden: int) -> tuple[list, dict, dict]:
    rows = {"q": m.heads * m.dim, "k": m.heads * m.dim, "v": m.out_features, "g": m.out_features, "i": m.heads, "f": m.heads}
    return ([(n, get(p + n, (r, hidden))) for n, r in rows.items()], {n: get(f"{p}{n}.b", (m.heads,)).float() for n in "if"},
            {"norm": get(p + "norm", (m.out_features,)).float().contiguous()})


def _plain_norm(get: Getter, name: str, cfg: ModelConfig) -> NormParams:
    return NormParams("rmsnorm", get(name, (cfg.hidden_size,)).float().contiguous(), eps=cfg.rms_norm_eps)


def _input_output_norm_layer(cfg: ModelConfig, i: int, spec: LayerSpec, get: Getter, device) -> LayeredLayerWeights:
    """A layer with a norm in front of and behind each sublayer, and perhaps a token side."""
    h, m, p = cfg.hidden_size, spec.mixer, f"l{i}."
    biases: dict = {}
    if isinstance(m, MemoryMixer):
        sections, biases, mix = _memory(m, get, p + "mix.", h)
    else:
        sections, mix = _windowed(m, get, p + "mix.", h)
    proj, offs = _fuse(sections)
    bias = None
    if biases:
        bias = torch.zeros(offs["end"], dtype=torch.float32, device=device)
        for n, b in biases.items():
            bias[offs[n]:offs[n] + b.shape[0]] = b
    lw = LayeredLayerWeights(spec, _plain_norm(get, p + "norm1", cfg), proj, bias, offs, pad_pitch(get(p + "mix.o", (h, m.out_features))), mix,
                             norm1b=_plain_norm(get, p + "norm1b", cfg), fp32_from=offs.get("i", 0))
    if spec.has_ffn:
        lw.norm2, lw.norm2b = (_plain_norm(get, p + n, cfg) for n in ("norm2", "norm2b"))
    if cfg.token_side:
        lw.side_gate = pad_pitch(get(p + "side.gate", (cfg.token_side, h)))
        lw.side_proj = pad_pitch(get(p + "side.proj", (h, cfg.token_side)))
        lw.side_norm = _plain_norm(get, p + "side.norm", cfg)
    return lw


def _scalar_norm(get: Getter, name: str, cfg: ModelConfig) -> NormParams:
    """An RMS norm with one weight for all coordinates."""
    return NormParams("rmsnorm", get(name, ()).float().expand(cfg.hidden_size).contiguous(), eps=cfg.rms_norm_eps)


def _input_norm_layer(cfg: ModelConfig, i: int, spec: LayerSpec, get: Getter, device, dtype: torch.dtype) -> LayeredLayerWeights:
    """A layer with norms in front of its sublayers only, whose results are added as they are."""
    h, m, p = cfg.hidden_size, spec.mixer, f"l{i}."
    biases: dict = {}
    if isinstance(m, LatentMixer):
        sections, mix = _latent(m, get, p + "mix.", h, dtype, device)
    else:
        sections, biases, mix = _scored(m, get, p + "mix.", h)
    proj, offs = _fuse(sections)
    if "v" not in offs and "k" in offs:
        offs["v"] = offs["k"]                            # values are the projected keys
    bias = torch.zeros(offs["end"], dtype=torch.float32, device=device) if biases else None
    for n, b in biases.items():
        bias[offs[n]:offs[n] + b.shape[0]] = b
    return LayeredLayerWeights(spec, _scalar_norm(get, p + "norm1", cfg), proj, bias, offs, pad_pitch(get(p + "mix.o", (h, m.out_features))), mix,
                               norm2=_scalar_norm(get, p + "norm2", cfg) if spec.has_ffn else None)


def _centred_norm(get: Getter, name: str, cfg: ModelConfig) -> NormParams:
    """An RMS norm whose weight is stored as its distance from one."""
    return NormParams("rmsnorm", 1.0 + get(name, (cfg.hidden_size,)).float(), eps=cfg.rms_norm_eps)


def _output_norm_layer(cfg: ModelConfig, i: int, spec: LayerSpec, get: Getter, device) -> LayeredLayerWeights:
    """A layer whose sublayers read the residual itself and are normed behind."""
    h, m, p = cfg.hidden_size, spec.mixer, f"l{i}.mix."
    biases: dict = {}
    extra: dict = {}
    if isinstance(m, ParallelMixer):
        left, biases, mix = _grouped(m.left, get, p + "left.", h)
        right, mix_r = _gated_linear(m.right, get, p + "right.", h)
        sections, mix = left + right, {**mix, **mix_r}
        o = get(p + "left.o", (h, m.left.out_features))
        extra = dict(o_bias=get(p + "left.o.b", (h,)).float().contiguous(), o_right=pad_pitch(get(p + "right.o", (h, m.right.out_features))),
                     branch_norms=tuple(NormParams("rmsnorm", get(f"{p}{side}.out", (h,)).float().contiguous(), eps=cfg.rms_norm_eps)
                                        for side in ("left", "right")))
    else:
        sections, mix = _delta(m, get, p, h)
        o = get(p + "o", (h, m.out_features))
    proj, offs = _fuse(sections)
    bias = torch.zeros(offs["end"], dtype=torch.float32, device=device) if biases else None
    for n, b in biases.items():
        bias[offs[n]:offs[n] + b.shape[0]] = b
    lw = LayeredLayerWeights(spec, _centred_norm(get, f"l{i}.norm1", cfg), proj, bias, offs, pad_pitch(o), mix, **extra)
    if spec.ff:
        lw.norm2 = _centred_norm(get, f"l{i}.norm2", cfg)
    return lw


def layered_attention_weights(cfg: ModelConfig, get: Getter, device, dtype: torch.dtype):
    """Everything but the FFNs of a layered decoder, from its named tensors (``l<i>.norm1``, ``l<i>.mix.*``,
    ``l<i>.rg1``, ...)."""
    from .weights import AttentionWeights

    h = cfg.hidden_size
    layers = []
    for i, spec in enumerate(cfg.layer_specs):
        if cfg.input_norm:
            layers.append(_input_output_norm_layer(cfg, i, spec, get, device))
            continue
        if cfg.output_norm:
            layers.append(_output_norm_layer(cfg, i, spec, get, device))
            continue
        if cfg.norm == "scalar":
            layers.append(_input_norm_layer(cfg, i, spec, get, device, dtype))
            continue
        p, m = f"l{i}", spec.mixer
        if isinstance(m, LatentMixer):
            sections, mix = _latent(m, get, p + ".mix.", h, dtype, device)
        else:
            sections, mix = _linear(m, get, p + ".mix.", h, device)
        sections.append(("rg", get(p + ".rg1", (h, h))))
        proj, offs = _fuse(sections)
        bias = torch.zeros(offs["end"], dtype=torch.float32, device=device)
        bias[offs["rg"]:offs["rg"] + h] = get(p + ".rg1.b", (h,)).float()
        lw = LayeredLayerWeights(spec, _norm(get, p + ".norm1", cfg), proj, bias, offs, pad_pitch(get(p + ".mix.o", (h, m.out_features))),
                                 mix)
        if spec.ff:
            lw.norm2 = _norm(get, p + ".norm2", cfg)
            lw.rg2, lw.rg2_bias = pad_pitch(get(p + ".rg2", (h, h))), get(p + ".rg2.b", (h,)).float().contiguous()
        if isinstance(m, LinearMixer):
            lw.silu_cols = offs["g"]            # q, k and v
        layers.append(lw)
    embed = get("embed", (cfg.vocab_size, h)).contiguous()
    norm = _scalar_norm if cfg.norm == "scalar" else _plain_norm if cfg.input_norm else _centred_norm if cfg.output_norm else _norm
    head = embed if cfg.tie_word_embeddings else get("head", (cfg.vocab_size, h))
    w = AttentionWeights(embed, layers, norm(get, "final.norm", cfg), pad_pitch(head))
    if cfg.token_side:
        # rows of whole 16-byte units, gathered for all layers at once
        n = cfg.num_layers * cfg.token_side
        w.extra["side_embed"] = torch.nn.functional.pad(get("side.embed", (cfg.vocab_size, n)), (0, ceil8(n) - n)).contiguous()
    return w


# stored around zero: norms behind sublayers; biases and decays of random models are zero too
_ZERO = (".b", "A_log", "dt_bias", ".pb")


def random_getter(gen: torch.Generator, dtype: torch.dtype, device, centred_norms: bool = False) -> Getter:
    """Random tensors by name: linear maps N(0, 0.02), norm weights one (``centred_norms``: layer norms are stored as zero),
    biases and decay parameters zero, dynamic-tanh scalars one, 16 rows where the checkpoint would say how many."""
    from .weights import _randn

    def get(name: str, shape: tuple[int, ...]) -> torch.Tensor:
        shape = tuple(n or 16 for n in shape)
        if len(shape) == 2:
            return _randn(gen, shape, dtype, device)
        zero = name.endswith(_ZERO) or centred_norms and name.rsplit(".", 1)[-1] in ("norm1", "norm2") or centred_norms and name == "final.norm"
        return (torch.zeros if zero else torch.ones)(shape, dtype=dtype, device=device)

    return get
