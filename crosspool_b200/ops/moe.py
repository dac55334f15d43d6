"""Mixture-of-experts FFN on the grouped tcgen05 GEMM.

Pipeline (all on the caller's stream, no host synchronisation, shapes independent of the routing):

    router logits GEMM -> top-k -> route ordering + tile tables -> row gather
    -> grouped gate/up GEMM with SwiGLU epilogue -> grouped down GEMM -> weighted combine

It replaces the reference's routing / bitmatrix / ordering / ragged-matmul / reduce chain
(src/xpool/runtime/ffnagent/operators/{routing,moe}.py). With ``expert_range=(lo, hi)`` only routes
to experts ``[lo, hi)`` are computed and the result is this rank's partial sum (expert parallelism);
``w.gate_up`` / ``w.down`` then hold just those experts.
"""

from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

from .. import native
from ..models.config import ModelConfig, MoeSpec, ceil8
from ..models.layered import pad_pitch
from ..models.weights import FfnLayerWeights
from . import gemm


@dataclass
class MoeWorkspace:
    cap_rows: int
    top_k: int
    logits: torch.Tensor
    ids: torch.Tensor
    weights: torch.Tensor
    counts: torch.Tensor
    offsets: torch.Tensor
    perm_token: torch.Tensor
    route_pos: torch.Tensor
    tiles_gu: torch.Tensor
    tiles_dn: torch.Tensor
    n_tiles: torch.Tensor
    xp: torch.Tensor
    act: torch.Tensor
    yp: torch.Tensor
    logits32: torch.Tensor | None = None   # fp32 router logits, allocated on first use by an fp32 router projection


ROUTER_PRECISIONS = {"payload": 0, "fp32_logits": 1, "fp32": 2}


def router_precision_code(w: FfnLayerWeights) -> int:
    """0: bf16 tensor-core projection with bf16 logits; 1: payload weights, fp32 accumulation and fp32 logits; 2: fp32
    weights (``w.extra["router_fp32"]``), fp32 accumulation and logits. Reference: ``RouterProjectionPrecision`` in
    src/xpool/ffn.py and its use in src/xpool/runtime/ffnagent/operators/routing.py."""
    p = w.extra.get("router_precision", "payload")
    p = getattr(p, "value", p)
    if p not in ROUTER_PRECISIONS:
        raise ValueError(f"unknown router projection precision {p!r}")
    if p == "fp32" and w.extra.get("router_fp32") is None:
        raise ValueError("router precision 'fp32' needs the fp32 router weights in extra['router_fp32']")
    return ROUTER_PRECISIONS[p]


def router_project_fp32(x: torch.Tensor, w: FfnLayerWeights, out: torch.Tensor) -> torch.Tensor:
    """``out[:, :num_experts] = x @ router^T`` accumulated and stored in fp32 (exact SIMT projection)."""
    code = router_precision_code(w)
    rw = w.extra["router_fp32"] if code == 2 else w.router
    assert rw.is_contiguous() and out.dtype == torch.float32 and x.stride(1) == 1
    assert rw.dtype == (torch.float32 if code == 2 else torch.bfloat16)
    native.check(native.kernels().xp_router_fp32(x.data_ptr(), x.stride(0), rw.data_ptr(), int(code == 2), out.data_ptr(),
                                                 out.stride(0), x.shape[0], x.shape[1], rw.shape[0], _stream(x.device)),
                 "xp_router_fp32")
    return out


_ws_cache: dict[tuple, MoeWorkspace] = {}


def workspace(device, cap_rows: int, cfg: ModelConfig, inter: int, n_local: int) -> MoeWorkspace:
    # one workspace per stream: Instances of one GPU that run concurrently must not share routing tables and scratch rows
    key = (str(device), torch.cuda.current_stream(device).cuda_stream if torch.device(device).type == "cuda" else 0,
           cap_rows, cfg.hidden_size, inter, cfg.num_experts_per_tok, n_local, cfg.num_experts)
    ws = _ws_cache.get(key)
    if ws is None:
        k, h = cfg.num_experts_per_tok, cfg.hidden_size
        routes = cap_rows * k
        e_pad = (cfg.num_experts + 127) // 128 * 128
        max_tiles = (max(inter, h) // 128) * (routes // 16 + n_local) + 8
        i32 = dict(dtype=torch.int32, device=device)
        bf = dict(dtype=torch.bfloat16, device=device)
        ws = MoeWorkspace(
            cap_rows, k, torch.zeros(cap_rows, e_pad, **bf), torch.zeros(cap_rows, k, **i32),
            torch.zeros(cap_rows, k, dtype=torch.float32, device=device), torch.zeros(n_local, **i32),
            torch.zeros(n_local + 1, **i32), torch.zeros(routes, **i32), torch.zeros(routes, **i32),
            torch.zeros(max_tiles, 4, **i32), torch.zeros(max_tiles, 4, **i32), torch.zeros(2, **i32),
            torch.zeros(routes, h, **bf), torch.zeros(routes, inter, **bf), torch.zeros(routes, h, **bf))
        _ws_cache[key] = ws
    return ws


def padded_router(w: FfnLayerWeights) -> torch.Tensor:
    """The layer's router weights with the expert dimension padded to a multiple of 128 rows (one UMMA
    tile); built once and kept with the layer."""
    router = w.router
    e = router.shape[0]
    if e % 128 == 0:
        return router
    t = w.extra.get("router_padded")
    if t is None or t.shape[1] != router.shape[1] or t.device != router.device:
        t = torch.zeros((e + 127) // 128 * 128, router.shape[1], dtype=router.dtype, device=router.device)
        t[:e] = router
        w.extra["router_padded"] = t
    return t


def _stream(dev) -> int:
    return torch.cuda.current_stream(dev).cuda_stream


def _router_args(logits: torch.Tensor, num_experts: int, top_k: int, out_ids: torch.Tensor, out_weights: torch.Tensor, sigmoid: int = False,
                 renormalize: bool = True, scale: float = 1.0, logit_bias: torch.Tensor | None = None,
                 correction_bias: torch.Tensor | None = None, round_weights_bf16: bool = False) -> "native.RouterArgs":
    a = native.RouterArgs()
    a.logits = logits.data_ptr()
    a.logit_bias = logit_bias.data_ptr() if logit_bias is not None else None
    a.correction_bias = correction_bias.data_ptr() if correction_bias is not None else None
    a.topk_ids, a.topk_weights = out_ids.data_ptr(), out_weights.data_ptr()
    a.rows, a.num_experts, a.top_k, a.ld_logits = logits.shape[0], num_experts, top_k, logits.stride(0)
    a.logits_fp32 = int(logits.dtype == torch.float32)
    a.sigmoid, a.renormalize, a.round_weights_bf16, a.scale = int(sigmoid), int(renormalize), int(round_weights_bf16), scale
    return a


def router_topk(logits: torch.Tensor, num_experts: int, top_k: int, *, out_ids: torch.Tensor, out_weights: torch.Tensor, **kw) -> None:
    """Scores (softmax, or ``sigmoid=True``; 2: the choice by logits, softmax over the chosen), the ``top_k`` largest after ``correction_bias``, their weights (``renormalize``,
    ``scale``)."""
    a = _router_args(logits, num_experts, top_k, out_ids, out_weights, **kw)
    native.check(native.kernels().xp_router_topk(C.byref(a), _stream(logits.device)), "xp_router_topk")


def _tile_width(rows: int, top_k: int, n_local: int, widest: int = 128) -> int:
    avg = max(1, rows * top_k // max(1, n_local))
    bn = 16
    while bn < avg and bn < widest:
        bn <<= 1
    return bn


def _grouped(x, w2d, out, *, n_out, rows_cap, bn, dual, up_offset, tiles, n_tiles, rows_per_group, epilogue, bias=None,
             transform=(0.0, 0.0, 0.0), relu2=0):
    """``bias``: fp32 ``[experts, rows_per_group]``, indexed by the weight row of the stacked tensor."""
    a = gemm._args(x, w2d, out, n_out=n_out, rows=rows_cap, epilogue=epilogue, dual=dual, up_offset=up_offset, splits=1, bn=bn,
                   bias=bias, gate_limit=transform[0], up_add=transform[1], act_alpha=transform[2])
    a.relu2 = relu2
    a.tile_table, a.n_tiles, a.w_rows_per_group = tiles.data_ptr(), n_tiles.data_ptr(), rows_per_group
    native.check(native.kernels().xp_gemm(C.byref(a)), "xp_gemm(grouped)")


def _route_args(ws: "MoeWorkspace | RoutedWorkspace", rows: int, k: int, lo: int, hi: int, gateup_features: int, down_features: int,
                bn: int) -> "native.RouteArgs":
    r = native.RouteArgs()
    r.topk_ids, r.counts, r.offsets = ws.ids.data_ptr(), ws.counts.data_ptr(), ws.offsets.data_ptr()
    r.perm_token, r.route_pos = ws.perm_token.data_ptr(), ws.route_pos.data_ptr()
    r.tiles_gateup, r.tiles_down = ws.tiles_gu.data_ptr(), ws.tiles_dn.data_ptr()
    r.n_tiles_gateup, r.n_tiles_down = ws.n_tiles.data_ptr(), ws.n_tiles.data_ptr() + 4
    r.rows, r.top_k, r.expert_lo, r.expert_hi = rows, k, lo, hi
    r.tm_gateup, r.bn_gateup, r.tm_down, r.bn_down = (gateup_features + 127) // 128, bn, (down_features + 127) // 128, bn
    return r


def moe_forward(x: torch.Tensor, w: FfnLayerWeights, cfg: ModelConfig, out: torch.Tensor | None = None,
                expert_range: tuple[int, int] | None = None, ws: MoeWorkspace | None = None) -> torch.Tensor:
    """``x`` [rows, hidden] bf16 -> MoE output [rows, hidden] (this rank's partial under EP)."""
    rows, h = x.shape
    k, e_total = cfg.num_experts_per_tok, cfg.num_experts
    lo, hi = expert_range or w.extra.get("experts") or (0, e_total)
    n_local = hi - lo
    inter = w.gate_up.shape[1] // 2
    assert w.gate_up.shape[0] == n_local and w.down.shape[0] == n_local
    dev = x.device
    ws = ws or workspace(dev, max(rows, 1), cfg, inter, n_local)
    if out is None:
        out = torch.empty(rows, h, dtype=torch.bfloat16, device=dev)
    lib, s = native.kernels(), _stream(dev)
    # 1. router (payload precision: bf16 logits; fp32 precisions: exact fp32 logits; scores always fp32)
    if router_precision_code(w) == 0:
        logits = ws.logits[:rows]
        gemm.linear(x, padded_router(w), out=logits)
    else:
        if ws.logits32 is None:
            ws.logits32 = torch.zeros(ws.cap_rows, ws.logits.shape[1], dtype=torch.float32, device=dev)
        logits = router_project_fp32(x, w, ws.logits32[:rows])
    router_topk(logits, e_total, k, out_ids=ws.ids[:rows], out_weights=ws.weights[:rows],
                sigmoid=cfg.router_scoring == "sigmoid", renormalize=cfg.norm_topk_prob, scale=cfg.routed_scaling_factor,
                correction_bias=w.extra.get("correction_bias"), logit_bias=w.extra.get("router_bias"),
                round_weights_bf16=bool(w.extra.get("round_topk_weights")))
    # 2. order the routes of the local experts, build the tile tables
    bn = _tile_width(rows, k, n_local)
    r = _route_args(ws, rows, k, lo, hi, inter, h, bn)
    native.check(lib.xp_moe_route(C.byref(r), s), "xp_moe_route", 3)
    # 3. gather rows into expert order
    routes = rows * k
    native.check(lib.xp_moe_gather(x.data_ptr(), ws.perm_token.data_ptr(), ws.offsets.data_ptr() + 4 * n_local,
                                   ws.xp.data_ptr(), routes, h, x.stride(0), s), "xp_moe_gather")
    # 4. grouped projections
    _grouped(ws.xp[:routes], w.gate_up.view(n_local * 2 * inter, h), ws.act[:routes], n_out=inter, rows_cap=routes, bn=bn,
             dual=1, up_offset=inter, tiles=ws.tiles_gu, n_tiles=ws.n_tiles[0:1], rows_per_group=2 * inter,
             epilogue=gemm.EPI_SWIGLU, bias=w.gate_up_bias, transform=w.extra.get("gate_transform", (0.0, 0.0, 0.0)))
    _grouped(ws.act[:routes], w.down.view(n_local * h, inter), ws.yp[:routes], n_out=h, rows_cap=routes, bn=bn, dual=0,
             up_offset=0, tiles=ws.tiles_dn, n_tiles=ws.n_tiles[1:2], rows_per_group=h, epilogue=gemm.EPI_STORE,
             bias=w.down_bias)
    # 5. weighted sum over the selected experts, fixed order
    native.check(lib.xp_moe_combine(ws.yp.data_ptr(), ws.route_pos.data_ptr(), ws.weights.data_ptr(), out.data_ptr(), rows, k,
                                    h, out.stride(0), s), "xp_moe_combine")
    if w.shared_gate_up is not None and (expert_range is None or lo == 0):
        sh = gemm.linear(gemm.gateup_swiglu(x, w.shared_gate_up), w.shared_down)
        out += sh
    return out


# ------------------------------------------------------------------------------------------ layered decoders

@dataclass
class RoutedWorkspace:
    """Scratch of :func:`routed_ffn`, sized for the widest routed layer of a model and ``cap`` rows."""

    ids: torch.Tensor
    weights: torch.Tensor
    counts: torch.Tensor
    offsets: torch.Tensor
    perm_token: torch.Tensor
    route_pos: torch.Tensor
    tiles_gu: torch.Tensor
    tiles_dn: torch.Tensor
    n_tiles: torch.Tensor
    logits: torch.Tensor          # fp32
    xp: torch.Tensor              # the others: activations
    act: torch.Tensor
    yp: torch.Tensor
    shared: torch.Tensor
    z: torch.Tensor | None = None # fp32 models: gate and up columns in front of their activation

    @classmethod
    def for_layers(cls, specs: list[MoeSpec], hidden: int, cap: int, dtype: torch.dtype, device) -> "RoutedWorkspace":
        def buf(n, dt=torch.int32):
            return torch.zeros(n, dtype=dt, device=device)

        top, experts, ff = max(s.top + s.folds_shared for s in specs), max(s.experts + s.folds_shared for s in specs), ceil8(max(max(s.ff, s.shared_ff) for s in specs))
        routes, wide = cap * top, (max(2 * ff, hidden) + 127) // 128    # (ungated experts need half the tiles)
        tiles = wide * (routes // 16 + experts + 1)
        f32 = dtype == torch.float32
        return cls(buf(routes), buf(routes, torch.float32), buf(experts), buf(experts + 1), buf(routes), buf(routes), buf(4 * tiles),
                   buf(4 * tiles), buf(2), buf(cap * (ceil8(max(s.routed for s in specs) + 1)), torch.float32), buf(routes * ceil8(hidden), dtype),
                   buf(routes * ff, dtype), buf(routes * ceil8(hidden), dtype), buf(cap * ceil8(hidden), dtype),
                   buf(max(routes, cap) * 2 * ff, dtype) if f32 else None)


def prepare_routed(w: FfnLayerWeights, spec: MoeSpec) -> None:
    """Puts a layer's weights in the layout of :func:`routed_ffn` (in place): the gate of the shared expert joins the router's
    rows, or the shared expert the routed ones; row pitches become whole 16-byte units."""
    if spec.folds_shared:
        pad = spec.ff - spec.shared_ff
        w.gate_up = torch.cat([w.gate_up, torch.nn.functional.pad(w.shared_gate_up, (0, 0, 0, pad))[None]])
        w.down = torch.cat([w.down, torch.nn.functional.pad(w.shared_down, (0, pad))[None]])
        w.shared_gate_up = w.shared_down = None
    w.gate_up, w.down = pad_pitch(w.gate_up), pad_pitch(w.down)
    scale = w.extra.get("shared_scale")
    w.extra["router_rows"] = pad_pitch(w.router if scale is None else torch.cat([w.router, scale.to(w.router.dtype)], 0))
    if w.shared_gate_up is not None:
        w.shared_gate_up, w.shared_down = pad_pitch(w.shared_gate_up), pad_pitch(w.shared_down)


def _grouped_f32(x, w, out, *, n, tiles, n_tiles, max_tiles) -> None:
    native.check(native.kernels().xp_gemm_f32_grouped(x.data_ptr(), w.data_ptr(), out.data_ptr(), tiles.data_ptr(), n_tiles.data_ptr(), max_tiles, n,
                                                      w.shape[2], x.stride(0), w.stride(1), out.stride(0), w.shape[1], _stream(x.device)),
                 "xp_gemm_f32_grouped")


def _hidden_rows(x: torch.Tensor, w_gate_up: torch.Tensor, act: torch.Tensor, z: torch.Tensor | None, relu2: bool) -> torch.Tensor:
    """``silu(gate) * up`` (or ``max(up, 0)^2``) of plain rows in the rows' element type."""
    if relu2:
        return gemm.linear_relu2(x, w_gate_up, act)
    if x.dtype == torch.float32:
        from . import mixers

        z = z[:x.shape[0] * w_gate_up.shape[0]].view(x.shape[0], w_gate_up.shape[0])
        gemm.linear(x, w_gate_up, out=z)
        return mixers.glu_f32(z, 0.0, 0.0, 1.0, act)
    return gemm.gateup_swiglu(x, w_gate_up, out=act)


def routed_ffn(x: torch.Tensor, w: FfnLayerWeights, spec: MoeSpec, out: torch.Tensor, ws: RoutedWorkspace) -> torch.Tensor:
    """Routed FFN of ``x`` ``[rows, hidden]`` (any width, bf16 or fp32): fp32 router logits of one product (the shared
    expert's gate is its last column), routes ordered by expert, two grouped products, and one kernel that adds up the
    chosen experts, the identity experts and the shared expert (which may be one more of the former). Few rows choose and order
    in one launch."""
    rows, h = x.shape
    f32, lib, s = x.dtype == torch.float32, native.kernels(), _stream(x.device)
    hp, ffp, fold = ceil8(h), ceil8(spec.ff), spec.folds_shared
    E, k = spec.experts + fold, spec.top + fold
    router = w.extra["router_rows"]
    ld = ceil8(router.shape[0])
    logits = ws.logits[:rows * ld].view(rows, ld)[:, :router.shape[0]]
    gemm.linear(x, router, out=logits)
    bn = 64 if f32 else _tile_width(rows, k, E, 256)
    bn_gu = min(bn, 256 if spec.relu2 else 128)            # a gated tile holds two accumulators
    n_gu = spec.in_features if f32 else spec.ff
    ids, wts = ws.ids[:rows * k].view(rows, k), ws.weights[:rows * k].view(rows, k)
    a = _router_args(logits, spec.routed, spec.top, ids, wts, sigmoid=2 if spec.logit_choice else 0, scale=spec.scale,
                     logit_bias=w.extra.get("router_bias"), correction_bias=w.extra.get("correction_bias"))
    a.always = int(fold)
    r = _route_args(ws, rows, k, 0, E, n_gu, h, bn)
    r.bn_gateup = bn_gu
    if rows <= 128:
        native.check(lib.xp_moe_topk_route(C.byref(a), C.byref(r), s), "xp_moe_topk_route")
    else:
        native.check(lib.xp_router_topk(C.byref(a), s), "xp_router_topk")
        native.check(lib.xp_moe_route(C.byref(r), s), "xp_moe_route", 3)
    routes = rows * k
    xp, yp = (t[:routes * hp].view(routes, hp)[:, :h] for t in (ws.xp, ws.yp))
    act = ws.act[:routes * ffp].view(routes, ffp)[:, :spec.ff]
    words = 2 if f32 else 1                               # the gather counts in 16-bit elements
    native.check(lib.xp_moe_gather(x.data_ptr(), ws.perm_token.data_ptr(), ws.offsets.data_ptr() + 4 * E, xp.data_ptr(), routes, hp * words,
                                   x.stride(0) * words, s), "xp_moe_gather")
    if f32:
        from . import mixers

        most = routes // bn + E
        z = ws.z[:routes * n_gu].view(routes, n_gu)
        _grouped_f32(xp, w.gate_up, z, n=n_gu, tiles=ws.tiles_gu, n_tiles=ws.n_tiles[0:1], max_tiles=most * r.tm_gateup)
        if spec.relu2:
            mixers.relu2_f32(z, act)
        else:
            mixers.glu_f32(z, 0.0, 0.0, 1.0, act)
        _grouped_f32(act, w.down, yp, n=h, tiles=ws.tiles_dn, n_tiles=ws.n_tiles[1:2], max_tiles=most * r.tm_down)
    else:
        _grouped(xp, w.gate_up.flatten(0, 1), act, n_out=spec.ff, rows_cap=routes, bn=bn_gu, dual=int(not spec.relu2),
                 up_offset=0 if spec.relu2 else spec.ff, tiles=ws.tiles_gu, n_tiles=ws.n_tiles[0:1], rows_per_group=spec.in_features,
                 epilogue=gemm.EPI_STORE if spec.relu2 else gemm.EPI_SWIGLU, relu2=int(spec.relu2))
        _grouped(act, w.down.flatten(0, 1), yp, n_out=h, rows_cap=routes, bn=bn, dual=0, up_offset=0, tiles=ws.tiles_dn,
                 n_tiles=ws.n_tiles[1:2], rows_per_group=h, epilogue=gemm.EPI_STORE)
    m = native.MoeMixArgs()
    if spec.shared_ff and not fold:
        # the experts' products are done with these rows
        sact = ws.act[:rows * ceil8(spec.shared_ff)].view(rows, ceil8(spec.shared_ff))[:, :spec.shared_ff]
        _hidden_rows(x, w.shared_gate_up, sact, ws.z, spec.relu2)
        shared = ws.shared[:rows * hp].view(rows, hp)[:, :h]
        gemm.linear(sact, w.shared_down, out=shared)
        m.shared, m.ld_shared = shared.data_ptr(), shared.stride(0)
        if spec.shared_gate:
            m.shared_gate, m.ld_gate = logits[:, spec.routed:].data_ptr(), ld
    m.y, m.x, m.topk_ids, m.route_pos, m.weights, m.out = (t.data_ptr() for t in (yp, x, ws.ids, ws.route_pos, ws.weights, out))
    m.rows, m.top_k, m.hidden, m.experts, m.ld_y, m.ld_x, m.ld_out, m.f32 = rows, k, h, E, hp, x.stride(0), out.stride(0), int(f32)
    native.check(lib.xp_moe_mix(C.byref(m), s), "xp_moe_mix")
    return out
