"""Row-wise and mixer operators of layered decoders (``csrc/kernels/{row_ops,latent_attn,linear_attn,grouped_attn,
recurrence,...}.cu``): fp32 residual streams with gates or norms behind the sublayers, PolyNorm, latent attention over a paged
latent cache, grouped-query attention with capped scores, and recurrences with per-sequence states (decayed linear attention,
per-channel decays, the gated delta rule). Every operator exists for bf16 and for fp32 activations; norms, scores, gates and states are fp32 in
both. The reference borrows such layers from its serving engine (pyproject.toml:17-35).
"""

from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Sequence

import torch

from .. import native
from ..models.config import GELU_ALPHA, GELU_CUBIC, attention_shape
from . import gemm

NORM_KINDS = {"rmsnorm": 0, "layernorm": 1, "dyt": 2}
# Rows of a recurrence computed with one set of matrix products (decay powers are tabulated up to this).
LINEAR_CHUNK = 64


@dataclass
class NormParams:
    """fp32 parameters of a norm: ``alpha`` is the scalar of dynamic tanh (one element on the device)."""

    kind: str
    weight: torch.Tensor
    bias: torch.Tensor | None = None
    alpha: torch.Tensor | None = None
    eps: float = 1e-6


def _stream(t: torch.Tensor) -> int:
    return torch.cuda.current_stream(t.device).cuda_stream


def _ptr(t: torch.Tensor | None):
    return t.data_ptr() if t is not None else None


def _f32(t: torch.Tensor) -> int:
    assert t.dtype in (torch.bfloat16, torch.float32)
    return int(t.dtype == torch.float32)


def resid_norm(resid: torch.Tensor, norm: NormParams | None, out: torch.Tensor | None, *, parts: Sequence[torch.Tensor] = (),
               gate: torch.Tensor | None = None, ids: torch.Tensor | None = None, table: torch.Tensor | None = None,
               sel: torch.Tensor | None = None, rows: int | None = None, dtype: torch.dtype | None = None) -> None:
    """``resid += sum(parts) * sigmoid(gate)`` (or ``resid = table[ids]``) in fp32, then ``out = norm(resid)``.

    With ``sel`` (int32) only the selected rows are normalised and the residual is left alone. ``out=None``: residual
    update only."""
    a = native.ResidNormArgs()
    act = out if out is not None else parts[0] if parts else table
    assert resid.dtype == torch.float32 and resid.is_contiguous()
    a.resid = resid.data_ptr()
    for i, p in enumerate(parts):
        assert p.dtype == act.dtype and p.stride(1) == 1 and p.stride(0) == parts[0].stride(0)
        a.parts[i] = p.data_ptr()
    a.gate, a.ids, a.table, a.sel = _ptr(gate), _ptr(ids), _ptr(table), _ptr(sel)
    a.out = _ptr(out)
    a.rows = rows if rows is not None else (sel.shape[0] if sel is not None else resid.shape[0])
    a.hidden, a.nparts = resid.shape[1], len(parts)
    a.ld_part = parts[0].stride(0) if parts else 0
    a.ld_gate = gate.stride(0) if gate is not None else 0
    a.ld_out = out.stride(0) if out is not None else 0
    a.vocab = table.shape[0] if table is not None else 0
    if norm is not None:
        a.weight, a.bias, a.alpha, a.kind, a.eps = norm.weight.data_ptr(), _ptr(norm.bias), _ptr(norm.alpha), NORM_KINDS[norm.kind], norm.eps
    a.f32 = _f32(act)
    native.check(native.kernels().xp_resid_norm(C.byref(a), _stream(resid)), "xp_resid_norm")


def post_norm(resid: torch.Tensor, out: torch.Tensor | None, *, norm: NormParams | None = None, branches: Sequence[torch.Tensor] = (),
              branch_norms: Sequence[NormParams] = (), ids: torch.Tensor | None = None, table: torch.Tensor | None = None,
              out_norm: NormParams | None = None, sel: torch.Tensor | None = None, rows: int | None = None, eps: float = 1e-6,
              embed_scale: float = 1.0) -> None:
    """``resid += norm(branch)`` (``branch_norms``: of the mean of the normed branches; ``ids``: ``resid = table[ids] *
    embed_scale``) in fp32, then ``out = resid``, or ``out_norm(resid)``. All norms are RMS norms with ``eps``. With ``sel`` (int32) only the
    selected rows are computed and the residual is left alone."""
    a = native.PostNormArgs()
    act = branches[0] if branches else table
    assert resid.dtype == torch.float32 and resid.is_contiguous() and len(branch_norms) in (0, len(branches))
    a.resid = resid.data_ptr()
    for i, b in enumerate(branches):
        assert b.dtype == act.dtype and b.stride(1) == 1
        a.branches[i], a.ld_branch[i] = b.data_ptr(), b.stride(0)
    for i, n in enumerate(branch_norms):
        a.branch_w[i] = n.weight.data_ptr()
    a.ids, a.table, a.sel, a.out = _ptr(ids), _ptr(table), _ptr(sel), _ptr(out)
    a.weight = norm.weight.data_ptr() if norm is not None else None
    a.out_weight = out_norm.weight.data_ptr() if out_norm is not None else None
    a.rows = rows if rows is not None else (sel.shape[0] if sel is not None else resid.shape[0])
    a.hidden, a.nbranches = resid.shape[1], len(branches)
    a.ld_out = out.stride(0) if out is not None else 0
    a.vocab = table.shape[0] if table is not None else 0
    a.eps, a.f32, a.embed_scale = norm.eps if norm is not None else out_norm.eps if out_norm is not None else eps, _f32(act), embed_scale
    native.check(native.kernels().xp_post_norm(C.byref(a), _stream(resid)), "xp_post_norm")


def head_gate(o: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, eps: float, out: torch.Tensor, heads: int = 0) -> torch.Tensor:
    """``rmsnorm(o) * weight * silu(gate)`` with the norm over every head of ``len(weight)`` columns; ``o`` fp32. With
    ``heads`` the weight covers all heads and the gate is a sigmoid."""
    assert o.dtype == torch.float32 and weight.dtype == torch.float32 and gate.dtype == out.dtype
    a = native.HeadGateArgs()
    a.o, a.weight, a.gate, a.out = o.data_ptr(), weight.data_ptr(), gate.data_ptr(), out.data_ptr()
    dim = weight.numel() // heads if heads else weight.numel()
    a.rows, a.heads, a.dim, a.per_head_weight, a.sigmoid_gate = o.shape[0], o.shape[1] // dim, dim, int(heads > 0), int(heads > 0)
    a.ld_o, a.ld_gate, a.ld_out, a.eps, a.f32 = o.stride(0), gate.stride(0), out.stride(0), eps, _f32(out)
    native.check(native.kernels().xp_head_gate(C.byref(a), _stream(o)), "xp_head_gate")
    return out


def glu_f32(z: torch.Tensor, limit: float, up_add: float, alpha: float, out: torch.Tensor, cubic: float = 0.0) -> torch.Tensor:
    """Gated activation of fp32 rows ``[g, u]`` (the bf16 product applies it in its epilogue)."""
    assert z.dtype == out.dtype == torch.float32
    a = native.GluArgs()
    a.z, a.out, a.rows, a.cols, a.ld_z, a.ld_out = z.data_ptr(), out.data_ptr(), z.shape[0], z.shape[1] // 2, z.stride(0), out.stride(0)
    a.limit, a.up_add, a.alpha, a.cubic = limit, up_add, alpha, cubic
    native.check(native.kernels().xp_glu_f32(C.byref(a), _stream(z)), "xp_glu_f32")
    return out


def gelu_gate(x: torch.Tensor, w: torch.Tensor, e: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``gelu_tanh(x @ w.T) * e``. bf16: one product with the gate in its epilogue; fp32: product, then a row kernel."""
    if x.dtype == torch.bfloat16:
        return gemm.linear_gate_mul(x, w, e, out, GELU_ALPHA, GELU_CUBIC)
    gemm.linear(x, w, out=out)
    a = native.GateMulArgs()
    a.z, a.e, a.out = out.data_ptr(), e.data_ptr(), out.data_ptr()
    a.rows, a.cols, a.ld_z, a.ld_e, a.ld_out = x.shape[0], w.shape[0], out.stride(0), e.stride(0), out.stride(0)
    a.alpha, a.cubic = GELU_ALPHA, GELU_CUBIC
    native.check(native.kernels().xp_gate_mul_f32(C.byref(a), _stream(x)), "xp_gate_mul_f32")
    return out


def sigmoid_mul_f32(z: torch.Tensor, e: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``z * sigmoid(e)`` of fp32 rows (the bf16 product applies it in its epilogue); ``out`` may be ``z``."""
    return _elementwise(z, e, out, 1)


def relu2_f32(z: torch.Tensor, out: torch.Tensor) -> torch.Tensor:
    """``max(z, 0)^2`` of fp32 rows (the bf16 product applies it in its epilogue); ``out`` may be ``z``."""
    return _elementwise(z, None, out, 2)


def _elementwise(z, e, out, kind: int) -> torch.Tensor:
    assert z.dtype == out.dtype == torch.float32 and z.stride(1) == out.stride(1) == 1
    a = native.GateMulArgs()
    a.z, a.e, a.out, a.kind = z.data_ptr(), _ptr(e), out.data_ptr(), kind
    a.rows, a.cols, a.ld_z, a.ld_e, a.ld_out = z.shape[0], z.shape[1], z.stride(0), e.stride(0) if e is not None else 0, out.stride(0)
    native.check(native.kernels().xp_gate_mul_f32(C.byref(a), _stream(z)), "xp_gate_mul_f32")
    return out


def polynorm(z: torch.Tensor, coef: torch.Tensor, eps: float, out: torch.Tensor) -> torch.Tensor:
    """``c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3`` per row, ``N`` dividing by the root mean square; ``out`` may be ``z``."""
    assert coef.dtype == torch.float32 and coef.numel() == 4 and out.dtype == z.dtype
    a = native.PolyNormArgs()
    a.z, a.coef, a.out = z.data_ptr(), coef.data_ptr(), out.data_ptr()
    a.rows, a.cols, a.ld_z, a.ld_out, a.eps, a.f32 = z.shape[0], z.shape[1], z.stride(0), out.stride(0), eps, _f32(z)
    native.check(native.kernels().xp_polynorm(C.byref(a), _stream(z)), "xp_polynorm")
    return out


def gated_rms(o: torch.Tensor, weight: torch.Tensor, gate: torch.Tensor, eps: float, out: torch.Tensor) -> torch.Tensor:
    """``rmsnorm(o) * weight * sigmoid(gate)``, ``o`` fp32."""
    assert o.dtype == torch.float32 and weight.dtype == torch.float32 and gate.dtype == out.dtype
    a = native.GatedRmsArgs()
    a.o, a.weight, a.gate, a.out = o.data_ptr(), weight.data_ptr(), gate.data_ptr(), out.data_ptr()
    a.rows, a.cols = o.shape
    a.ld_o, a.ld_gate, a.ld_out, a.eps, a.f32 = o.stride(0), gate.stride(0), out.stride(0), eps, _f32(out)
    native.check(native.kernels().xp_gated_rms(C.byref(a), _stream(o)), "xp_gated_rms")
    return out


# ------------------------------------------------------------------------------------------ latent attention

def latent_prep(proj: torch.Tensor, norm_w: torch.Tensor, freq: torch.Tensor, positions: torch.Tensor, slots: torch.Tensor,
                cache: torch.Tensor, *, heads: int, dim: int, rot: int, kv_rank: int, q_off: int, kv_off: int, eps: float,
                abs_rows: int, q_plain: torch.Tensor | None, q_abs: torch.Tensor | None, q_exp: torch.Tensor | None,
                q: torch.Tensor | None = None, q_rank: int = 0, interleaved: bool = False) -> None:
    """Latent norm, rotary positions, cache write and query layouts of ``proj`` ``[rows, ...]``. ``cache`` ``[pages, page,
    1, width]``. Queries are the columns at ``q_off``, or ``q`` ``[rows, heads * (dim + rot)]``, a map of the ``q_rank`` columns at
    ``q_off`` that is divided by their root mean square here. Rows below ``abs_rows`` go to ``q_plain`` ``[heads, abs_rows, dim_p]`` and the rotary columns of ``q_abs``
    ``[heads, abs_rows, width]``; the others to ``q_exp`` ``[rows, heads, dq]`` (zero-padded)."""
    a = native.LatentPrepArgs()
    assert freq.dtype == torch.float64 and norm_w.dtype == torch.float32 and cache.dtype == proj.dtype
    a.proj, a.norm_w, a.freq, a.positions, a.slots = (t.data_ptr() for t in (proj, norm_w, freq, positions, slots))
    a.cache, a.q_plain, a.q_abs, a.q_exp = cache.data_ptr(), _ptr(q_plain), _ptr(q_abs), _ptr(q_exp)
    a.rows, a.heads, a.dim, a.rot, a.rot_dims, a.kv_rank = proj.shape[0], heads, dim, rot, 2 * freq.numel(), kv_rank
    a.ld_proj, a.q_off, a.kv_off, a.ld_cache = proj.stride(0), q_off, kv_off, cache.shape[-1]
    if q_plain is not None:
        a.qp_rows, a.dim_p, a.ld_abs = q_plain.shape[1], q_plain.shape[2], q_abs.shape[2]
    a.dq_pad = q_exp.shape[2] if q_exp is not None else 0
    a.abs_rows, a.eps, a.f32, a.interleaved = abs_rows, eps, _f32(proj), int(interleaved)
    if q is not None:
        a.q, a.ld_q, a.q_rank, a.ql_off = q.data_ptr(), q.stride(0), q_rank, q_off
    native.check(native.kernels().xp_latent_prep(C.byref(a), _stream(proj)), "xp_latent_prep")


def latent_attn_plan(rows: int, heads: int, max_len: int, width: int = 576) -> tuple[int, int]:
    """(num_splits, chunk_tokens) of the absorbed decode kernel: the split count that finishes first, counting a CTA as its
    64-token tiles plus three for start and merge, with one CTA per SM for wide cache rows and two for narrow ones."""
    ctas = rows * ((heads + 15) // 16 if heads <= 16 else (heads + 31) // 32)
    slots = 148 if width > 288 else 296
    tiles = (max_len + 63) // 64
    best, best_cost = 1, None
    for s in range(1, min(64, max(1, tiles // 2)) + 1):
        per = (tiles + s - 1) // s
        if s > 1 and (s - 1) * per >= tiles:
            continue
        cost = ((ctas * s + slots - 1) // slots) * (per + 3) + (2 if s > 1 else 0)
        if best_cost is None or cost < best_cost:
            best, best_cost = s, cost
    return (best, (tiles + best - 1) // best * 64) if best > 1 else (1, 0)


def latent_attn(q: torch.Tensor, cache: torch.Tensor, out: torch.Tensor, block_table: torch.Tensor, positions: torch.Tensor,
                slots: torch.Tensor, *, kv_rank: int, rot: int, scale: float, gate: torch.Tensor | None = None,
                row_seq: torch.Tensor | None = None, num_splits: int = 1, chunk_tokens: int = 0, ws: torch.Tensor | None = None,
                force_simt: bool = False, window: int = 0) -> torch.Tensor:
    """Rows of latent-space queries ``q`` ``[heads, rows, width]`` against the latent cache; ``out`` ``[heads, rows, >= kv_rank]``.
    Row ``r`` attends to the first ``positions[r] + 1`` tokens of its sequence (``window`` > 0: to the last ``window`` of those).
    ``force_simt`` selects the plain kernel."""
    a = native.LatentAttnArgs()
    heads, rows = q.shape[0], q.shape[1]
    a.q, a.cache, a.out, a.gate, a.row_seq = q.data_ptr(), cache.data_ptr(), out.data_ptr(), _ptr(gate), _ptr(row_seq)
    a.positions, a.slots, a.block_table, a.ws = positions.data_ptr(), slots.data_ptr(), block_table.data_ptr(), _ptr(ws)
    a.rows, a.heads, a.kv_rank, a.rot, a.q_rows = rows, heads, kv_rank, rot, rows
    a.ld_q, a.ld_cache, a.ld_out = q.shape[2], cache.shape[-1], out.shape[2]
    a.ld_gate = gate.stride(0) if gate is not None else 0
    a.page_size, a.max_blocks, a.num_splits, a.chunk_tokens = cache.shape[1], block_table.stride(0), num_splits, chunk_tokens
    assert num_splits == 1 or ws.numel() >= rows * heads * num_splits * (kv_rank + 2)
    a.scale, a.f32, a.force_simt, a.window = scale, _f32(q), int(force_simt), window
    a.status = gemm.status_words(q.device).data_ptr()
    native.check(native.kernels().xp_latent_attn(C.byref(a), _stream(q)), "xp_latent_attn", 2 if num_splits > 1 else 1)
    return out


def latent_gather(cache: torch.Tensor, out: torch.Tensor, block_table: torch.Tensor, ctx_lens: torch.Tensor, q_lens: torch.Tensor,
                  starts: torch.Tensor, max_len: int, window: int = 0) -> None:
    """Dense copies of the sequences' cached rows: sequence i's tokens start at row ``starts[i]`` of ``out``. With a ``window`` only
    those from the 64-token boundary at or before the first token that the first query sees; ``max_len`` bounds the rows of a
    sequence."""
    a = native.LatentGatherArgs()
    a.cache, a.out, a.block_table = cache.data_ptr(), out.data_ptr(), block_table.data_ptr()
    a.ctx_lens, a.q_lens, a.starts = ctx_lens.data_ptr(), q_lens.data_ptr(), starts.data_ptr()
    a.n_seqs, a.max_len, a.page_size, a.max_blocks = q_lens.shape[0], max_len, cache.shape[1], block_table.stride(0)
    a.ld_cache, a.elem_bytes, a.window = cache.shape[-1], cache.element_size(), window
    native.check(native.kernels().xp_latent_gather(C.byref(a), _stream(cache)), "xp_latent_gather")


def expanded_shape(dim: int, rot: int, vdim: int) -> tuple[int, int] | None:
    """Padded widths of the expanded (per-head keys and values) prefill form, None when no kernel covers the sizes."""
    return attention_shape(dim + rot, vdim)


def expanded_prefill(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, out: torch.Tensor, q_starts: torch.Tensor, q_lens: torch.Tensor,
                     ctx_lens: torch.Tensor, starts: torch.Tensor, max_q: int, *, scale: float, vdim: int,
                     gate: torch.Tensor | None = None, window: int = 0) -> None:
    """Causal attention of chunk queries ``q`` ``[rows, heads, dq]`` over dense per-head keys ``k`` ``[tokens, heads, dq]``
    and values ``v`` ``[tokens, heads, dv]`` (sequence i's tokens start at row ``starts[i]``, a multiple of 64; with a ``window``
    those that :func:`latent_gather` leaves); ``out`` ``[rows, heads * vdim]``, multiplied by the sigmoid of ``gate``, which has
    one column per head or one per output."""
    a = native.PrefillAttnArgs()
    a.q, a.k_cache, a.v_cache, a.out = q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr()
    a.q_starts, a.q_lens, a.ctx_lens, a.seq_starts = q_starts.data_ptr(), q_lens.data_ptr(), ctx_lens.data_ptr(), starts.data_ptr()
    a.num_seqs, a.max_q_len, a.q_heads, a.kv_heads = q_lens.shape[0], max_q, q.shape[1], k.shape[1]
    a.head_dim, a.v_dim, a.v_valid, a.ld_out = q.shape[2], v.shape[2], vdim, out.stride(0)
    a.page_size, a.max_blocks, a.num_pages = 64, 0, k.shape[0] // 64
    a.scale, a.total_q, a.p_pair = scale, q.shape[0], 1
    a.gate, a.window, a.gate_elems = _ptr(gate), window, _gate_elems(gate, a.q_heads, vdim)
    a.ld_gate = gate.stride(0) if gate is not None else 0
    a.status = gemm.status_words(q.device).data_ptr()
    lib = native.kernels()
    native.check(lib.xp_prefill_attn_umma(C.byref(a), _stream(q)), "xp_prefill_attn_umma")


# ------------------------------------------------------------------------------------------ linear attention

def decay_powers(decay: Sequence[float], chunk: int = LINEAR_CHUNK) -> torch.Tensor:
    """``decay[h] ** j`` for j = 0 .. chunk, fp32 rounded from double."""
    d = torch.tensor(list(decay), dtype=torch.float64)
    return (d[:, None] ** torch.arange(chunk + 1, dtype=torch.float64)).to(torch.float32)


def _linear_args(proj, state, decay, decay_pow, out, positions, slots, state_slots, heads, dim, vdim, offs) -> "native.LinearAttnArgs":
    assert state.dtype == torch.float32 and out.dtype == torch.float32 and decay.dtype == torch.float32
    a = native.LinearAttnArgs()
    a.proj, a.state, a.decay, a.decay_pow, a.out = (t.data_ptr() for t in (proj, state, decay, decay_pow, out))
    a.positions, a.slots, a.state_slots = positions.data_ptr(), slots.data_ptr(), state_slots.data_ptr()
    a.heads, a.dim, a.vdim, a.ld_proj = heads, dim, vdim, proj.stride(0)
    a.q_off, a.k_off, a.v_off = offs
    a.f32 = _f32(proj)
    return a


def linear_attn_decode(proj, state, decay, decay_pow, out, positions, slots, state_slots, *, heads: int, dim: int, vdim: int,
                       offs: tuple[int, int, int]) -> None:
    """One token per row: row r updates state slot ``state_slots[r]`` and writes ``out`` ``[rows, heads * vdim]`` (fp32)."""
    a = _linear_args(proj, state, decay, decay_pow, out, positions, slots, state_slots, heads, dim, vdim, offs)
    a.rows = proj.shape[0]
    native.check(native.kernels().xp_linear_attn_decode(C.byref(a), _stream(proj)), "xp_linear_attn_decode")


def linear_attn_plan(seqs: int, heads: int, dim: int, vdim: int, max_q: int) -> tuple[int, int]:
    """(segments, tokens per segment) of the chunked prefill: enough CTAs for the 148 SMs when sequences and heads are few.
    A segmented run reads keys and values twice and passes its states through memory."""
    slices = (vdim + 127) // 128 if dim <= 128 else (vdim + 31) // 32
    ctas, chunks = seqs * heads * slices, (max_q + LINEAR_CHUNK - 1) // LINEAR_CHUNK
    best, best_cost = 1, None
    for s in range(1, min(chunks, 64) + 1):
        per = (chunks + s - 1) // s
        if s > 1 and (ctas * s > 2 * 148 or (s - 1) * per >= chunks):
            continue
        cost = ((ctas * s + 147) // 148) * per * (1.0 if s == 1 else 1.4) + (0 if s == 1 else 4)
        if best_cost is None or cost < best_cost:
            best, best_cost = s, cost
    return best, (chunks + best - 1) // best * LINEAR_CHUNK


def linear_attn_ws_elems(dim: int, vdim: int) -> int:
    """Bound on the workspace of any plan (fp32 elements)."""
    return 2 * 148 * dim * vdim


def linear_attn_prefill(proj, state, decay, decay_pow, out, positions, slots, state_slots, q_starts, q_lens, *, heads: int,
                        dim: int, vdim: int, offs: tuple[int, int, int], force_sequential: bool = False, segs: int = 1, seg_tokens: int = 0,
                        ws: torch.Tensor | None = None) -> None:
    """Portions of sequences: portion i covers rows ``q_starts[i] .. + q_lens[i]`` and continues state ``state_slots[i]``.
    ``segs`` and ``seg_tokens`` as planned for the longest portion (:func:`linear_attn_plan`), with ``ws`` of
    ``seqs * heads * segs * dim * vdim`` fp32 elements when ``segs`` > 1."""
    a = _linear_args(proj, state, decay, decay_pow, out, positions, slots, state_slots, heads, dim, vdim, offs)
    a.q_starts, a.q_lens, a.seqs = q_starts.data_ptr(), q_lens.data_ptr(), q_lens.shape[0]
    a.rows, a.force_sequential = proj.shape[0], int(force_sequential)
    if segs > 1 and a.f32 == 0 and not force_sequential:
        assert ws is not None and ws.numel() >= q_lens.shape[0] * heads * segs * dim * vdim
        a.segs, a.seg_tokens, a.ws = segs, seg_tokens, ws.data_ptr()
    native.check(native.kernels().xp_linear_attn_prefill(C.byref(a), _stream(proj)), "xp_linear_attn_prefill", 3 if a.segs > 1 else 1)


# ------------------------------------------------------------------------------------------ grouped-query attention

def group_pad(heads: int, kv_heads: int) -> int:
    """Query heads of a group rounded up to a power of two (the tiles of the prefill kernel)."""
    n = 1
    while n < heads // kv_heads:
        n *= 2
    return n


@dataclass
class BlockMeans:
    """Means of whole blocks of ``size`` cached tokens, keys and values ``[pages, rows beside a page, kv_heads, width]``: block b of a
    sequence is row ``b % rows`` beside page ``b // rows`` of its table."""

    k: torch.Tensor
    v: torch.Tensor
    size: int

    def put(self, a) -> None:
        a.k_pool, a.v_pool, a.pool, a.pool_page = self.k.data_ptr(), self.v.data_ptr(), self.size, self.k.shape[1]


def grouped_prep(proj: torch.Tensor, q_norm: torch.Tensor | None, k_norm: torch.Tensor | None, slots: torch.Tensor, k_cache: torch.Tensor,
                 v_cache: torch.Tensor, q_out: torch.Tensor, *, heads: int, dim: int, vdim: int, offs: tuple[int, int, int], eps: float,
                 unit: bool = False, rot: torch.Tensor | None = None, interleaved: bool = False, positions: torch.Tensor | None = None,
                 pool: BlockMeans | None = None, pool_rows: int = 0, block_table: torch.Tensor | None = None) -> None:
    """Query and key norms (with weights, or ``unit`` without any), rotation (``rot`` fp32 ``[positions, pairs, 2]``), cache
    write and the padded query layout ``q_out`` ``[rows, kv_heads, group_pad, dq]``; caches ``[pages, page, kv_heads, dq]`` and
    ``[..., dv]``. The first ``pool_rows`` rows (row r is sequence r) store the block means that they complete."""
    assert k_cache.dtype == proj.dtype == q_out.dtype and (q_norm is None or q_norm.dtype == torch.float32)
    a = native.GroupedPrepArgs()
    a.proj, a.q_norm, a.k_norm, a.slots = proj.data_ptr(), _ptr(q_norm), _ptr(k_norm), slots.data_ptr()
    a.k_cache, a.v_cache, a.q_out = k_cache.data_ptr(), v_cache.data_ptr(), q_out.data_ptr()
    a.rows, a.heads, a.kv_heads, a.group_pad = proj.shape[0], heads, k_cache.shape[2], q_out.shape[2]
    a.dim, a.vdim, a.dq, a.dv, a.ld_proj = dim, vdim, k_cache.shape[3], v_cache.shape[3], proj.stride(0)
    a.q_off, a.k_off, a.v_off = offs
    a.eps, a.f32, a.norm, a.interleaved, a.positions = eps, _f32(proj), int(unit or q_norm is not None), int(interleaved), _ptr(positions)
    if rot is not None:
        assert rot.dtype == torch.float32
        a.rot, a.rot_positions, a.rot_pairs = rot.data_ptr(), rot.shape[0], rot.shape[1]
    if pool is not None and pool_rows:
        pool.put(a)
        a.pool_rows, a.block_table, a.page_size, a.max_blocks = pool_rows, block_table.data_ptr(), k_cache.shape[1], block_table.stride(0)
    native.check(native.kernels().xp_grouped_prep(C.byref(a), _stream(proj)), "xp_grouped_prep")


def block_means(k_cache: torch.Tensor, v_cache: torch.Tensor, pool: BlockMeans, block_table: torch.Tensor, positions: torch.Tensor,
                slots: torch.Tensor, row_seq: torch.Tensor | None = None) -> None:
    """Every row whose position completes a block stores the means of the block's cached keys and values."""
    a = native.BlockMeanArgs()
    a.k_cache, a.v_cache, a.row_seq, a.positions, a.slots = k_cache.data_ptr(), v_cache.data_ptr(), _ptr(row_seq), positions.data_ptr(), slots.data_ptr()
    a.block_table, a.rows, a.kv_heads, a.dq, a.dv = block_table.data_ptr(), positions.shape[0], k_cache.shape[2], k_cache.shape[3], v_cache.shape[3]
    a.page_size, a.max_blocks, a.f32 = k_cache.shape[1], block_table.stride(0), _f32(k_cache)
    pool.put(a)
    native.check(native.kernels().xp_block_mean(C.byref(a), _stream(k_cache)), "xp_block_mean")


def _score_forms(a, heads: int, sink: torch.Tensor | None, sigmoid_bias: torch.Tensor | None, pool: BlockMeans | None) -> None:
    for t in (sink, sigmoid_bias):
        assert t is None or t.dtype == torch.float32 and t.numel() == heads
    a.sink, a.sigmoid_bias = _ptr(sink), _ptr(sigmoid_bias)
    if pool is not None:
        pool.put(a)


def _gate_elems(gate: torch.Tensor | None, heads: int, vdim: int) -> int:
    """Whether a gate has one logit per output element: as many columns as the output, and more than heads."""
    return int(gate is not None and vdim > 1 and gate.shape[1] == heads * vdim)


def conv_rope(proj: torch.Tensor, conv_w: torch.Tensor | None, ring: torch.Tensor | None, rot: torch.Tensor | None, positions: torch.Tensor,
              slots: torch.Tensor, state_slots: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, q_out: torch.Tensor, *, heads: int,
              dim: int, vdim: int, offs: tuple[int, ...], q_starts: torch.Tensor | None = None, q_lens: torch.Tensor | None = None,
              max_q: int = 0) -> None:
    """Convolution over time (``conv_w`` fp32 ``[taps, channels]``, inputs behind every sequence in ``ring`` ``[slots, taps,
    channels]``), rotation (``rot`` fp32 ``[positions, pairs, 2]``), cache write and the padded query layout ``q_out`` ``[rows,
    kv_heads, group_pad, dq]``. ``offs``: columns of q, k, v in ``proj``, or of q alone (nothing is cached). One token per row,
    or with ``q_lens`` the portions that start at rows ``q_starts``."""
    a = native.ConvRopeArgs()
    assert k_cache.dtype == proj.dtype == q_out.dtype and (rot is None or rot.dtype == torch.float32)
    a.proj, a.conv_w, a.ring, a.rot = proj.data_ptr(), _ptr(conv_w), _ptr(ring), _ptr(rot)
    a.positions, a.slots, a.state_slots = positions.data_ptr(), slots.data_ptr(), state_slots.data_ptr()
    a.k_cache, a.v_cache, a.q_out = k_cache.data_ptr(), v_cache.data_ptr(), q_out.data_ptr()
    a.rows, a.heads, a.kv_heads, a.group_pad = proj.shape[0], heads, k_cache.shape[2], q_out.shape[2]
    a.dim, a.vdim, a.dq, a.dv, a.ld_proj, a.own_kv = dim, vdim, k_cache.shape[3], v_cache.shape[3], proj.stride(0), int(len(offs) == 3)
    a.q_off, a.k_off, a.v_off = offs if len(offs) == 3 else (offs[0], 0, 0)
    if conv_w is not None:
        assert conv_w.dtype == torch.float32 and conv_w.is_contiguous() and ring.dtype == proj.dtype and tuple(conv_w.shape) == tuple(ring.shape[1:])
        a.taps = conv_w.shape[0]
    if rot is not None:
        a.rot_positions, a.rot_pairs = rot.shape[0], rot.shape[1]
    a.f32 = _f32(proj)
    lib = native.kernels()
    if q_lens is None:
        native.check(lib.xp_conv_rope_decode(C.byref(a), _stream(proj)), "xp_conv_rope_decode")
        return
    a.q_starts, a.q_lens, a.seqs, a.max_q = q_starts.data_ptr(), q_lens.data_ptr(), q_lens.shape[0], max_q
    native.check(lib.xp_conv_rope_prefill(C.byref(a), _stream(proj)), "xp_conv_rope_prefill")


def grouped_attn(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor, block_table: torch.Tensor,
                 positions: torch.Tensor, slots: torch.Tensor, *, heads: int, dim: int, vdim: int, scale: float, softcap: float = 0.0,
                 gate: torch.Tensor | None = None, row_seq: torch.Tensor | None = None, window: int = 0, keep_first: int = 0,
                 sink: torch.Tensor | None = None, sigmoid_bias: torch.Tensor | None = None, pool: BlockMeans | None = None) -> torch.Tensor:
    """Rows of queries ``[rows, kv_heads, group_pad, dq]`` against the first ``positions[r] + 1`` cached tokens of their
    sequences (``window`` > 0: the last ``window`` of those and the first ``keep_first``, or with ``pool`` the means of the blocks
    behind the window), any sizes and types; ``out`` ``[rows, heads * vdim]``, multiplied by the sigmoid of ``gate``, which has one
    column per head or one per output. ``sink``: a number per head that joins the softmax's sum; ``sigmoid_bias``: weights are
    ``sigmoid(score + bias)``, not normalised."""
    step = 32768
    for lo in range(0, q.shape[0], step):
        n = min(step, q.shape[0] - lo)
        a = native.GroupedAttnArgs()
        a.q, a.k_cache, a.v_cache, a.out = q[lo:].data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out[lo:].data_ptr()
        a.gate = gate[lo:].data_ptr() if gate is not None else None
        a.row_seq = row_seq[lo:].data_ptr() if row_seq is not None else None
        a.positions, a.slots = positions[lo:].data_ptr(), slots[lo:].data_ptr()
        a.block_table = block_table[lo:].data_ptr() if row_seq is None else block_table.data_ptr()
        a.rows, a.heads, a.kv_heads, a.group_pad, a.dim, a.vdim = n, heads, q.shape[1], q.shape[2], dim, vdim
        a.dq, a.dv, a.ld_gate, a.ld_out = q.shape[3], v_cache.shape[3], gate.stride(0) if gate is not None else 0, out.stride(0)
        a.page_size, a.max_blocks, a.scale, a.softcap, a.f32 = k_cache.shape[1], block_table.stride(0), scale, softcap, _f32(q)
        a.window, a.keep_first, a.gate_elems = window, keep_first, _gate_elems(gate, heads, vdim)
        _score_forms(a, heads, sink, sigmoid_bias, pool)
        native.check(native.kernels().xp_grouped_attn(C.byref(a), _stream(q)), "xp_grouped_attn")
    return out


def grouped_decode(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor, block_table: torch.Tensor,
                   positions: torch.Tensor, slots: torch.Tensor, *, heads: int, dim: int, vdim: int, scale: float, softcap: float = 0.0,
                   gate: torch.Tensor | None = None, row_seq: torch.Tensor | None = None, num_splits: int = 1, chunk_tokens: int = 0,
                   ws: torch.Tensor | None = None, window: int = 0, keep_first: int = 0, sink: torch.Tensor | None = None,
                   sigmoid_bias: torch.Tensor | None = None, pool: BlockMeans | None = None) -> torch.Tensor:
    """:func:`grouped_attn` on the tensor cores (bf16, widths of ``ATTENTION_SHAPES``, at most 16 query heads per key head).
    ``ws``: fp32, ``rows * heads * num_splits * (dv + 2)`` elements when ``num_splits`` > 1."""
    r = native.DecodeRowsArgs()
    a = r.a
    a.q, a.k_cache, a.v_cache, a.out, a.ws = q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), _ptr(ws)
    assert q.dtype == out.dtype == torch.bfloat16 and (num_splits == 1 or ws.numel() >= q.shape[0] * heads * num_splits * (v_cache.shape[3] + 2))
    a.block_table, a.batch, a.q_heads, a.kv_heads, a.head_dim = block_table.data_ptr(), q.shape[0], heads, q.shape[1], q.shape[3]
    a.page_size, a.max_blocks, a.num_splits, a.chunk_tokens, a.num_pages = k_cache.shape[1], block_table.stride(0), num_splits, chunk_tokens, k_cache.shape[0]
    a.scale, a.status = scale, gemm.status_words(q.device).data_ptr()
    r.row_seq, r.positions, r.slots, r.gate = _ptr(row_seq), positions.data_ptr(), slots.data_ptr(), _ptr(gate)
    r.group_pad, r.v_dim, r.v_valid, r.ld_out, r.softcap = q.shape[2], v_cache.shape[3], vdim, out.stride(0), softcap
    r.ld_gate = gate.stride(0) if gate is not None else 0
    r.window, r.keep_first, r.gate_elems = window, keep_first, _gate_elems(gate, heads, vdim)
    _score_forms(r, heads, sink, sigmoid_bias, pool)
    native.check(native.kernels().xp_decode_rows(C.byref(r), _stream(q)), "xp_decode_rows", 2 if num_splits > 1 else 1)
    return out


def grouped_prefill(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, out: torch.Tensor, block_table: torch.Tensor,
                    q_starts: torch.Tensor, q_lens: torch.Tensor, ctx_lens: torch.Tensor, max_q: int, *, heads: int, vdim: int, scale: float,
                    softcap: float = 0.0, gate: torch.Tensor | None = None, window: int = 0, keep_first: int = 0, sink: torch.Tensor | None = None,
                    sigmoid_bias: torch.Tensor | None = None, pool: BlockMeans | None = None) -> torch.Tensor:
    """Causal attention of portions (rows of ``q`` ``[rows, kv_heads, group_pad, dq]``) over the paged cache, which holds the
    portions' own tokens already, on tcgen05; ``out`` ``[rows, heads * vdim]``."""
    a = native.PrefillAttnArgs()
    a.q, a.k_cache, a.v_cache, a.out, a.block_table = (t.data_ptr() for t in (q, k_cache, v_cache, out, block_table))
    a.q_starts, a.q_lens, a.ctx_lens = q_starts.data_ptr(), q_lens.data_ptr(), ctx_lens.data_ptr()
    a.num_seqs, a.max_q_len, a.kv_heads, a.q_heads = q_lens.shape[0], max_q, q.shape[1], q.shape[1] * q.shape[2]
    a.head_dim, a.v_dim, a.v_valid, a.ld_out = q.shape[3], v_cache.shape[3], vdim, out.stride(0)
    a.page_size, a.max_blocks, a.num_pages = k_cache.shape[1], block_table.stride(0), k_cache.shape[0]
    a.scale, a.total_q, a.p_pair, a.group_valid, a.softcap = scale, q.shape[0], 1, heads // q.shape[1], softcap
    a.gate, a.ld_gate = _ptr(gate), gate.stride(0) if gate is not None else 0
    a.window, a.keep_first, a.gate_elems = window, keep_first, _gate_elems(gate, heads, vdim)
    _score_forms(a, heads, sink, sigmoid_bias, pool)
    a.status = gemm.status_words(q.device).data_ptr()
    native.check(native.kernels().xp_prefill_attn_umma(C.byref(a), _stream(q)), "xp_prefill_attn_umma")
    return out


# ------------------------------------------------------------------------------------------ input-dependent recurrences

def _recurrent(a, proj, state, out, positions, slots, state_slots, heads, dim, vdim):
    assert state.dtype == torch.float32
    a.proj, a.state, a.out, a.positions, a.slots, a.state_slots = (t.data_ptr() for t in (proj, state, out, positions, slots, state_slots))
    a.heads, a.dim, a.vdim, a.ld_proj, a.ld_out, a.f32, a.rows = heads, dim, vdim, proj.stride(0), out.stride(0), _f32(proj), proj.shape[0]
    return a


def gated_linear_decode(proj, state, a2, a2_bias, norm, out, positions, slots, state_slots, *, heads: int, dim: int, vdim: int,
                        offs: tuple[int, int, int, int, int], tau: float, eps: float) -> None:
    """One token per row from the projection (q, k, v, gate and the decay's first map at ``offs``) to the gated heads
    ``out`` ``[rows, heads * vdim]``; row r updates state slot ``state_slots[r]``."""
    a = _recurrent(native.GatedLinearArgs(), proj, state, out, positions, slots, state_slots, heads, dim, vdim)
    assert a2.dtype == proj.dtype == out.dtype and a2_bias.dtype == norm.dtype == torch.float32
    a.a2, a.a2_bias, a.norm = a2.data_ptr(), a2_bias.data_ptr(), norm.data_ptr()
    a.q_off, a.k_off, a.v_off, a.g_off, a.a_off = offs
    a.rank, a.ld_a2, a.inv_tau, a.qscale, a.eps = a2.shape[1], a2.stride(0), 1.0 / tau, dim ** -0.5, eps
    native.check(native.kernels().xp_gated_linear_decode(C.byref(a), _stream(proj)), "xp_gated_linear_decode")


def gated_linear_plan(seqs: int, heads: int, vdim: int, max_q: int) -> tuple[int, int]:
    """(segments, tokens per segment) of the chunked prefill: enough CTAs for the 148 SMs when sequences and heads are few. A
    segmented run walks the chunks twice, the first time without outputs."""
    slices = (vdim + 63) // 64
    ctas, chunks = seqs * heads * slices, (max_q + LINEAR_CHUNK - 1) // LINEAR_CHUNK
    best, best_cost = 1, None
    for s in range(1, min(chunks, 64) + 1):
        per = (chunks + s - 1) // s
        if s > 1 and (ctas * s > 2 * 148 or (s - 1) * per >= chunks):
            continue
        cost = ((ctas * s + 147) // 148) * per * (1.0 if s == 1 else 1.6) + (0 if s == 1 else 4)
        if best_cost is None or cost < best_cost:
            best, best_cost = s, cost
    return best, (chunks + best - 1) // best * LINEAR_CHUNK


@dataclass
class GatedLinearScratch:
    """What the chunked prefill kernels hand on: scores of every (chunk, head), states and decays between segments."""

    records: torch.Tensor
    ws: torch.Tensor

    @classmethod
    def for_rows(cls, rows: int, seqs: int, heads: int, dim: int, vdim: int, device) -> "GatedLinearScratch":
        """For batches of at most ``rows`` rows in ``seqs`` portions; any plan of :func:`gated_linear_plan` fits."""
        n = native.kernels().xp_gated_linear_record_bytes(rows, seqs, heads)
        return cls(torch.zeros(n, dtype=torch.uint8, device=device), torch.zeros(2 * 148 * dim * (vdim + 1), dtype=torch.float32, device=device))


def gated_linear_prefill(proj, z, state, out, positions, slots, state_slots, q_starts, q_lens, max_q: int, scratch: GatedLinearScratch | None,
                         *, heads: int, dim: int, vdim: int, offs: tuple[int, int, int], tau: float, segs: int = 1, seg_tokens: int = 0,
                         force_sequential: bool = False) -> None:
    """Portions of sequences (the longest has ``max_q`` rows): portion i covers rows ``q_starts[i] .. + q_lens[i]`` and
    continues state ``state_slots[i]``; ``z`` fp32 ``[rows, heads * dim]`` is the decay map's value and is used up, ``out`` fp32
    ``[rows, heads * vdim]``. ``segs`` and ``seg_tokens`` as planned. bf16 rows with widths in multiples of 8 and at most 128
    key dimensions run the chunked tensor-core kernels when there is ``scratch``, everything else the sequential kernel."""
    a = _recurrent(native.GatedLinearArgs(), proj, state, out, positions, slots, state_slots, heads, dim, vdim)
    assert z.dtype == out.dtype == torch.float32 and z.is_contiguous()
    a.z, a.q_starts, a.q_lens, a.seqs, a.max_q = z.data_ptr(), q_starts.data_ptr(), q_lens.data_ptr(), q_lens.shape[0], max_q
    a.q_off, a.k_off, a.v_off = offs
    a.inv_tau, a.qscale, a.force_sequential = 1.0 / tau, dim ** -0.5, int(force_sequential)
    n = 1
    if scratch is not None:
        a.records, a.segs, a.seg_tokens, a.ws = scratch.records.data_ptr(), segs, seg_tokens, scratch.ws.data_ptr()
        assert segs <= 1 or scratch.ws.numel() >= q_lens.shape[0] * heads * segs * dim * (vdim + 1)
        n = 4 if segs > 1 else 2
    native.check(native.kernels().xp_gated_linear_prefill(C.byref(a), _stream(proj)), "xp_gated_linear_prefill", n)


@dataclass
class MemoryScratch:
    """What the prefill kernels hand on: the gates of every (token, head), key sums and maxima before every portion, states
    between segments."""

    planes: torch.Tensor
    before: torch.Tensor
    ws: torch.Tensor

    @classmethod
    def for_rows(cls, rows: int, seqs: int, heads: int, dim: int, vdim: int, device) -> "MemoryScratch":
        """For batches of at most ``rows`` rows in ``seqs`` portions; any plan of :func:`linear_attn_plan` fits."""
        return cls(*(torch.zeros(n, dtype=torch.float32, device=device)
                     for n in (3 * heads * rows, seqs * heads * (dim + 1), 2 * 148 * (dim * (vdim + 1) + 4))))


def _memory(proj, gates, state, out, positions, slots, state_slots, heads, dim, vdim, offs, cap) -> "native.MemoryArgs":
    assert gates.dtype == torch.float32 and state.shape[1] == heads and state.is_contiguous()
    a = _recurrent(native.MemoryArgs(), proj, state, out, positions, slots, state_slots, heads, dim, vdim)
    a.gates, a.ld_gates, a.head_state, a.cap, a.qscale = gates.data_ptr(), gates.stride(0), state.shape[2], cap, dim ** -0.5
    a.q_off, a.k_off, a.v_off, a.g_off, a.i_off, a.f_off = offs
    return a


def memory_decode(proj, gates, state, norm, out, positions, slots, state_slots, *, heads: int, dim: int, vdim: int,
                  offs: tuple[int, int, int, int, int, int], cap: float, eps: float) -> None:
    """One token per row from the projection (q, k, v, output gate in ``proj``, input and forget gate in the fp32 rows of
    ``gates``, at ``offs``) to the normed and gated heads ``out``; row r updates state slot ``state_slots[r]``."""
    a = _memory(proj, gates, state, out, positions, slots, state_slots, heads, dim, vdim, offs, cap)
    assert out.dtype == proj.dtype and norm.dtype == torch.float32 and norm.numel() == heads * vdim
    a.norm, a.eps = norm.data_ptr(), eps
    native.check(native.kernels().xp_memory_decode(C.byref(a), _stream(proj)), "xp_memory_decode")


def memory_prefill(proj, gates, state, out, positions, slots, state_slots, q_starts, q_lens, max_q: int, scratch: MemoryScratch, *, heads: int,
                   dim: int, vdim: int, offs: tuple[int, int, int, int, int, int], cap: float, segs: int = 1, seg_tokens: int = 0,
                   force_sequential: bool = False) -> None:
    """Portions of sequences (the longest has ``max_q`` rows) continue state ``state_slots[i]``; ``out`` fp32 ``[rows, heads *
    vdim]``. bf16 rows with widths in multiples of 8 and at most 256 key dimensions run the chunked tensor-core kernel, with
    ``segs`` and ``seg_tokens`` as planned for the longest portion (:func:`linear_attn_plan`)."""
    a = _memory(proj, gates, state, out, positions, slots, state_slots, heads, dim, vdim, offs, cap)
    n = q_lens.shape[0]
    assert out.dtype == torch.float32 and scratch.planes.numel() >= 3 * heads * proj.shape[0] and scratch.before.numel() >= n * heads * (dim + 1)
    a.planes, a.before, a.ws = scratch.planes.data_ptr(), scratch.before.data_ptr(), scratch.ws.data_ptr()
    a.q_starts, a.q_lens, a.seqs, a.max_q, a.force_sequential = q_starts.data_ptr(), q_lens.data_ptr(), n, max_q, int(force_sequential)
    if segs > 1 and not a.f32 and not force_sequential:
        assert scratch.ws.numel() >= n * heads * segs * state.shape[2]
        a.segs, a.seg_tokens = segs, seg_tokens
    native.check(native.kernels().xp_memory_prefill(C.byref(a), _stream(proj)), "xp_memory_prefill", 4 if a.segs > 1 else 2)


@dataclass
class DeltaWeights:
    """Parameters of the gated delta rule around its projections, fp32: convolution ``[channels, taps]`` over queries, keys
    and values, ``-exp(A_log)`` and the step bias per head, the output norm ``[vdim]``."""

    conv: torch.Tensor
    neg_a: torch.Tensor
    dt_bias: torch.Tensor
    norm: torch.Tensor


@dataclass
class DeltaScratch:
    """What the prefill kernels hand on: convolved rows, unit-vector factors, ``beta`` and ``log g``, and the solved systems
    of every (chunk, head)."""

    qkv: torch.Tensor
    qk_scale: torch.Tensor
    beta_g: torch.Tensor
    ws: torch.Tensor | None = None

    @classmethod
    def for_rows(cls, rows: int, seqs: int, heads: int, kv_heads: int, dim: int, vdim: int, dtype: torch.dtype, device) -> "DeltaScratch":
        """For batches of at most ``rows`` rows in ``seqs`` portions."""
        def buf(n, dt):
            return torch.zeros(n, dtype=dt, device=device)

        ws = buf(native.kernels().xp_delta_ws_bytes(rows, seqs, heads), torch.uint8) if dtype == torch.bfloat16 else None
        return cls(buf(rows * (2 * kv_heads * dim + heads * vdim), dtype), buf(rows * 2 * kv_heads, torch.float32),
                   buf(rows * 2 * heads, torch.float32), ws)


def _delta(proj, conv_state, w: DeltaWeights, state, out, positions, slots, state_slots, heads, kv_heads, dim, vdim, offs, eps):
    a = _recurrent(native.DeltaArgs(), proj, state, out, positions, slots, state_slots, heads, dim, vdim)
    assert conv_state.dtype == proj.dtype and w.conv.dtype == torch.float32
    a.conv_w, a.conv_state, a.neg_a, a.dt_bias, a.norm = (t.data_ptr() for t in (w.conv, conv_state, w.neg_a, w.dt_bias, w.norm))
    a.kv_heads, a.taps, a.qscale, a.eps = kv_heads, w.conv.shape[1], dim ** -0.5, eps
    a.q_off, a.k_off, a.v_off, a.g_off, a.b_off, a.a_off = offs
    return a


def delta_decode(proj, conv_state, w: DeltaWeights, state, out, positions, slots, state_slots, *, heads: int, kv_heads: int, dim: int,
                 vdim: int, offs: tuple[int, int, int, int, int, int], eps: float) -> None:
    """One token per row from the projection (q, k, v, gate, b, a at ``offs``) to the gated heads ``out``; row r updates
    state and convolution slot ``state_slots[r]``."""
    a = _delta(proj, conv_state, w, state, out, positions, slots, state_slots, heads, kv_heads, dim, vdim, offs, eps)
    assert out.dtype == proj.dtype
    native.check(native.kernels().xp_delta_decode(C.byref(a), _stream(proj)), "xp_delta_decode")


def delta_prefill(proj, conv_state, w: DeltaWeights, state, out, positions, slots, state_slots, q_starts, q_lens, max_q: int,
                  scratch: DeltaScratch, *, heads: int, kv_heads: int, dim: int, vdim: int, offs: tuple[int, int, int, int, int, int],
                  eps: float, force_sequential: bool = False) -> None:
    """Portions of sequences (the longest has ``max_q`` rows): convolution and recurrence; ``out`` fp32 ``[rows, heads * vdim]``.
    bf16 rows with widths in multiples of 8 and at most 128 key dimensions run the chunked tensor-core kernels."""
    a = _delta(proj, conv_state, w, state, out, positions, slots, state_slots, heads, kv_heads, dim, vdim, offs, eps)
    assert out.dtype == torch.float32 and scratch.qkv.dtype == proj.dtype
    a.qkv, a.qk_scale, a.beta_g = scratch.qkv.data_ptr(), scratch.qk_scale.data_ptr(), scratch.beta_g.data_ptr()
    a.ws = _ptr(scratch.ws)
    a.q_starts, a.q_lens, a.seqs, a.max_q, a.force_sequential = q_starts.data_ptr(), q_lens.data_ptr(), q_lens.shape[0], max_q, int(force_sequential)
    lib = native.kernels()
    native.check(lib.xp_delta_prep(C.byref(a), _stream(proj)), "xp_delta_prep")
    native.check(lib.xp_delta_prefill(C.byref(a), _stream(proj)), "xp_delta_prefill", 1 if scratch.ws is None else 2)
