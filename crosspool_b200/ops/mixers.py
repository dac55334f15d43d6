"""Row-wise and mixer operators of layered decoders (``csrc/kernels/{row_ops,latent_attn,linear_attn}.cu``): gated fp32
residual streams with a fused norm, PolyNorm, latent attention over a paged latent cache, decayed linear attention with
per-sequence states. Every operator exists for bf16 and for fp32 activations; norms, scores, gates and states are fp32 in
both. The reference borrows such layers from its serving engine (pyproject.toml:17-35).
"""

from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Sequence

import torch

from .. import native

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
                abs_rows: int, q_plain: torch.Tensor | None, q_abs: torch.Tensor | None, q_exp: torch.Tensor | None) -> None:
    """Latent norm, rotary positions, cache write and query layouts of ``proj`` ``[rows, ...]``. ``cache`` ``[pages, page,
    1, width]``. Rows below ``abs_rows`` go to ``q_plain`` ``[heads, abs_rows, dim_p]`` and the rotary columns of ``q_abs``
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
    a.abs_rows, a.eps, a.f32 = abs_rows, eps, _f32(proj)
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
                force_simt: bool = False) -> torch.Tensor:
    """Rows of latent-space queries ``q`` ``[heads, rows, width]`` against the latent cache; ``out`` ``[heads, rows, >= kv_rank]``.
    Row ``r`` attends to the first ``positions[r] + 1`` tokens of its sequence. ``force_simt`` selects the plain kernel."""
    a = native.LatentAttnArgs()
    heads, rows = q.shape[0], q.shape[1]
    a.q, a.cache, a.out, a.gate, a.row_seq = q.data_ptr(), cache.data_ptr(), out.data_ptr(), _ptr(gate), _ptr(row_seq)
    a.positions, a.slots, a.block_table, a.ws = positions.data_ptr(), slots.data_ptr(), block_table.data_ptr(), _ptr(ws)
    a.rows, a.heads, a.kv_rank, a.rot, a.q_rows = rows, heads, kv_rank, rot, rows
    a.ld_q, a.ld_cache, a.ld_out = q.shape[2], cache.shape[-1], out.shape[2]
    a.ld_gate = gate.stride(0) if gate is not None else 0
    a.page_size, a.max_blocks, a.num_splits, a.chunk_tokens = cache.shape[1], block_table.stride(0), num_splits, chunk_tokens
    assert num_splits == 1 or ws.numel() >= rows * heads * num_splits * (kv_rank + 2)
    a.scale, a.f32, a.force_simt = scale, _f32(q), int(force_simt)
    from .gemm import status_words

    a.status = status_words(q.device).data_ptr()
    native.check(native.kernels().xp_latent_attn(C.byref(a), _stream(q)), "xp_latent_attn", 2 if num_splits > 1 else 1)
    return out


def latent_gather(cache: torch.Tensor, out: torch.Tensor, block_table: torch.Tensor, ctx_lens: torch.Tensor, q_lens: torch.Tensor,
                  starts: torch.Tensor, max_len: int) -> None:
    """Dense copies of the sequences' cached rows: sequence i's tokens start at row ``starts[i]`` of ``out``."""
    a = native.LatentGatherArgs()
    a.cache, a.out, a.block_table = cache.data_ptr(), out.data_ptr(), block_table.data_ptr()
    a.ctx_lens, a.q_lens, a.starts = ctx_lens.data_ptr(), q_lens.data_ptr(), starts.data_ptr()
    a.n_seqs, a.max_len, a.page_size, a.max_blocks = q_lens.shape[0], max_len, cache.shape[1], block_table.stride(0)
    a.ld_cache, a.elem_bytes = cache.shape[-1], cache.element_size()
    native.check(native.kernels().xp_latent_gather(C.byref(a), _stream(cache)), "xp_latent_gather")


# tcgen05 prefill shapes (query/key width, value width), narrowest first
EXPANDED_SHAPES = ((64, 64), (128, 64), (128, 128), (192, 128))


def expanded_shape(dim: int, rot: int, vdim: int) -> tuple[int, int] | None:
    """Padded widths of the expanded (per-head keys and values) prefill form, None when no kernel covers the sizes."""
    if vdim % 8:
        return None
    for dq, dv in EXPANDED_SHAPES:
        if dim + rot <= dq and vdim <= dv:
            return dq, dv
    return None


def expanded_prefill(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, out: torch.Tensor, q_starts: torch.Tensor, q_lens: torch.Tensor,
                     ctx_lens: torch.Tensor, starts: torch.Tensor, max_q: int, *, scale: float, vdim: int,
                     gate: torch.Tensor | None = None) -> None:
    """Causal attention of chunk queries ``q`` ``[rows, heads, dq]`` over dense per-head keys ``k`` ``[tokens, heads, dq]``
    and values ``v`` ``[tokens, heads, dv]`` (sequence i's tokens start at row ``starts[i]``, a multiple of 64); ``out``
    ``[rows, heads * vdim]``, head h multiplied by ``sigmoid(gate[:, h])``."""
    from .gemm import status_words

    a = native.PrefillAttnArgs()
    a.q, a.k_cache, a.v_cache, a.out = q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr()
    a.q_starts, a.q_lens, a.ctx_lens, a.seq_starts = q_starts.data_ptr(), q_lens.data_ptr(), ctx_lens.data_ptr(), starts.data_ptr()
    a.num_seqs, a.max_q_len, a.q_heads, a.kv_heads = q_lens.shape[0], max_q, q.shape[1], k.shape[1]
    a.head_dim, a.v_dim, a.v_valid, a.ld_out = q.shape[2], v.shape[2], vdim, out.stride(0)
    a.page_size, a.max_blocks, a.num_pages = 64, 0, k.shape[0] // 64
    a.scale, a.total_q, a.p_pair = scale, q.shape[0], 1
    a.gate = _ptr(gate)
    a.ld_gate = gate.stride(0) if gate is not None else 0
    a.status = status_words(q.device).data_ptr()
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
