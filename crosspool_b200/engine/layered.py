"""Forward pass of layered decoders inside :class:`AttentionEngine`: every layer brings its own mixer.

One batch (:class:`RowBatch`) holds single decoded tokens first, then portions of prompts. The products and row kernels run
over all rows together; a mixer splits the rows where its decode and prefill kernels differ:

* latent attention: decoded tokens and short portions run in the absorbed form (queries multiplied into the latent space,
  one pass over the cached rows); long portions in the expanded form (the sequence's latents are expanded to per-head keys
  and values with one product each, then the tcgen05 prefill kernel; of a windowed layer only what the portion sees);
* grouped-query attention: decoded tokens and short portions as single rows, long portions in the tcgen05 prefill kernel; a layer
  that pools stores the means of the blocks that the batch completes before it attends;
* recurrences (decayed linear attention, gated linear attention, gated delta rule, matrix memory): one kernel advances the
  states of the decoded tokens, others those of the portions;
* a parallel pair runs both of its sides on the columns of one projection.

The residual stream is fp32. Where a norm stands in front of a sublayer, one kernel gates and adds the previous sublayer's
output and normalises for the next; where it stands behind, one kernel norms the output (of both sides of a pair), adds it and
hands the residual itself on, or its norm where one stands in front as well.
"""

from __future__ import annotations

from dataclasses import dataclass

import torch

from ..models.config import (DeltaMixer, GatedLinearMixer, GroupedMixer, LatentMixer, LinearMixer, MemoryMixer, ParallelMixer,
                             attention_shape, ceil8, sub_mixers)
from ..models.layered import LayeredLayerWeights, rotary_table
from ..ops import gemm
from ..ops import mixers as M
from ..ops.attention import decode_plan, embedding, window_plan

# Portions of at most this many tokens run as single rows (latent attention: in the absorbed form, expanding the whole context
# costs more).
SHORT_PORTION = 16


@dataclass
class ExpandGroup:
    """Consecutive sequences whose contexts are expanded together: ``seq0 .. seq0 + n``."""

    seq0: int
    n: int
    max_len: int      # bound on the workspace rows of a sequence
    max_q: int
    tokens: int       # workspace rows, every sequence starting on a multiple of 64


@dataclass
class RowBatch:
    rows: int
    n_seqs: int
    n_dec: int                           # leading rows that are one token each (= leading sequences)
    n_abs: int                           # leading rows that attend as single rows (decoded tokens, then short portions)
    n_short: int                         # leading sequences that do
    max_q: int                           # longest portion behind the decoded tokens
    max_len: int                         # bound on positions + 1 of those rows
    positions: torch.Tensor              # [rows]
    slots: torch.Tensor                  # [rows] cache row, -1: padding
    table: torch.Tensor                  # [seqs, max_blocks]
    state_slots: torch.Tensor            # [seqs]
    row_seq: torch.Tensor | None = None  # [rows]; None: row r is sequence r
    q_starts: torch.Tensor | None = None
    q_lens: torch.Tensor | None = None
    ctx_lens: torch.Tensor | None = None
    starts: torch.Tensor | None = None   # [seqs] first workspace row of an expanded context
    groups: tuple[ExpandGroup, ...] = ()


class LayeredForward:
    def __init__(self, engine):
        self.e = engine
        cfg, dev, dt, cap = engine.cfg, engine.device, engine.dtype, engine.cap
        self.dtype = dt
        h8 = ceil8(cfg.hidden_size)
        layers: list[LayeredLayerWeights] = engine.w.layers
        self.layers = layers

        def buf(n, dtype=dt):
            return torch.zeros(n, dtype=dtype, device=dev)

        self.resid = torch.zeros(cap, cfg.hidden_size, dtype=torch.float32, device=dev)
        self.x, self.x2, self.y, self.rg2 = (torch.zeros(cap, h8, dtype=dt, device=dev)[:, :cfg.hidden_size] for _ in range(4))
        self.proj = buf(cap * max(lw.offs["end"] for lw in layers))
        self.mix_out = torch.zeros(cap * max(sum(ceil8(m.out_features) for m in sub_mixers(lw.spec.mixer)) for lw in layers),
                                   dtype=dt, device=dev)
        mixers = [m for lw in layers for m in sub_mixers(lw.spec.mixer)]

        def of(kind):
            return [m for m in mixers if isinstance(m, kind)]

        lat, lin, grp, gla, delta, mem = (of(k) for k in (LatentMixer, LinearMixer, GroupedMixer, GatedLinearMixer, DeltaMixer, MemoryMixer))
        self.expands = [("exp_k" in lw.mix) for lw in layers]
        # only decoded tokens and short portions attend as single rows, in every layer
        self.all_expand = all(ex for lw, ex in zip(layers, self.expands) if isinstance(lw.spec.mixer, LatentMixer)) and \
            all(self._tiled(m) for m in grp)
        if cfg.output_norm:
            self.y2 = torch.zeros(cap, h8, dtype=dt, device=dev)[:, :cfg.hidden_size]
        if lat:
            self.q_plain = buf(cap * max(m.heads * ceil8(m.dim) for m in lat))
            self.q_abs = buf(cap * max(m.heads * m.cache_width for m in lat))
            self.o_lat = buf(cap * max(m.heads * ceil8(m.kv_rank) for m in lat))
            buckets = engine._buckets
            need = max(b * M.latent_attn_plan(b, m.heads, m.visible(engine.ecfg.max_seq_len), m.cache_width)[0] * m.heads * (m.kv_rank + 2)
                       for b in buckets for m in lat)
            self.attn_ws = buf(max(need, 1 << 20), torch.float32)
            if any(m.q_rank for m in lat):
                self.q_lat = buf(cap * max(ceil8(m.heads * (m.dim + m.rot_dim)) for m in lat if m.q_rank))
        self.ws_tokens = 0
        # tokens that the widest latent layer sees (0: all of them)
        self.latent_window = 0 if any(not m.window for m in lat) else max((m.window for m in lat), default=0)
        if any(self.expands):
            shapes = [(m.heads, *M.expanded_shape(m.dim, m.rot_dim, m.vdim), m.cache_width)
                      for m, ex in ((lw.spec.mixer, ex) for lw, ex in zip(layers, self.expands)) if ex]
            self.ws_tokens = (max(engine.ecfg.max_seq_len, cap) + 63) // 64 * 64 + 64
            self.q_exp = buf(cap * max(H * dq for H, dq, _, _ in shapes))
            self.lat_ws = buf(self.ws_tokens * max(w for *_, w in shapes))
            self.k_exp = buf(self.ws_tokens * max(H * dq for H, dq, _, _ in shapes))
            self.v_exp = buf(self.ws_tokens * max(H * dv for H, _, dv, _ in shapes))
        # cos and sin of every position, one table for all layers of the same rotation
        self.rot_tables = {rot: rotary_table(rot, engine.ecfg.max_seq_len, dev) for rot in {m.rot for m in grp if m.rot is not None}}
        if grp:
            self.q_grp = buf(cap * max(m.kv_heads * M.group_pad(m.heads, m.kv_heads) * m.row_shapes[0][1] for m in grp))
            need = max(b * m.heads * self._splits(m, b, engine.ecfg.max_seq_len)[0] * (m.row_shapes[1][1] + 2)
                       for b in engine._buckets for m in grp)
            self.grp_ws = buf(max(need, 1 << 20), torch.float32)
        if gla:
            self.z = buf(cap * max(m.heads * m.dim for m in gla), torch.float32)
            self.gla_ws = None
            if dt == torch.bfloat16:
                self.gla_ws = M.GatedLinearScratch.for_rows(cap, engine.max_seqs, max(m.heads for m in gla), max(m.dim for m in gla),
                                                            max(m.vdim for m in gla), dev)
        if delta:
            self.delta_ws = M.DeltaScratch.for_rows(cap, engine.max_seqs, max(m.heads for m in delta), max(m.kv_heads for m in delta),
                                                    max(m.dim for m in delta), max(m.vdim for m in delta), dt, dev)
        if mem:
            self.mem_ws = M.MemoryScratch.for_rows(cap, engine.max_seqs, max(m.heads for m in mem), max(m.dim for m in mem),
                                                   max(m.vdim for m in mem), dev)
        self.tails = buf(cap * max((lw.offs["end"] - lw.fp32_from for lw in layers if lw.fp32_from), default=0), torch.float32)
        if cfg.token_side:
            self.side = torch.zeros(cap, ceil8(cfg.token_side), dtype=dt, device=dev)[:, :cfg.token_side]
            self.side_e = torch.zeros(cap, engine.w.extra["side_embed"].shape[1], dtype=dt, device=dev)
        if lin or gla or delta or mem:
            self.o_lin = buf(cap * max(m.out_features for m in lin + gla + delta + mem), torch.float32)
        if lin:
            self.lin_ws = buf(max(M.linear_attn_ws_elems(m.dim, m.vdim) for m in lin) if dt == torch.bfloat16 else 1, torch.float32)

    def expand_rows(self, computed: int, n: int) -> int:
        """Workspace rows in which the expanded form holds what a portion of ``n`` tokens behind ``computed`` ones sees."""
        behind = computed
        if self.latent_window:
            behind -= max(0, computed - self.latent_window + 1) // 64 * 64
        return (behind + n + 63) // 64 * 64

    # ------------------------------------------------------------------ mixers
    def _latent(self, l: int, lw: LayeredLayerWeights, m: LatentMixer, proj: torch.Tensor, out: torch.Tensor, b: RowBatch) -> None:
        rows, H, R, W = b.rows, m.heads, m.kv_rank, m.cache_width
        n_abs = b.n_abs if self.expands[l] else rows
        dp, rp = ceil8(m.dim), ceil8(R)
        cache = self.e.kv.k[l]
        q_plain = self.q_plain[:H * n_abs * dp].view(H, n_abs, dp) if n_abs else None
        q_abs = self.q_abs[:H * n_abs * W].view(H, n_abs, W) if n_abs else None
        q_exp = None
        if n_abs < rows:
            dq, dv = M.expanded_shape(m.dim, m.rot_dim, m.vdim)
            q_exp = self.q_exp[:rows * H * dq].view(rows, H, dq)
        gate = proj[:, lw.offs["g"]:lw.offs["g"] + m.gate_features]
        q, q_off = None, lw.offs["q"]
        if m.q_rank:
            n = m.heads * (m.dim + m.rot_dim)
            q = self.q_lat[:rows * ceil8(n)].view(rows, ceil8(n))[:, :n]
            gemm.linear(proj[:, q_off:q_off + m.q_rank], lw.mix["uq"], out=q)
        M.latent_prep(proj, lw.mix["norm"], lw.mix["freq"], b.positions, b.slots, cache, heads=H, dim=m.dim, rot=m.rot_dim, kv_rank=R,
                      q_off=q_off, kv_off=lw.offs["kv"], eps=self.e.cfg.rms_norm_eps, abs_rows=n_abs, q_plain=q_plain,
                      q_abs=q_abs, q_exp=q_exp, q=q, q_rank=m.q_rank, interleaved=m.rot.interleaved)
        if n_abs:
            gemm.linear_batched(q_plain[:, :, :m.dim], lw.mix["uk_t"], q_abs, n_abs * W)
            splits, chunk = M.latent_attn_plan(n_abs, H, m.visible(b.max_len), W)
            if splits > 1 and n_abs * H * splits * (R + 2) > self.attn_ws.numel():
                splits, chunk = 1, 0
            o_lat = self.o_lat[:H * n_abs * rp].view(H, n_abs, rp)
            M.latent_attn(q_abs, cache, o_lat, b.table, b.positions, b.slots, kv_rank=R, rot=m.rot_dim, scale=m.scale,
                          gate=None if m.gate_elems else gate, row_seq=b.row_seq, num_splits=splits, chunk_tokens=chunk, ws=self.attn_ws,
                          window=m.window)
            gemm.linear_batched(o_lat[:, :, :R], lw.mix["uv"], out[:n_abs], m.vdim, gate=gate[:n_abs] if m.gate_elems else None)
        if n_abs < rows:
            for g in b.groups:
                s = slice(g.seq0, g.seq0 + g.n)
                starts = b.starts[s]
                lat = self.lat_ws[:g.tokens * W].view(g.tokens, W)
                M.latent_gather(cache, lat, b.table[s], b.ctx_lens[s], b.q_lens[s], starts, g.max_len, m.window)
                k = self.k_exp[:g.tokens * H * dq].view(g.tokens, H, dq)
                v = self.v_exp[:g.tokens * H * dv].view(g.tokens, H, dv)
                gemm.linear(lat[:, :R + m.rot_dim], lw.mix["exp_k"], out=k.view(g.tokens, H * dq))
                gemm.linear(lat[:, :R], lw.mix["exp_v"], out=v.view(g.tokens, H * dv))
                M.expanded_prefill(q_exp, k, v, out, b.q_starts[s], b.q_lens[s], b.ctx_lens[s], starts, g.max_q, scale=m.scale,
                                   vdim=m.vdim, gate=gate, window=m.window)

    def _linear(self, l: int, lw: LayeredLayerWeights, m: LinearMixer, proj: torch.Tensor, out: torch.Tensor, b: RowBatch) -> None:
        n = m.out_features
        o = self.o_lin[:b.rows * n].view(b.rows, n)
        kw = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, offs=(lw.offs["q"], lw.offs["k"], lw.offs["v"]))
        state, dec, pw = self.e.kv.states[l], lw.mix["decay"], lw.mix["decay_pow"]
        if b.n_dec:
            M.linear_attn_decode(proj[:b.n_dec], state, dec, pw, o[:b.n_dec], b.positions, b.slots, b.state_slots, **kw)
        if b.n_dec < b.n_seqs:
            s = slice(b.n_dec, b.n_seqs)
            segs, seg_tokens = M.linear_attn_plan(b.n_seqs - b.n_dec, m.heads, m.dim, m.vdim, b.max_q)
            M.linear_attn_prefill(proj, state, dec, pw, o, b.positions, b.slots, b.state_slots[s], b.q_starts[s], b.q_lens[s], segs=segs,
                                  seg_tokens=seg_tokens, ws=self.lin_ws, **kw)
        M.gated_rms(o, lw.mix["norm"], proj[:, lw.offs["g"]:lw.offs["g"] + n], self.e.cfg.rms_norm_eps, out)

    def _tiled(self, m: GroupedMixer) -> bool:
        """Whether the tensor-core attention kernels cover the mixer."""
        shape, page = attention_shape(m.dim, m.vdim), self.e.ecfg.page_size
        return (self.dtype == torch.bfloat16 and shape is not None and m.heads // m.kv_heads <= 16 and page & (page - 1) == 0
                and page >= (16 if shape[0] == shape[1] else 64) and (not m.sigmoid or shape[0] == shape[1]) and (m.sigmoid or not m.pool))

    @staticmethod
    def _splits(m: GroupedMixer, rows: int, max_len: int) -> tuple[int, int]:
        seen = m.visible(max_len)
        return window_plan(rows, m.kv_heads, seen + 32) if seen < max_len else decode_plan(rows, m.kv_heads, max_len)   # edges lie inside tiles

    def _grouped(self, l: int, lw: LayeredLayerWeights, m: GroupedMixer, proj: torch.Tensor, out: torch.Tensor, b: RowBatch) -> None:
        rows, o, kv = b.rows, lw.offs, self.e.kv
        k, v = kv.k[l], kv.v[l]
        gp = M.group_pad(m.heads, m.kv_heads)
        q = self.q_grp[:rows * m.kv_heads * gp * k.shape[3]].view(rows, m.kv_heads, gp, k.shape[3])
        pool = M.BlockMeans(kv.k_pool[l], kv.v_pool[l], m.pool) if m.pool else None
        if m.norm:
            rot = self.rot_tables.get(m.rot)
            M.grouped_prep(proj, lw.mix.get("q_norm"), lw.mix.get("k_norm"), b.slots, k, v, q, heads=m.heads, dim=m.dim, vdim=m.vdim,
                           offs=(o["q"], o["k"], o["v"]), eps=self.e.cfg.rms_norm_eps, unit=m.norm == "unit", rot=rot, interleaved=rot is not None and m.rot.interleaved,
                           positions=b.positions, pool=pool, pool_rows=b.n_dec, block_table=b.table)
        else:
            self._conv_rope(l, lw, m, proj, q, b)
        if pool is not None and b.n_dec < rows:
            s = slice(b.n_dec, rows)
            M.block_means(k, v, pool, b.table, b.positions[s], b.slots[s], b.row_seq[s])
        g_at = o["hg" if m.gate == "head" else "g"] if m.gate else 0
        gate = proj[:, g_at:g_at + m.gate_features] if m.gate else None
        kw = dict(heads=m.heads, vdim=m.vdim, scale=m.scale, softcap=m.softcap, window=m.window, keep_first=m.keep_first,
                  sink=lw.mix.get("sink"), sigmoid_bias=lw.mix.get("bias"), pool=pool)
        if not self._tiled(m):
            M.grouped_attn(q, k, v, out, b.table, b.positions, b.slots, dim=m.dim, gate=gate, row_seq=b.row_seq, **kw)
            return
        n = b.n_abs
        if n:
            splits, chunk = self._splits(m, n, b.max_len)
            if splits > 1 and n * m.heads * splits * (v.shape[3] + 2) > self.grp_ws.numel():
                splits, chunk = 1, 0
            M.grouped_decode(q[:n], k, v, out[:n], b.table, b.positions, b.slots, dim=m.dim, gate=gate, row_seq=b.row_seq, num_splits=splits,
                             chunk_tokens=chunk, ws=self.grp_ws, **kw)
        if n < rows:
            s = slice(b.n_short, b.n_seqs)
            M.grouped_prefill(q, k, v, out, b.table[s], b.q_starts[s], b.q_lens[s], b.ctx_lens[s], b.max_q, gate=gate, **kw)

    def _conv_rope(self, l: int, lw: LayeredLayerWeights, m: GroupedMixer, proj: torch.Tensor, q: torch.Tensor, b: RowBatch) -> None:
        o, kv, nd = lw.offs, self.e.kv, b.n_dec
        offs = (o["q"], o["k"], o["v"]) if m.kv_from is None else (o["q"],)
        kw = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, offs=offs)
        args = (lw.mix["conv"], kv.conv[l], self.rot_tables.get(m.rot))
        if nd:
            M.conv_rope(proj[:nd], *args, b.positions, b.slots, b.state_slots, kv.k[l], kv.v[l], q, **kw)
        if nd < b.n_seqs:
            s = slice(nd, b.n_seqs)
            M.conv_rope(proj, *args, b.positions, b.slots, b.state_slots[s], kv.k[l], kv.v[l], q, q_starts=b.q_starts[s], q_lens=b.q_lens[s],
                        max_q=b.max_q, **kw)

    def _memory(self, l: int, lw: LayeredLayerWeights, m: MemoryMixer, proj: torch.Tensor, out: torch.Tensor, b: RowBatch) -> None:
        o, n, nd, eps = lw.offs, m.out_features, b.n_dec, self.e.cfg.rms_norm_eps
        state = self.e.kv.states[l]
        gates = self._tail(lw, proj, b.rows)
        kw = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, cap=m.gate_cap,
                  offs=(*(o[c] for c in "qkvg"), o["i"] - lw.fp32_from, o["f"] - lw.fp32_from))
        if nd:
            M.memory_decode(proj[:nd], gates, state, lw.mix["norm"], out[:nd], b.positions, b.slots, b.state_slots, eps=eps, **kw)
        if nd < b.n_seqs:
            s = slice(nd, b.n_seqs)
            y = self.o_lin[:b.rows * n].view(b.rows, n)
            segs, seg_tokens = M.linear_attn_plan(b.n_seqs - nd, m.heads, m.dim, m.vdim, b.max_q)
            M.memory_prefill(proj, gates, state, y, b.positions, b.slots, b.state_slots[s], b.q_starts[s], b.q_lens[s], b.max_q, self.mem_ws,
                             segs=segs, seg_tokens=seg_tokens, **kw)
            M.head_gate(y[nd:], lw.mix["norm"], proj[nd:, o["g"]:o["g"] + n], eps, out[nd:], heads=m.heads)

    def _gated_linear(self, l: int, lw: LayeredLayerWeights, m: GatedLinearMixer, proj: torch.Tensor, out: torch.Tensor, b: RowBatch) -> None:
        o, w, n, nd, eps = lw.offs, lw.mix, m.out_features, b.n_dec, self.e.cfg.rms_norm_eps
        state = self.e.kv.states[l]
        kw = dict(heads=m.heads, dim=m.dim, vdim=m.vdim, tau=m.tau)
        qkv = (o["lin_q"], o["lin_k"], o["lin_v"])
        if nd:
            M.gated_linear_decode(proj[:nd], state, w["a2"], w["a2_bias"], w["norm"], out[:nd], b.positions, b.slots, b.state_slots,
                                  offs=(*qkv, o["lin_g"], o["lin_a"]), eps=eps, **kw)
        if nd < b.n_seqs:
            s = slice(nd, b.n_seqs)
            z = self.z[:b.rows * m.heads * m.dim].view(b.rows, m.heads * m.dim)
            gemm.linear(proj[nd:, o["lin_a"]:o["lin_a"] + w["a2"].shape[1]], w["a2"], out=z[nd:], bias=w["a2_bias"])
            y = self.o_lin[:b.rows * n].view(b.rows, n)
            segs, seg_tokens = M.gated_linear_plan(b.n_seqs - nd, m.heads, m.vdim, b.max_q)
            M.gated_linear_prefill(proj, z, state, y, b.positions, b.slots, b.state_slots[s], b.q_starts[s], b.q_lens[s], b.max_q, self.gla_ws,
                                   offs=qkv, segs=segs, seg_tokens=seg_tokens, **kw)
            M.head_gate(y[nd:], w["norm"], proj[nd:, o["lin_g"]:o["lin_g"] + n], eps, out[nd:])

    def _delta(self, l: int, lw: LayeredLayerWeights, m: DeltaMixer, proj: torch.Tensor, out: torch.Tensor, b: RowBatch) -> None:
        o, w, n, nd, eps = lw.offs, lw.mix["delta"], m.out_features, b.n_dec, self.e.cfg.rms_norm_eps
        state, conv = self.e.kv.states[l], self.e.kv.conv[l]
        kw = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, offs=tuple(o[c] for c in "qkvgba"), eps=eps)
        if nd:
            M.delta_decode(proj[:nd], conv, w, state, out[:nd], b.positions, b.slots, b.state_slots, **kw)
        if nd < b.n_seqs:
            s = slice(nd, b.n_seqs)
            y = self.o_lin[:b.rows * n].view(b.rows, n)
            M.delta_prefill(proj, conv, w, state, y, b.positions, b.slots, b.state_slots[s], b.q_starts[s], b.q_lens[s], b.max_q, self.delta_ws, **kw)
            M.head_gate(y[nd:], w.norm, proj[nd:, o["g"]:o["g"] + n], eps, out[nd:])

    _RUN = {LatentMixer: _latent, LinearMixer: _linear, GroupedMixer: _grouped, GatedLinearMixer: _gated_linear, DeltaMixer: _delta,
            MemoryMixer: _memory}

    # ------------------------------------------------------------------ layers
    def _tail(self, lw: LayeredLayerWeights, proj: torch.Tensor, rows: int) -> torch.Tensor | None:
        """Where the layer's fp32 columns of the product are: a buffer of their own, or the product itself in an fp32 model."""
        if not lw.fp32_from:
            return None
        n = lw.offs["end"] - lw.fp32_from
        return proj[:, lw.fp32_from:] if self.dtype == torch.float32 else self.tails[:rows * n].view(rows, n)

    def _mix(self, l: int, lw: LayeredLayerWeights, x: torch.Tensor, b: RowBatch) -> tuple[torch.Tensor, list[torch.Tensor]]:
        """The layer's projection, and the outputs of its mixer (of both sides of a pair) behind their output products."""
        rows = b.rows
        proj = self.proj[:rows * lw.offs["end"]].view(rows, lw.offs["end"])
        tail = self._tail(lw, proj, rows) if self.dtype != torch.float32 else None
        gemm.linear(x, lw.proj, out=proj, bias=lw.proj_bias, silu_cols=lw.silu_cols, tail=tail)
        ys, at = [], 0
        for i, m in enumerate(sub_mixers(lw.spec.mixer)):
            n = m.out_features
            out = self.mix_out[at:][:rows * ceil8(n)].view(rows, ceil8(n))[:, :n]
            at += rows * ceil8(n)
            self._RUN[type(m)](self, l, lw, m, proj, out, b)
            y = (self.y2 if i else self.y)[:rows]
            gemm.linear(out, lw.o_right if i else lw.o, out=y, bias=None if i else lw.o_bias)
            ys.append(y)
        return proj, ys

    def _enter(self, resid: torch.Tensor, norm, x: torch.Tensor, pending: dict) -> None:
        """Adds the pending sublayer output to the residual and prepares the next sublayer's input (``norm``: the one in front
        of it)."""
        if self.e.cfg.output_norm:
            M.post_norm(resid, x, out_norm=norm if self.e.cfg.input_norm else None, **pending)
        else:
            M.resid_norm(resid, norm, x, **pending)

    def forward(self, ids: torch.Tensor, b: RowBatch, mode: int) -> None:
        """Embedding and all layers over the batch's rows; the last sublayer's output stays pending for :meth:`head`."""
        rows, hid = b.rows, self.e.cfg.hidden_size
        resid, x, x2 = self.resid[:rows], self.x[:rows], self.x2[:rows]
        cfg = self.e.cfg
        post = cfg.output_norm
        pending: dict = dict(ids=ids, table=self.e.w.embed)
        if cfg.embed_scale != 1.0:
            pending["embed_scale"] = cfg.embed_scale
        if cfg.token_side:
            embedding(ids, self.e.w.extra["side_embed"], out=self.side_e[:rows])
        for l, lw in enumerate(self.layers):
            self._enter(resid, lw.norm1, x, pending)
            proj, ys = self._mix(l, lw, x, b)
            if post:
                pending = dict(branches=ys, branch_norms=lw.branch_norms, norm=lw.norm1b or lw.norm1)
            else:
                pending = dict(parts=ys, gate=proj[:, lw.offs["rg"]:lw.offs["rg"] + hid] if cfg.residual_gate else None)
            if lw.norm2 is not None:
                self._enter(resid, lw.norm2, x2, pending)
                if post:
                    pending = dict(branches=self.e.port.run(l, x2, rows, mode), norm=lw.norm2b or lw.norm2)
                elif not cfg.residual_gate:
                    pending = dict(parts=self.e.port.run(l, x2, rows, mode))
                else:
                    rg2 = self.rg2[:rows]
                    gemm.linear(x2, lw.rg2, out=rg2, bias=lw.rg2_bias)
                    pending = dict(parts=self.e.port.run(l, x2, rows, mode), gate=rg2)
            if lw.side_gate is not None:
                pending = self._token_side(l, lw, resid, x, pending)
            self.tap(l, rows, pending)
        self._pending = pending

    def _token_side(self, l: int, lw: LayeredLayerWeights, resid: torch.Tensor, x: torch.Tensor, pending: dict) -> dict:
        """``gelu_tanh(side_gate x)`` times the layer's part of the token's second embedding, mapped back to the model width;
        ``x`` is the residual itself."""
        rows, n = x.shape[0], self.e.cfg.token_side
        M.post_norm(resid, x, **pending)
        e = self.side[:rows]
        M.gelu_gate(x, lw.side_gate, self.side_e[:rows, l * n:(l + 1) * n], e)
        gemm.linear(e, lw.side_proj, out=self.y[:rows])
        return dict(branches=[self.y[:rows]], norm=lw.side_norm)

    def tap(self, layer: int, rows: int, pending: dict) -> None:
        """Called after every layer with its output still pending; a debugging subclass or test may look at it."""

    def head(self, rows: int, sel: torch.Tensor | None, n_sel: int, out: torch.Tensor, logits: torch.Tensor) -> None:
        """Final norm of the selected rows (all of the first ``n_sel`` without ``sel``) and their scaled logits (fp32)."""
        e = self.e
        if e.cfg.output_norm:
            # (without a selection the rows are their own; a selection leaves the residual of the others alone)
            M.post_norm(self.resid[:rows], out[:n_sel], out_norm=e.w.final_norm, sel=sel, rows=n_sel, **self._pending)
        else:
            M.resid_norm(self.resid[:rows], e.w.final_norm, out[:n_sel], sel=sel, rows=n_sel, **self._pending)
        gemm.linear(out[:n_sel], e.w.lm_head, out=logits[:n_sel], out_scale=e.cfg.logit_scale)
