"""Saninex for ``bench.py --layered saninex``: a model of the classic one's width, vocabulary and FFN, and each of its kernels
alone beside the like kernels of the classic model and of Segirax (decayed linear attention)."""

from __future__ import annotations

import torch

from ..models.config import DeltaMixer, GatedLinearMixer, GroupedMixer, LayerSpec, ModelConfig, ParallelMixer

DIM = 128
TAPS = 4
RANK = 16
LIMIT = 7.0


def twin(classic: ModelConfig, heads: int, layers: int) -> ModelConfig:
    """Gated delta rule layers and parallel layers in turn, the classic model's query and key heads on the attention side."""
    delta = DeltaMixer(heads, heads // 2, DIM, DIM, TAPS)
    pair = ParallelMixer(GroupedMixer(classic.num_q_heads, classic.num_kv_heads, classic.head_dim, classic.head_dim, classic.head_dim ** -0.5, 50.0),
                         GatedLinearMixer(heads // 2, DIM, DIM, 16.0))
    specs = tuple(LayerSpec(pair if i % 2 else delta, classic.intermediate_size, LIMIT) for i in range(layers))
    return ModelConfig(name=f"saninex-{classic.name}", architecture="Saninex", hidden_size=classic.hidden_size, num_layers=layers,
                       num_q_heads=heads, num_kv_heads=heads // 2, head_dim=DIM, intermediate_size=classic.intermediate_size,
                       vocab_size=classic.vocab_size, rms_norm_eps=1e-6, tie_word_embeddings=True, hidden_act="clamped_glu",
                       layer_specs=specs, output_norm=True)


def kernel_table(classic: ModelConfig, cfg: ModelConfig, timer, context: int, chunk: int, row, batch: int = 64) -> list[dict]:
    """``row(name, us, bytes, flops, like)`` makes one line; bytes and flops are those the operation needs at least."""
    from ..ops import attention as A
    from ..ops import gemm, norm
    from ..ops import mixers as M

    dev, bf = torch.device("cuda"), torch.bfloat16
    delta = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, DeltaMixer))
    left, right = next((s.mixer.left, s.mixer.right) for s in cfg.layer_specs if isinstance(s.mixer, ParallelMixer))
    W, ff, T, out = cfg.hidden_size, cfg.intermediate_size, chunk, []

    def rnd(*shape, dtype=bf, scale=1.0):
        return (torch.randn(*shape, device=dev) * scale).to(dtype)

    def i32(x):
        return torch.tensor(x, dtype=torch.int32, device=dev)

    def add(name, fn, byts, flops=0.0, like=""):
        out.append(row(name, timer(fn), byts, flops, like))

    blocks = context // 64
    table = torch.randperm(batch * blocks, device=dev).int().view(batch, blocks)
    pos, slots = i32([context - 1] * batch), torch.arange(batch, dtype=torch.int32, device=dev)
    p0, one, st = torch.arange(T, dtype=torch.int32, device=dev), i32([0]), i32([T])

    # ---- decode: attention, and the recurrences from projection to gated heads
    hq, hk, d = left.heads, left.kv_heads, left.dim
    G = hq // hk
    kc, vc, q = rnd(batch * blocks, 64, hk, d), rnd(batch * blocks, 64, hk, d), rnd(batch, hk, G, d)
    o, gate, lens = torch.empty(batch, hq * d, dtype=bf, device=dev), rnd(T, hq), i32([context] * batch)
    sp, ck = A.decode_plan(batch, hk, context)
    ws = torch.empty(max(1, batch * hq * sp * (d + 2)), device=dev)
    kvb = (kc.numel() + vc.numel()) * 2
    add(f"capped decode b{batch}", lambda: M.grouped_decode(q, kc, vc, o, table, pos, slots, heads=hq, dim=d, vdim=d, scale=left.scale,
                                                           softcap=left.softcap, gate=gate[:batch], num_splits=sp, chunk_tokens=ck, ws=ws),
        kvb, 4.0 * batch * hq * context * d, "paged decode")
    add(f"paged decode b{batch}", lambda: A.paged_decode(q.view(batch, hq, d), kc, vc, table, lens, out=o.view(batch, hq, d), num_splits=sp,
                                                         chunk_tokens=ck, ws=ws), kvb, 4.0 * batch * hq * context * d)
    H, Gd, D = delta.heads, delta.kv_heads, delta.dim
    nq, nv = Gd * D, H * delta.vdim
    doffs = (0, nq, 2 * nq, 2 * nq + nv, 2 * nq + 2 * nv, 2 * nq + 2 * nv + (H + 7) // 8 * 8)
    dproj = rnd(T, doffs[5] + (H + 7) // 8 * 8)
    dw = M.DeltaWeights(rnd(2 * nq + nv, TAPS, dtype=torch.float32), -torch.ones(H, device=dev), torch.zeros(H, device=dev) - 2, torch.ones(delta.vdim, device=dev))
    state = torch.zeros(batch, H, D, delta.vdim, device=dev)
    ring = torch.zeros(batch, TAPS, 2 * nq + nv, dtype=bf, device=dev)
    dout = torch.empty(T, nv, dtype=bf, device=dev)
    dkw = dict(heads=H, kv_heads=Gd, dim=D, vdim=delta.vdim, offs=doffs, eps=1e-6)
    add(f"delta decode b{batch}", lambda: M.delta_decode(dproj[:batch], ring, dw, state, dout[:batch], pos, slots, slots, **dkw),
        state.numel() * 8 + batch * (doffs[5] + 3 * (2 * nq + nv) + nv) * 2, 8.0 * state.numel(), "linear decode")
    Hr, Dr = right.heads, right.dim
    nr = Hr * Dr
    roffs = (0, nr, 2 * nr, 3 * nr, 4 * nr)
    rproj, a2, a2b, nw = rnd(T, 4 * nr + RANK), rnd(nr, RANK), torch.ones(nr, device=dev), torch.ones(right.vdim, device=dev)
    rstate = torch.zeros(batch, Hr, Dr, right.vdim, device=dev)
    rout = torch.empty(T, nr, dtype=bf, device=dev)
    rkw = dict(heads=Hr, dim=Dr, vdim=right.vdim, tau=right.tau)
    add(f"gated linear decode b{batch}", lambda: M.gated_linear_decode(rproj[:batch], rstate, a2, a2b, nw, rout[:batch], pos, slots, slots, offs=roffs,
                                                                      eps=1e-6, **rkw),
        rstate.numel() * 8 + batch * 5 * nr * 2 + a2.numel() * 2, 4.0 * rstate.numel(), "linear decode")
    lproj, dec = rnd(T, 4 * H * D), torch.full((H,), 0.98, device=dev)
    pw, lo = M.decay_powers([0.98] * H).to(dev), torch.empty(T, H * D, device=dev)
    lkw = dict(heads=H, dim=D, vdim=D, offs=(0, H * D, 2 * H * D))
    add(f"linear decode b{batch}", lambda: M.linear_attn_decode(lproj[:batch], state, dec, pw, lo[:batch], pos, slots, slots, **lkw), state.numel() * 8,
        4.0 * state.numel())

    # ---- one prefill chunk of one sequence
    pairs = T * (T + 1) / 2
    qp, op, tp = rnd(T, hk, G, d), torch.empty(T, hq * d, dtype=bf, device=dev), table.flatten()[:T // 64].view(1, -1).contiguous()
    byts = 4 * qp.numel() + 4 * T * hk * d
    for x, tag in ((1.0, ""), (8.0, ", scores up to the cap")):
        qx = (qp * x).to(bf)
        add(f"capped prefill {T}{tag}", lambda: M.grouped_prefill(qx, kc, vc, op, tp, one, st, one, T, heads=hq, vdim=d, scale=left.scale,
                                                                  softcap=left.softcap, gate=gate), byts, 4.0 * pairs * hq * d, "paged prefill")
    add(f"paged prefill {T}", lambda: A.paged_prefill(qp.view(T, hq, d), kc, vc, tp, one, st, one, T, out=op.view(T, hq, d)), byts,
        4.0 * pairs * hq * d)
    scratch, do = M.DeltaScratch.for_rows(T, 1, H, Gd, D, delta.vdim, bf, dev), torch.empty(T, nv, device=dev)
    add(f"delta prefill {T} (convolution, systems, scan)", lambda: M.delta_prefill(dproj, ring, dw, state, do, p0, p0, one, one, st, T, scratch, **dkw),
        T * ((2 * nq + nv) * 2 + 2 * H * 2 + nv * 4), 2.0 * T * H * (3 * D * delta.vdim + 32 * (2 * D + 2 * delta.vdim)), "linear prefill")
    z, ro, gs = torch.zeros(T, nr, device=dev), torch.empty(T, nr, device=dev), M.GatedLinearScratch.for_rows(T, 1, Hr, Dr, right.vdim, dev)
    segs, seg_tokens = M.gated_linear_plan(1, Hr, right.vdim, T)

    def gla():
        gemm.linear(rproj[:, roffs[4]:roffs[4] + RANK], a2, out=z, bias=a2b)
        M.gated_linear_prefill(rproj, z, rstate, ro, p0, p0, one, one, st, T, gs, offs=roffs[:3], segs=segs, seg_tokens=seg_tokens, **rkw)

    add(f"gated linear prefill {T} (decay map, scores, scan)", gla, T * (3 * nr * 2 + RANK * 2 + nr * 4),
        2.0 * T * Hr * (2 * Dr * right.vdim + 32 * (Dr + right.vdim)), "linear prefill")
    lsegs, lst = M.linear_attn_plan(1, H, D, D, T)
    lws = torch.empty(M.linear_attn_ws_elems(D, D), device=dev)
    add(f"linear prefill {T}", lambda: M.linear_attn_prefill(lproj, state, dec, pw, lo, p0, p0, one, one, st, segs=lsegs, seg_tokens=lst, ws=lws, **lkw),
        T * H * 3 * D * 2 + lo.numel() * 4, 2.0 * T * H * (2 * D * D + 64 / 2 * 2 * D))

    # ---- row kernels and products
    resid, x, y, y2 = torch.zeros(T, W, device=dev), rnd(T, W), rnd(T, W), rnd(T, W)
    P = M.NormParams("rmsnorm", torch.ones(W, device=dev))
    rb, wn = rnd(T, W), torch.ones(W, dtype=bf, device=dev)
    aproj, qn = rnd(T, (hq + 2 * hk) * d), torch.ones(d, device=dev)
    qkv, qo = rnd(T, (hq + 2 * hk) * d), rnd(T, hq, d)
    for n in (batch, T):
        add(f"q/k norm + kv write {n}", lambda: M.grouped_prep(aproj[:n], qn, qn, p0[:n], kc, vc, qp[:n], heads=hq, dim=d, vdim=d,
                                                              offs=(0, hq * d, (hq + hk) * d), eps=1e-6), 4 * n * (hq + 2 * hk) * d, 0.0, "rope + kv write")
        add(f"rope + kv write {n}", lambda: A.rope_kv_write(qkv[:n], qo[:n], kc, vc, p0[:n], p0[:n], q_heads=hq, kv_heads=hk, head_dim=d, theta=1e6),
            4 * n * (hq + 2 * hk) * d)
        add(f"norm + residual {n}", lambda: M.post_norm(resid[:n], x[:n], branches=[y[:n]], norm=P), n * W * 12, 0.0, "residual + norm")
        add(f"two norms + norm + residual {n}", lambda: M.post_norm(resid[:n], x[:n], branches=[y[:n], y2[:n]], branch_norms=[P, P], norm=P), n * W * 14,
            0.0, "residual + norm")
        add(f"residual + norm {n}", lambda: norm.add_rmsnorm([y[:n]], wn, 1e-6, resid=rb[:n], out=x[:n]), n * W * 8)
        np_ = doffs[5]
        wp, wg, wu = rnd(np_, W), rnd(2 * ff, W), rnd(2 * ff, W)
        outp, outg = torch.empty(n, np_, dtype=bf, device=dev), torch.empty(n, ff, dtype=bf, device=dev)
        add(f"delta projection product {n}", lambda: gemm.linear(x[:n], wp, out=outp), 2 * (wp.numel() + n * (W + np_)), 2.0 * n * W * np_, "gate/up product")
        add(f"clamped gate/up product {n}", lambda: gemm.gateup_swiglu(x[:n], wu, out=outg, gate_limit=LIMIT, up_add=1.0, act_alpha=1.702),
            2 * (wu.numel() + n * (W + ff)), 2.0 * n * W * 2 * ff, "gate/up product")
        add(f"gate/up product {n}", lambda: gemm.gateup_swiglu(x[:n], wg, out=outg), 2 * (wg.numel() + n * (W + ff)), 2.0 * n * W * 2 * ff)
        del wp, wg, wu
    add(f"norm per head + gate {T}", lambda: M.head_gate(do, nw, dproj[:, doffs[3]:doffs[3] + nv], 1e-6, dout), T * nv * 8, 0.0, "residual + norm")
    gemm.check_status(dev)
    return out
