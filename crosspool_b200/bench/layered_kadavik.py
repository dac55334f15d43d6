"""Kadavik for ``bench.py --layered kadavik``: a model of the classic one's width, vocabulary, FFN and attention heads, and each of
its kernels alone beside the like kernels of the classic model, of Segirax (decayed linear attention) and of a classic routed
FFN."""

from __future__ import annotations

from types import SimpleNamespace

import torch

from ..models.config import (GELU_ALPHA, GELU_CUBIC, GroupedMixer, LayerSpec, MemoryMixer, ModelConfig, MoeSpec, RotaryScaling, RotarySpec)

DIM = 128
TAPS = 4
WINDOW = 1024
KEEP = 64
SIDE = 256
EXPERTS, TOP, IDENTITY = 32, 4, 4


def twin(classic: ModelConfig, heads: int, layers: int) -> ModelConfig:
    """Memories with dense and routed FFNs, windowed attention, and attention that reads the former's keys, in turn. A routed
    layer's active experts (the shared one too) hold as many weights as the classic FFN."""
    ff = classic.intermediate_size
    memory = MemoryMixer(heads, DIM, DIM, 15.0)
    att = dict(heads=classic.num_q_heads, kv_heads=classic.num_kv_heads, dim=classic.head_dim, vdim=classic.head_dim, scale=classic.head_dim ** -0.5,
               norm="", biases=False, gate="element", conv=TAPS, rot=RotarySpec(64, 5e5, RotaryScaling(8.0, 1.0, 4.0, 8192)), window=WINDOW, keep_first=KEEP)
    moe = MoeSpec(EXPERTS, TOP, ff // 4, IDENTITY, 2.5, ff // 4)
    specs = []
    for i in range(layers):
        mixer = memory if i % 4 < 2 else GroupedMixer(**att, kv_from=i - 1 if i % 4 == 3 else None)
        specs.append(LayerSpec(mixer, moe=moe) if i % 4 in (1, 3) else LayerSpec(mixer, ff, gelu=True))
    return ModelConfig(name=f"kadavik-{classic.name}", architecture="Kadavik", hidden_size=classic.hidden_size, num_layers=layers, num_q_heads=heads,
                       num_kv_heads=classic.num_kv_heads, head_dim=DIM, intermediate_size=ff, vocab_size=classic.vocab_size, rms_norm_eps=1e-6,
                       qk_norm=False, tie_word_embeddings=True, hidden_act="gelu_pytorch_tanh", layer_specs=tuple(specs), output_norm=True,
                       input_norm=True, token_side=SIDE, embed_scale=16.0)


def kernel_table(classic: ModelConfig, cfg: ModelConfig, timer, context: int, chunk: int, row, batch: int = 64) -> list[dict]:
    """``row(name, us, bytes, flops, like)`` makes one line; bytes and flops are those the operation needs at least."""
    from ..models.layered import rotary_table
    from ..models.weights import FfnLayerWeights
    from ..ops import attention as A
    from ..ops import gemm, moe, norm
    from ..ops import mixers as M

    dev, bf = torch.device("cuda"), torch.bfloat16
    att = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, GroupedMixer))
    mem = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, MemoryMixer))
    spec = next(s.moe for s in cfg.layer_specs if s.moe is not None)
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

    # ---- decode: attention, memory
    hq, hk, d = att.heads, att.kv_heads, att.dim
    G, no = hq // hk, att.out_features
    kc, vc, q = rnd(batch * blocks, 64, hk, d), rnd(batch * blocks, 64, hk, d), rnd(batch, hk, G, d)
    o, gate, lens = torch.empty(batch, no, dtype=bf, device=dev), rnd(T, no), i32([context] * batch)
    seen = att.visible(context)
    sp, ck = A.window_plan(batch, hk, seen + 32)
    ws = torch.empty(max(1, batch * hq * sp * (d + 2)), device=dev)
    kw = dict(heads=hq, vdim=d, scale=att.scale, window=WINDOW, keep_first=KEEP)
    add(f"windowed decode b{batch}", lambda: M.grouped_decode(q, kc, vc, o, table, pos, slots, dim=d, gate=gate[:batch], num_splits=sp, chunk_tokens=ck,
                                                             ws=ws, **kw), batch * seen * hk * d * 4, 4.0 * batch * hq * seen * d, "paged decode")
    sp2, ck2 = A.decode_plan(batch, hk, context)
    ws2 = torch.empty(max(1, batch * hq * sp2 * (d + 2)), device=dev)
    add(f"paged decode b{batch}", lambda: A.paged_decode(q.view(batch, hq, d), kc, vc, table, lens, out=o.view(batch, hq, d), num_splits=sp2,
                                                         chunk_tokens=ck2, ws=ws2), (kc.numel() + vc.numel()) * 2, 4.0 * batch * hq * context * d)
    H, D = mem.heads, mem.dim
    n = H * D
    proj, gates = rnd(T, 4 * n), rnd(T, 2 * H, dtype=torch.float32)
    gates[:, H:] += 3.0
    moffs = (0, n, 2 * n, 3 * n, 0, H)
    state, nw, mout = torch.zeros(batch, H, mem.head_state, device=dev), torch.ones(n, device=dev), torch.empty(T, n, dtype=bf, device=dev)
    mkw = dict(heads=H, dim=D, vdim=mem.vdim, offs=moffs, cap=mem.gate_cap)
    add(f"memory decode b{batch}", lambda: M.memory_decode(proj[:batch], gates, state, nw, mout[:batch], pos, slots, slots, eps=1e-6, **mkw),
        state.numel() * 8 + batch * 5 * n * 2, 4.0 * state.numel(), "linear decode")
    lstate = torch.zeros(batch, H, D, D, device=dev)
    dec, pw, lo = torch.full((H,), 0.98, device=dev), M.decay_powers([0.98] * H).to(dev), torch.empty(T, n, device=dev)
    lkw = dict(heads=H, dim=D, vdim=D, offs=(0, n, 2 * n))
    add(f"linear decode b{batch}", lambda: M.linear_attn_decode(proj[:batch], lstate, dec, pw, lo[:batch], pos, slots, slots, **lkw), lstate.numel() * 8,
        4.0 * lstate.numel())

    # ---- one prefill chunk of one sequence
    pairs = sum(att.visible(t + 1) for t in range(T))
    qp, op, tp = rnd(T, hk, G, d), torch.empty(T, no, dtype=bf, device=dev), table.flatten()[:T // 64].view(1, -1).contiguous()
    byts = 4 * qp.numel() + 4 * T * hk * d
    add(f"windowed prefill {T}", lambda: M.grouped_prefill(qp, kc, vc, op, tp, one, st, one, T, gate=gate, **kw), byts + 2 * gate.numel(),
        4.0 * pairs * hq * d, "paged prefill")
    add(f"paged prefill {T}", lambda: A.paged_prefill(qp.view(T, hq, d), kc, vc, tp, one, st, one, T, out=op.view(T, hq, d)), byts,
        4.0 * T * (T + 1) / 2 * hq * d)
    scratch = M.MemoryScratch.for_rows(T, 1, H, D, mem.vdim, dev)
    segs, seg_tokens = M.linear_attn_plan(1, H, D, D, T)
    flops = 2.0 * T * H * (2 * D * D + 64 / 2 * 2 * D)
    add(f"memory prefill {T} (gates, segments)", lambda: M.memory_prefill(proj, gates, state, lo, p0, p0, one, one, st, T, scratch, segs=segs,
                                                                         seg_tokens=seg_tokens, **mkw), T * (3 * n * 2 + 2 * H * 4 + n * 4), flops, "linear prefill")
    lws = torch.empty(M.linear_attn_ws_elems(D, D), device=dev)
    add(f"linear prefill {T}", lambda: M.linear_attn_prefill(proj, lstate, dec, pw, lo, p0, p0, one, one, st, segs=segs, seg_tokens=seg_tokens, ws=lws, **lkw),
        T * (3 * n * 2 + n * 4), flops)
    add(f"norm per head + gate {T}", lambda: M.head_gate(lo, nw, proj[:, 3 * n:], 1e-6, mout, heads=H), T * n * 8, 0.0, "residual + norm")

    # ---- row kernels and products
    resid, x, y = torch.zeros(T, W, device=dev), rnd(T, W), rnd(T, W)
    P, rb, wn = M.NormParams("rmsnorm", torch.ones(W, device=dev)), rnd(T, W), torch.ones(W, dtype=bf, device=dev)
    C = att.conv_channels
    aproj, conv, ring = rnd(T, C + no), rnd(TAPS, C, dtype=torch.float32), torch.zeros(batch, TAPS, C, dtype=bf, device=dev)
    rot = rotary_table(att.rot, max(T, context), dev)
    qkv, qo, aoffs = rnd(T, (hq + 2 * hk) * d), rnd(T, hq, d), (0, hq * d, (hq + hk) * d)
    side = rnd(T, 8 * SIDE)[:, SIDE:2 * SIDE]
    add(f"convolution + rope + kv write {batch}", lambda: M.conv_rope(aproj[:batch], conv, ring, rot, pos, slots, slots, kc, vc, qp[:batch], heads=hq,
                                                                     dim=d, vdim=d, offs=aoffs), 2 * batch * C * (2 + TAPS), 0.0, "rope + kv write")
    add(f"convolution + rope + kv write {T}", lambda: M.conv_rope(aproj, conv, ring, rot, p0, p0, one, kc, vc, qp, heads=hq, dim=d, vdim=d, offs=aoffs,
                                                                 q_starts=one, q_lens=st, max_q=T), 4 * T * C, 0.0, "rope + kv write")
    for r in (batch, T):
        add(f"rope + kv write {r}", lambda: A.rope_kv_write(qkv[:r], qo[:r], kc, vc, p0[:r], p0[:r], q_heads=hq, kv_heads=hk, head_dim=d, theta=1e6),
            4 * r * (hq + 2 * hk) * d)
        add(f"norm + residual + norm {r}", lambda: M.post_norm(resid[:r], x[:r], branches=[y[:r]], norm=P, out_norm=P), r * W * 12, 0.0, "residual + norm")
        add(f"residual + norm {r}", lambda: norm.add_rmsnorm([y[:r]], wn, 1e-6, resid=rb[:r], out=x[:r]), r * W * 8)
        wm, wg, wu, wo = rnd(4 * n + 2 * H, W), rnd(2 * ff, W), rnd(2 * ff, W), rnd(W, hq * d)
        outm, tail, outg = torch.empty(r, 4 * n + 2 * H, dtype=bf, device=dev), torch.empty(r, 2 * H, device=dev), torch.empty(r, ff, dtype=bf, device=dev)
        add(f"memory projection product {r}", lambda: gemm.linear(x[:r], wm, out=outm, tail=tail), 2 * (wm.numel() + r * (W + 4 * n)), 2.0 * r * wm.numel(),
            "gate/up product")
        add(f"gelu gate/up product {r}", lambda: gemm.gateup_swiglu(x[:r], wu, out=outg, act_alpha=GELU_ALPHA, act_cubic=GELU_CUBIC),
            2 * (wu.numel() + r * (W + ff)), 2.0 * r * wu.numel(), "gate/up product")
        add(f"gate/up product {r}", lambda: gemm.gateup_swiglu(x[:r], wg, out=outg), 2 * (wg.numel() + r * (W + ff)), 2.0 * r * wg.numel())
        ws1, ws2, es = rnd(SIDE, W), rnd(W, SIDE), torch.empty(r, SIDE, dtype=bf, device=dev)
        add(f"token side gate product {r}", lambda: M.gelu_gate(x[:r], ws1, side[:r], es), 2 * (ws1.numel() + r * (W + 2 * SIDE)),
            2.0 * r * ws1.numel(), "o product")
        add(f"token side projection {r}", lambda: gemm.linear(es, ws2, out=y[:r]), 2 * (ws2.numel() + r * (W + SIDE)), 2.0 * r * ws2.numel(), "o product")
        xo = rnd(r, hq * d)
        add(f"o product {r}", lambda: gemm.linear(xo, wo, out=y[:r]), 2 * (wo.numel() + r * (W + hq * d)), 2.0 * r * wo.numel())
        del wm, wg, wu, wo
    # routed FFN, and a classic one of the same experts: without identity and shared experts, logits in bf16
    E, k, f = spec.experts, spec.top, spec.ff
    shape = SimpleNamespace(num_experts_per_tok=k, num_experts=E, router_scoring="softmax", norm_topk_prob=True, routed_scaling_factor=1.0, hidden_size=W)
    w = FfnLayerWeights(rnd(E, 2 * f, W, scale=0.02), rnd(E, W, f, scale=0.02), router=rnd(spec.routed, W, scale=0.02))
    plain = FfnLayerWeights(w.gate_up, w.down, router=w.router[:E].contiguous())
    w.shared_gate_up, w.shared_down, w.extra["shared_scale"] = rnd(2 * f, W, scale=0.02), rnd(W, f, scale=0.02), rnd(1, W, scale=0.02)
    w.extra["correction_bias"] = torch.zeros(spec.routed, device=dev)
    moe.prepare_routed(w, spec)
    rws = moe.RoutedWorkspace.for_layers([spec], W, T, bf, dev)
    cws = moe.workspace(dev, T, shape, f, E)
    for r in (batch, T):
        use = min(E, r * k)
        per = 2.0 * 3 * W * f
        byts = 2 * (use * 3 * W * f + 2 * r * W)
        live = k * E / spec.routed                        # of a token's choices are real experts
        add(f"routed ffn {r} (identity, shared)", lambda: moe.routed_ffn(x[:r], w, spec, y[:r], rws), byts + 2 * 3 * W * f, r * per * (live + 1),
            "classic routed ffn")
        add(f"classic routed ffn {r}", lambda: moe.moe_forward(x[:r], plain, shape, out=y[:r], ws=cws), byts, r * per * k)
    gemm.check_status(dev)
    return out
