"""Dofevik for ``bench.py --layered dofevik``: a model of the classic one's width, vocabulary, FFN weight count and attention heads, and
each of its kernels alone beside the like kernels of Kadavik (windowed attention, routed FFNs), Segirax (latent attention) and the
classic model."""

from __future__ import annotations

import torch

from ..models.config import GroupedMixer, LatentMixer, LayerSpec, ModelConfig, MoeSpec, RotaryScaling, RotarySpec

WINDOW = 1024
POOL = 16
Q_RANK, KV_RANK, DIM, ROT = 768, 512, 128, 64
EXPERTS, TOP = 32, 4


def twin(classic: ModelConfig, heads: int, layers: int) -> ModelConfig:
    """Windowed attention with sinks, sigmoid attention over a window and pooled blocks, and windowed latent attention in turn, each with
    a routed FFN whose active experts (the shared one too) hold about as many weights as the classic FFN."""
    ff = classic.intermediate_size * 3 // (2 * (TOP + 1)) // 128 * 128
    shape = dict(heads=classic.num_q_heads, kv_heads=classic.num_kv_heads, dim=classic.head_dim, vdim=classic.head_dim, scale=classic.head_dim ** -0.5,
                 gate="", window=WINDOW)
    mixers = (GroupedMixer(**shape, norm="unit", rot=RotarySpec(classic.head_dim, 5e5, RotaryScaling(4.0), True), sink=True),
              GroupedMixer(**shape, biases=False, sigmoid=True, pool=POOL, tied=True),
              LatentMixer(heads, DIM, ROT, DIM, KV_RANK, RotarySpec(ROT, 1e6), (DIM + ROT) ** -0.5, Q_RANK, WINDOW, True))
    moe = MoeSpec(EXPERTS, TOP, ff, shared_ff=ff, shared_gate=False, relu2=True, logit_choice=True)
    return ModelConfig(name=f"dofevik-{classic.name}", architecture="Dofevik", hidden_size=classic.hidden_size, num_layers=layers, num_q_heads=classic.num_q_heads,
                       num_kv_heads=classic.num_kv_heads, head_dim=classic.head_dim, intermediate_size=ff, vocab_size=classic.vocab_size, rms_norm_eps=1e-6,
                       qk_norm=False, hidden_act="relu2", norm="scalar", layer_specs=tuple(LayerSpec(mixers[i % 3], moe=moe) for i in range(layers)))


def kernel_table(classic: ModelConfig, cfg: ModelConfig, timer, context: int, chunk: int, row, batch: int = 64) -> list[dict]:
    """``row(name, us, bytes, flops, like)`` makes one line; bytes and flops are those the operation needs at least."""
    from ..models.layered import rotary_table, scaled_frequencies
    from ..models.weights import FfnLayerWeights
    from ..ops import attention as A
    from ..ops import gemm, moe, norm
    from ..ops import mixers as M

    dev, bf = torch.device("cuda"), torch.bfloat16
    att, pooled, lat = (s.mixer for s in cfg.layer_specs[:3])
    spec, W, T, out = cfg.layer_specs[0].moe, cfg.hidden_size, chunk, []

    def rnd(*shape, dtype=bf, scale=1.0):
        return (torch.randn(*shape, device=dev) * scale).to(dtype)

    def i32(x):
        return torch.tensor(x, dtype=torch.int32, device=dev)

    def add(name, fn, byts, flops=0.0, like=""):
        out.append(row(name, timer(fn), byts, flops, like))

    blocks = max(context, T) // 64
    table = torch.randperm(batch * blocks, device=dev).int().view(batch, blocks)
    pos, slots = i32([context - 1] * batch), torch.arange(batch, dtype=torch.int32, device=dev)
    p0, one, st = torch.arange(T, dtype=torch.int32, device=dev), i32([0]), i32([T])
    tp = table[:1].contiguous()

    # ---- grouped attention, decode
    hq, hk, d = att.heads, att.kv_heads, att.dim
    G, no = hq // hk, att.out_features
    kc, vc, q = rnd(batch * blocks, 64, hk, d), rnd(batch * blocks, 64, hk, d), rnd(batch, hk, G, d)
    page = pooled.pool_page(64)
    means = M.BlockMeans(rnd(batch * blocks, page, hk, d), rnd(batch * blocks, page, hk, d), POOL)
    o, gate, lens = torch.empty(batch, no, dtype=bf, device=dev), rnd(T, no), i32([context] * batch)
    sink, bias = rnd(hq, dtype=torch.float32), rnd(hq, dtype=torch.float32) - 4
    kw = dict(heads=hq, vdim=d, scale=att.scale, window=WINDOW)
    forms = {"windowed, sinks": (att, dict(sink=sink)), "window and blocks, sigmoid": (pooled, dict(sigmoid_bias=bias, pool=means)),
             "windowed, gate (Kadavik)": (att, dict(gate=gate[:batch]))}
    for name, (m, form) in forms.items():
        seen = m.visible(context)
        sp, ck = A.window_plan(batch, hk, seen + 32)
        ws = torch.empty(max(1, batch * hq * sp * (d + 2)), device=dev)
        add(f"decode b{batch}: {name}", lambda: M.grouped_decode(q, kc, vc, o, table, pos, slots, dim=d, num_splits=sp, chunk_tokens=ck, ws=ws, **kw, **form),
            batch * seen * hk * d * 4, 4.0 * batch * hq * seen * d, "" if "Kadavik" in name else "windowed, gate (Kadavik)")
    sp2, ck2 = A.decode_plan(batch, hk, context)
    ws2 = torch.empty(max(1, batch * hq * sp2 * (d + 2)), device=dev)
    add(f"decode b{batch}: paged (classic)", lambda: A.paged_decode(q.view(batch, hq, d), kc, vc, table, lens, out=o.view(batch, hq, d), num_splits=sp2,
                                                                   chunk_tokens=ck2, ws=ws2), batch * context * hk * d * 4, 4.0 * batch * hq * context * d)

    # ---- one prefill chunk of one sequence
    qp, op = rnd(T, hk, G, d), torch.empty(T, no, dtype=bf, device=dev)
    byts = 4 * qp.numel() + 4 * T * hk * d
    forms["windowed, gate (Kadavik)"] = (att, dict(gate=gate))
    for name, (m, form) in forms.items():
        pairs = sum(m.visible(t + 1) for t in range(T))
        add(f"prefill {T}: {name}", lambda: M.grouped_prefill(qp, kc, vc, op, tp, one, st, one, T, **kw, **form), byts, 4.0 * pairs * hq * d,
            "" if "Kadavik" in name else "windowed, gate (Kadavik)")
    add(f"prefill {T}: paged (classic)", lambda: A.paged_prefill(qp.view(T, hq, d), kc, vc, tp, one, st, one, T, out=op.view(T, hq, d)), byts,
        4.0 * T * (T + 1) / 2 * hq * d)

    # ---- latent attention
    H, R, r, vd = lat.heads, lat.kv_rank, lat.rot_dim, lat.vdim
    cache = rnd(batch * blocks, 64, 1, lat.cache_width)
    ql, ol = rnd(H, batch, lat.cache_width), torch.empty(H, batch, R, dtype=bf, device=dev)
    for name, window in (("windowed", WINDOW), ("whole (Segirax)", 0)):
        seen = min(context, window or context)
        splits, ck = M.latent_attn_plan(batch, H, seen, lat.cache_width)
        lws = torch.empty(batch * H * splits * (R + 2), device=dev)
        add(f"latent decode b{batch}: {name}", lambda: M.latent_attn(ql, cache, ol, table, pos, slots, kv_rank=R, rot=r, scale=lat.scale, num_splits=splits,
                                                                    chunk_tokens=ck, ws=lws, window=window),
            2 * (batch * seen * lat.cache_width + ql.numel() + ol.numel()), 2.0 * batch * H * seen * (2 * R + r), "" if not window else "whole (Segirax)")
    dq, dv = M.expanded_shape(lat.dim, r, vd)
    qe, ke, ve, oe = rnd(T, H, dq), rnd(T, H, dq), rnd(T, H, dv), torch.empty(T, H * vd, dtype=bf, device=dev)
    ge = rnd(T, H * vd)
    for name, window, g in (("windowed, gate per element", WINDOW, ge), ("whole, gate per head (Segirax)", 0, ge[:, :H])):
        pairs = sum(min(t + 1, window or T) for t in range(T))
        add(f"expanded prefill {T}: {name}", lambda: M.expanded_prefill(qe, ke, ve, oe, one, st, one, one, T, scale=lat.scale, vdim=vd, gate=g, window=window),
            (qe.numel() + ke.numel() + ve.numel() + oe.numel() + (g.numel() if window else 0)) * 2, 2.0 * pairs * H * (lat.dim + r + vd),
            "whole, gate per head (Segirax)" if window else "")
    wv, gl, ov = rnd(H * vd, R), rnd(batch, H * vd), torch.empty(batch, H * vd, dtype=bf, device=dev)
    need = 2 * (wv.numel() + batch * H * (R + vd))
    add(f"expand value b{batch}: times a gate", lambda: gemm.linear_batched(ol, wv, ov, vd, gate=gl), need + 2 * gl.numel(), 2.0 * batch * wv.numel(), "plain (Segirax)")
    add(f"expand value b{batch}: plain (Segirax)", lambda: gemm.linear_batched(ol, wv, ov, vd), need, 2.0 * batch * wv.numel())

    # ---- row kernels and products
    resid, x, y = torch.zeros(T, W, device=dev), rnd(T, W), rnd(T, W)
    P, rb, wn = M.NormParams("rmsnorm", torch.ones(W, device=dev)), rnd(T, W), torch.ones(W, dtype=bf, device=dev)
    rot, ones = rotary_table(att.rot, max(T, context), dev), torch.ones(d, device=dev)
    qkv, qo = rnd(T, (hq + 2 * hk) * d), rnd(T, hq, d)
    n_lat = H * (lat.dim + r)
    lproj, lnorm, freq = rnd(T, Q_RANK + R + r), torch.ones(R, device=dev), scaled_frequencies(lat.rot).to(dev)
    lq, sproj = rnd(T, n_lat), rnd(T, n_lat + R + r)
    for n in (batch, T):
        dec = n == batch
        ab = n if dec else 0
        ps, sl, tb = (pos, slots, table) if dec else (p0, p0, tp)
        add(f"unit norm + rope + kv write {n}", lambda: M.grouped_prep(qkv[:n], None, None, sl, kc, vc, qp[:n], heads=hq, dim=d, vdim=d,
                                                                      offs=(0, hq * d, (hq + hk) * d), eps=1e-6, unit=True, rot=rot, interleaved=True, positions=ps),
            4 * n * (hq + 2 * hk) * d, 0.0, "rope + kv write")
        add(f"norm + kv write, tied{', block means' if dec else ''} {n}",
            lambda: M.grouped_prep(qkv[:n], ones, ones, sl, kc, vc, qp[:n], heads=hq, dim=d, vdim=d, offs=(0, hq * d, hq * d), eps=1e-6, positions=ps,
                                   pool=means if dec else None, pool_rows=ab, block_table=tb),
            2 * n * (2 * hq + 3 * hk) * d + (2 * n * 2 * hk * d * POOL if dec else 0), 0.0, "rope + kv write")
        add(f"rope + kv write {n}", lambda: A.rope_kv_write(qkv[:n], qo[:n], kc, vc, p0[:n], p0[:n], q_heads=hq, kv_heads=hk, head_dim=d, theta=1e6),
            4 * n * (hq + 2 * hk) * d)
        qpl, qab = rnd(H, max(ab, 1), lat.dim), rnd(H, max(ab, 1), lat.cache_width)
        lay = dict(heads=H, dim=lat.dim, rot=r, kv_rank=R, eps=1e-6, abs_rows=ab, q_plain=qpl if ab else None, q_abs=qab if ab else None, q_exp=None if ab else qe)
        add(f"latent prep, query latent {n}", lambda: M.latent_prep(lproj[:n], lnorm, freq, p0[:n], p0[:n], cache, q_off=0, kv_off=Q_RANK, q=lq[:n], q_rank=Q_RANK, **lay),
            2 * n * (2 * n_lat + Q_RANK + 2 * (R + r)), 0.0, "latent prep (Segirax)")
        add(f"latent prep (Segirax) {n}", lambda: M.latent_prep(sproj[:n], lnorm, freq, p0[:n], p0[:n], cache, q_off=0, kv_off=n_lat, **lay),
            2 * n * (2 * n_lat + 2 * (R + r)))
        add(f"residual + norm, 32 bits {n}", lambda: M.resid_norm(resid[:n], P, x[:n], parts=[y[:n]]), n * W * 12, 0.0, "residual + norm")
        add(f"residual + norm {n}", lambda: norm.add_rmsnorm([y[:n]], wn, 1e-6, resid=rb[:n], out=x[:n]), n * W * 8)
        for name, k, no_ in (("projection, attention", W, (hq + 2 * hk) * d), ("projection, tied", W, (hq + hk) * d), ("projection, latent", W, Q_RANK + R + r + H * vd),
                             ("query map", Q_RANK, n_lat), ("o product", hq * d, W)):
            w1, x1, o1 = rnd(no_, k), rnd(n, k), torch.empty(n, no_, dtype=bf, device=dev)
            add(f"{name} {n}", lambda: gemm.linear(x1, w1, out=o1), 2 * (w1.numel() + n * (k + no_)), 2.0 * n * w1.numel(), "" if name == "o product" else "o product")
            del w1, x1, o1
    seq = torch.zeros_like(p0)
    add(f"block means {T}", lambda: M.block_means(kc, vc, means, tp, p0, p0, seq), 2 * 2 * T * hk * d * (1 + 1 / POOL), 0.0, "rope + kv write")
    lat_d = rnd(T, lat.cache_width)
    wek, kx = rnd(H * dq, R + r), torch.empty(T, H * dq, dtype=bf, device=dev)
    add(f"expand keys {T} (as Segirax)", lambda: gemm.linear(lat_d[:, :R + r], wek, out=kx), 2 * (wek.numel() + T * (R + r + H * dq)), 2.0 * T * wek.numel())

    # ---- routed FFN, and Kadavik's of the same experts' width with gated experts
    E, k, f = spec.experts, spec.top, spec.ff
    gated = MoeSpec(E, k, f, shared_ff=f)
    for name, sp, like in (("squared relu", spec, "gated (Kadavik)"), ("gated (Kadavik)", gated, "")):
        w = FfnLayerWeights(rnd(E, sp.in_features, W, scale=0.02), rnd(E, W, f, scale=0.02), router=rnd(E, W, scale=0.02))
        w.shared_gate_up, w.shared_down = rnd((sp.maps - 1) * f, W, scale=0.02), rnd(W, f, scale=0.02)
        if sp.shared_gate:
            w.extra["shared_scale"] = rnd(1, W, scale=0.02)
        w.extra["router_bias" if sp.logit_choice else "correction_bias"] = torch.zeros(E, device=dev)
        moe.prepare_routed(w, sp)
        rws = moe.RoutedWorkspace.for_layers([sp], W, T, bf, dev)
        for n in (batch, T):
            use, per = min(E, n * k), 2.0 * sp.maps * W * f
            add(f"routed ffn {n}: {name}", lambda: moe.routed_ffn(x[:n], w, sp, y[:n], rws), 2 * ((use + 1) * sp.maps * W * f + 2 * n * W), n * per * (k + 1), like)
        del w
    gemm.check_status(dev)
    return out
