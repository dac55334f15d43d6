"""Layered decoders beside the closest classic model of equal size on one GPU: ``bench.py --layered`` (Segirax),
``--layered saninex`` and ``--layered kadavik`` (also beside Segirax), ``--layered dofevik`` (also beside Kadavik); their sizes and
kernels are in ``layered_saninex.py``, ``layered_kadavik.py`` and ``layered_dofevik.py``.

Two sizes whose layers resemble a real model's (random weights, a few layers): latent attention and decayed linear attention
alternate, each with a PolyNorm FFN that holds as many weights as the gated FFN of the classic model. For both models, in
the same engine with the same limits: prompt tokens per second of one prefill chunk and output tokens per second of decode
steps (captured graphs) at several batch sizes. Then every kernel of the layered model, and the like kernel of the classic
one, alone: microseconds and the fraction of its roofline (measured copy bandwidth and cuBLAS throughput).
"""

from __future__ import annotations

import json
import statistics

import torch

from ..models.config import LatentMixer, LayerSpec, LinearMixer, ModelConfig, RotarySpec
from ..models.config import preset as mc_preset
from .kernels import Timer, peaks

SIZES = {"small": ("Qwen/Qwen3-0.6B", 16), "large": ("Qwen/Qwen3-8B", 32)}
CONTEXT = 2048          # cached tokens per sequence in decode
CHUNK = 4096            # prompt tokens of a prefill step
BATCHES = (1, 64, 256)


def layered_twin(classic: ModelConfig, heads: int, layers: int) -> ModelConfig:
    """A layered decoder of the classic model's width, vocabulary and FFN weight count."""
    latent = LatentMixer(heads=heads, dim=128, rot_dim=64, vdim=128, kv_rank=512, rot=RotarySpec(64, 1e6), scale=192 ** -0.5)
    linear = LinearMixer(heads=heads, dim=128, vdim=128, decay=tuple(1.0 - 2.0 ** -(1 + 7 * h / heads) for h in range(heads)))
    ff = classic.intermediate_size * 3 // 2
    specs = tuple(LayerSpec(linear if i % 2 == 0 else latent, ff) for i in range(layers))
    return ModelConfig(name=f"segirax-{classic.name}", architecture="Segirax", hidden_size=classic.hidden_size, num_layers=layers,
                       num_q_heads=heads, num_kv_heads=1, head_dim=128, intermediate_size=ff, vocab_size=classic.vocab_size,
                       rms_norm_eps=1e-6, qk_norm=False, tie_word_embeddings=True, hidden_act="polynorm", norm="dyt",
                       layer_specs=specs, residual_gate=True)


def _engine(cfg: ModelConfig, batch: int):
    from ..deployment import build_loopback
    from ..engine.atn_engine import EngineConfig

    pages = (batch * (CONTEXT + 64) + CHUNK + 1024) // 64
    ecfg = EngineConfig(max_batch=batch, prefill_chunk=CHUNK, max_seq_len=CHUNK + 64, page_size=64, num_pages=pages,
                        decode_buckets=[b for b in BATCHES if b <= batch])
    return build_loopback([(cfg.name, cfg, 0)], ecfg).instances[0].engine


def _event_ms(stream, fn) -> float:
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record(stream)
    fn()
    b.record(stream)
    torch.cuda.synchronize()
    return a.elapsed_time(b)


def throughput(cfg: ModelConfig, steps: int, warmup: int) -> dict:
    """Prefill and decode rates of one model. Decode sequences count ``CONTEXT`` tokens as cached already."""
    from ..engine.atn_engine import Sequence
    from ..ops import gemm

    e = _engine(cfg, max(BATCHES))
    e.warmup()
    g = torch.Generator().manual_seed(0)
    ms = []
    for i in range(warmup + steps):
        e.add_request(torch.randint(0, cfg.vocab_size, (CHUNK,), generator=g).tolist(), 1)
        t = _event_ms(e.stream, e.step)
        if i >= warmup:
            ms.append(t)
        assert not e.has_work
    out = {"prefill_ms": round(statistics.median(ms), 3), "prefill_tok_s": round(CHUNK / statistics.median(ms) * 1e3)}
    seqs = [Sequence(1000 + i, [1] * CONTEXT, 8, generated=[1]) for i in range(max(BATCHES))]
    for s in seqs:
        e.kv.ensure(s.seq_id, s.total_len)
    for b in BATCHES:
        e._fill_decode(seqs[:b])
        with torch.cuda.stream(e.stream):
            e.dec_meta.copy_(e.dec_meta_host, non_blocking=True)
            for _ in range(max(3, warmup)):
                e._replay_decode(b)
        t = _event_ms(e.stream, lambda: [_replay(e, b) for _ in range(steps)]) / steps
        out[f"decode_b{b}_ms"], out[f"decode_b{b}_tok_s"] = round(t, 3), round(b / t * 1e3)
    gemm.check_status(e.device)
    out["cache_bytes_per_token"], out["state_bytes_per_sequence"] = cfg.kv_bytes_per_token(), cfg.state_bytes_per_sequence()
    return out


def _replay(e, b: int) -> None:
    with torch.cuda.stream(e.stream):
        e._replay_decode(b)


# ------------------------------------------------------------------------------------------ kernels alone

def _row(name: str, us: float, byts: float, flops: float, like: str = "") -> dict:
    pk = peaks()
    need = max(byts / pk["hbm_gbs"] / 1e3, flops / pk["bf16_tflops"] / 1e6)      # microseconds at the roofline
    return {"kernel": name, "us": round(us, 2), "roofline_us": round(need, 2), "frac": round(need / us, 3), **({"like": like} if like else {})}


def kernel_table(classic: ModelConfig, cfg: ModelConfig, timer: Timer, batch: int = 64) -> list[dict]:
    from ..ops import attention as A
    from ..ops import gemm, norm
    from ..ops import mixers as M

    dev, bf = torch.device("cuda"), torch.bfloat16
    lat = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, LatentMixer))
    lin = next(s.mixer for s in cfg.layer_specs if isinstance(s.mixer, LinearMixer))
    W, ff, H, R, r = cfg.hidden_size, cfg.layer_specs[0].ff, lat.heads, lat.kv_rank, lat.rot_dim
    rows_out: list[dict] = []

    def rnd(*shape, dtype=bf, scale=1.0):
        return (torch.randn(*shape, device=dev) * scale).to(dtype)

    def i32(x):
        return torch.tensor(x, dtype=torch.int32, device=dev)

    def add(name, fn, byts, flops=0.0, like=""):
        rows_out.append(_row(name, timer(fn), byts, flops, like))

    # ---- attention and recurrence, decode
    blocks = CONTEXT // 64
    table = torch.randperm(batch * blocks, device=dev).int().view(batch, blocks)
    pos, slots = i32([CONTEXT - 1] * batch), torch.arange(batch, dtype=torch.int32, device=dev)
    cache = rnd(batch * blocks, 64, 1, lat.cache_width)
    q, o = rnd(H, batch, lat.cache_width), torch.empty(H, batch, R, dtype=bf, device=dev)
    gate = rnd(batch, H)
    splits, chunk = M.latent_attn_plan(batch, H, CONTEXT, lat.cache_width)
    ws = torch.empty(batch * H * splits * (R + 2), device=dev)
    add(f"latent decode b{batch}", lambda: M.latent_attn(q, cache, o, table, pos, slots, kv_rank=R, rot=r, scale=lat.scale, gate=gate,
                                                        num_splits=splits, chunk_tokens=chunk, ws=ws),
        cache.numel() * 2 + 2 * (q.numel() + o.numel()), 2.0 * batch * H * CONTEXT * (2 * R + r), "paged decode")
    hq, hk, d = classic.num_q_heads, classic.num_kv_heads, classic.head_dim
    kc, vc, qd = rnd(batch * blocks, 64, hk, d), rnd(batch * blocks, 64, hk, d), rnd(batch, hq, d)
    od, lens = torch.empty_like(qd), i32([CONTEXT] * batch)
    sp, ck = A.decode_plan(batch, hk, CONTEXT)
    wsd = torch.empty(max(1, batch * hq * sp * (d + 2)), device=dev)
    add(f"paged decode b{batch}", lambda: A.paged_decode(qd, kc, vc, table, lens, out=od, num_splits=sp, chunk_tokens=ck, ws=wsd),
        (kc.numel() + vc.numel()) * 2, 4.0 * batch * hq * CONTEXT * d)
    Hl, dl, vl = lin.heads, lin.dim, lin.vdim
    pl = rnd(CHUNK, Hl * (2 * dl + 2 * vl))
    offs = (0, Hl * dl, 2 * Hl * dl)
    state = torch.zeros(batch, Hl, dl, vl, device=dev)
    dec, pw = torch.tensor(lin.decay, device=dev), M.decay_powers(lin.decay).to(dev)
    ol = torch.empty(CHUNK, Hl * vl, device=dev)
    kw = dict(heads=Hl, dim=dl, vdim=vl, offs=offs)
    add(f"linear decode b{batch}", lambda: M.linear_attn_decode(pl[:batch], state, dec, pw, ol[:batch], pos, slots, slots, **kw),
        state.numel() * 8, 4.0 * state.numel(), "paged decode")

    # ---- attention and recurrence, one prefill chunk of one sequence
    T = CHUNK
    p0, one, st = torch.arange(T, dtype=torch.int32, device=dev), i32([0]), i32([T])
    segs, seg_tokens = M.linear_attn_plan(1, Hl, dl, vl, T)
    lws = torch.empty(M.linear_attn_ws_elems(dl, vl), device=dev)
    add(f"linear prefill {T}", lambda: M.linear_attn_prefill(pl, state, dec, pw, ol, p0, p0, one, one, st, segs=segs, seg_tokens=seg_tokens,
                                                            ws=lws, **kw),
        T * Hl * (2 * dl + vl) * 2 + ol.numel() * 4, 2.0 * T * Hl * (2 * dl * vl + 64 / 2 * (dl + vl)), "paged prefill")
    dq, dv = M.expanded_shape(lat.dim, r, lat.vdim)
    qe, ke, ve = rnd(T, H, dq), rnd(T, H, dq), rnd(T, H, dv)
    oe, ge = torch.empty(T, H * lat.vdim, dtype=bf, device=dev), rnd(T, H)
    pairs = T * (T + 1) / 2
    add(f"expanded prefill {T}", lambda: M.expanded_prefill(qe, ke, ve, oe, one, st, one, one, T, scale=lat.scale, vdim=lat.vdim, gate=ge),
        (qe.numel() + ke.numel() + ve.numel() + oe.numel()) * 2, 2.0 * pairs * H * (lat.dim + r + lat.vdim), "paged prefill")
    qp = rnd(T, hq, d)
    op, tp = torch.empty_like(qp), table.flatten()[:T // 64].view(1, -1).contiguous()
    add(f"paged prefill {T}", lambda: A.paged_prefill(qp, kc, vc, tp, one, st, one, T, out=op), 4 * qp.numel() + 4 * T * hk * d,
        4.0 * pairs * hq * d)

    # ---- row kernels and small products, prefill rows and decode rows
    n_proj = H * (lat.dim + r) + R + r + H + W
    proj, nw = rnd(T, (n_proj + 15) // 8 * 8), torch.ones(max(R, Hl * vl), device=dev)
    freq = 1e6 ** (-torch.arange(r // 2, dtype=torch.float64, device=dev) / (r // 2))
    resid, x, y, g = torch.zeros(T, W, device=dev), rnd(T, W), rnd(T, W), rnd(T, W)
    dyt = M.NormParams("dyt", torch.ones(W, device=dev), torch.zeros(W, device=dev), torch.ones(1, device=dev))
    rb, wn = rnd(T, W), torch.ones(W, dtype=bf, device=dev)
    z, coef = rnd(T, ff), torch.ones(4, device=dev)
    gl, oo = rnd(T, Hl * vl), torch.empty(T, Hl * vl, dtype=bf, device=dev)
    qkv = rnd(T, (hq + 2 * hk) * d)
    for n in (batch, T):
        ab = n if n == batch else 0
        qpl, qab = rnd(H, max(ab, 1), lat.dim), rnd(H, max(ab, 1), lat.cache_width)
        add(f"latent prep {n}", lambda: M.latent_prep(
            proj[:n], nw[:R], freq, p0[:n], p0[:n], cache, heads=H, dim=lat.dim, rot=r, kv_rank=R, q_off=0, kv_off=H * (lat.dim + r),
            eps=1e-6, abs_rows=ab, q_plain=qpl if ab else None, q_abs=qab if ab else None, q_exp=None if ab else qe),
            2 * n * (2 * H * (lat.dim + r) + 2 * (R + r)), 0.0, "rope + kv write")
        add(f"rope + kv write {n}", lambda: A.rope_kv_write(qkv[:n], qp[:n], kc, vc, p0[:n], p0[:n], q_heads=hq, kv_heads=hk, head_dim=d,
                                                           theta=1e6), 4 * n * (hq + 2 * hk) * d)
        add(f"gate + residual + norm {n}", lambda: M.resid_norm(resid[:n], dyt, x[:n], parts=[y[:n]], gate=g[:n]), n * W * (8 + 6), 0.0,
            "residual + norm")
        add(f"residual + norm {n}", lambda: norm.add_rmsnorm([y[:n]], wn, 1e-6, resid=rb[:n], out=x[:n]), n * W * 8)
        add(f"polynorm {n}", lambda: M.polynorm(z[:n], coef, 1e-6, z[:n]), n * ff * 4, 0.0, "residual + norm")
        add(f"norm + gate (linear) {n}", lambda: M.gated_rms(ol[:n], nw[:Hl * vl], gl[:n], 1e-6, oo[:n]), n * Hl * vl * 8, 0.0,
            "residual + norm")
        wp, wg, wu, wd = rnd(n_proj, W), rnd(2 * classic.intermediate_size, W), rnd(ff, W), rnd(W, ff)
        outp, outg = torch.empty(n, n_proj, dtype=bf, device=dev), torch.empty(n, classic.intermediate_size, dtype=bf, device=dev)
        add(f"projection product {n}", lambda: gemm.linear(x[:n], wp, out=outp, silu_cols=256), 2 * (wp.numel() + n * (W + n_proj)),
            2.0 * n * W * n_proj, "gate/up product")
        add(f"up product {n}", lambda: gemm.linear(x[:n], wu, out=z[:n]), 2 * (wu.numel() + n * (W + ff)), 2.0 * n * W * ff, "gate/up product")
        add(f"down product {n}", lambda: gemm.linear(z[:n], wd, out=y[:n]), 2 * (wd.numel() + n * (W + ff)), 2.0 * n * W * ff, "gate/up product")
        add(f"gate/up product {n}", lambda: gemm.gateup_swiglu(x[:n], wg, out=outg), 2 * (wg.numel() + n * (W + classic.intermediate_size)),
            2.0 * n * W * wg.shape[0])
        del wp, wg, wu, wd
    wk = rnd(H * R, lat.dim)
    qpl, qab = rnd(H, batch, lat.dim), rnd(H, batch, lat.cache_width)
    add(f"absorb query b{batch}", lambda: gemm.linear_batched(qpl, wk, qab, batch * lat.cache_width),
        2 * (wk.numel() + batch * H * (R + lat.dim)), 2.0 * batch * wk.numel(), "o product")
    wv, ov = rnd(H * lat.vdim, R), torch.empty(batch, H * lat.vdim, dtype=bf, device=dev)
    add(f"expand value b{batch}", lambda: gemm.linear_batched(o, wv, ov, lat.vdim), 2 * (wv.numel() + batch * H * (R + lat.vdim)),
        2.0 * batch * wv.numel(), "o product")
    wo, xo = rnd(W, hq * d), rnd(batch, hq * d)
    add(f"o product b{batch}", lambda: gemm.linear(xo, wo, out=y[:batch]), 2 * (wo.numel() + batch * (W + hq * d)), 2.0 * batch * wo.numel())
    lat_d = rnd(T, lat.cache_width)
    wek, kx = rnd(H * dq, R + r), torch.empty(T, H * dq, dtype=bf, device=dev)
    add(f"expand keys {T}", lambda: gemm.linear(lat_d[:, :R + r], wek, out=kx), 2 * (wek.numel() + T * (R + r + H * dq)),
        2.0 * T * wek.numel(), "gate/up product")
    add(f"gather latents {T}", lambda: M.latent_gather(cache, lat_d, tp, one, st, one, T), 4 * T * lat.cache_width, 0.0, "rope + kv write")
    gemm.check_status(dev)
    return rows_out


def run(steps: int = 20, warmup: int = 5, layers: int = 8, sizes=tuple(SIZES), design: str = "segirax") -> dict:
    from . import layered_dofevik, layered_kadavik, layered_saninex
    from .decode_bench import ClockSampler

    torch.cuda.set_device(0)
    sampler = ClockSampler(0)
    sampler.start()
    out = {"metric": "prefill and decode tok/s of layered decoders beside the closest classic model of equal size", "unit": "tok/s",
           "dtype": "bf16", "data": "synthetic: random-init weights, random token ids", "context": CONTEXT, "chunk": CHUNK,
           "layers": layers, "design": design, "sizes": {}}
    for size in sizes:
        name, heads = SIZES[size]
        classic = mc_preset(name).with_layers(layers)
        segirax = layered_twin(classic, heads, layers)
        other = {"saninex": layered_saninex, "kadavik": layered_kadavik, "dofevik": layered_dofevik}.get(design)
        cfg = segirax if other is None else other.twin(classic, heads, layers)
        beside = ("kadavik", layered_kadavik.twin(classic, heads, layers)) if design == "dofevik" else ("segirax", segirax)
        res = {"classic": name, "layered": throughput(cfg, steps, warmup), "classic_rates": throughput(classic, steps, warmup)}
        torch.cuda.empty_cache()
        timer = Timer(max(10, steps), max(3, warmup), True)
        if other is None:
            res["kernels"] = kernel_table(classic, cfg, timer)
        else:
            res[beside[0] + "_rates"] = throughput(beside[1], steps, warmup)
            torch.cuda.empty_cache()
            res["kernels"] = other.kernel_table(classic, cfg, timer, CONTEXT, CHUNK, _row)
        torch.cuda.empty_cache()
        out["sizes"][size] = res
    out["clocks"] = sampler.stop()
    return out


if __name__ == "__main__":
    print(json.dumps(run()))
