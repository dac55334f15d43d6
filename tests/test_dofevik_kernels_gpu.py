"""Each kernel that Dofevik added to the layered decoders, or extended, alone against its plain restatement (float64 on the CPU)."""
import math

import pytest
import torch

import dofevik_oracle as oracle

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _rnd(*shape, seed=0, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype).cuda()


def _close(got, want, dtype, tol=0.0):
    t = tol or (2e-5 if dtype == torch.float32 else 1.2e-2)
    got, want = got.double().cpu(), want.double().cpu()
    assert torch.allclose(got, want, rtol=t, atol=t), (got - want).abs().max()


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _status():
    from crosspool_b200.ops import gemm

    gemm.check_status(torch.device("cuda"))


def _pitched(rows, n, dtype, seed):
    """Rows whose pitch is a whole number of 16-byte units; what lies between them must not matter."""
    x = torch.full((rows, (n + 7) // 8 * 8), float("nan"), dtype=dtype, device="cuda")[:, :n]
    x.copy_(_rnd(rows, n, seed=seed))
    return x


def _cpu(t):
    return t.double().cpu()


# ------------------------------------------------------------------ products and routed FFNs

@pytest.mark.parametrize("rows,n,k", [(1, 37, 52), (5, 136, 96), (70, 72, 40), (300, 200, 192), (3, 1000, 1024)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_squared_relu_products_of_any_shape(rows, n, k, dtype):
    from crosspool_b200.models.layered import pad_pitch
    from crosspool_b200.ops import gemm

    x, w = _pitched(rows, k, dtype, 1), pad_pitch(_rnd(n, k, seed=2, dtype=dtype, scale=k ** -0.5))
    out = torch.full((rows, (n + 7) // 8 * 8 + 8), 7.0, dtype=dtype, device="cuda")
    gemm.linear_relu2(x, w, out[:, :n])
    _close(out[:, :n], (_cpu(x) @ _cpu(w).T).clamp(min=0) ** 2, dtype, 2e-2 if dtype == torch.bfloat16 else 1e-4)
    assert (out[:, n:] == 7.0).all()
    _status()


@pytest.mark.parametrize("rows,heads,n,k", [(1, 3, 13, 30), (16, 2, 128, 512), (40, 5, 56, 80), (130, 17, 24, 136)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_product_per_head_times_a_sigmoid_per_element(rows, heads, n, k, dtype):
    """The gate is a column range of wider rows."""
    from crosspool_b200.models.layered import pad_pitch
    from crosspool_b200.ops import gemm

    kp = (k + 7) // 8 * 8
    x = torch.zeros(heads, rows, kp, dtype=dtype, device="cuda")
    x[..., :k] = _rnd(heads, rows, k, seed=1, dtype=dtype)
    w = pad_pitch(_rnd(heads * n, k, seed=2, dtype=dtype, scale=k ** -0.5))
    gate = _rnd(rows, heads * n + 8 + (-heads * n) % 8, seed=3, dtype=dtype, scale=2.0)[:, 8:8 + heads * n]
    wide = torch.full((rows, (heads * n + 7) // 8 * 8 + 8), 7.0, dtype=dtype, device="cuda")
    out = wide[:, :heads * n]
    gemm.linear_batched(x[:, :, :k], w, out, n, gate=gate)
    want = torch.einsum("hrk,hnk->rhn", _cpu(x[..., :k]), _cpu(w).view(heads, n, k)).reshape(rows, -1) * torch.sigmoid(_cpu(gate))
    _close(out, want, dtype, 1e-4 if dtype == torch.float32 else 0)
    assert (wide[:, heads * n:] == 7.0).all()
    _status()


@pytest.mark.parametrize("rows", [1, 3, 128, 129, 400])
@pytest.mark.parametrize("h,E,top,ff,shared", [(96, 5, 2, 40, 56), (52, 4, 3, 11, 7), (256, 16, 4, 136, 0), (64, 1, 1, 24, 8), (128, 40, 32, 8, 200)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_routed_ffn_of_squared_relu_experts(rows, h, E, top, ff, shared, dtype):
    from crosspool_b200.models.config import MoeSpec
    from crosspool_b200.models.weights import FfnLayerWeights
    from crosspool_b200.ops import moe

    kw = dict(shared_gate=False, relu2=True, logit_choice=True)
    spec = MoeSpec(E, top, ff, shared_ff=shared, **kw)
    cfg = {"router": {"experts": E, "top": top}, "shared": shared}
    bf = torch.bfloat16
    t = {"router": _rnd(E, h, seed=1, dtype=bf, scale=2 * h ** -0.5), "router.b": _rnd(E, seed=2, scale=2.0)}
    for e in range(E):
        t.update({f"e{e}.up": _rnd(ff, h, seed=100 + e, dtype=bf, scale=h ** -0.5), f"e{e}.down": _rnd(h, ff, seed=200 + e, dtype=bf, scale=ff ** -0.5)})
    w = FfnLayerWeights(torch.stack([t[f"e{e}.up"] for e in range(E)]).to(dtype), torch.stack([t[f"e{e}.down"] for e in range(E)]).to(dtype),
                        router=t["router"].to(dtype))
    w.extra["router_bias"] = t["router.b"]
    if shared:
        t.update({"shared.up": _rnd(shared, h, seed=6, dtype=bf, scale=h ** -0.5), "shared.down": _rnd(h, shared, seed=7, dtype=bf, scale=shared ** -0.5)})
        w.shared_gate_up, w.shared_down = t["shared.up"].to(dtype), t["shared.down"].to(dtype)
    moe.prepare_routed(w, spec)
    x = _pitched(rows, h, dtype, 3)
    ws = moe.RoutedWorkspace.for_layers([spec, MoeSpec(2, 1, 8, **kw)], h, 400, dtype, torch.device("cuda"))
    out = torch.full((rows, (h + 7) // 8 * 8), 7.0, dtype=dtype, device="cuda")
    tt = {k: _cpu(v) for k, v in t.items()}
    for n in (rows, max(1, rows // 2)):                       # the second call finds the first one's tables
        moe.routed_ffn(x[:n], w, spec, out[:n, :h], ws)
        margins: list = []
        want = oracle.experts(_cpu(x[:n]), cfg, lambda k: tt[k], margins)
        ok = (margins[0] > 1e-5).cuda() if margins else torch.ones(n, dtype=torch.bool, device="cuda")   # router logits are fp32 in both types
        assert ok.float().mean() > 0.9
        _close(out[:n, :h][ok], want[ok.cpu()], dtype, 3e-2 if dtype == torch.bfloat16 else 1e-4)
    assert (out[:, h:] == 7.0).all()
    _status()


@pytest.mark.parametrize("rows", [2, 200])
def test_choice_by_logits_far_apart(rows):
    """Logits whose softmax over all experts would leave nothing of the second choice still order the choice."""
    from crosspool_b200.ops import moe

    z = torch.tensor([[300.0, -500.0, 0.0, 10.0], [-1.0, -2.0, -400.0, -300.0]]).repeat(rows // 2, 1).cuda()
    ids, w = _i32([[0] * 3] * rows), torch.zeros(rows, 3, device="cuda")
    moe.router_topk(z, 4, 3, out_ids=ids, out_weights=w, sigmoid=2, logit_bias=torch.tensor([0.0, 0.0, 0.0, 1.0], device="cuda"))
    assert ids[:2].tolist() == [[0, 3, 2], [0, 1, 3]]
    _close(w[:2], torch.tensor([[1.0, 0.0, 0.0], [1 / (1 + math.exp(-1)), 1 / (1 + math.e), 0.0]]), torch.float32)


# ------------------------------------------------------------------ between projection and attention

def _blocks(k, v, G, dq, dv, pool, table, lens, page, dtype, stray=float("nan")):
    """Pooled caches of whole sequences, unused rows NaN; returns the object and the plain means."""
    from crosspool_b200.models.config import GroupedMixer
    from crosspool_b200.ops import mixers as M

    n = GroupedMixer(G, G, dq, dv, 1.0, window=1, pool=pool).pool_page(page)
    pages = int(table.max()) + 1
    bm = M.BlockMeans(*(torch.full((pages, n, G, w), stray, dtype=dtype, device="cuda") for w in (dq, dv)), pool)
    plain = []
    for i in range(len(lens)):
        means = [oracle.block_means(_cpu(x[i]), pool).to(dtype).cuda() for x in (k, v)]
        for b in range(lens[i] // pool):
            at = int(table[i, b // n])
            bm.k[at, b % n], bm.v[at, b % n] = means[0][b], means[1][b]
        plain.append([_cpu(m) for m in means])
    return bm, plain


@pytest.mark.parametrize("H,G,d,e,pairs,form", [(6, 2, 24, 40, 8, "unit"), (4, 1, 64, 64, 32, "unit"), (3, 3, 128, 72, 20, "unit"), (5, 1, 10, 13, 3, "unit"),
                                                (4, 2, 40, 40, 0, "tied"), (3, 1, 10, 10, 0, "tied"), (8, 8, 128, 128, 0, "tied"), (2, 1, 200, 200, 0, "tied"),
                                                (4, 2, 32, 32, 12, "weight"), (6, 2, 24, 24, 12, "half")])
@pytest.mark.parametrize("dtype", DTYPES)
def test_norms_rotation_cache_rows_and_block_means(H, G, d, e, pairs, form, dtype):
    from crosspool_b200.models.config import attention_shape, ceil8
    from crosspool_b200.ops import mixers as M

    page, pool, tied = 16, 5, form == "tied"
    positions = [0, 4, 14, 15, 63, 79]
    lens, rows = [p + 1 for p in positions], len(positions)
    dq, dv = attention_shape(d, e) or (ceil8(d), ceil8(e))
    blocks = 5
    table = torch.randperm(rows * blocks, generator=torch.Generator().manual_seed(1)).view(rows, blocks).int().cuda()
    kc, vc = (torch.full((rows * blocks, page, G, w), 9.0, dtype=dtype, device="cuda") for w in (dq, dv))
    hist = [[torch.cat([_rnd(n, G, w, seed=s + i, dtype=dtype), torch.zeros(n, G, pad - w, dtype=dtype, device="cuda")], -1)
             for i, n in enumerate(lens)] for s, w, pad in ((10, d, dq), (30, e, dv))]
    for i, p in enumerate(positions):
        for t in range(p):
            at = int(table[i, t // page]) * page + t % page
            kc.flatten(0, 1)[at], vc.flatten(0, 1)[at] = hist[0][i][t], hist[1][i][t]
    off_q, off_k = 8, 8 + (H * d + 7) // 8 * 8
    off_v = off_k if tied else off_k + (G * d + 7) // 8 * 8
    proj = _rnd(rows + 1, (off_v + max(G * d, G * e) + 7) // 8 * 8, seed=5, dtype=dtype)
    slots = _i32([int(table[i, p // page]) * page + p % page for i, p in enumerate(positions)] + [-1])
    pos = _i32(positions + [3])
    qn, kn = (None, None) if form == "unit" else (_rnd(d, seed=6), _rnd(d, seed=7))
    neighbours = form != "half"
    freq = oracle.frequencies({"dims": 2 * pairs, "base": 50.0})
    a = torch.arange(100, dtype=torch.float64)[:, None] * freq
    rot = torch.stack([a.cos(), a.sin()], -1).float().cuda() if pairs else None
    bm, _ = _blocks([h[:n - 1] for h, n in zip(hist[0], lens)], [h[:n - 1] for h, n in zip(hist[1], lens)], G, dq, dv, pool, table, [n - 1 for n in lens], page, dtype, 9.0)
    before = bm.k.clone(), bm.v.clone()
    q = torch.full((rows + 1, G, M.group_pad(H, G), dq), 9.0, dtype=dtype, device="cuda")
    M.grouped_prep(proj, qn, kn, slots, kc, vc, q, heads=H, dim=d, vdim=e, offs=(off_q, off_k, off_v), eps=1e-3, unit=form == "unit", rot=rot, interleaved=neighbours and pairs > 0,
                   positions=pos, pool=bm, pool_rows=rows, block_table=table)
    x = _cpu(proj)

    def turned(u, p, w):                                     # u [heads, d] at position p
        if form in ("unit",):
            u = oracle.rms(oracle.rotate(u.expand(p + 1, -1, -1), freq, True)[p], 1e-3) if pairs else oracle.rms(u, 1e-3)
        else:
            u = oracle.rms(u, 1e-3) * _cpu(w)
            u = oracle.rotate(u.expand(p + 1, -1, -1), freq, neighbours)[p] if pairs else u
        return u

    for r, p in enumerate(positions):
        want = turned(x[r, off_q:off_q + H * d].view(H, d), p, qn).view(G, H // G, d)
        _close(q[r, :, :H // G, :d], want, dtype)
        assert (q[r, :, :, d:] == 0).all() and (q[r, :, H // G:] == 0).all()
        key, val = turned(x[r, off_k:off_k + G * d].view(G, d), p, kn), x[r, off_v:off_v + G * e].view(G, e)
        gk, gv = kc.flatten(0, 1)[int(slots[r])], vc.flatten(0, 1)[int(slots[r])]
        _close(gk[:, :d], key, dtype)
        assert torch.equal(_cpu(gv[:, :e]), val) and (gk[:, d:] == 0).all() and (gv[:, e:] == 0).all()
        if (p + 1) % pool == 0:
            b, n = p // pool, bm.k.shape[1]
            for cache, means, own, h in ((bm.k, before[0], gk, hist[0][r]), (bm.v, before[1], gv, hist[1][r])):
                m = (_cpu(h[b * pool:p]).sum(0) + _cpu(own)) / pool
                at = int(table[r, b // n])
                _close(cache[at, b % n], m, dtype, 5e-3 if dtype == torch.bfloat16 else 0)
                means[at, b % n] = cache[at, b % n]
    assert torch.equal(bm.k, before[0]) and torch.equal(bm.v, before[1])      # no other block is touched
    used = set(slots.tolist()) | {int(table[i, t // page]) * page + t % page for i, p in enumerate(positions) for t in range(p)}
    assert all((kc.flatten(0, 1)[i] == 9).all() for i in range(rows * blocks * page) if i not in used)
    # the same means by the kernel of portions, from the cached rows alone
    again = M.BlockMeans(torch.full_like(bm.k, 9.0), torch.full_like(bm.v, 9.0), pool)
    M.block_means(kc, vc, again, table, pos, slots, _i32(list(range(rows)) + [0]))
    for r, p in enumerate(positions):
        if (p + 1) % pool == 0:
            b, n = p // pool, bm.k.shape[1]
            at = int(table[r, b // n])
            assert torch.equal(again.k[at, b % n], bm.k[at, b % n]) and torch.equal(again.v[at, b % n], bm.v[at, b % n])
    done = sum((p + 1) % pool == 0 for p in positions)
    assert ((again.k != 9).flatten(2).any(-1)).sum() == done


@pytest.mark.parametrize("dim,rot,q_rank,rank,heads", [(24, 16, 40, 56, 3), (10, 6, 21, 30, 2), (128, 64, 96, 512, 9)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_queries_from_a_latent(dim, rot, q_rank, rank, heads, dtype):
    """A map of the query latent without its norm, which the row kernel applies; neighbours or halves turn."""
    from crosspool_b200.ops import mixers as M

    rows, ab = 5, 2
    width, dp, dq = (rank + rot + 15) // 16 * 16, (dim + 7) // 8 * 8, (dim + rot + 63) // 64 * 64
    ql, kv_off = 8, 8 + (q_rank + 7) // 8 * 8
    proj = _rnd(rows, (kv_off + rank + rot + 7) // 8 * 8, seed=1, dtype=dtype, scale=3.0)
    raw = _pitched(rows, heads * (dim + rot), dtype, 4)
    nw = _rnd(rank, seed=2)
    freq = oracle.frequencies({"dims": rot, "base": 1e4})
    pos, slots = [0, 1, 17, 1000, 3], _i32([5, 0, 31, 32, 9])
    for neighbours in (False, True):
        cache = torch.full((4, 16, 1, width), 9.0, dtype=dtype, device="cuda")
        qp, qa = torch.full((heads, ab, dp), 9.0, dtype=dtype, device="cuda"), torch.full((heads, ab, width), 9.0, dtype=dtype, device="cuda")
        qe = torch.full((rows, heads, dq), 9.0, dtype=dtype, device="cuda")
        M.latent_prep(proj, nw, freq.cuda(), _i32(pos), slots, cache, heads=heads, dim=dim, rot=rot, kv_rank=rank, q_off=ql, kv_off=kv_off, eps=1e-3,
                      abs_rows=ab, q_plain=qp, q_abs=qa, q_exp=qe, q=raw, q_rank=q_rank, interleaved=neighbours)
        x = _cpu(proj)
        inv = 1 / (x[:, ql:ql + q_rank].pow(2).mean(-1) + 1e-3).sqrt()
        q = _cpu(raw).view(rows, heads, dim + rot) * inv[:, None, None]
        q[..., dim:] = torch.stack([oracle.rotate(q[r:r + 1, :, dim:].expand(p + 1, -1, -1), freq, neighbours)[p] for r, p in enumerate(pos)])
        _close(qp[:, :, :dim].transpose(0, 1), q[:ab, :, :dim], dtype)
        _close(qa[:, :, rank:rank + rot].transpose(0, 1), q[:ab, :, dim:], dtype)
        _close(qe[ab:, :, :dim + rot], q[ab:], dtype)
        for r, p in enumerate(pos):
            key = oracle.rotate(x[r:r + 1, None, kv_off + rank:kv_off + rank + rot].expand(p + 1, -1, -1), freq, neighbours)[p, 0]
            _close(cache.view(-1, width)[int(slots[r]), rank:rank + rot], key, dtype)


# ------------------------------------------------------------------ attention

def _paged(lens, G, dq, dv, page, dtype, seed=1):
    """Caches whose pages are shuffled and whose unused rows hold NaN, the table, and the plain keys and values."""
    blocks = max((n + page - 1) // page for n in lens)
    perm = torch.randperm(len(lens) * blocks, generator=torch.Generator().manual_seed(seed)).view(len(lens), blocks)
    k, v = (torch.full((len(lens) * blocks, page, G, w), float("nan"), dtype=dtype, device="cuda") for w in (dq, dv))
    ks = [_rnd(n, G, dq, seed=10 * seed + i, dtype=dtype) for i, n in enumerate(lens)]
    vs = [_rnd(n, G, dv, seed=20 * seed + i, dtype=dtype) for i, n in enumerate(lens)]
    table = perm.int().cuda()

    def fill():
        for i, n in enumerate(lens):
            rows = torch.tensor([int(perm[i, p // page]) * page + p % page for p in range(n)]).cuda()
            k.flatten(0, 1)[rows], v.flatten(0, 1)[rows] = ks[i], vs[i]

    return k, v, table, ks, vs, fill


def _attend(q, k, v, scale, first, window, sink, bias, pool, means):
    """Rows first .. of a sequence (q ``[n, H, d]``, all of its keys and values) by the plain equations."""
    T, H, G = k.shape[0], q.shape[1], k.shape[1]
    seen = oracle.in_window(T, window or T)
    if pool:
        k, v = torch.cat([k, means[0]]), torch.cat([v, means[1]])
        seen = torch.cat([seen, oracle.blocks_behind_window(T, window, pool)], 1)
    seen = seen[first:]
    out = torch.zeros(q.shape[0], H, v.shape[-1], dtype=torch.float64)
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].T * scale
        w = oracle.sigmoid_weights(s, seen, bias[h]) if bias is not None else oracle.softmax_with_sink(s, seen, None if sink is None else sink[h])
        out[:, h] = w @ v[:, h // (H // G)]
    return out.reshape(q.shape[0], -1)


# (window, block, kind of weights)
FORMS = [(40, 0, "sink"), (0, 0, "sink"), (1, 0, "sink"), (64, 0, "sigmoid"), (0, 0, "sigmoid"), (40, 5, "sigmoid"), (16, 16, "sigmoid"), (100, 1, "sigmoid"),
         (33, 70, "sigmoid"), (1, 3, "sigmoid"), (64, 8, "sigmoid"), (500, 4, "sigmoid"), (50, 7, "sink")]


@pytest.mark.parametrize("window,pool,kind", FORMS)
@pytest.mark.parametrize("H,G,d,dtype", [(6, 2, 64, torch.bfloat16), (4, 1, 128, torch.bfloat16), (16, 1, 64, torch.bfloat16), (3, 3, 24, torch.float32),
                                         (3, 1, 16, torch.bfloat16)])
@pytest.mark.parametrize("page", [16, 64])
def test_rows_with_sinks_sigmoid_weights_and_blocks(window, pool, kind, H, G, d, dtype, page):
    from crosspool_b200.ops import mixers as M

    e = d
    lens = [1, 15, 40, 41, 63, 64, 65, 129, 300, 420]
    k, v, table, ks, vs, fill = _paged(lens, G, d, e, page, dtype)
    pad = M.group_pad(H, G)
    q = _rnd(len(lens), G, pad, d, seed=3, dtype=dtype)
    q[:, :, H // G:] = 0
    for i, n in enumerate(lens):                              # tokens on both sides of the window's and the blocks' edges stand out in turn
        last = (n - window) // pool * pool if pool else 0
        edge = [n - window, n - window - 1, last - 1, last, 0][i % 5] if window else n // 2
        if 0 <= edge < n:
            ks[i][edge] = q[i, :, :H // G].float().mean(1).to(dtype) * 3 * max(1, pool)
            vs[i][edge] *= 3
    fill()
    sink = _rnd(H, seed=6, scale=2.0) if kind == "sink" else None
    bias = _rnd(H, seed=7) - 2 if kind == "sigmoid" else None
    bm, plain = _blocks(ks, vs, G, d, e, pool, table, lens, page, dtype) if pool else (None, None)
    out = torch.full((len(lens) + 1, H * e), 7.0, dtype=dtype, device="cuda")
    order = [3, 0, 1, 2, 9, 8, 7, 6, 5, 4]                    # rows in another order than their table rows
    pos, slots = _i32([lens[i] - 1 for i in order] + [0]), _i32([0] * len(lens) + [-1])
    seq = _i32(order + [0])
    qq = torch.cat([q[order], q[:1]])
    want = torch.cat([_attend(_cpu(q[i:i + 1, :, :H // G].reshape(1, H, d)), _cpu(ks[i]), _cpu(vs[i]), 0.2, lens[i] - 1, window,
                              None if sink is None else _cpu(sink), None if bias is None else _cpu(bias), pool, plain[i] if pool else None) for i in order])
    kw = dict(heads=H, dim=d, vdim=e, scale=0.2, window=window, row_seq=seq, sink=sink, sigmoid_bias=bias, pool=bm)
    tol = dict(tol=2e-4) if dtype == torch.float32 else dict(tol=1.6e-2)
    M.grouped_attn(qq, k, v, out, table, pos, slots, **kw)
    _close(out[:-1], want, dtype, **tol)
    assert (out[-1] == 0).all()
    if dtype == torch.bfloat16 and d >= 64 and not (pool and kind == "sink"):
        for splits, chunk in ((1, 0), (4, 0), (4, 112), (30, 16)):
            ws = torch.empty((len(lens) + 1) * H * splits * (e + 2), device="cuda")
            out.fill_(7.0)
            M.grouped_decode(qq, k, v, out, table, pos, slots, num_splits=splits, chunk_tokens=chunk, ws=ws, **kw)
            _close(out[:-1], want, dtype, **tol)
    _status()


@pytest.mark.parametrize("window,pool,kind", [f for f in FORMS if not (f[1] and f[2] == "sink")])
@pytest.mark.parametrize("H,G,d", [(6, 2, 64), (4, 1, 128), (16, 1, 64), (3, 3, 128)])
@pytest.mark.parametrize("page", [16, 64])
def test_portions_with_sinks_sigmoid_weights_and_blocks(window, pool, kind, H, G, d, page):
    from crosspool_b200.ops import mixers as M

    dtype, e = torch.bfloat16, d
    lens, ctx = [20, 64, 65, 200, 333, 700], [0, 0, 17, 64, 300, 33]
    k, v, table, ks, vs, fill = _paged(lens, G, d, e, page, dtype)
    q_lens = [n - c for n, c in zip(lens, ctx)]
    starts = [sum(q_lens[:i]) for i in range(len(lens))]
    T, pad, vd = sum(q_lens), M.group_pad(H, G), e - 8
    q = _rnd(T, G, pad, d, seed=3, dtype=dtype)
    for i, n in enumerate(lens):
        for edge in (0, 63, 64, n - 1 - window, n // 2):
            if 0 <= edge < n:
                ks[i][edge] *= 2.5                            # stands out for many rows
                vs[i][edge] *= 2
    fill()
    sink = _rnd(H, seed=6, scale=2.0) if kind == "sink" else None
    bias = _rnd(H, seed=7) - 3 if kind == "sigmoid" else None
    bm, plain = _blocks(ks, vs, G, d, e, pool, table, lens, page, dtype) if pool else (None, None)
    out = torch.full((T + 1, H * vd), 7.0, dtype=dtype, device="cuda")
    M.grouped_prefill(q, k, v, out[:T], table, _i32(starts), _i32(q_lens), _i32(ctx), max(q_lens), heads=H, vdim=vd, scale=0.15, window=window, sink=sink,
                      sigmoid_bias=bias, pool=bm)
    _status()
    assert (out[T] == 7.0).all()
    for i, n in enumerate(lens):
        s = slice(starts[i], starts[i] + q_lens[i])
        means = [plain[i][0], plain[i][1][..., :vd]] if pool else None
        want = _attend(_cpu(q[s, :, :H // G].reshape(-1, H, d)), _cpu(ks[i]), _cpu(vs[i][..., :vd]), 0.15, ctx[i], window,
                       None if sink is None else _cpu(sink), None if bias is None else _cpu(bias), pool, means)
        _close(out[s], want, dtype, 1.6e-2)


@pytest.mark.parametrize("sink", [-300.0, 0.0, 300.0])
def test_sinks_far_from_the_scores(sink):
    """A sink that vanishes beside the scores, and one beside which they vanish."""
    from crosspool_b200.ops import mixers as M

    k, v, table, ks, vs, fill = _paged([80], 1, 64, 64, 64, torch.bfloat16)
    fill()
    q, sinks = _rnd(80, 1, 4, 64, seed=3, dtype=torch.bfloat16), torch.full((4,), sink, device="cuda")
    want = _attend(_cpu(q.view(80, 4, 64)), _cpu(ks[0]), _cpu(vs[0]), 0.2, 0, 30, _cpu(sinks), None, 0, None)
    out, pos = torch.empty(80, 256, dtype=torch.bfloat16, device="cuda"), torch.arange(80, dtype=torch.int32, device="cuda")
    seq = torch.zeros_like(pos)
    kw = dict(heads=4, vdim=64, scale=0.2, window=30, sink=sinks)
    M.grouped_attn(q, k, v, out, table, pos, pos, dim=64, row_seq=seq, **kw)
    _close(out, want, torch.bfloat16)
    M.grouped_decode(q, k, v, out, table, pos, pos, dim=64, row_seq=seq, num_splits=3, chunk_tokens=16, ws=torch.empty(80 * 4 * 3 * 66, device="cuda"), **kw)
    _close(out, want, torch.bfloat16)
    M.grouped_prefill(q, k, v, out, table, _i32([0]), _i32([80]), _i32([0]), 80, **kw)
    _close(out, want, torch.bfloat16)
    _status()


@pytest.mark.parametrize("shift", [-200.0, 200.0])
def test_sigmoid_weights_that_saturate(shift):
    from crosspool_b200.ops import mixers as M

    k, v, table, ks, vs, fill = _paged([150], 2, 64, 64, 64, torch.bfloat16)
    fill()
    q, bias = _rnd(150, 2, 2, 64, seed=3, dtype=torch.bfloat16), torch.full((4,), shift, device="cuda")
    want = _attend(_cpu(q.view(150, 4, 64)), _cpu(ks[0]), _cpu(vs[0]), 0.2, 0, 20, None, _cpu(bias), 0, None)
    out, pos = torch.empty(150, 256, dtype=torch.bfloat16, device="cuda"), torch.arange(150, dtype=torch.int32, device="cuda")
    kw = dict(heads=4, vdim=64, scale=0.2, window=20, sigmoid_bias=bias)
    M.grouped_attn(q, k, v, out, table, pos, pos, dim=64, row_seq=torch.zeros_like(pos), **kw)
    _close(out, want, torch.bfloat16)
    M.grouped_decode(q, k, v, out, table, pos, pos, dim=64, row_seq=torch.zeros_like(pos), **kw)
    _close(out, want, torch.bfloat16)
    M.grouped_prefill(q, k, v, out, table, _i32([0]), _i32([150]), _i32([0]), 150, **kw)
    _close(out, want, torch.bfloat16)
    _status()


# ------------------------------------------------------------------ latent attention over a window

@pytest.mark.parametrize("window", [1, 40, 64, 130, 1000])
@pytest.mark.parametrize("rank,rot,heads", [(56, 16, 3), (512, 64, 17), (136, 24, 16), (30, 6, 2), (600, 64, 2)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_absorbed_rows_over_a_window(window, rank, rot, heads, dtype):
    from crosspool_b200.ops import mixers as M

    width, page = (rank + rot + 15) // 16 * 16, 64
    lens = [1, 40, 41, 64, 65, 129, 300, 500]
    c, _, table, cs, _, fill = _paged(lens, 1, width, 8, page, dtype)
    q = torch.zeros(heads, len(lens), width, dtype=dtype, device="cuda")
    q[..., :rank + rot] = _rnd(heads, len(lens), rank + rot, seed=3, dtype=dtype, scale=0.5)
    for i, n in enumerate(lens):
        cs[i][..., rank + rot:] = 0
        edge = [n - window, n - window - 1][i % 2]
        if 0 <= edge < n:
            cs[i][edge, 0] = q[:, i].float().mean(0).to(dtype) * 3
    fill()
    pos, slots = _i32([n - 1 for n in lens]), _i32([0] * len(lens))
    scale = (rank + rot) ** -0.5 * 2
    want = torch.zeros(heads, len(lens), rank, dtype=torch.float64)
    for i, n in enumerate(lens):
        seen = oracle.in_window(n, window)[-1:]
        x = _cpu(cs[i][:, 0])
        want[:, i] = oracle.softmax_with_sink(_cpu(q[:, i, :rank + rot]) @ x[:, :rank + rot].T * scale, seen.expand(heads, -1), None) @ x[:, :rank]
    for splits, chunk, simt in ((1, 0, False), (3, 192, False), (8, 64, False), (1, 0, True)):
        if (splits > 1 and (dtype == torch.float32 or rank > 512)) or splits * chunk and splits * chunk < min(window, 500):
            continue                                          # slices are a form of the tensor-core kernel and must cover what is seen
        out = torch.full((heads, len(lens), (rank + 7) // 8 * 8), 7.0, dtype=dtype, device="cuda")
        ws = torch.empty(max(1, len(lens) * heads * splits * (rank + 2)), device="cuda")
        M.latent_attn(q, c, out, table, pos, slots, kv_rank=rank, rot=rot, scale=scale, num_splits=splits, chunk_tokens=chunk, ws=ws, window=window,
                      force_simt=simt)
        _close(out[..., :rank], want, dtype, 1e-4 if dtype == torch.float32 else 0)
    _status()


@pytest.mark.parametrize("window", [1, 40, 64, 100, 1000])
@pytest.mark.parametrize("dim,rot,vdim,heads", [(24, 16, 40, 3), (64, 32, 64, 2), (128, 64, 128, 2)])
@pytest.mark.parametrize("page", [16, 64])
def test_expanded_portions_over_a_window(window, dim, rot, vdim, heads, page):
    """Only what a portion sees is gathered and expanded; every element has a gate of its own."""
    from crosspool_b200.ops import gemm
    from crosspool_b200.ops import mixers as M

    width = 80
    ctx, qn = [0, 37, 128, 5, 300], [130, 27, 64, 300, 40]
    cache, _, table, cs, _, fill = _paged([c + n for c, n in zip(ctx, qn)], 1, width, 8, page, torch.bfloat16, 3)
    fill()
    dq, dv = M.expanded_shape(dim, rot, vdim)
    wk, wv = torch.zeros(heads, dq, width), torch.zeros(heads, dv, width)
    wk[:, :dim + rot] = torch.randn(heads, dim + rot, width, generator=torch.Generator().manual_seed(4)) * width ** -0.5
    wv[:, :vdim] = torch.randn(heads, vdim, width, generator=torch.Generator().manual_seed(5)) * width ** -0.5
    wk, wv = wk.bfloat16().cuda(), wv.bfloat16().cuda()
    base = [max(0, c - window + 1) // 64 * 64 for c in ctx]
    starts, at = [], 0
    for c, n, b in zip(ctx, qn, base):
        starts.append(at)
        at += (c - b + n + 63) // 64 * 64
    lat = torch.zeros(at, width, dtype=torch.bfloat16, device="cuda")
    c_, n_, s_ = _i32(ctx), _i32(qn), _i32(starts)
    M.latent_gather(cache, lat, table, c_, n_, s_, max(c - b + n for c, n, b in zip(ctx, qn, base)), window)
    for i, x in enumerate(cs):
        assert torch.equal(lat[starts[i]:starts[i] + len(x) - base[i]], x[base[i]:, 0])
    k = gemm.linear(lat, wk.view(heads * dq, width)).view(at, heads, dq)
    v = gemm.linear(lat, wv.view(heads * dv, width)).view(at, heads, dv)
    rows, off = sum(qn) + 3, 3                                # three rows of other sequences come first
    q = torch.zeros(rows, heads, dq, dtype=torch.bfloat16, device="cuda")
    q[..., :dim + rot] = _rnd(rows, heads, dim + rot, seed=6, dtype=torch.bfloat16)
    q_starts = [off + sum(qn[:i]) for i in range(5)]
    for i in range(5):                                        # the last token looks for the one before its window, the one before that for its first
        for back in (0, 1):
            j = ctx[i] + qn[i] - 1 - back - window + back
            if j >= base[i]:
                q[q_starts[i] + qn[i] - 1 - back] = 4.0 * k[starts[i] + j - base[i]]
    gate = _rnd(rows, heads * vdim + 8, seed=7, dtype=torch.bfloat16)[:, 8:]
    out = torch.full((rows, heads * vdim), 5.0, dtype=torch.bfloat16, device="cuda")
    M.expanded_prefill(q, k, v, out, _i32(q_starts), n_, c_, s_, max(qn), scale=0.2, vdim=vdim, gate=gate, window=window)
    _status()
    assert (out[:3] == 5.0).all()
    for i in range(5):
        n = ctx[i] + qn[i] - base[i]
        ki, vi = _cpu(k[starts[i]:starts[i] + n]), _cpu(v[starts[i]:starts[i] + n, :, :vdim])
        r = slice(q_starts[i], q_starts[i] + qn[i])
        seen = oracle.in_window(n, window)[ctx[i] - base[i]:]
        want = torch.stack([oracle.softmax_with_sink(_cpu(q[r, h]) @ ki[:, h].T * 0.2, seen, None) @ vi[:, h] for h in range(heads)], 1)
        _close(out[r], want.reshape(qn[i], -1) * torch.sigmoid(_cpu(gate[r])), torch.bfloat16)
