"""Each kernel of the layered decoders alone against its plain restatement (float64 on the CPU)."""
import pytest
import torch

import segirax_oracle as oracle

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _tol(dtype):
    return dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1.2e-2, atol=1.2e-2)


def _rnd(*shape, seed=0, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype).cuda()


def _close(got, want, dtype, scale=1.0):
    t = _tol(dtype)
    assert torch.allclose(got.double().cpu() / scale, want.double().cpu() / scale, **t), (got.double().cpu() - want.double().cpu()).abs().max()


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


# ------------------------------------------------------------------ products

@pytest.mark.parametrize("rows,n,k", [(1, 6, 40), (5, 130, 64), (70, 320, 136), (300, 200, 72), (3, 1000, 1024)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_products_of_any_shape_with_scale_bias_and_silu(rows, n, k, dtype):
    from crosspool_b200.models.layered import ceil8, pad_pitch
    from crosspool_b200.ops import gemm

    x = torch.full((rows, ceil8(k)), float("nan"), dtype=dtype, device="cuda")[:, :k]   # the pitch's padding is never read
    x.copy_(_rnd(rows, k, seed=1))
    w, bias = pad_pitch(_rnd(n, k, seed=2, dtype=dtype, scale=k ** -0.5)), _rnd(n, seed=3)
    out = torch.full((rows, n + 8), 7.0, device="cuda")
    got = gemm.linear(x, w, out=out[:, :n], bias=bias, out_scale=0.5, silu_cols=n // 2)
    want = x.double() @ w.double().T * 0.5 + bias.double()
    want[:, :n // 2] = oracle.silu(want[:, :n // 2])
    _close(got, want, torch.float32 if dtype == torch.float32 else dtype)
    assert (out[:, n:] == 7.0).all()
    gemm.check_status(torch.device("cuda"))


@pytest.mark.parametrize("groups,rows,n,k", [(3, 5, 56, 24), (17, 1, 200, 16), (2, 70, 130, 128), (6, 20, 12, 40)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_batched_products_store_each_group_at_its_stride(groups, rows, n, k, dtype):
    from crosspool_b200.ops import gemm

    x, w = _rnd(groups, rows, k, seed=1, dtype=dtype), _rnd(groups * n, k, seed=2, dtype=dtype, scale=k ** -0.5)
    out = torch.full((rows, groups * n + 16), 7.0, dtype=dtype, device="cuda")
    gemm.linear_batched(x, w, out, n)                      # head after head in one row
    want = torch.einsum("grk,gnk->rgn", x.double(), w.double().view(groups, n, k)).reshape(rows, groups * n)
    _close(out[:, :groups * n], want, dtype)
    assert (out[:, groups * n:] == 7.0).all()
    gemm.check_status(torch.device("cuda"))


# ------------------------------------------------------------------ rows

@pytest.mark.parametrize("width", [64, 52, 1030, 4096])
@pytest.mark.parametrize("kind", ["rmsnorm", "layernorm", "dyt"])
@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_residual_and_norm(width, kind, dtype):
    from crosspool_b200.ops import mixers as M

    R = 7
    resid, y, z = _rnd(R, width, seed=1, scale=2.0), _rnd(R, width, seed=2, dtype=dtype), _rnd(R, width, seed=3, dtype=dtype)
    gate, w, b, alpha = _rnd(R, width + 8, seed=4, dtype=dtype, scale=2.0)[:, :width], _rnd(width, seed=5), _rnd(width, seed=6), _rnd(1, seed=7)
    p = M.NormParams(kind, w, b, alpha, 1e-3)

    def norm(x):
        x, W, B = x.double(), w.double(), b.double()
        if kind == "dyt":
            return oracle.dynamic_tanh(x, alpha.double(), W, B)
        return oracle.rms(x - x.mean(-1, keepdim=True) if kind == "layernorm" else x, 1e-3) * W + B

    new = resid.double() + (y.double() + z.double()) * torch.sigmoid(gate.double())
    out = torch.empty(R, width, dtype=dtype, device="cuda")
    sel = _i32([5, 0, 5])
    before = resid.clone()
    M.resid_norm(resid, p, out[:3], parts=[y, z], gate=gate, sel=sel)
    assert torch.equal(resid, before)
    _close(out[:3], norm(new)[sel.long()], dtype)
    M.resid_norm(resid, p, out, parts=[y, z], gate=gate)
    assert torch.allclose(resid.double(), new, rtol=1e-5, atol=1e-5)
    _close(out, norm(resid), dtype)
    table = _rnd(11, width, seed=8, dtype=dtype)
    ids = _i32([3, 10, 0, 3, 7, 1, 2])
    M.resid_norm(resid, p, out, ids=ids, table=table)
    assert torch.equal(resid, table[ids.long()].float())
    _close(out, norm(resid), dtype)
    M.resid_norm(resid, None, None, parts=[y])
    assert torch.allclose(resid, table[ids.long()].float() + y.float())


@pytest.mark.parametrize("cols", [37, 136, 4100, 9000])
@pytest.mark.parametrize("dtype", DTYPES)
def test_polynorm(cols, dtype):
    from crosspool_b200.ops import mixers as M

    z, coef = _rnd(5, cols, seed=1, dtype=dtype, scale=1.5), torch.tensor([0.7, -0.4, 0.3, 0.2], device="cuda")
    z[1] *= 1e-3                                             # eps matters inside the root
    want = oracle.poly_norm(z.double(), coef.double(), 1e-4)
    got = M.polynorm(z, coef, 1e-4, torch.empty_like(z))
    _close(got, want, dtype, scale=max(1.0, want.abs().max().item()))
    M.polynorm(z, coef, 1e-4, z)
    assert torch.equal(z, got)


@pytest.mark.parametrize("cols", [21, 128, 2048])
@pytest.mark.parametrize("dtype", DTYPES)
def test_gated_rms(cols, dtype):
    from crosspool_b200.ops import mixers as M

    o, w, g = _rnd(4, cols, seed=1, scale=3.0), _rnd(cols, seed=2), _rnd(4, cols + 3, seed=3, dtype=dtype)[:, :cols]
    got = M.gated_rms(o, w, g, 1e-2, torch.empty(4, cols, dtype=dtype, device="cuda"))
    _close(got, oracle.rms(o.double(), 1e-2) * w.double() * torch.sigmoid(g.double()), dtype)


# ------------------------------------------------------------------ latent attention

def _paged(lens, page, width, dtype, seed):
    """Random cache rows of several sequences in shuffled pages; every page holds NaN outside its live rows."""
    g = torch.Generator().manual_seed(seed)
    need = [(n + page - 1) // page for n in lens]
    perm = torch.randperm(sum(need) + 3, generator=g)
    cache = torch.full((sum(need) + 3, page, 1, width), float("nan"), dtype=dtype)
    table = torch.zeros(len(lens), max(need), dtype=torch.int32)
    rows, at = [], 0
    for i, n in enumerate(lens):
        pages = perm[at:at + need[i]]
        at += need[i]
        table[i, :need[i]] = pages.int()
        x = torch.randn(n, width, generator=g).to(dtype)
        slot = pages[torch.arange(n) // page] * page + torch.arange(n) % page
        cache.view(-1, width)[slot] = x
        rows.append(x)
    return cache.cuda(), table.cuda(), rows


@pytest.mark.parametrize("heads,rank,rot", [(1, 30, 6), (3, 56, 16), (17, 200, 32), (16, 512, 64), (2, 120, 8)])
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("form", ["f32", "bf16", "bf16-plain", "bf16-split6", "bf16-split3"])
def test_latent_attention_of_single_rows(heads, rank, rot, page, form):
    from crosspool_b200.ops import mixers as M

    dtype = torch.float32 if form == "f32" else torch.bfloat16
    width = (rank + rot + 15) // 16 * 16
    lens = [1, 15, 16, 17, 64, 65, 200, 333]
    cache, table, kv = _paged(lens, page, width, dtype, 1)
    for x in kv:
        x[:, rank + rot:] = 0
    cache.view(-1, width)[:, rank + rot:] = 0                # what the writer of the cache guarantees
    rows = len(lens) + 2                                     # row 8: a second query of sequence 6, row 9: padding
    q = _rnd(heads, rows, width, seed=2, dtype=dtype)
    # one far, one near and one page-border key stand out by far for some queries
    for r, j in ((4, 0), (5, 64), (6, 15), (7, 16)):
        q[:, r] = 3.0 * cache.view(-1, width)[int(table[r, j // page]) * page + j % page]
    pos = _i32([n - 1 for n in lens] + [99, 0])
    seq, slots = _i32(list(range(8)) + [6, 0]), _i32([0] * 9 + [-1])
    gate = _rnd(rows, heads + 5, seed=3, dtype=dtype)
    out = torch.full((heads, rows, (rank + 7) // 8 * 8), 5.0, dtype=dtype, device="cuda")
    splits, chunk = {"6": (6, 64), "3": (3, 128)}.get(form[-1], (1, 0)) if "split" in form else (1, 0)
    ws = torch.empty(rows * heads * splits * (rank + 2), device="cuda")
    M.latent_attn(q, cache, out, table, pos, slots, kv_rank=rank, rot=rot, scale=0.11, gate=gate, row_seq=seq, num_splits=splits,
                  chunk_tokens=chunk, ws=ws, force_simt=form == "bf16-plain")
    from crosspool_b200.ops import gemm

    gemm.check_status(torch.device("cuda"))
    for r in range(9):
        k = kv[int(seq[r])][:int(pos[r]) + 1].double()
        s = q[:, r, :rank + rot].double().cpu() @ k[:, :rank + rot].T * 0.11
        want = s.softmax(-1) @ k[:, :rank] * torch.sigmoid(gate[r, :heads].double().cpu())[:, None]
        _close(out[:, r, :rank], want, dtype)
    assert (out[:, 9, :rank] == 0).all()


@pytest.mark.parametrize("dim,rot,dims,rank,heads", [(24, 16, 16, 56, 3), (10, 6, 4, 30, 2), (128, 64, 64, 512, 2)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_latent_prep_writes_cache_and_query_layouts(dim, rot, dims, rank, heads, dtype):
    from crosspool_b200.models.layered import rotary_frequencies
    from crosspool_b200.ops import mixers as M

    rows, ab = 6, 2
    width, dp, dq = (rank + rot + 15) // 16 * 16, (dim + 7) // 8 * 8, (dim + rot + 63) // 64 * 64
    q_off, kv_off = 8, 8 + heads * (dim + rot)
    proj = _rnd(rows, kv_off + rank + rot, seed=1, dtype=dtype)
    nw, freq = _rnd(rank, seed=2), rotary_frequencies(dims, 1e4).cuda()
    pos, slots = _i32([0, 1, 17, 1000, 100000, 3]), _i32([5, 0, 31, 32, -1, 9])
    cache = torch.full((4, 16, 1, width), 9.0, dtype=dtype, device="cuda")
    qp, qa = torch.full((heads, ab, dp), 9.0, dtype=dtype, device="cuda"), torch.full((heads, ab, width), 9.0, dtype=dtype, device="cuda")
    qe = torch.full((rows, heads, dq), 9.0, dtype=dtype, device="cuda")
    M.latent_prep(proj, nw, freq, pos, slots, cache, heads=heads, dim=dim, rot=rot, kv_rank=rank, q_off=q_off, kv_off=kv_off, eps=1e-3,
                  abs_rows=ab, q_plain=qp, q_abs=qa, q_exp=qe)
    x, P = proj.double().cpu(), pos.cpu()
    kv = torch.cat([oracle.rms(x[:, kv_off:kv_off + rank], 1e-3) * nw.double().cpu(), oracle.rotate_half(x[:, kv_off + rank:], P, dims, 1e4)], -1)
    q = x[:, q_off:kv_off].view(rows, heads, dim + rot)
    q = torch.cat([q[..., :dim], oracle.rotate_half(q[..., dim:], P, dims, 1e4)], -1)
    flat = cache.view(-1, width)
    for r in (0, 1, 2, 3, 5):
        _close(flat[slots[r], :rank + rot], kv[r], dtype)
        assert (flat[slots[r], rank + rot:] == 0).all()
    live = set(slots.tolist())
    assert all((flat[i] == 9).all() for i in range(64) if i not in live)
    _close(qp[:, :, :dim].transpose(0, 1), q[:ab, :, :dim], dtype)
    assert (qp[:, :, dim:] == 0).all() and (qa[:, :, :rank] == 9).all() and (qa[:, :, rank + rot:] == 0).all()
    _close(qa[:, :, rank:rank + rot].transpose(0, 1), q[:ab, :, dim:], dtype)
    _close(qe[ab:, :, :dim + rot], q[ab:], dtype)
    assert (qe[ab:, :, dim + rot:] == 0).all() and (qe[:ab] == 9).all()


@pytest.mark.parametrize("dim,rot,vdim,heads", [(24, 16, 40, 3), (64, 32, 64, 2), (40, 40, 128, 2), (128, 64, 128, 2), (16, 8, 8, 5)])
@pytest.mark.parametrize("page", [16, 64])
def test_expanded_prefill_over_gathered_latents(dim, rot, vdim, heads, page):
    """Portions of several sequences (first chunks, later chunks, a chunk that ends a page) through gather, expansion and the
    tcgen05 kernel; per-head keys are random maps of the cached row, so a wrong row or head shows."""
    from crosspool_b200.ops import gemm
    from crosspool_b200.ops import mixers as M

    width = 80
    ctx, qn = [0, 37, 128, 5], [130, 27, 64, 300]
    cache, table, kv = _paged([c + n for c, n in zip(ctx, qn)], page, width, torch.bfloat16, 3)
    dq, dv = M.expanded_shape(dim, rot, vdim)
    wk = torch.zeros(heads, dq, width)
    wk[:, :dim + rot] = torch.randn(heads, dim + rot, width, generator=torch.Generator().manual_seed(4)) * width ** -0.5
    wv = torch.zeros(heads, dv, width)
    wv[:, :vdim] = torch.randn(heads, vdim, width, generator=torch.Generator().manual_seed(5)) * width ** -0.5
    wk, wv = wk.bfloat16().cuda(), wv.bfloat16().cuda()
    starts, at = [], 0
    for c, n in zip(ctx, qn):
        starts.append(at)
        at += (c + n + 63) // 64 * 64
    lat = torch.zeros(at, width, dtype=torch.bfloat16, device="cuda")
    c_, n_, s_ = _i32(ctx), _i32(qn), _i32(starts)
    M.latent_gather(cache, lat, table, c_, n_, s_, max(c + n for c, n in zip(ctx, qn)))
    for i, x in enumerate(kv):
        assert torch.equal(lat[starts[i]:starts[i] + len(x)].cpu(), x)
    k = gemm.linear(lat, wk.view(heads * dq, width)).view(at, heads, dq)
    v = gemm.linear(lat, wv.view(heads * dv, width)).view(at, heads, dv)
    rows, off = sum(qn) + 3, 3                                # three rows of other sequences come first
    q = torch.zeros(rows, heads, dq, dtype=torch.bfloat16, device="cuda")
    q[..., :dim + rot] = _rnd(rows, heads, dim + rot, seed=6, dtype=torch.bfloat16)
    q_starts = [off + sum(qn[:i]) for i in range(4)]
    far = {1: (0, 26), 2: (64, 0), 3: (5, 200)}               # (key, query) that stands out in sequence i
    for i, (j, p) in far.items():
        q[q_starts[i] + p] = 4.0 * k[starts[i] + j]
    gate = _rnd(rows, heads, seed=7, dtype=torch.bfloat16)
    out = torch.full((rows, heads * vdim), 5.0, dtype=torch.bfloat16, device="cuda")
    M.expanded_prefill(q, k, v, out, _i32(q_starts), n_, c_, s_, max(qn), scale=0.2, vdim=vdim, gate=gate)
    gemm.check_status(torch.device("cuda"))
    assert (out[:3] == 5.0).all()
    for i in range(4):
        T = ctx[i] + qn[i]
        ki, vi = k[starts[i]:starts[i] + T].double().cpu(), v[starts[i]:starts[i] + T, :, :vdim].double().cpu()
        r = slice(q_starts[i], q_starts[i] + qn[i])
        s = torch.einsum("thd,nhd->htn", q[r].double().cpu(), ki) * 0.2
        s = s.masked_fill(torch.arange(T)[None, :] > (ctx[i] + torch.arange(qn[i]))[:, None], float("-inf"))
        want = torch.einsum("htn,nhd->thd", s.softmax(-1), vi) * torch.sigmoid(gate[r].double().cpu())[..., None]
        _close(out[r], want.reshape(qn[i], -1), torch.bfloat16)


# ------------------------------------------------------------------ linear attention

@pytest.mark.parametrize("heads,dim,vdim", [(2, 48, 24), (3, 20, 7), (1, 200, 136), (4, 128, 128), (2, 64, 32), (1, 8, 16)])
@pytest.mark.parametrize("form", ["f32", "bf16", "bf16-sequential", "bf16-segments"])
def test_linear_attention_portions_and_single_tokens(heads, dim, vdim, form):
    """Three sequences of unequal length in unequal portions, some of two tokens, with single tokens at the end; slots are
    shuffled and hold garbage before."""
    from crosspool_b200.ops import mixers as M

    dtype = torch.float32 if form == "f32" else torch.bfloat16
    decay = [0.5, 0.98, 1.0, 0.0][:heads]
    nq, nk = heads * dim, heads * vdim
    offs = (8, 8 + (nq + 7) // 8 * 8, 8 + 2 * ((nq + 7) // 8 * 8))
    ld = offs[2] + (nk + 7) // 8 * 8
    total = [203, 66, 64]
    x = [_rnd(n, ld, seed=i, dtype=dtype) for i, n in enumerate(total)]
    state = torch.full((4, heads, dim, vdim), float("nan"), device="cuda")
    dec, pw = torch.tensor(decay, device="cuda"), M.decay_powers(decay).cuda()
    kw = dict(heads=heads, dim=dim, vdim=vdim, offs=offs)
    slot, done, got = [2, 0, 3], [0, 0, 0], [[], [], []]
    for portions in ([2, 64, 0], [64, 0, 63], [130, 2, 0], [5, 0, 0]):
        live = [i for i in range(3) if portions[i]]
        rows = torch.cat([x[i][done[i]:done[i] + portions[i]] for i in live])
        pos = _i32([done[i] + j for i in live for j in range(portions[i])])
        lens = [portions[i] for i in live]
        out = torch.full((len(rows), heads * vdim), 5.0, device="cuda")
        # segments of one chunk: portions of 64 tokens end with their first segment, longer ones do not
        segs = dict(segs=3, seg_tokens=64, ws=torch.full((len(live) * 3 * heads * dim * vdim,), float("nan"), device="cuda")) \
            if form == "bf16-segments" else {}
        M.linear_attn_prefill(rows, state, dec, pw, out, pos, pos, _i32([slot[i] for i in live]), _i32([sum(lens[:j]) for j in range(len(lens))]),
                              _i32(lens), force_sequential=form == "bf16-sequential", **segs, **kw)
        for i, o in zip(live, out.split(lens)):
            got[i].append(o)
            done[i] += portions[i]
    while any(d < n for d, n in zip(done, total)):            # single tokens, one padding row among them
        live = [i for i in range(3) if done[i] < total[i]]
        rows = torch.cat([x[i][done[i]:done[i] + 1] for i in live] + [x[0][:1]])
        out = torch.full((len(rows), heads * vdim), 5.0, device="cuda")
        M.linear_attn_decode(rows, state, dec, pw, out, _i32([done[i] for i in live] + [0]), _i32([0] * len(live) + [-1]),
                             _i32([slot[i] for i in live] + [slot[live[0]]]), **kw)
        assert (out[-1] == 0).all()
        for i, o in zip(live, out):
            got[i].append(o[None])
            done[i] += 1
    assert state[1].isnan().all()
    for i in range(3):
        xs = x[i].double().cpu()
        q, k = (xs[:, o:o + nq].view(-1, heads, dim) for o in offs[:2])
        want, S = oracle.decayed_recurrence(q, k, xs[:, offs[2]:offs[2] + nk].reshape(-1, heads, vdim), decay)
        # the state and everything around it is fp32 (or a bf16 pair) also for bf16 inputs: far tighter than bf16
        scale = want.pow(2).mean().sqrt().item()
        assert (torch.cat(got[i]).double().cpu().view_as(want) - want).abs().max().item() < 2e-4 * scale
        assert (state[slot[i]].double().cpu() - S).abs().max().item() < 2e-4 * S.pow(2).mean().sqrt().item()


def test_segment_plans_cover_the_portion_and_fit_the_workspace():
    from crosspool_b200.ops import mixers as M

    for seqs, heads, dim, vdim, q in [(1, 16, 128, 128, 4096), (1, 1, 64, 32, 64), (3, 2, 200, 136, 1000), (40, 16, 128, 128, 100), (1, 1, 256, 256, 9000)]:
        segs, tokens = M.linear_attn_plan(seqs, heads, dim, vdim, q)
        assert tokens % 64 == 0 and segs * tokens >= q and (segs - 1) * tokens < q
        assert segs == 1 or seqs * heads * segs * dim * vdim <= M.linear_attn_ws_elems(dim, vdim)
