"""Each kernel that Saninex added to the layered decoders alone against its plain restatement (float64 on the CPU)."""
import functools

import pytest
import torch

import saninex_oracle as oracle

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def _rnd(*shape, seed=0, dtype=torch.float32, scale=1.0):
    return (torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale).to(dtype).cuda()


def _close(got, want, dtype):
    t = dict(rtol=2e-5, atol=2e-5) if dtype == torch.float32 else dict(rtol=1.2e-2, atol=1.2e-2)
    assert torch.allclose(got.double().cpu(), want.double().cpu(), **t), (got.double().cpu() - want.double().cpu()).abs().max()


def _i32(x):
    return torch.tensor(x, dtype=torch.int32, device="cuda")


def _status():
    from crosspool_b200.ops import gemm

    gemm.check_status(torch.device("cuda"))


# ------------------------------------------------------------------ products and rows

@pytest.mark.parametrize("rows,ff,k", [(1, 37, 52), (5, 136, 96), (70, 72, 40), (300, 200, 192), (3, 1000, 1024)])
def test_clamped_gated_products_of_any_shape(rows, ff, k):
    from crosspool_b200.models.layered import pad_pitch
    from crosspool_b200.ops import gemm

    x = torch.full((rows, (k + 7) // 8 * 8), float("nan"), dtype=torch.bfloat16, device="cuda")[:, :k]
    x.copy_(_rnd(rows, k, seed=1))
    w = pad_pitch(_rnd(2 * ff, k, seed=2, dtype=torch.bfloat16, scale=k ** -0.5))
    out = torch.full((rows, ff + 8), 7.0, dtype=torch.bfloat16, device="cuda")
    gemm.gateup_swiglu(x, w, out=out[:, :ff], gate_limit=0.7, up_add=1.0, act_alpha=1.702)
    z = x.double() @ w.double().T
    _close(out[:, :ff], oracle.clamped_glu(z[:, :ff], z[:, ff:], 0.7), torch.bfloat16)
    assert (out[:, ff:] == 7.0).all()
    _status()


def test_clamped_gated_activation_in_32_bit():
    from crosspool_b200.ops import mixers as M

    z = _rnd(5, 2 * 37, seed=1, scale=3.0)
    got = M.glu_f32(z, 1.1, 1.0, 1.702, torch.empty(5, 40, device="cuda")[:, :37])
    _close(got, oracle.clamped_glu(z[:, :37].double(), z[:, 37:].double(), 1.1), torch.float32)


@pytest.mark.parametrize("width", [64, 52, 1030, 4096, 6000])
@pytest.mark.parametrize("two", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
def test_norms_behind_a_sublayer(width, two, dtype):
    from crosspool_b200.ops import mixers as M

    R, eps = 7, 1e-3
    resid = _rnd(R, width, seed=1, scale=2.0)
    ys = [_rnd(R, width + 8 * i, seed=2 + i, dtype=dtype, scale=[1.0, 1e-2][i])[:, :width] for i in range(2 if two else 1)]
    w, ow, bw = _rnd(width, seed=5), _rnd(width, seed=6), [_rnd(width, seed=7 + i) for i in range(2)]

    def P(x):
        return M.NormParams("rmsnorm", x, eps=eps)

    y = ys[0].double()
    if two:                                              # the second branch is small: its own norm brings it up, eps counts
        y = 0.5 * sum(oracle.rms(v.double(), eps) * b.double() for v, b in zip(ys, bw))
    new = resid.double() + oracle.rms(y, eps) * w.double()
    kw = dict(branches=ys, branch_norms=[P(b) for b in bw] if two else [], norm=P(w))
    out = torch.full((R, width), 5.0, dtype=dtype, device="cuda")
    sel, before = _i32([5, 0, 5]), resid.clone()
    M.post_norm(resid, out[:3], out_norm=P(ow), sel=sel, **kw)
    assert torch.equal(resid, before) and (out[3:] == 5.0).all()
    _close(out[:3], (oracle.rms(new, eps) * ow.double())[sel.long()], dtype)
    M.post_norm(resid, out, **kw)
    assert torch.allclose(resid.double(), new, rtol=1e-5, atol=1e-5)
    _close(out, new, dtype)
    table, ids = _rnd(11, width, seed=8, dtype=dtype), _i32([3, 10, 0, 3, 7, 1, 2])
    M.post_norm(resid, out, ids=ids, table=table)
    assert torch.equal(resid, table[ids.long()].float()) and torch.equal(out, table[ids.long()])
    M.post_norm(resid, None, **kw)
    _close(resid, table[ids.long()].double() + oracle.rms(y, eps) * w.double(), torch.float32)


@pytest.mark.parametrize("heads,dim", [(3, 7), (4, 128), (1, 40), (5, 264)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_per_head_and_silu_gate(heads, dim, dtype):
    from crosspool_b200.ops import mixers as M

    o, w, g = _rnd(6, heads * dim, seed=1, scale=3.0), _rnd(dim, seed=2), _rnd(6, heads * dim + 3, seed=3, dtype=dtype)[:, :heads * dim]
    o[2] *= 1e-3
    got = M.head_gate(o, w, g, 1e-2, torch.empty(6, heads * dim, dtype=dtype, device="cuda"))
    _close(got, oracle.gated_heads(o.double().view(6, heads, dim), w.double(), g.double(), 1e-2), dtype)


# ------------------------------------------------------------------ grouped-query attention

@pytest.mark.parametrize("heads,kv,dim,vdim", [(6, 2, 24, 40), (3, 1, 10, 13), (4, 4, 128, 128), (5, 1, 160, 72)])
@pytest.mark.parametrize("normed", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
def test_grouped_prep_writes_cache_and_query_layout(heads, kv, dim, vdim, normed, dtype):
    from crosspool_b200.models.config import GroupedMixer
    from crosspool_b200.ops import mixers as M

    (_, dq), (_, dv) = GroupedMixer(heads, kv, dim, vdim, 1.0).cache_rows
    rows, gp, G = 5, M.group_pad(heads, kv), heads // kv
    offs = (8, 16 + heads * dim, 24 + (heads + kv) * dim)
    proj = _rnd(rows, offs[2] + kv * vdim + 5, seed=1, dtype=dtype)
    qn, kn = (_rnd(dim, seed=2), _rnd(dim, seed=3)) if normed else (None, None)
    slots = _i32([5, 0, -1, 31, 32])
    kc, vc = (torch.full((4, 16, kv, n), 9.0, dtype=dtype, device="cuda") for n in (dq, dv))
    q = torch.full((rows, kv, gp, dq), 9.0, dtype=dtype, device="cuda")
    M.grouped_prep(proj, qn, kn, slots, kc, vc, q, heads=heads, dim=dim, vdim=vdim, offs=offs, eps=1e-3)
    x = proj.double().cpu()

    def norm(v, w):
        return v if w is None else oracle.rms(v, 1e-3) * w.double().cpu()

    wq = norm(x[:, offs[0]:offs[0] + heads * dim].view(rows, kv, G, dim), qn)
    _close(q[:, :, :G, :dim], wq, dtype)
    assert (q[:, :, G:] == 0).all() and (q[..., dim:] == 0).all()
    wk = norm(x[:, offs[1]:offs[1] + kv * dim].view(rows, kv, dim), kn)
    wv = x[:, offs[2]:offs[2] + kv * vdim].view(rows, kv, vdim)
    live = [0, 1, 3, 4]
    for cache, want, n in ((kc, wk, dim), (vc, wv, vdim)):
        flat = cache.view(64, kv, -1)
        _close(flat[slots[live].long(), :, :n], want[live], dtype)
        assert (flat[slots[live].long(), :, n:] == 0).all()
        assert all((flat[i] == 9).all() for i in range(64) if i not in slots[live].tolist())


def _caches(lens, page, kv, dim, vdim, dq, dv, dtype, seed, pad_nan=True):
    """Random cache rows of several sequences in shuffled pages; rows that hold no token are NaN."""
    g = torch.Generator().manual_seed(seed)
    need = [(n + page - 1) // page for n in lens]
    perm = torch.randperm(sum(need) + 3, generator=g)
    kc, vc = (torch.full((sum(need) + 3, page, kv, n), float("nan"), dtype=dtype) for n in (dq, dv))
    table, rows, at = torch.zeros(len(lens), max(need), dtype=torch.int32), [], 0
    for i, n in enumerate(lens):
        pages = perm[at:at + need[i]]
        at += need[i]
        table[i, :need[i]] = pages.int()
        slot = pages[torch.arange(n) // page] * page + torch.arange(n) % page
        k, v = torch.zeros(n, kv, dq), torch.zeros(n, kv, dv)
        k[..., :dim], v[..., :vdim] = torch.randn(n, kv, dim, generator=g), torch.randn(n, kv, vdim, generator=g)
        kc.view(-1, kv, dq)[slot], vc.view(-1, kv, dv)[slot] = k.to(dtype), v.to(dtype)
        rows.append((k.to(dtype)[..., :dim].double(), v.to(dtype)[..., :vdim].double()))
    return kc.cuda(), vc.cuda(), table.cuda(), rows


def _attend(q, k, v, n, scale, cap, gate):
    """q ``[H, d]`` against the first n tokens of k ``[T, G, d]``, v ``[T, G, e]``."""
    H, G = q.shape[0], k.shape[1]
    out = []
    for h in range(H):
        s = k[:n, h // (H // G)] @ q[h] * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        out.append(s.softmax(-1) @ v[:n, h // (H // G)] * torch.sigmoid(gate[h]))
    return torch.cat(out)


ATTN_SHAPES = [(6, 2, 24, 40), (3, 1, 10, 13), (8, 2, 128, 128), (5, 1, 160, 72), (4, 4, 64, 64), (12, 1, 100, 64), (17, 1, 16, 24)]


@pytest.mark.parametrize("heads,kv,dim,vdim", ATTN_SHAPES)
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("form", ["f32", "bf16", "bf16-plain", "bf16-split6", "bf16-split3"])
def test_attention_of_single_rows(heads, kv, dim, vdim, page, form):
    from crosspool_b200.models.config import GroupedMixer, attention_shape
    from crosspool_b200.ops import mixers as M

    dtype = torch.float32 if form == "f32" else torch.bfloat16
    (_, dq), (_, dv) = GroupedMixer(heads, kv, dim, vdim, 1.0).cache_rows
    G, gp = heads // kv, M.group_pad(heads, kv)
    lens = [1, 15, 16, 17, 64, 65, 200, 333]
    kc, vc, table, kvs = _caches(lens, page, kv, dim, vdim, dq, dv, dtype, 1)
    rows = len(lens) + 2                                 # row 8: a second query of sequence 6, row 9: padding
    q = torch.zeros(rows, kv, gp, dq)
    q[:, :, :G, :dim] = torch.randn(rows, kv, G, dim, generator=torch.Generator().manual_seed(2))
    for r, j in ((4, 0), (5, 64), (6, 15), (7, 16), (7, 64)):     # far, near and page-border keys that stand out
        q[r, :, :G, :dim] = 4.0 * kvs[r][0][j][:, None].float()
    q = q.to(dtype).cuda()
    pos, seq, slots = _i32([n - 1 for n in lens] + [99, 0]), _i32(list(range(8)) + [6, 0]), _i32([0] * 9 + [-1])
    gate = _rnd(rows, heads + 5, seed=3, dtype=dtype)
    out = torch.full((rows, (heads * vdim + 7) // 8 * 8), 5.0, dtype=dtype, device="cuda")
    kw = dict(heads=heads, dim=dim, vdim=vdim, scale=dim ** -0.5, softcap=9.0, gate=gate, row_seq=seq)
    if form in ("f32", "bf16-plain"):
        M.grouped_attn(q, kc, vc, out, table, pos, slots, **kw)
    else:
        if attention_shape(dim, vdim) is None or gp > 16:
            pytest.skip("no tensor-core kernel for these sizes")
        splits, chunk = {"6": (6, 64), "3": (3, 128)}.get(form[-1], (1, 0)) if "split" in form else (1, 0)
        ws = torch.full((rows * heads * splits * (dv + 2),), float("nan"), device="cuda")
        M.grouped_decode(q, kc, vc, out, table, pos, slots, num_splits=splits, chunk_tokens=chunk, ws=ws, **kw)
    _status()
    for r in range(9):
        k, v = kvs[int(seq[r])]
        want = _attend(q[r, :, :G, :dim].double().cpu().reshape(heads, dim), k, v, int(pos[r]) + 1, dim ** -0.5, 9.0, gate[r].double().cpu())
        _close(out[r, :heads * vdim], want, dtype)
    assert (out[9, :heads * vdim] == 0).all() and (out[:, heads * vdim:] == 5.0).all()


@pytest.mark.parametrize("heads,kv,dim,vdim", [s for s in ATTN_SHAPES if s[3] % 8 == 0 and s[0] // s[1] <= 16])
@pytest.mark.parametrize("page", [16, 64])
@pytest.mark.parametrize("cap", [0.0, 9.0, 0.7])
def test_attention_of_portions(heads, kv, dim, vdim, page, cap):
    """First chunks, later chunks, a chunk that ends a page; marked keys stand out for marked queries."""
    from crosspool_b200.models.config import attention_shape
    from crosspool_b200.ops import mixers as M

    dq, dv = attention_shape(dim, vdim)
    if page < 64 and dq != dv:
        pytest.skip("pages of less than a tile need equal widths")
    G, gp, scale = heads // kv, M.group_pad(heads, kv), dim ** -0.5
    ctx, qn = [0, 37, 128, 5], [130, 27, 64, 300]
    kc, vc, table, kvs = _caches([c + n for c, n in zip(ctx, qn)], page, kv, dim, vdim, dq, dv, torch.bfloat16, 3)
    rows, off = sum(qn) + 3, 3                           # three rows of other sequences come first
    q = torch.zeros(rows, kv, gp, dq)
    q[:, :, :G, :dim] = torch.randn(rows, kv, G, dim, generator=torch.Generator().manual_seed(6))
    q_starts = [off + sum(qn[:i]) for i in range(4)]
    for i, (j, p) in {1: (0, 26), 2: (64, 0), 3: (5, 200), 0: (63, 129)}.items():    # (key, query) of sequence i
        q[q_starts[i] + p, :, :G, :dim] = 4.0 * kvs[i][0][j][:, None].float()
    q = q.bfloat16().cuda()
    gate = _rnd(rows, heads + 3, seed=7, dtype=torch.bfloat16)
    out = torch.full((rows, heads * vdim + 8), 5.0, dtype=torch.bfloat16, device="cuda")
    M.grouped_prefill(q, kc, vc, out, table, _i32(q_starts), _i32(qn), _i32(ctx), max(qn), heads=heads, vdim=vdim, scale=scale, softcap=cap,
                      gate=gate)
    _status()
    assert (out[:3] == 5.0).all() and (out[:, heads * vdim:] == 5.0).all()
    for i in range(4):
        k, v = kvs[i]
        r = slice(q_starts[i], q_starts[i] + qn[i])
        qq = q[r, :, :G, :dim].double().cpu().reshape(qn[i], heads, dim)
        s = torch.einsum("thd,nhd->htn", qq, k.repeat_interleave(G, 1)) * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        s = s.masked_fill(torch.arange(len(k))[None, :] > (ctx[i] + torch.arange(qn[i]))[:, None], float("-inf"))
        want = torch.einsum("htn,nhd->thd", s.softmax(-1), v.repeat_interleave(G, 1)) * torch.sigmoid(gate[r, :heads].double().cpu())[..., None]
        _close(out[r, :heads * vdim], want.reshape(qn[i], -1), torch.bfloat16)


# ------------------------------------------------------------------ recurrences

PORTIONS = [[2, 64, 0], [64, 0, 63], [130, 2, 0], [5, 0, 0]]
TOTAL = [204, 69, 66]


def _schedule():
    """Portions of three sequences, then their tokens one by one with a padding row at the end."""
    done = [0, 0, 0]
    for portions in PORTIONS:
        live = [i for i in range(3) if portions[i]]
        yield live, list(done), [portions[i] for i in live], False
        for i in live:
            done[i] += portions[i]
    while any(d < n for d, n in zip(done, TOTAL)):
        live = [i for i in range(3) if done[i] < TOTAL[i]]
        yield live, list(done), [1] * len(live), True
        for i in live:
            done[i] += 1


def _meta(live, done, lens, slot):
    pos = _i32([done[i] + j for i, n in zip(live, lens) for j in range(n)])
    return pos, _i32([slot[i] for i in live]), _i32([sum(lens[:j]) for j in range(len(lens))]), _i32(lens)


def _compare(o, y, want_o, want_y, state, S, tol):
    """Portions: the recurrence's own fp32 outputs, up to its rounding. Single tokens: the normed and gated heads in the
    activation type. And the last states."""
    for i in range(3):
        n = len(o[i])
        w = want_o[i][:n]
        e = (o[i].double().cpu().view_as(w) - w).abs().max().item() / w.pow(2).mean().sqrt().item()
        assert e < tol, (i, e)
        e = (y[i].double().cpu() - want_y[i][n:]).pow(2).mean(-1).sqrt() / want_y[i][n:].pow(2).mean(-1).sqrt()
        assert e.max().item() < (tol if y[i].dtype == torch.float32 else 1e-2), (i, n + e.argmax().item(), e.max().item())
        e = (state[i].double().cpu() - S[i]).abs().max().item() / S[i].pow(2).mean().sqrt().item()
        assert e < tol, (i, e)


def _offsets(sizes):
    offs = [8]
    for n in sizes:
        offs.append(offs[-1] + (n + 7) // 8 * 8)
    return offs


GLA_SHAPES = [(3, 16, 24), (2, 9, 5), (1, 200, 136), (4, 128, 128), (2, 64, 32), (1, 264, 8), (2, 128, 24)]


@functools.lru_cache(maxsize=None)
def _gla_case(heads, dim, vdim, tau, bias, dtype):
    """Inputs on the device and the plain implementation's outputs."""
    nq, nv, rank, eps = heads * dim, heads * vdim, 12, 1e-3
    offs = _offsets((nq, nq, nv, nv, rank))
    x = [_rnd(n, offs[5], seed=i, dtype=dtype) for i, n in enumerate(TOTAL)]
    a2, b, norm = _rnd(nq, rank, seed=5, dtype=dtype, scale=0.5), _rnd(nq, seed=6, scale=1.5) + bias, _rnd(vdim, seed=7)
    b[::7] += 6.0                                        # channels that hardly forget
    if bias < 0:
        b[3::11] -= 30.0                                 # channels that forget at once: more than a chunk's factors can hold
    zs, o, y, S = [], [], [], []
    for t in x:
        f = t.double().cpu()
        z = f[:, offs[4]:offs[4] + rank] @ a2.double().cpu().T + b.double().cpu()
        q, k = (f[:, c:c + nq].view(-1, heads, dim) for c in offs[:2])
        oo, s = oracle.channel_recurrence(q * dim ** -0.5, k, f[:, offs[2]:offs[2] + nv].reshape(-1, heads, vdim),
                                          torch.sigmoid(z).view_as(q) ** (1 / tau))
        zs.append(z.float().cuda()), o.append(oo), S.append(s)
        y.append(oracle.gated_heads(oo, norm.double().cpu(), f[:, offs[3]:offs[3] + nv], eps))
    return offs, x, a2, b, norm, zs, o, y, S


@pytest.mark.parametrize("form", ["f32", "bf16", "bf16-sequential", "bf16-segments"])
@pytest.mark.parametrize("tau,bias", [(8.0, 1.0), (1.0, 0.0), (1.0, -6.0)])
@pytest.mark.parametrize("heads,dim,vdim", GLA_SHAPES)
def test_gated_linear_attention_portions_and_single_tokens(heads, dim, vdim, tau, bias, form):
    """Three sequences of unequal length in unequal portions, some of two tokens, with single tokens at the end; slots are
    shuffled and hold garbage before. The decays reach from almost one to almost zero, also within a chunk."""
    from crosspool_b200.models.layered import pad_pitch
    from crosspool_b200.ops import mixers as M

    dtype = torch.float32 if form == "f32" else torch.bfloat16
    offs, x, a2, b, norm, zs, want_o, want_y, S = _gla_case(heads, dim, vdim, tau, bias, dtype)
    a2, nv = pad_pitch(a2), heads * vdim
    state = torch.full((4, heads, dim, vdim), float("nan"), device="cuda")
    kw = dict(heads=heads, dim=dim, vdim=vdim, tau=tau)
    slot, o, y = [2, 0, 3], [[], [], []], [[], [], []]
    for live, done, lens, single in _schedule():
        rows = torch.cat([x[i][done[i]:done[i] + n] for i, n in zip(live, lens)])
        pos, ss, starts, ln = _meta(live, done, lens, slot)
        if single:
            rows, pos, ss = torch.cat([rows, x[0][:1]]), torch.cat([pos, _i32([0])]), torch.cat([ss, ss[-1:]])
            out = torch.full((len(rows), nv), 5.0, dtype=dtype, device="cuda")
            M.gated_linear_decode(rows, state, a2, b, norm, out, pos, _i32([0] * len(live) + [-1]), ss, offs=tuple(offs[:5]), eps=1e-3, **kw)
            assert (out[-1] == 0).all()
        else:
            z = torch.cat([zs[i][done[i]:done[i] + n] for i, n in zip(live, lens)])
            out = torch.full((len(rows), nv), 5.0, device="cuda")
            # segments of one chunk: portions of 64 tokens end with their first segment, longer ones do not
            scratch = M.GatedLinearScratch.for_rows(len(rows), len(live), heads, dim, vdim, "cuda")
            scratch.ws = torch.full((len(live) * 3 * heads * dim * (vdim + 1),), float("nan"), device="cuda")
            M.gated_linear_prefill(rows, z, state, out, pos, pos, ss, starts, ln, max(lens), None if form == "f32" else scratch,
                                   offs=tuple(offs[:3]), force_sequential=form == "bf16-sequential",
                                   **(dict(segs=3, seg_tokens=64) if form == "bf16-segments" else {}), **kw)
        for i, t in zip(live, out[:sum(lens)].split(lens)):
            (y if single else o)[i].append(t)
    _status()
    assert state[1].isnan().all()
    # the state and everything around it is fp32 (or a bf16 pair) also for bf16 inputs: far tighter than bf16
    _compare([torch.cat(t) for t in o], [torch.cat(t) for t in y], want_o, want_y, [state[i] for i in slot], S, 3e-4)


DELTA_CASES = [(6, 3, 24, 40, 4), (3, 1, 20, 7, 2), (2, 2, 48, 16, 3), (4, 2, 128, 128, 4), (2, 1, 256, 256, 4), (3, 3, 72, 136, 1), (4, 4, 128, 24, 6)]


@functools.lru_cache(maxsize=None)
def _delta_case(heads, kv, dim, vdim, taps, strong, dtype):
    nq, nv, eps = kv * dim, heads * vdim, 1e-3
    offs = _offsets((nq, nq, nv, nv, heads, heads))
    x = [_rnd(n, offs[6], seed=i, dtype=dtype) for i, n in enumerate(TOTAL)]
    conv = _rnd(2 * nq + nv, taps, seed=4, scale=taps ** -0.5)
    if strong:
        conv = conv.abs()
        for t in x:
            t[:, offs[1]:offs[1] + nq] += 2.0 * t[:1, offs[1]:offs[1] + nq]      # keys share a direction
            t[:, offs[4]:offs[4] + heads] += 3.0
            t[:, offs[5]:offs[5] + heads] -= 4.0
    neg_a, dt_bias, norm = -_rnd(heads, seed=5).exp(), _rnd(heads, seed=6), _rnd(vdim, seed=7)
    rows = []
    for t in x:
        f, cw = t.double().cpu(), conv.double().cpu()
        rows.append(torch.cat([oracle.silu(oracle.short_convolution(f[:, c:c + n], cw[at:at + n]))
                               for c, n, at in ((offs[0], nq, 0), (offs[1], nq, nq), (offs[2], nv, 2 * nq))], 1))
    return offs, x, conv, neg_a, dt_bias, norm, rows


def _delta_expected(case, heads, kv, dim, vdim, rows, eps=1e-3):
    """The plain implementation behind the convolution, for convolved ``rows`` of every sequence."""
    offs, x, _, neg_a, dt_bias, norm, _ = case
    nq, nv, of = kv * dim, heads * vdim, torch.arange(heads) // (heads // kv)
    o, y, S = [], [], []
    for t, r in zip(x, rows):
        f = t.double().cpu()
        q, k = (oracle.unit(p.view(-1, kv, dim))[:, of] for p in (r[:, :nq], r[:, nq:2 * nq]))
        step = torch.nn.functional.softplus(f[:, offs[5]:offs[5] + heads] + dt_bias.double().cpu())
        oo, s = oracle.delta_recurrence(q * dim ** -0.5, k, r[:, 2 * nq:].reshape(-1, heads, vdim), torch.sigmoid(f[:, offs[4]:offs[4] + heads]),
                                        torch.exp(neg_a.double().cpu() * step))
        o.append(oo), S.append(s), y.append(oracle.gated_heads(oo, norm.double().cpu(), f[:, offs[3]:offs[3] + nv], eps))
    return o, y, S


@pytest.mark.parametrize("form", ["f32", "bf16", "bf16-sequential"])
@pytest.mark.parametrize("strong", [False, True])
@pytest.mark.parametrize("heads,kv,dim,vdim,taps", DELTA_CASES)
def test_delta_rule_portions_and_single_tokens(heads, kv, dim, vdim, taps, strong, form):
    """As above. Strong: writes that replace almost everything under keys that come again and again, slow decay, so that
    hundreds of writes correct one another."""
    from crosspool_b200.ops import mixers as M

    dtype = torch.float32 if form == "f32" else torch.bfloat16
    case = _delta_case(heads, kv, dim, vdim, taps, strong, dtype)
    offs, x, conv, neg_a, dt_bias, norm, exact = case
    conved = [[], [], []]
    nv, channels = heads * vdim, conv.shape[0]
    w = M.DeltaWeights(conv, neg_a, dt_bias, norm)
    state = torch.full((4, heads, dim, vdim), float("nan"), device="cuda")
    ring = torch.full((4, taps, channels), float("nan"), dtype=dtype, device="cuda")
    kw = dict(heads=heads, kv_heads=kv, dim=dim, vdim=vdim, offs=tuple(offs[:6]), eps=1e-3)
    slot, o, y = [2, 0, 3], [[], [], []], [[], [], []]
    for live, done, lens, single in _schedule():
        rows = torch.cat([x[i][done[i]:done[i] + n] for i, n in zip(live, lens)])
        pos, ss, starts, ln = _meta(live, done, lens, slot)
        if single:
            rows, pos, ss = torch.cat([rows, x[0][:1]]), torch.cat([pos, _i32([0])]), torch.cat([ss, ss[-1:]])
            out = torch.full((len(rows), nv), 5.0, dtype=dtype, device="cuda")
            M.delta_decode(rows, ring, w, state, out, pos, _i32([0] * len(live) + [-1]), ss, **kw)
            assert (out[-1] == 0).all()
        else:
            out = torch.full((len(rows), nv), 5.0, device="cuda")
            scratch = M.DeltaScratch.for_rows(len(rows), len(live), heads, kv, dim, vdim, dtype, "cuda")
            M.delta_prefill(rows, ring, w, state, out, pos, pos, ss, starts, ln, max(lens), scratch, force_sequential=form == "bf16-sequential", **kw)
            for i, t in zip(live, scratch.qkv.view(-1, channels).split(lens)):
                conved[i].append(t.double().cpu())
        for i, t in zip(live, out[:sum(lens)].split(lens)):
            (y if single else o)[i].append(t)
    _status()
    assert state[1].isnan().all() and ring[1].isnan().all()
    # the convolution by itself, then the recurrence on the rows as the convolution left them (single tokens keep fp32 rows)
    for i in range(3):
        conved[i] = torch.cat(conved[i])
        _close(conved[i], exact[i][:len(conved[i])], dtype)
        conved[i] = torch.cat([conved[i], exact[i][len(conved[i]):]])
    want_o, want_y, S = _delta_expected(case, heads, kv, dim, vdim, conved)
    _compare([torch.cat(t) for t in o], [torch.cat(t) for t in y], want_o, want_y, [state[i] for i in slot], S,
             1e-3 if strong and form == "bf16" else 3e-4)


def test_segment_plans_cover_the_portion_and_fit_the_workspace():
    from crosspool_b200.ops import mixers as M

    for seqs, heads, vdim, q in [(1, 16, 128, 4096), (1, 1, 32, 64), (3, 2, 136, 1000), (40, 16, 128, 100), (1, 1, 256, 9000), (1, 32, 128, 4096)]:
        segs, tokens = M.gated_linear_plan(seqs, heads, vdim, q)
        assert tokens % 64 == 0 and segs * tokens >= q and (segs - 1) * tokens < q
        assert segs == 1 or seqs * heads * segs <= 2 * 148
