"""Each kernel that Kadavik added to the layered decoders, or extended, alone against its plain restatement (float64 on the
CPU)."""
import math

import pytest
import torch

import kadavik_oracle as oracle

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


# ------------------------------------------------------------------ products and rows

@pytest.mark.parametrize("rows,ff,k", [(1, 37, 52), (5, 136, 96), (70, 72, 40), (300, 200, 192), (3, 1000, 1024)])
def test_gelu_products_of_any_shape(rows, ff, k):
    from crosspool_b200.models.config import GELU_ALPHA, GELU_CUBIC
    from crosspool_b200.models.layered import pad_pitch
    from crosspool_b200.ops import gemm

    x, w = _pitched(rows, k, torch.bfloat16, 1), pad_pitch(_rnd(2 * ff, k, seed=2, dtype=torch.bfloat16, scale=2 * k ** -0.5))
    out = torch.full((rows, ff + 8), 7.0, dtype=torch.bfloat16, device="cuda")
    gemm.gateup_swiglu(x, w, out=out[:, :ff], act_alpha=GELU_ALPHA, act_cubic=GELU_CUBIC)
    z = x.double() @ w.double().T
    _close(out[:, :ff], oracle.gelu_tanh(z[:, :ff]) * z[:, ff:], torch.bfloat16, 2e-2)
    assert (out[:, ff:] == 7.0).all()
    _status()


def test_gelu_far_from_zero():
    from crosspool_b200.models.config import GELU_ALPHA, GELU_CUBIC
    from crosspool_b200.ops import gemm, mixers as M

    g = torch.tensor([-1e3, -60.0, -20.0, -6.0, -1.0, 0.0, 1.0, 6.0, 20.0, 60.0, 1e3])
    w = torch.zeros(2 * 11, 64, dtype=torch.bfloat16)
    w[:11, 0], w[11:, 1] = g.bfloat16(), 1.0
    x = torch.zeros(3, 64, dtype=torch.bfloat16)
    x[:, :2] = 1.0
    out = gemm.gateup_swiglu(x.cuda(), w.cuda(), out=torch.empty(3, 16, dtype=torch.bfloat16, device="cuda")[:, :11], act_alpha=GELU_ALPHA,
                             act_cubic=GELU_CUBIC)
    _close(out, oracle.gelu_tanh(g.bfloat16().double()).expand(3, 11), torch.bfloat16)
    z = torch.cat([g, torch.ones(11)]).cuda().expand(3, 22).contiguous()
    _close(M.glu_f32(z, 0.0, 0.0, GELU_ALPHA, torch.empty(3, 11, device="cuda"), GELU_CUBIC), oracle.gelu_tanh(g.double()).expand(3, 11), torch.float32)
    _status()


@pytest.mark.parametrize("rows,n,k", [(1, 10, 52), (4, 24, 96), (130, 40, 160), (37, 300, 512)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_gelu_gate(rows, n, k, dtype):
    """Product, activation and a column range of other rows."""
    from crosspool_b200.models.layered import pad_pitch
    from crosspool_b200.ops import mixers as M

    x, w = _pitched(rows, k, dtype, 1), pad_pitch(_rnd(n, k, seed=2, dtype=dtype, scale=k ** -0.5))
    e = _rnd(rows, 3 * n, seed=3, dtype=dtype)[:, n:2 * n]
    out = torch.full((rows, (n + 7) // 8 * 8), 7.0, dtype=dtype, device="cuda")
    M.gelu_gate(x, w, e, out[:, :n])
    want = oracle.gelu_tanh(x.double() @ w.double().T) * e.double()
    _close(out[:, :n], want, dtype, 2e-2 if dtype == torch.bfloat16 else 0)
    assert (out[:, n:] == 7.0).all()
    _status()


@pytest.mark.parametrize("rows", [1, 7, 200])
@pytest.mark.parametrize("n,tail", [(784, 16), (96, 40), (1032, 9)])
def test_product_with_fp32_columns(rows, n, tail):
    """The last features of a bf16 product keep their 32 bits, biases included."""
    from crosspool_b200.ops import gemm

    x, w, bias = _rnd(rows, 256, seed=1, dtype=torch.bfloat16), _rnd(n, 256, seed=2, dtype=torch.bfloat16), _rnd(n, seed=3)
    pitch = (n + 7) // 8 * 8
    out = torch.full((rows, pitch), 7.0, dtype=torch.bfloat16, device="cuda")
    t = torch.full((rows, tail + 3), 7.0, device="cuda")
    gemm.linear(x, w, out=out[:, :n], bias=bias, tail=t[:, :tail])
    want = x.double() @ w.double().T + bias.double()
    _close(out[:, :n - tail], want[:, :-tail], torch.bfloat16)
    _close(t[:, :tail], want[:, -tail:], torch.float32, 1e-4)
    assert (out[:, n - tail:] == 7.0).all() and (t[:, tail:] == 7.0).all()
    _status()


@pytest.mark.parametrize("heads,dim", [(1, 5), (3, 40), (4, 128)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_norm_per_head_with_its_own_weights_and_a_sigmoid(heads, dim, dtype):
    from crosspool_b200.ops import mixers as M

    n = heads * dim
    o, w, gate = _rnd(9, n, seed=1), _rnd(n, seed=2), _rnd(9, n + 8, seed=3, dtype=dtype)[:, 8:]
    out = torch.empty(9, n, dtype=dtype, device="cuda")
    M.head_gate(o, w, gate, 1e-3, out, heads=heads)
    _close(out, oracle.rms(o.double().view(9, heads, dim), 1e-3).reshape(9, n) * w.double() * torch.sigmoid(gate.double()), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [52, 256])
def test_scaled_embedding_behind_its_norm(width, dtype):
    from crosspool_b200.ops import mixers as M

    table, w, ids = _rnd(20, width, seed=1, dtype=dtype), _rnd(width, seed=2), _i32([3, 19, 0])
    resid, out = torch.full((3, width), 9.0, device="cuda"), torch.empty(3, width, dtype=dtype, device="cuda")
    M.post_norm(resid, out, ids=ids, table=table, out_norm=M.NormParams("rmsnorm", w, eps=1e-2), embed_scale=5.5)
    want = table.double()[ids.long()] * 5.5
    _close(resid, want, torch.float32)
    _close(out, oracle.rms(want, 1e-2) * w.double(), dtype)


# ------------------------------------------------------------------ routed FFNs

@pytest.mark.parametrize("rows", [1, 3, 128, 129, 400])
@pytest.mark.parametrize("h,E,top,ff,ident,shared", [(96, 5, 2, 40, 2, 56), (52, 4, 3, 11, 1, 7), (256, 16, 4, 136, 0, 0), (64, 1, 1, 24, 3, 8), (128, 40, 32, 8, 5, 200)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_routed_ffn(rows, h, E, top, ff, ident, shared, dtype):
    from crosspool_b200.models.config import MoeSpec
    from crosspool_b200.models.weights import FfnLayerWeights
    from crosspool_b200.ops import moe

    spec = MoeSpec(E, top, ff, ident, 2.5, shared)
    cfg = {"router": {"experts": E, "top": top, "identity": ident, "scale": 2.5}, "shared": shared}
    t = {"router": _rnd(E + ident, h, seed=1, dtype=torch.bfloat16, scale=2 * h ** -0.5), "correction": _rnd(E + ident, seed=2, scale=0.1)}
    for e in range(E):
        t.update({f"e{e}.gate": _rnd(ff, h, seed=10 + e, dtype=torch.bfloat16, scale=h ** -0.5), f"e{e}.up": _rnd(ff, h, seed=100 + e, dtype=torch.bfloat16, scale=h ** -0.5),
                  f"e{e}.down": _rnd(h, ff, seed=200 + e, dtype=torch.bfloat16, scale=ff ** -0.5)})
    w = FfnLayerWeights(torch.stack([torch.cat([t[f"e{e}.gate"], t[f"e{e}.up"]]) for e in range(E)]).to(dtype),
                        torch.stack([t[f"e{e}.down"] for e in range(E)]).to(dtype), router=t["router"].to(dtype))
    w.extra["correction_bias"] = t["correction"]
    if shared:
        t.update({"shared.gate": _rnd(shared, h, seed=5, dtype=torch.bfloat16, scale=h ** -0.5), "shared.up": _rnd(shared, h, seed=6, dtype=torch.bfloat16, scale=h ** -0.5),
                  "shared.down": _rnd(h, shared, seed=7, dtype=torch.bfloat16, scale=shared ** -0.5), "shared.sg": _rnd(1, h, seed=8, dtype=torch.bfloat16)})
        w.shared_gate_up, w.shared_down = torch.cat([t["shared.gate"], t["shared.up"]]).to(dtype), t["shared.down"].to(dtype)
        w.extra["shared_scale"] = t["shared.sg"].to(dtype)
    moe.prepare_routed(w, spec)
    x = _pitched(rows, h, torch.bfloat16, 3).to(dtype)
    if x.stride(0) % 8:
        x = _pitched(rows, h, dtype, 3).copy_(x)
    ws = moe.RoutedWorkspace.for_layers([spec, MoeSpec(2, 1, 8)], h, 400, dtype, torch.device("cuda"))
    out = torch.full((rows, (h + 7) // 8 * 8), 7.0, dtype=dtype, device="cuda")
    tt = {k: v.double().cpu() for k, v in t.items()}
    for n in (rows, max(1, rows // 2)):                       # the second call finds the first one's tables
        moe.routed_ffn(x[:n], w, spec, out[:n, :h], ws)
        margins: list = []
        want = oracle.experts(x[:n].double().cpu(), cfg, lambda k: tt[k], margins)
        ok = (margins[0] > 1e-5).cuda() if margins else torch.ones(n, dtype=torch.bool, device="cuda")   # router logits are fp32 in both types
        assert ok.float().mean() > 0.9
        _close(out[:n, :h][ok], want[ok.cpu()], dtype, 3e-2 if dtype == torch.bfloat16 else 1e-4)
    assert (out[:, h:] == 7.0).all()
    _status()


# ------------------------------------------------------------------ convolution, rotation, cache write

@pytest.mark.parametrize("H,G,d,e,taps,pairs,own", [(6, 2, 24, 40, 4, 8, True), (3, 1, 10, 13, 3, 3, True), (4, 4, 128, 64, 1, 64, True), (5, 1, 40, 16, 6, 11, False),
                                                  (2, 1, 16, 24, 0, 8, True), (4, 2, 32, 32, 2, 0, False)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_convolution_and_rotation_in_portions(H, G, d, e, taps, pairs, own, dtype):
    """Two sequences in portions of several lengths (single tokens through the decode kernel), rings that held other inputs."""
    from crosspool_b200.ops import mixers as M

    lens, pad, page = [150, 83], M.group_pad(H, G), 16
    dq, dv = (d + 7) // 8 * 8, (e + 7) // 8 * 8
    rows = {"q": H * d, **({"k": G * d, "v": G * e} if own else {})}
    offs, at = [], 8
    for n in rows.values():
        offs.append(at)
        at += (n + 7) // 8 * 8
    proj = [_rnd(n, at, seed=i + 1, dtype=dtype) for i, n in enumerate(lens)]
    C = sum(rows.values())
    conv = _rnd(taps, C, seed=5) if taps else None
    ring = torch.full((3, max(taps, 1), C), 1e4, dtype=dtype, device="cuda") if taps else None
    freq = oracle.rotary_frequencies(2 * pairs, 50.0)
    ang = torch.arange(200, dtype=torch.float64)[:, None] * freq
    rot = torch.stack([ang.cos(), ang.sin()], -1).float().cuda() if pairs else None
    kc, vc = torch.zeros(20, page, G, dq, dtype=dtype, device="cuda"), torch.zeros(20, page, G, dv, dtype=dtype, device="cuda")
    base, slot = [0, 160], [2, 0]
    got = [[], []]
    done = [0, 0]
    for step in ([70, 1], [1, 2], [1, 1], [64, 63], [2, 1], [3, 15], [9, 0]):
        order = sorted((i for i in (0, 1) if step[i]), key=lambda i: step[i] > 1)
        x = torch.cat([proj[i][done[i]:done[i] + step[i]] for i in order])
        pos = _i32([p for i in order for p in range(done[i], done[i] + step[i])])
        slots = _i32([base[i] + p for i in order for p in range(done[i], done[i] + step[i])])
        q = torch.full((x.shape[0], G, pad, dq), 7.0, dtype=dtype, device="cuda")
        nd = sum(step[i] == 1 for i in order)
        kw = dict(heads=H, dim=d, vdim=e, offs=tuple(offs))
        sl = _i32([slot[i] for i in order])
        if nd:
            M.conv_rope(x[:nd], conv, ring, rot, pos, slots, sl, kc, vc, q, **kw)
        if nd < len(order):
            n = [step[i] for i in order]
            starts = [sum(n[:j]) for j in range(len(n))]
            M.conv_rope(x, conv, ring, rot, pos, slots, sl[nd:], kc, vc, q, q_starts=_i32(starts[nd:]), q_lens=_i32(n[nd:]), max_q=max(n[nd:]), **kw)
        at0 = 0
        for i in order:
            got[i].append(q[at0:at0 + step[i]])
            at0 += step[i]
            done[i] += step[i]
    assert done == lens
    for i, n in enumerate(lens):
        at0 = 0
        for (name, r), o in zip(rows.items(), offs):
            u = proj[i][:, o:o + r].double().cpu()
            if taps:
                u = oracle.short_convolution(u, conv[:, at0:at0 + r].double().cpu().T)
            at0 += r
            heads, w = (H, d) if name == "q" else (G, d) if name == "k" else (G, e)
            u = u.view(n, heads, w)
            if name != "v" and pairs:
                u = oracle.rotate(u, freq)
            if name == "q":
                y = torch.cat(got[i])
                _close(y[:, :, :H // G, :d].reshape(n, H, d), u, dtype)
                assert (y[:, :, H // G:] == 0).all() and (y[..., d:] == 0).all()
            else:
                c = (kc if name == "k" else vc).flatten(0, 1)[base[i]:base[i] + n]
                _close(c[..., :w], u, dtype)
                assert (c[..., w:] == 0).all()
    if taps:
        assert (ring[1] == 1e4).all()                        # nobody's slot


# ------------------------------------------------------------------ windows

SPANS = [(1, 0), (16, 0), (40, 5), (64, 64), (100, 17), (33, 70), (500, 3), (0, 0)]


def _paged(lens, G, dq, dv, page, dtype, seed=1):
    """Caches whose pages are shuffled and whose unused rows hold NaN, the table, and the plain keys and values."""
    blocks = max((n + page - 1) // page for n in lens)
    perm = torch.randperm(len(lens) * blocks, generator=torch.Generator().manual_seed(seed)).view(len(lens), blocks)
    k, v = (torch.full((len(lens) * blocks, page, G, w), float("nan"), dtype=dtype, device="cuda") for w in (dq, dv))
    ks, vs = [], []
    for i, n in enumerate(lens):
        ks.append(_rnd(n, G, dq, seed=10 * seed + i, dtype=dtype))
        vs.append(_rnd(n, G, dv, seed=20 * seed + i, dtype=dtype))
        rows = torch.tensor([int(perm[i, p // page]) * page + p % page for p in range(n)]).cuda()
        k.flatten(0, 1)[rows], v.flatten(0, 1)[rows] = ks[-1], vs[-1]
    return k, v, perm.int().cuda(), ks, vs


def _one_key(ks, q, places, row):
    """Makes one key stand out for a row's queries, so that the edge it lies at decides the result."""
    for p in places:
        ks[p] = q[row].float().mean(1).to(ks.dtype) * 3


@pytest.mark.parametrize("window,keep", SPANS)
@pytest.mark.parametrize("H,G,d,e,dtype", [(6, 2, 64, 64, torch.bfloat16), (4, 1, 128, 128, torch.bfloat16), (16, 1, 192, 128, torch.bfloat16),
                                           (3, 3, 24, 40, torch.float32), (3, 1, 16, 16, torch.bfloat16)])
@pytest.mark.parametrize("page", [16, 64])
def test_rows_see_their_window_and_the_first_tokens(window, keep, H, G, d, e, dtype, page):
    from crosspool_b200.ops import mixers as M

    tc = dtype == torch.bfloat16 and d >= 64
    lens = [1, 15, 40, 41, 63, 64, 65, 129, 300, 420]
    k, v, table, ks, vs = _paged(lens, G, d, e, page, dtype)
    pad = M.group_pad(H, G)
    q = _rnd(len(lens), G, pad, d, seed=3, dtype=dtype)
    q[:, :, H // G:] = 0
    for i, n in enumerate(lens):                              # the tokens on both sides of every edge stand out in turn
        edge = [keep - 1, keep, n - window - 1, n - window, 0][i % 5] if window else n // 2
        if 0 <= edge < n:
            _one_key(ks[i], q[:, :, :H // G], [edge], i)
            k.flatten(0, 1)[int(table[i, edge // page]) * page + edge % page] = ks[i][edge]
    gate = _rnd(len(lens), H * e, seed=4, dtype=dtype)
    out = torch.full((len(lens), H * e), 7.0, dtype=dtype, device="cuda")
    pos, slots = _i32([n - 1 for n in lens]), _i32(list(range(len(lens))))
    want = []
    for i, n in enumerate(lens):
        qi = torch.zeros(n, H, d, dtype=torch.float64)
        qi[-1] = q[i, :, :H // G].reshape(H, d).double().cpu()
        want.append(oracle.windowed_attention(qi, ks[i].double().cpu(), vs[i].double().cpu(), 0.2, window or n, keep)[-1].reshape(-1))
    want = torch.stack(want) * torch.sigmoid(gate.double().cpu())
    kw = dict(heads=H, dim=d, vdim=e, scale=0.2, gate=gate, window=window, keep_first=keep)
    M.grouped_attn(q, k, v, out, table, pos, slots, **kw)
    _close(out, want, dtype)
    if tc:
        for splits, chunk in ((1, 0), (4, 0), (4, 112), (27, 16)):
            ws = torch.empty(len(lens) * H * splits * (e + 2), device="cuda")
            out.fill_(7.0)
            M.grouped_decode(q, k, v, out, table, pos, slots, num_splits=splits, chunk_tokens=chunk, ws=ws, **kw)
            _close(out, want, dtype)
    _status()


@pytest.mark.parametrize("window,keep", SPANS)
@pytest.mark.parametrize("H,G,d,e", [(6, 2, 64, 64), (4, 1, 128, 128), (2, 1, 192, 128), (16, 1, 128, 64)])
@pytest.mark.parametrize("page", [64, 128])
def test_portions_see_their_window_and_the_first_tokens(window, keep, H, G, d, e, page):
    from crosspool_b200.ops import mixers as M

    lens, ctx = [20, 64, 65, 200, 333, 420], [0, 0, 17, 64, 300, 33]
    k, v, table, ks, vs = _paged(lens, G, d, e, page, torch.bfloat16)
    q_lens = [n - c for n, c in zip(lens, ctx)]
    starts = [sum(q_lens[:i]) for i in range(len(lens))]
    T, pad, vd = sum(q_lens), M.group_pad(H, G), e - 8
    q = _rnd(T, G, pad, d, seed=3, dtype=torch.bfloat16)
    for i, n in enumerate(lens):
        for edge in (keep - 1, keep, 63, 64, n - 1 - window if window else 0):
            if 0 <= edge < n and window:
                ks[i][edge] *= 2.5                            # stands out for many rows
                k.flatten(0, 1)[int(table[i, edge // page]) * page + edge % page] = ks[i][edge]
    gate = _rnd(T, H * vd + 8, seed=4, dtype=torch.bfloat16)[:, 8:]
    out = torch.full((T + 1, H * vd), 7.0, dtype=torch.bfloat16, device="cuda")
    M.grouped_prefill(q, k, v, out[:T], table, _i32(starts), _i32(q_lens), _i32(ctx), max(q_lens), heads=H, vdim=vd, scale=0.15, gate=gate,
                      window=window, keep_first=keep)
    _status()
    assert (out[T] == 7.0).all()
    for i, n in enumerate(lens):
        s = slice(starts[i], starts[i] + q_lens[i])
        qi = torch.zeros(n, H, d, dtype=torch.float64)
        qi[ctx[i]:] = q[s, :, :H // G].reshape(-1, H, d).double().cpu()
        want = oracle.windowed_attention(qi, ks[i].double().cpu(), vs[i][..., :vd].double().cpu(), 0.15, window or n, keep)[ctx[i]:]
        _close(out[s], want.reshape(q_lens[i], -1) * torch.sigmoid(gate[s].double().cpu()), torch.bfloat16)


# ------------------------------------------------------------------ matrix memory

def _memory_case(H, d, e, n, cap, seed=0, kind="plain"):
    """Projection rows, gates and the plain result; kinds of gates: what a trained model may do, saturated, drifting."""
    offs, at = [], 0
    for w in (H * d, H * d, H * e, H * e):
        offs.append(at)
        at += (w + 7) // 8 * 8
    proj = torch.randn(n, at, generator=torch.Generator().manual_seed(seed))
    proj[:, offs[1]:offs[1] + H * d] = 0.8 * proj[:, :H * d] + 0.6 * proj[:, offs[1]:offs[1] + H * d]
    z = torch.randn(n, 2 * H + 3, generator=torch.Generator().manual_seed(seed + 1)) * 2
    z[:, H + 3:] += 2.0
    if kind == "saturated":
        z *= 100
    if kind == "shut":                                       # nothing comes in for long, and what is there is forgotten
        z[:, :H] -= 12
        z[:, H + 3:] -= 4
        z[n // 2] += 20
    if kind == "open":
        z[:, H + 3:] += 8
    return proj, z, offs + [0, H + 3]


def _memory_want(proj, z, offs, H, d, e, cap):
    n = proj.shape[0]
    q, k, v = (proj[:, o:o + H * w].double().cpu().view(n, H, w) for o, w in zip(offs, (d, d, e)))
    z = z.double().cpu()
    i, f = oracle.soft_cap(z[:, :H], cap), oracle.log_sigmoid(oracle.soft_cap(z[:, H + 3:2 * H + 3], cap))
    o, _ = oracle.stabilised_memory(q * d ** -0.5, k, v, i, f)
    # the sums of magnitudes behind what is read and behind its divisor, both over the divisor: what rounding is relative to
    F, t = f.cumsum(0), torch.arange(n)
    diff = (F[:, None] - F[None] + i[None]).masked_fill((t[None] > t[:, None])[..., None], -math.inf)          # [T, T, H]
    m = torch.maximum(F, diff.max(1).values)
    s = torch.einsum("thd,jhd->tjh", q * d ** -0.5, k) * (diff - m[:, None]).exp()
    size = torch.maximum(s.sum(1).abs(), (-m).exp()) + 1e-6
    mags = torch.einsum("tjh,jhe->the", s.abs(), v.abs()) / size[..., None]
    return o, _size(mags) + _size(o) * s.abs().sum(1) / size


def _size(x):
    return x.pow(2).mean(-1).sqrt()


def _heads_close(got, want, scale, dtype, kind):
    """Per row and head. Open gates near the cap change a maximum by less than its last bit, token after token."""
    err = _size(got.double().cpu() - want) / scale
    limit = 5e-4 if kind == "saturated" else 1e-5 if dtype == torch.float32 else 1e-4
    assert err.max() < limit, (err.max(), err.argmax())


@pytest.mark.parametrize("kind", ["plain", "saturated", "shut", "open"])
@pytest.mark.parametrize("H,d,e", [(3, 24, 40), (2, 128, 128), (1, 256, 72), (2, 64, 264), (3, 9, 5), (1, 264, 24), (2, 8, 16)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_memory_in_portions_and_token_by_token(H, d, e, kind, dtype):
    """Two sequences in portions (also cut into segments), single tokens, and slots that held something else. The state is
    carried in 32 bits: outputs of bf16 rows are as exact as the rows."""
    from crosspool_b200.ops import mixers as M

    lens, cap = [340, 150], 15.0
    cases = [_memory_case(H, d, e, n, cap, seed=7 * i, kind=kind) for i, n in enumerate(lens)]
    offs = cases[0][2]
    proj, z = [c[0].to(dtype).cuda() for c in cases], [c[1].float().cuda() for c in cases]
    want = [_memory_want(p, g, offs, H, d, e, cap) for p, g in zip(proj, z)]
    hs = (d * e + d + 4) // 4 * 4
    norm = torch.ones(H * e, device="cuda")
    kw = dict(heads=H, dim=d, vdim=e, offs=tuple(offs), cap=cap)
    scratch = M.MemoryScratch.for_rows(sum(lens), 2, H, d, e, torch.device("cuda"))
    for plan in ([(340, 150)], [(64, 3), (1, 1), (130, 2), (2, 64), (1, 1), (70, 79), (72, 0)], [(1, 1)] * 40 + [(300, 110)]):
        state = torch.full((3, H, hs), 1e3, device="cuda")
        slot, done, got = [2, 0], [0, 0], [[], []]
        for step in plan:
            order = sorted((i for i in (0, 1) if step[i]), key=lambda i: step[i] > 1)
            x, g = (torch.cat([t[i][done[i]:done[i] + step[i]] for i in order]) for t in (proj, z))
            pos = _i32([p for i in order for p in range(done[i], done[i] + step[i])])
            slots, sl = pos * 0, _i32([slot[i] for i in order])
            n = [step[i] for i in order]
            nd = sum(c == 1 for c in n)
            out = torch.full((x.shape[0], H * e), float("nan"), device="cuda")
            if nd:
                o = torch.empty(nd, H * e, dtype=dtype, device="cuda")
                M.memory_decode(x[:nd], g, state, norm, o, pos, slots, sl, eps=1e-30, **kw)
                gate = torch.sigmoid(x[:nd, offs[3]:offs[3] + H * e].float())
                out[:nd] = o.float() / gate                   # the norm leaves the direction of every head
            if nd < len(order):
                most = max(n[nd:])
                segs, seg_tokens = M.linear_attn_plan(len(n) - nd, H, d, e, most)
                M.memory_prefill(x, g, state, out, pos, slots, sl[nd:], _i32([sum(n[:j]) for j in range(len(n))][nd:]), _i32(n[nd:]), most, scratch,
                                 segs=segs, seg_tokens=seg_tokens, **kw)
            at = 0
            for j, i in enumerate(order):
                got[i].append((out[at:at + n[j]], n[j] == 1))
                at += n[j]
                done[i] += n[j]
        assert done == lens and (state[1] == 1e3).all()
        for i in (0, 1):
            at = 0
            for o, single in got[i]:
                w, scale = (x[at:at + o.shape[0]] for x in want[i])
                o = o.view(-1, H, e)
                if single:
                    err = _size(o.double().cpu() - oracle.rms(w, 1e-60)) / (scale / _size(w))
                    assert err.max() < (5e-4 if kind == "saturated" else 1e-5) + 5e-3 * (dtype == torch.bfloat16), (at, err)
                else:
                    _heads_close(o, w, scale, dtype, kind)
                at += o.shape[0]


@pytest.mark.parametrize("segs,seg_tokens", [(1, 0), (2, 192), (3, 128), (6, 64)])
def test_memory_segments_agree_with_the_sequential_kernel(segs, seg_tokens):
    from crosspool_b200.ops import mixers as M

    H, d, e, n, cap = 2, 72, 136, 340, 8.0
    proj, z, offs = _memory_case(H, d, e, n, cap, kind="open")
    proj, z, hs = proj.bfloat16().cuda(), z.float().cuda(), (d * e + d + 4) // 4 * 4
    kw = dict(heads=H, dim=d, vdim=e, offs=tuple(offs), cap=cap)
    res = []
    for force in (False, True):
        state = _rnd(1, H, hs, seed=9, scale=0.3)
        out, pos = torch.empty(n, H * e, device="cuda"), torch.arange(5, 5 + n, dtype=torch.int32, device="cuda")
        M.memory_prefill(proj, z, state, out, pos, pos, _i32([0]), _i32([0]), _i32([n]), n, M.MemoryScratch.for_rows(n, 1, H, d, e, torch.device("cuda")),
                         segs=segs, seg_tokens=seg_tokens, force_sequential=force, **kw)
        res.append((out, state[:, :, :d * e + d + 1]))
    assert torch.allclose(res[0][0], res[1][0], rtol=2e-3, atol=2e-3) and torch.allclose(res[0][1], res[1][1], rtol=2e-3, atol=2e-3)


def test_memory_padding_rows_touch_nothing():
    from crosspool_b200.ops import mixers as M

    H, d, e = 2, 16, 24
    proj, z, offs = _memory_case(H, d, e, 3, 15.0)
    state = torch.full((2, H, (d * e + d + 4) // 4 * 4), 3.0, device="cuda")
    out = torch.full((3, H * e), 7.0, device="cuda")
    M.memory_decode(proj.cuda(), z.cuda(), state, torch.ones(H * e, device="cuda"), out, _i32([0, 0, 0]), _i32([-1, 5, -1]), _i32([0, 1, 0]), heads=H,
                    dim=d, vdim=e, offs=tuple(offs), cap=15.0, eps=1e-5)
    assert (state[0] == 3.0).all() and (out[0] == 0).all() and (out[2] == 0).all() and math.isfinite(out[1].sum().item()) and not (state[1, :, :d * e + d + 1] == 3.0).any()
