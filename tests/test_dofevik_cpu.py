"""Dofevik without a GPU: the plain implementation against independent forms of the same equations, configuration, FFN description,
weight layout, cache bookkeeping."""
import json
import math

import pytest
import torch

import dofevik_cases as dc
import dofevik_oracle as oracle


def _cfg(name):
    from crosspool_b200.models import config as mc

    return mc.from_hf_config(dc.CASES[name], name)


def _r(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


# ------------------------------------------------------------------ the plain implementation itself

def test_oracle_rotation_pairs_and_scaling():
    rot = {"dims": 4, "base": 100.0}
    f = oracle.frequencies(rot)
    assert torch.allclose(f, torch.tensor([1.0, 0.1], dtype=torch.float64))
    assert torch.allclose(oracle.frequencies({**rot, "scaling": {"factor": 4.0}}), f / 4)
    x = _r(1, 1, 6, seed=1).expand(9, 1, 6)
    for neighbours, (a, b) in ((True, (2, 3)), (False, (1, 3))):
        y = oracle.rotate(x, f, neighbours)[:, 0]
        assert torch.equal(y[0], x[0, 0]) and torch.equal(y[:, 4:], x[:, 0, 4:])
        assert torch.allclose(y[5] @ y[2], y[8] @ y[5]) and not torch.allclose(y[5] @ y[2], y[5] @ y[3])
        u, w = x[0, 0, a], x[0, 0, b]                        # the pair that turns by a tenth per position
        assert torch.allclose(y[7, a], u * math.cos(0.7) - w * math.sin(0.7)) and torch.allclose(y[7, b], w * math.cos(0.7) + u * math.sin(0.7))


def test_oracle_windows_and_blocks():
    for T, W, P in ((30, 5, 4), (23, 1, 1), (40, 7, 12), (12, 50, 3)):
        w, b = oracle.in_window(T, W), oracle.blocks_behind_window(T, W, P)
        for i in range(T):
            seen = [j for j in range(T) if w[i, j]]
            assert seen == list(range(max(0, i - W + 1), i + 1))
            whole = [n for n in range(T // P) if all(j < i - W + 1 for j in range(n * P, n * P + P))]
            assert [n for n in range(T // P) if b[i, n]] == whole
    x = _r(11, 2, 3)
    m = oracle.block_means(x, 4)
    assert m.shape == (2, 2, 3) and torch.allclose(m[1, 1], (x[4, 1] + x[5, 1] + x[6, 1] + x[7, 1]) / 4)


def test_oracle_weights():
    s, seen = _r(5, 7, seed=1), _r(5, 7, seed=2) > -1
    seen[:, 0] = True
    sink = torch.tensor(0.7, dtype=torch.float64)
    w = oracle.softmax_with_sink(s, seen, sink)
    e = torch.exp(s) * seen
    assert torch.allclose(w, e / (e.sum(-1, keepdim=True) + math.exp(0.7)))
    assert torch.allclose(oracle.softmax_with_sink(s, seen, None).sum(-1), torch.ones(5, dtype=torch.float64))
    assert torch.allclose(oracle.softmax_with_sink(s, seen, torch.tensor(900.0, dtype=torch.float64)), torch.zeros(5, 7, dtype=torch.float64))
    assert torch.allclose(oracle.sigmoid_weights(s, seen, 0.3), seen / (1 + torch.exp(-s - 0.3)))


def test_oracle_unit_heads_commute_with_rotation():
    x, f = _r(6, 2, 8), oracle.frequencies({"dims": 6, "base": 10.0})
    assert torch.allclose(oracle.rms(oracle.rotate(x, f, True), 1e-3), oracle.rotate(oracle.rms(x, 1e-3), f, True))


def test_oracle_latent_attention_equals_its_absorbed_form():
    """Queries multiplied into the latent space, one pass over the latents, values behind the sum."""
    m = dc.latent(3, 10, 4, 6, 12, 15, 9)["mixer"]
    t = {k.removeprefix("l0.mix."): v.double() for k, v in oracle.random_tensors(dc.model(20, 30, [({"type": "latent_attention", "mixer": m}, None)]), 3).items()}
    t["o"] = torch.eye(18, dtype=torch.float64)
    h, H, d, e, R = _r(25, 20, seed=1), 3, 10, 6, 15
    q = (oracle.rms(h @ t["dq"].T, 1e-5) * t["dq.norm"] @ t["uq"].T).view(25, H, d + 4)
    kv = h @ t["dkv"].T
    c, f = oracle.rms(kv[:, :R], 1e-5) * t["dkv.norm"], oracle.frequencies(m["rot"])
    qa = torch.cat([torch.einsum("thd,hdr->thr", q[..., :d], t["uk"].view(H, d, R)), oracle.rotate(q[..., d:], f, False)], -1)
    ka = torch.cat([c, oracle.rotate(kv[:, None, R:], f, False)[:, 0]], -1)
    s = torch.einsum("thr,nr->htn", qa, ka) * m["scale"]
    w = s.masked_fill(~oracle.in_window(25, 9), -math.inf).softmax(-1)
    o = torch.einsum("htr,hvr->thv", w @ c, t["uv"].view(H, e, R)).reshape(25, -1)
    assert torch.allclose(oracle.latent_attention(h, m, lambda n: t[n], 1e-5), o * torch.sigmoid(h @ t["g"].T))


def test_oracle_routing():
    z = torch.tensor([[2.0, 1.0, 0.0, -1.0]], dtype=torch.float64)
    w = oracle.routing(z, 2)[0]
    assert torch.allclose(w, torch.tensor([math.e / (1 + math.e), 1 / (1 + math.e), 0, 0], dtype=torch.float64))
    m: list = []
    oracle.routing(z, 3, m)
    assert m[0].item() == 1.0
    t = {"up": torch.tensor([[1.0], [-1.0]], dtype=torch.float64), "down": torch.tensor([[1.0, 10.0]], dtype=torch.float64)}
    assert oracle.squared_relu(torch.tensor([[3.0], [-2.0]], dtype=torch.float64), lambda n: t[n]).flatten().tolist() == [9.0, 40.0]


@pytest.mark.parametrize("name", ["mixed", "odd", "edges"])
def test_oracle_is_causal(name):
    c, t = dc.CASES[name], dc.tensors(name)
    ids = dc.prompt(c, 90, 3)
    assert torch.allclose(oracle.forward(c, t, ids)[:70], oracle.forward(c, t, ids[:70]), atol=1e-10)


@pytest.mark.parametrize("kind,size,pool", [("attention", 40, 0), ("pooled", 40, 5), ("pooled", 33, 12), ("latent", 40, 0)])
def test_the_marked_token_shows_where_it_is_seen(kind, size, pool):
    """What the engine tests rest on: one token more or less in a window, one block more or less behind it moves the logits far
    beyond rounding."""
    c, t = dc.marked_model(kind, size, pool)
    ids = [i for i in dc.prompt(c, 200, 6) if i != dc.MARK][:160]
    for place in (0, 5, 64):
        a, b = ids[:place] + [dc.MARK] + ids[place + 1:], ids[:place] + [8] + ids[place + 1:]
        e = dc.error(oracle.forward(c, t, a), oracle.forward(c, t, b))
        edge = place + size
        assert e[place + 1:edge].min() > 0.4
        if pool:
            first = place // pool * pool + pool - 1 + size    # the first token that sees the mark's block
            assert edge <= first and (e[edge:first] < 1e-6).all() and e[first:].min() > 0.1
        else:
            assert e[edge:].max() < 1e-6


# ------------------------------------------------------------------ configuration and FFN description

def test_config_reads_every_layer():
    c = _cfg("mixed")
    assert c.layered and not c.recurrent and not c.output_norm and not c.residual_gate and c.norm == "scalar" and not c.tie_word_embeddings
    a, p, l, p2 = (s.mixer for s in c.layer_specs)
    assert (a.norm, a.biases, a.gate, a.window, a.sink, a.sigmoid, a.pool, a.tied) == ("unit", True, "", 37, True, False, 0, False)
    assert (a.rot.dims, a.rot.interleaved, a.rot.scaling.factor, a.rot.scaling.original) == (16, True, 3.0, 0.0)
    assert (p.norm, p.biases, p.gate, p.window, p.sink, p.sigmoid, p.pool, p.tied, p.rot, p.vdim) == ("weight", False, "", 50, False, True, 7, True, None, 40)
    assert (l.q_rank, l.kv_rank, l.window, l.gate_elems, l.gate_features, l.rot.interleaved, l.rot.scaling) == (56, 72, 45, True, 120, False, None)
    m = c.layer_specs[0].moe
    assert (m.experts, m.top, m.ff, m.shared_ff, m.relu2, m.logit_choice, m.shared_gate, m.maps, m.routed) == (5, 2, 40, 56, True, True, False, 2, 5)
    assert [s.has_ffn for s in c.layer_specs] == [True, False, True, True] and c.layer_specs[2].moe.shared_ff == 0
    assert a.visible(30) == 30 and a.visible(1000) == 37 and p.visible(50) == 50 and p.visible(64) == 52 and l.visible(1000) == 45 and p2.visible(63) == 25
    assert c.kv_bytes_per_token() == 2 * (2 * 2 * 64 + 2 * 2 * 64 + 80 + 2 * 64) and c.state_bytes_per_sequence() == 0


def test_block_means_fit_beside_their_pages():
    """Every block that a sequence's pages complete has a row beside a page that the sequence holds."""
    from crosspool_b200.models.config import GroupedMixer

    for page in (16, 64, 128):
        for pool in (1, 3, 7, 8, 12, 16, 50, 64, 200):
            n = GroupedMixer(2, 1, 24, 24, 1.0, pool=pool, window=9).pool_page(page)
            assert n >= 8 and n & (n - 1) == 0
            for tokens in range(1, 1000):
                blocks, pages = tokens // pool, (tokens + page - 1) // page
                assert blocks == 0 or (blocks - 1) // n < pages


def test_pages_that_hold_whole_blocks_can_be_shared():
    from crosspool_b200.models import config as mc

    for page, pool, ok in ((16, 2, True), (64, 8, True), (64, 4, True), (64, 7, False), (64, 16, False), (128, 16, True), (16, 8, False)):
        c = mc.from_hf_config(dc.model(32, 40, [(dc.pooled(2, 1, 16, 9, pool), None)]))
        assert c.pages_shareable(page) == ok, (page, pool)
    assert mc.from_hf_config(dc.model(32, 40, [(dc.attention(2, 1, 16, 16, 9), None)])).pages_shareable(64)


def test_parameter_counts_match_the_checkpoint():
    for name in dc.CASES:
        t, c = dc.tensors(name), _cfg(name)
        assert c.attention_param_bytes() == 2 * sum(v.numel() for k, v in t.items() if ".mlp." not in k), name
        for i in range(c.num_layers):
            assert c.ffn_param_bytes_per_layer(i) == 2 * sum(v.numel() for k, v in t.items() if k.startswith(f"l{i}.mlp.")), (name, i)


@pytest.mark.parametrize("layer,change", [
    (0, lambda l: l.update(type="lightning")), (0, lambda l: l["mixer"].update(kv_heads=4)), (1, lambda l: l["mixer"].update(kv_heads=3)),
    (0, lambda l: l["mixer"]["rot"].update(dims=26)), (0, lambda l: l["mixer"]["rot"].update(dims=15)), (1, lambda l: l["mixer"].update(vdim=32)),
    (0, lambda l: l["mixer"]["mask"].update(size=0)), (1, lambda l: l["mixer"]["mask"].update(pool=-1)), (2, lambda l: l["mixer"].update(q_rank=0)),
    (2, lambda l: l["mixer"]["rot"].update(dims=10)), (0, lambda l: l["mlp"]["router"].update(top=6)), (0, lambda l: l["mlp"].update(kind="dense"))])
def test_config_refuses_what_it_does_not_know(layer, change):
    from crosspool_b200.models import config as mc

    c = json.loads(json.dumps(dc.CASES["mixed"]))
    change(c["layers"][layer])
    with pytest.raises(ValueError):
        mc.from_hf_config(c)


def test_ffn_description_covers_the_checkpoint_and_loads(tmp_path):
    from crosspool_b200.deployment import load_ffn_weights

    t = dc.tensors("mixed")
    fw = load_ffn_weights(_cfg("mixed"), dc.write_checkpoint(tmp_path / "m", dc.CASES["mixed"], t), "cpu", torch.float32)
    assert fw[1] is None and fw[2].shared_gate_up is None
    w = fw[0]
    assert w.is_moe and tuple(w.gate_up.shape) == (5, 40, 96) and tuple(w.router.shape) == (5, 96)
    assert torch.equal(w.gate_up[3], t["l0.mlp.e3.up"].float()) and torch.equal(w.down[4], t["l0.mlp.e4.down"].float())
    assert torch.equal(w.extra["router_bias"], t["l0.mlp.router.b"].float()) and "correction_bias" not in w.extra and "shared_scale" not in w.extra
    assert torch.equal(w.shared_gate_up, t["l0.mlp.shared.up"].float()) and torch.equal(w.shared_down, t["l0.mlp.shared.down"].float())
    for bad in ("l0.mlp.e4.down", "l3.mlp.shared.up", "l0.mlp.router.b"):
        less = {k: v for k, v in t.items() if k != bad}
        with pytest.raises(ValueError, match=bad):
            load_ffn_weights(_cfg("mixed"), dc.write_checkpoint(tmp_path / bad, dc.CASES["mixed"], less), "cpu", torch.float32)
    with pytest.raises(ValueError, match="e5"):
        load_ffn_weights(_cfg("mixed"), dc.write_checkpoint(tmp_path / "more", dc.CASES["mixed"], {**t, "l0.mlp.e5.up": t["l0.mlp.e4.up"].clone()}), "cpu",
                         torch.float32)


# ------------------------------------------------------------------ weight layout

@pytest.mark.parametrize("name", list(dc.CASES))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_fused_projection_holds_every_map_at_its_offset(tmp_path, name, dtype):
    from crosspool_b200.models.weights import load_attention_from_safetensors

    c, t = dc.CASES[name], dc.tensors(name)
    w = load_attention_from_safetensors(_cfg(name), dc.write_checkpoint(tmp_path, c, t), "cpu", dtype)
    assert torch.equal(w.embed, t["embed"].to(dtype)) and torch.equal(w.lm_head, t["head"].to(dtype)) and w.lm_head.stride(0) % 8 == 0
    assert (w.final_norm.weight == t["final.norm"].float()).all() and w.final_norm.weight.shape == (c["width"],)
    for i, (lw, l) in enumerate(zip(w.layers, c["layers"])):
        mix = {k.split(".mix.")[1]: v.to(dtype) for k, v in t.items() if k.startswith(f"l{i}.mix.")}
        want = {"attention": ["q", "k", "v"], "attention_2": ["q", "k"], "latent_attention": ["dq", "dkv", "g"]}[l["type"]]
        for n in want:
            o = lw.offs[{"dq": "q", "dkv": "kv"}.get(n, n)]
            assert o % 8 == 0 and torch.equal(lw.proj[o:o + mix[n].shape[0]], mix[n])
        if l["type"] == "attention":
            bias = torch.zeros_like(lw.proj_bias)
            for n in "qkv":
                bias[lw.offs[n]:lw.offs[n] + mix[n].shape[0]] = t[f"l{i}.mix.{n}.b"].float()
            assert torch.equal(lw.proj_bias, bias) and torch.equal(lw.mix["sink"], t[f"l{i}.mix.sink"].float()) and "bias" not in lw.mix
        elif l["type"] == "attention_2":
            assert lw.offs["v"] == lw.offs["k"] and lw.proj_bias is None and torch.equal(lw.mix["bias"], t[f"l{i}.mix.pb"].float())
            assert torch.equal(lw.mix["q_norm"], t[f"l{i}.mix.q.norm"].float()) and torch.equal(lw.mix["k_norm"], t[f"l{i}.mix.k.norm"].float())
        else:
            folded = t[f"l{i}.mix.uq"].float() * t[f"l{i}.mix.dq.norm"].float()
            assert torch.equal(lw.mix["uq"], folded.to(dtype)) and lw.mix["uq"].stride(0) % 8 == 0
        assert lw.proj.stride(0) % 8 == 0 and lw.o.stride(0) % 8 == 0 and torch.equal(lw.o, mix["o"])
        assert (lw.norm1.weight == t[f"l{i}.norm1"].float()).all() and (lw.norm2 is None) == (l["mlp"] is None)


def test_weights_of_the_wrong_shape_are_refused(tmp_path):
    from crosspool_b200.models.weights import load_attention_from_safetensors

    for i, key in enumerate(("l0.mix.sink", "l1.mix.k.norm", "l2.mix.uq", "head", "l1.mix.pb")):
        t = dc.tensors("mixed")
        t[key] = t[key][..., :-1]
        d = dc.write_checkpoint(tmp_path / str(i), dc.CASES["mixed"], t)
        with pytest.raises(ValueError, match=key):
            load_attention_from_safetensors(_cfg("mixed"), d, "cpu", torch.float32)


def test_rotary_table_with_linear_scaling():
    from crosspool_b200.models.config import _rotary
    from crosspool_b200.models.layered import rotary_table

    r = {"dims": 24, "base": 5e3, "scaling": {"factor": 6.0}}
    tab = rotary_table(_rotary(r, 32, True), 3000, "cpu")
    a = torch.arange(3000, dtype=torch.float64)[:, None] * oracle.frequencies(r)
    assert torch.allclose(tab[..., 0].double(), a.cos(), atol=1e-7) and torch.allclose(tab[..., 1].double(), a.sin(), atol=1e-7)


def test_random_models_have_every_part():
    from crosspool_b200.models.weights import random_attention_weights, random_ffn_weights

    c = _cfg("mixed")
    w, f = random_attention_weights(c, 1, "cpu", torch.float32), random_ffn_weights(c, 1, "cpu")
    assert (w.layers[0].norm1.weight == 1).all() and (w.final_norm.weight == 1).all() and w.lm_head is not w.embed
    assert w.layers[0].mix["sink"].shape == (6,) and w.layers[2].mix["uq"].shape == (96, 56)
    assert f[1] is None and tuple(f[3].shared_gate_up.shape) == (16, 96) and tuple(f[0].gate_up.shape) == (5, 40, 96) and "router_bias" in f[0].extra


# ------------------------------------------------------------------ cache

def test_pages_and_block_means():
    from crosspool_b200.engine.kv_cache import PagedKvCache

    kv = PagedKvCache.fixed(_cfg("mixed"), 6, 16, "cpu", torch.float32, state_slots=2)
    assert [tuple(k.shape) for k in kv.k] == [(6, 16, 2, 64), (6, 16, 2, 64), (6, 16, 1, 80), (6, 16, 1, 64)] and kv.slots is None
    assert [None if k is None else tuple(k.shape) for k in kv.k_pool] == [None, (6, 8, 2, 64), None, (6, 8, 1, 64)]
    assert [None if v is None else tuple(v.shape) for v in kv.v_pool] == [None, (6, 8, 2, 64), None, (6, 8, 1, 64)]
    assert kv.layout.bytes_per_page_all_layers == 4 * (16 * (256 + 256 + 80 + 128) + 8 * 256 + 8 * 128)
    kv.ensure(1, 20)
    kv.release(1)
    assert kv.allocator.free_pages == 6
