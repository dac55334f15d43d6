"""Saninex without a GPU: the plain implementation against independent forms of the same equations, configuration, FFN
description, weight layout, cache and state bookkeeping."""
import json
import math

import pytest
import torch

import saninex_cases as sc
import saninex_oracle as oracle


def _cfg(name):
    from crosspool_b200.models import config as mc

    return mc.from_hf_config(sc.CASES[name], name)


def _r(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


# ------------------------------------------------------------------ the plain implementation itself

def test_oracle_delta_rule_equals_its_triangular_form():
    """All writes of a stretch at once: (1 + strictly lower part of beta decay k k^T) U = beta (V - decayed reads)."""
    T, d, e = 19, 6, 5
    q, k, v = _r(T, 1, d, seed=1), oracle.unit(_r(T, 1, d, seed=2)), _r(T, 1, e, seed=3)
    beta, g = torch.sigmoid(_r(T, 1, seed=4)), torch.sigmoid(_r(T, 1, seed=5) + 1)
    o, S = oracle.delta_recurrence(q, k, v, beta, g)
    cum = g[:, 0].log().cumsum(0)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    decay = torch.where(j <= i, (cum[:, None] - cum[None, :]).exp(), torch.zeros((), dtype=torch.float64))
    L = torch.tril(beta * decay * (k[:, 0] @ k[:, 0].T), -1)
    U = torch.linalg.solve_triangular(L + torch.eye(T, dtype=torch.float64), beta * v[:, 0], upper=False)
    assert torch.allclose(o[:, 0], (decay * (q[:, 0] @ k[:, 0].T)) @ U)
    assert torch.allclose(S[0], (decay[-1][:, None] * k[:, 0]).T @ U)


def test_oracle_delta_rule_replaces_what_a_key_holds():
    """beta = 1 and no decay: writing under a key again leaves the new value only, and it is read in the same step."""
    k = oracle.unit(_r(1, 1, 8)).expand(3, 1, 8)
    v = _r(3, 1, 4, seed=1)
    one = torch.ones(3, 1, dtype=torch.float64)
    o, _ = oracle.delta_recurrence(k, k, v, one, one)
    assert torch.allclose(o, v, atol=1e-5)


def test_oracle_channel_decays_reduce_to_one_decay_and_to_none():
    q, k, v = _r(15, 2, 4, seed=1), _r(15, 2, 4, seed=2), _r(15, 2, 3, seed=3)
    i, j = torch.arange(15)[:, None], torch.arange(15)[None, :]
    for a in (1.0, 0.7):
        o, _ = oracle.channel_recurrence(q, k, v, torch.full_like(q, a))
        m = torch.where(j <= i, a ** (i - j).double(), torch.zeros((), dtype=torch.float64))
        for h in range(2):
            assert torch.allclose(o[:, h], (m * (q[:, h] @ k[:, h].T)) @ v[:, h])
    a = torch.ones_like(q)
    a[:, :, 0] = 0
    o, S = oracle.channel_recurrence(q, k, v, a)
    assert torch.allclose(S[:, 0], k[-1, :, :1] * v[-1])        # a channel with decay zero remembers the last token only


def test_oracle_convolution_starts_from_zeros_and_ends_with_the_current_token():
    x = _r(5, 2)
    w = torch.tensor([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]], dtype=torch.float64)
    y = oracle.short_convolution(x, w)
    assert torch.allclose(y[0, 0], 100 * x[0, 0]) and torch.allclose(y[1, 0], 100 * x[1, 0] + 10 * x[0, 0])
    assert torch.allclose(y[4, 0], 100 * x[4, 0] + 10 * x[3, 0] + x[2, 0]) and torch.equal(y[:, 1], x[:, 1])


def test_oracle_capped_scores_saturate():
    q, k, v = 100 * _r(4, 1, 3, seed=1), _r(4, 1, 3, seed=2), _r(4, 1, 2, seed=3)
    o = oracle.capped_attention(q, k, v, 1.0, 1e-3)             # all scores within a thousandth: the mean of the values
    assert torch.allclose(o[3, 0], v.mean((0, 1)), atol=1e-2)
    o = oracle.capped_attention(q / 100, k, v, 0.5, 1e9)
    s = (q[3, 0] / 100 @ k[:, 0].T) * 0.5
    assert torch.allclose(o[3, 0], s.softmax(-1) @ v[:, 0])
    assert torch.equal(o[0, 0], v[0, 0])


def test_oracle_activation_and_norms():
    g, u = torch.tensor([3.0, -3.0, 0.5]), torch.tensor([3.0, -3.0, 0.25])
    y = oracle.clamped_glu(g, u, 2.0)
    want = [2 / (1 + math.exp(-3.404)) * 3, -3 / (1 + math.exp(5.106)) * -1, 0.5 / (1 + math.exp(-0.851)) * 1.25]
    assert torch.allclose(y, torch.tensor(want), atol=1e-6)
    x = torch.tensor([[3.0, -4.0]], dtype=torch.float64)
    assert torch.allclose(oracle.centred_norm(x, torch.zeros(2), 0.0), x / math.sqrt(12.5))
    assert torch.allclose(oracle.unit(x), x / math.sqrt(25 + 1e-6))


@pytest.mark.parametrize("name", ["mixed", "odd"])
def test_oracle_is_causal(name):
    c, t = sc.CASES[name], sc.tensors(name)
    ids = sc.prompt(c, 20, 3)
    assert torch.allclose(oracle.forward(c, t, ids)[:12], oracle.forward(c, t, ids[:12]), atol=1e-10)


# ------------------------------------------------------------------ configuration and FFN description

def test_config_reads_every_layer():
    c = _cfg("mixed")
    assert c.layered and c.recurrent and c.output_norm and c.gpu_attention_supported and c.num_layers == 4
    assert [s.mixer.kind for s in c.layer_specs] == ["parallel", "delta", "delta", "parallel"]
    assert [(s.ff, s.gate_limit) for s in c.layer_specs] == [(136, 0.9), (0, 0.0), (72, 7.0), (0, 0.0)]
    m = c.layer_specs[3].mixer
    assert (m.left.heads, m.left.kv_heads, m.left.dim, m.left.vdim, m.left.softcap, m.right.tau) == (3, 3, 40, 16, 4.0, 16.0)
    # cached heads are padded to the tensor-core kernels' widths (64 each here)
    assert c.kv_bytes_per_token() == 2 * (2 + 3) * 128
    states = 3 * 16 * 24 + 6 * 24 * 40 + 2 * 48 * 16 + 2 * 48 * 32
    assert c.state_bytes_per_sequence() == 4 * states + 2 * (4 * (2 * 3 * 24 + 6 * 40) + 3 * (2 * 2 * 48 + 2 * 16))
    assert c.rms_norm_eps == 1e-5 and c.tie_word_embeddings
    assert [s.ff for s in c.with_layers(6).layer_specs] == [136, 0, 72, 0, 136, 0]
    assert c.ffn_param_bytes_per_layer(0) == 2 * 3 * 96 * 136


def test_attention_parameter_count_matches_the_checkpoint():
    for name in sc.CASES:
        t, c = sc.tensors(name), _cfg(name)
        n = sum(v.numel() for k, v in t.items() if ".mlp." not in k)
        rank = sum(v.numel() for k, v in t.items() if k.endswith((".a1", ".a2")))     # the configuration does not know the rank
        assert c.attention_param_bytes() == 2 * (n - rank), name


@pytest.mark.parametrize("change", [lambda l: l.update(type="latent_attention"), lambda l: l.update(mlp={"kind": "moe", "ff": 8}),
                                    lambda l: l["mlp"].update(limit=0.0), lambda l: l["mixer"]["left"].update(kv_heads=4)])
def test_config_refuses_what_it_does_not_know(change):
    from crosspool_b200.models import config as mc

    c = json.loads(json.dumps(sc.CASES["mixed"]))
    change(c["layers"][0])
    with pytest.raises(ValueError):
        mc.from_hf_config(c)


def test_config_refuses_uneven_delta_heads():
    from crosspool_b200.models import config as mc

    c = json.loads(json.dumps(sc.CASES["mixed"]))
    c["layers"][1]["mixer"]["kv_heads"] = 4
    with pytest.raises(ValueError, match="evenly"):
        mc.from_hf_config(c)


def test_ffn_description_covers_the_checkpoint_and_loads(tmp_path):
    from crosspool_b200.deployment import load_ffn_weights

    t = sc.tensors("mixed")
    d = sc.write_checkpoint(tmp_path / "m", sc.CASES["mixed"], t)
    fw = load_ffn_weights(_cfg("mixed"), d, "cpu", torch.float32)
    assert fw[1] is None and fw[3] is None
    for i, limit in ((0, 0.9), (2, 7.0)):
        assert torch.equal(fw[i].gate_up, torch.cat([t[f"l{i}.mlp.gate"], t[f"l{i}.mlp.up"]]).float())
        assert torch.equal(fw[i].down, t[f"l{i}.mlp.down"].float()) and fw[i].extra["gate_transform"] == (limit, 1.0, 1.702)
    del t["l2.mlp.up"]
    with pytest.raises(ValueError, match="l2.mlp.up"):
        load_ffn_weights(_cfg("mixed"), sc.write_checkpoint(tmp_path / "less", sc.CASES["mixed"], t), "cpu", torch.float32)


# ------------------------------------------------------------------ weight layout

@pytest.mark.parametrize("name", list(sc.CASES))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_fused_projection_holds_every_map_at_its_offset(tmp_path, name, dtype):
    from crosspool_b200.models.weights import load_attention_from_safetensors

    c, t = sc.CASES[name], sc.tensors(name)
    w = load_attention_from_safetensors(_cfg(name), sc.write_checkpoint(tmp_path, c, t), "cpu", dtype)
    assert torch.equal(w.embed, t["embed"].to(dtype)) and torch.equal(w.final_norm.weight, 1 + t["final.norm"].float())
    for i, (lw, l) in enumerate(zip(w.layers, c["layers"])):
        mix = {k.split(".mix.")[1]: v.to(dtype) for k, v in t.items() if k.startswith(f"l{i}.mix.")}
        if l["type"] == "delta":
            names = {n: n for n in "qkvgba"}
            d = lw.mix["delta"]
            assert torch.equal(d.conv, torch.cat([t[f"l{i}.mix.{n}.conv"] for n in "qkv"]).float())
            assert torch.allclose(d.neg_a, -t[f"l{i}.mix.A_log"].float().exp()) and lw.proj_bias is None and lw.o_right is None
            assert torch.equal(lw.o, mix["o"])
        else:
            names = {"q": "left.q", "k": "left.k", "v": "left.v", "hg": "left.g", **{"lin_" + n: "right." + n for n in "qkvg"}, "lin_a": "right.a1"}
            bias = torch.zeros_like(lw.proj_bias)
            for n in "qkv":
                b = t[f"l{i}.mix.left.{n}.b"].float()
                bias[lw.offs[n]:lw.offs[n] + len(b)] = b
            assert torch.equal(lw.proj_bias, bias) and torch.equal(lw.o_bias, t[f"l{i}.mix.left.o.b"].float())
            assert torch.equal(lw.o, mix["left.o"]) and torch.equal(lw.o_right, mix["right.o"]) and torch.equal(lw.mix["a2"], mix["right.a2"])
            assert torch.equal(lw.branch_norms[1].weight, t[f"l{i}.mix.right.out"].float())
        for sec, key in names.items():
            o = lw.offs[sec]
            assert o % 8 == 0 and torch.equal(lw.proj[o:o + mix[key].shape[0]], mix[key])
        assert lw.proj.stride(0) % 8 == 0 and lw.o.stride(0) % 8 == 0 and (lw.norm2 is None) == (l["mlp"] is None)
        assert torch.equal(lw.norm1.weight, 1 + t[f"l{i}.norm1"].float())


def test_weights_of_the_wrong_shape_are_refused(tmp_path):
    from crosspool_b200.models.weights import load_attention_from_safetensors

    for i, key in enumerate(("l0.mix.right.a1", "l0.mix.right.a2", "l1.mix.k.conv")):
        t = sc.tensors("mixed")
        t[key] = t[key][:, :-1]
        d = sc.write_checkpoint(tmp_path / str(i), sc.CASES["mixed"], t)
        with pytest.raises(ValueError, match=key):
            load_attention_from_safetensors(_cfg("mixed"), d, "cpu", torch.float32)


def test_random_models_start_from_norms_of_one():
    from crosspool_b200.models.weights import random_attention_weights, random_ffn_weights

    c = _cfg("mixed")
    w = random_attention_weights(c, 1, "cpu", torch.float32)
    assert (w.layers[0].norm1.weight == 1).all() and (w.final_norm.weight == 1).all() and (w.layers[0].branch_norms[0].weight == 1).all()
    assert (w.layers[1].mix["delta"].neg_a == -1).all() and w.layers[0].mix["a2"].shape == (48, 16)
    assert random_ffn_weights(c, 1, "cpu")[2].extra["gate_transform"] == (7.0, 1.0, 1.702)


# ------------------------------------------------------------------ cache and states

def test_pages_states_and_convolution_inputs_follow_their_sequences():
    from crosspool_b200.engine.kv_cache import OutOfPages, PagedKvCache

    kv = PagedKvCache.fixed(_cfg("mixed"), 6, 16, "cpu", torch.float32, state_slots=2)
    assert [None if k is None else tuple(k.shape) for k in kv.k] == [(6, 16, 2, 64), None, None, (6, 16, 3, 64)]
    assert [None if v is None else tuple(v.shape) for v in kv.v] == [(6, 16, 2, 64), None, None, (6, 16, 3, 64)]
    assert [tuple(s.shape) for s in kv.states] == [(2, 3, 16, 24), (2, 6, 24, 40), (2, 2, 48, 16), (2, 2, 48, 32)]
    assert [None if s is None else tuple(s.shape) for s in kv.conv] == [None, (2, 4, 384), (2, 3, 224), None]
    assert kv.layout.bytes_per_page_all_layers == 16 * (256 + 384) * 4
    kv.ensure(1, 20)
    kv.ensure(2, 5)
    with pytest.raises(OutOfPages):
        kv.ensure(3, 1)
    slot = kv.seq_slots[1]
    kv.release(1)
    kv.ensure(3, 1)
    assert kv.seq_slots[3] == slot
    kv.release(2), kv.release(3)
    assert kv.allocator.free_pages == 6 and kv.slots.free_slots == 2


def test_attention_shapes_pad_to_a_kernel_or_not_at_all():
    from crosspool_b200.models.config import GroupedMixer, attention_shape

    assert attention_shape(24, 40) == (64, 64) and attention_shape(65, 64) == (128, 64) and attention_shape(160, 72) == (192, 128)
    assert attention_shape(24, 41) is None and attention_shape(193, 64) is None and attention_shape(64, 136) is None
    assert GroupedMixer(4, 2, 9, 13, 1.0).cache_rows == ((2, 16), (2, 16))
    from crosspool_b200.ops.mixers import group_pad

    assert [group_pad(h, 2) for h in (2, 4, 6, 10, 34)] == [1, 2, 4, 8, 32]
