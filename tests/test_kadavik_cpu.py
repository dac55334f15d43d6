"""Kadavik without a GPU: the plain implementation against independent forms of the same equations, configuration, FFN
description, weight layout, cache and state bookkeeping."""
import json
import math

import pytest
import torch

import kadavik_cases as kc
import kadavik_oracle as oracle


def _cfg(name):
    from crosspool_b200.models import config as mc

    return mc.from_hf_config(kc.CASES[name], name)


def _r(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


# ------------------------------------------------------------------ the plain implementation itself

def test_oracle_memory_equals_its_unscaled_sum():
    """Without the running maximum: S_t = sum_j e^(i_j + f_(j+1) + .. + f_t) k_j v_j^T, and the floor of the divisor is one."""
    T, d, e = 23, 6, 5
    q, k, v = _r(T, 1, d, seed=1), _r(T, 1, d, seed=2), _r(T, 1, e, seed=3)
    i, f = 2 * _r(T, 1, seed=4), -_r(T, 1, seed=5).abs()
    o, (S, n, m) = oracle.stabilised_memory(q, k, v, i, f)
    F = f[:, 0].cumsum(0)
    a, b = torch.arange(T)[:, None], torch.arange(T)[None, :]
    w = torch.where(b <= a, (F[:, None] - F[None, :] + i[None, :, 0]).exp(), torch.zeros((), dtype=torch.float64))
    s = w * (q[:, 0] @ k[:, 0].T)
    top = torch.stack([torch.maximum(F[t], (F[t] - F[:t + 1] + i[:t + 1, 0]).max()) for t in range(T)])
    size = torch.maximum(s.sum(1).abs(), torch.ones(T, dtype=torch.float64)) + 1e-6 * top.exp()
    assert torch.allclose(o[:, 0], (s @ v[:, 0]) / size[:, None]) and torch.allclose(m[0], top[-1])
    assert torch.allclose(S[0] * m.exp(), (w[-1][:, None] * k[:, 0]).T @ v[:, 0]) and torch.allclose(n[0] * m.exp(), w[-1] @ k[:, 0])


def test_oracle_memory_maximum_starts_at_zero():
    """A first input gate far below zero: the maximum follows the forget gate down from zero, not the input gate."""
    o, (S, n, m) = oracle.stabilised_memory(torch.ones(1, 1, 1), torch.ones(1, 1, 1), torch.ones(1, 1, 1), torch.full((1, 1), -9.0), torch.full((1, 1), -0.25))
    assert m.item() == -0.25 and abs(n.item() - math.exp(-8.75)) < 1e-9
    assert abs(o.item() - math.exp(-8.75) / (math.exp(0.25) + 1e-6)) < 1e-9


def test_oracle_gates_saturate():
    z = torch.tensor([-1e4, -3.0, 0.0, 3.0, 1e4], dtype=torch.float64)
    assert torch.allclose(oracle.soft_cap(z, 2.0)[[0, 2, 4]], torch.tensor([-2.0, 0.0, 2.0], dtype=torch.float64))
    assert torch.allclose(oracle.log_sigmoid(z[1:4]), torch.sigmoid(z[1:4]).log()) and oracle.log_sigmoid(z[:1]).item() == -1e4


def test_oracle_window_and_first_tokens():
    T, W, K = 12, 4, 2
    q, k, v = _r(T, 2, 3, seed=1), _r(T, 1, 3, seed=2), _r(T, 1, 2, seed=3)
    o = oracle.windowed_attention(q, k, v, 0.7, W, K)
    for i in range(T):
        seen = [j for j in range(i + 1) if i - j < W or j < K]
        assert len(seen) == min(i + 1, W + min(K, max(0, i + 1 - W)))
        for h in range(2):
            assert torch.allclose(o[i, h], (0.7 * k[seen, 0] @ q[i, h]).softmax(0) @ v[seen, 0])
    assert torch.allclose(oracle.windowed_attention(q, k, v, 0.7, 1, 0)[:, 1], v[:, 0])


def test_oracle_rotation_keeps_distances():
    f = oracle.rotary_frequencies(4, 100.0)
    assert torch.allclose(f, torch.tensor([1.0, 0.1], dtype=torch.float64))
    x = _r(1, 1, 6, seed=1).expand(9, 1, 6)
    y = oracle.rotate(x, f)[:, 0]
    assert torch.equal(y[0], x[0, 0]) and torch.equal(y[:, 4:], x[:, 0, 4:])
    assert torch.allclose(y[5] @ y[2], y[8] @ y[5]) and not torch.allclose(y[5] @ y[2], y[5] @ y[3])
    u, w = x[0, 0, 1], x[0, 0, 3]                            # pair 1: dimensions 1 and 3
    assert torch.allclose(y[7, 1], u * math.cos(0.7) - w * math.sin(0.7)) and torch.allclose(y[7, 3], w * math.cos(0.7) + u * math.sin(0.7))


def test_oracle_frequency_scaling_bands():
    sc = {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 100}
    plain, f = oracle.rotary_frequencies(16, 1000.0), oracle.rotary_frequencies(16, 1000.0, sc)
    wave = 2 * math.pi / plain
    assert torch.equal(f[wave < 25], plain[wave < 25]) and torch.allclose(f[wave > 100], plain[wave > 100] / 8)
    mid = (wave >= 25) & (wave <= 100)
    assert mid.any() and (f[mid] < plain[mid]).all() and (f[mid] > plain[mid] / 8).all()


def test_oracle_routing():
    z = torch.tensor([[2.0, 1.0, 0.0, -1.0]], dtype=torch.float64)
    s = z.softmax(-1)[0]
    w = oracle.routing(z, torch.tensor([0.0, 0.0, 0.0, 5.0], dtype=torch.float64), 2, 3.0)[0]
    assert torch.allclose(w, 3.0 * torch.stack([s[0], 0 * s[0], 0 * s[0], s[3]]) / (s[0] + s[3]))     # chosen with, weighed without
    m: list = []
    oracle.routing(z, torch.zeros(4), 2, 1.0, m)
    assert torch.allclose(m[0], s[1] - s[2])


def test_oracle_convolution_and_activations():
    x = _r(5, 2)
    w = torch.tensor([[1.0, 10.0, 100.0], [0.0, 0.0, 1.0]], dtype=torch.float64)
    y = oracle.short_convolution(x, w)
    assert torch.allclose(y[0, 0], 100 * x[0, 0]) and torch.allclose(y[4, 0], 100 * x[4, 0] + 10 * x[3, 0] + x[2, 0]) and torch.equal(y[:, 1], x[:, 1])
    z = _r(50)
    assert torch.allclose(oracle.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    assert torch.allclose(oracle.silu(z), torch.nn.functional.silu(z))


@pytest.mark.parametrize("name", ["mixed", "odd", "plain"])
def test_oracle_is_causal(name):
    c, t = kc.CASES[name], kc.tensors(name)
    ids = kc.prompt(c, 20, 3)
    assert torch.allclose(oracle.forward(c, t, ids)[:12], oracle.forward(c, t, ids[:12]), atol=1e-10)


def test_the_marked_token_shows_where_it_is_seen():
    """What the engine tests rest on: one token more or less in the window moves the logits far beyond rounding."""
    c, t = kc.marked_model(40, 5)
    ids = [i for i in kc.prompt(c, 200, 6) if i != kc.MARK][:160]
    for place in (4, 5, 64, 100):
        a, b = ids[:place] + [kc.MARK] + ids[place + 1:], ids[:place] + [8] + ids[place + 1:]
        e = kc.error(oracle.forward(c, t, a), oracle.forward(c, t, b))
        inside = e[place:place + 40].min()
        assert inside > 0.5 and (e[place + 40:].min() > 0.5 if place < 5 else e[place + 40] < 0.6 * inside)   # memories still hold some


# ------------------------------------------------------------------ configuration and FFN description

def test_config_reads_every_layer():
    c = _cfg("mixed")
    assert c.layered and c.recurrent and c.output_norm and c.input_norm and c.gpu_attention_supported and c.num_layers == 4
    assert [s.mixer.kind for s in c.layer_specs] == ["grouped_attention", "mlstm", "grouped_attention", "mlstm"]
    a, b = c.layer_specs[0].mixer, c.layer_specs[2].mixer
    assert (a.window, a.keep_first, a.conv, a.kv_from, a.head_norms) == (40, 5, 4, None, False)
    assert (b.window, b.keep_first, b.conv, b.kv_from) == (70, 0, 2, 0) and a.rot == b.rot
    assert (a.rot.dims, a.rot.base, a.rot.scaling.factor, a.rot.scaling.original) == (16, 1e4, 4.0, 64.0)
    m = c.layer_specs[0].moe
    assert (m.experts, m.top, m.ff, m.identity, m.shared_ff, m.scale, m.routed) == (5, 2, 40, 2, 56, 1.5, 7)
    assert [s.has_ffn for s in c.layer_specs] == [True, False, True, True] and c.layer_specs[2].gelu and c.layer_specs[2].ff == 136
    assert (c.token_side, c.embed_scale, c.logit_scale, c.rms_norm_eps) == (16, 4.0, 0.8, 1e-5)
    # one cached layer, heads padded to the tensor-core kernels' widths; the layer that reads it adds nothing
    assert c.kv_bytes_per_token() == 2 * 2 * 128
    states = 3 * 988 + 2 * 820                                # matrix, key sum and maximum, in whole 16 bytes
    assert c.layer_specs[1].mixer.head_state == 988 and c.layer_specs[3].mixer.head_state == 820
    assert c.state_bytes_per_sequence() == 4 * states + 2 * (4 * (6 * 24 + 2 * 64) + 2 * 6 * 24)
    assert a.visible(30) == 30 and a.visible(1000) == 45


def test_a_plain_model_needs_no_slots():
    c = _cfg("plain")
    assert not c.recurrent and c.token_side == 0 and c.layer_specs[0].mixer.window == 0 and c.layer_specs[0].mixer.visible(1000) == 1000


def test_parameter_counts_match_the_checkpoint():
    for name in kc.CASES:
        t, c = kc.tensors(name), _cfg(name)
        assert c.attention_param_bytes() == 2 * sum(v.numel() for k, v in t.items() if ".mlp." not in k), name
        for i in range(c.num_layers):
            assert c.ffn_param_bytes_per_layer(i) == 2 * sum(v.numel() for k, v in t.items() if k.startswith(f"l{i}.mlp.")), (name, i)


@pytest.mark.parametrize("layer,change", [
    (0, lambda l: l.update(type="lightning")), (0, lambda l: l["mixer"].update(kv_heads=4)), (0, lambda l: l["mixer"].update(kv_from=0)),
    (2, lambda l: l["mixer"].update(kv_from=1)), (2, lambda l: l["mixer"].update(vdim=32)), (0, lambda l: l["mixer"]["rot"].update(dims=26)),
    (0, lambda l: l["mixer"]["rot"].update(dims=15)), (1, lambda l: l["mixer"].update(gate_cap=0.0)), (0, lambda l: l["mlp"]["router"].update(top=8)),
    (2, lambda l: l["mlp"].update(kind="sparse")), (0, lambda l: l["mixer"]["mask"].update(size=0))])
def test_config_refuses_what_it_does_not_know(layer, change):
    from crosspool_b200.models import config as mc

    c = json.loads(json.dumps(kc.CASES["mixed"]))
    change(c["layers"][layer])
    with pytest.raises(ValueError):
        mc.from_hf_config(c)


def test_ffn_description_covers_the_checkpoint_and_loads(tmp_path):
    from crosspool_b200.deployment import load_ffn_weights
    from crosspool_b200.models.config import GELU_ALPHA, GELU_CUBIC

    t = kc.tensors("mixed")
    fw = load_ffn_weights(_cfg("mixed"), kc.write_checkpoint(tmp_path / "m", kc.CASES["mixed"], t), "cpu", torch.float32)
    assert fw[1] is None and fw[2].extra["gate_transform"] == pytest.approx((0.0, 0.0, GELU_ALPHA, GELU_CUBIC))
    assert torch.equal(fw[2].gate_up, torch.cat([t["l2.mlp.gate"], t["l2.mlp.up"]]).float())
    w = fw[0]
    assert w.is_moe and tuple(w.gate_up.shape) == (5, 80, 96) and tuple(w.router.shape) == (7, 96)
    assert torch.equal(w.gate_up[3], torch.cat([t["l0.mlp.e3.gate"], t["l0.mlp.e3.up"]]).float()) and torch.equal(w.down[4], t["l0.mlp.e4.down"].float())
    assert torch.equal(w.extra["correction_bias"], t["l0.mlp.correction"].float()) and torch.equal(w.extra["shared_scale"], t["l0.mlp.shared.sg"].float())
    for bad in ("l0.mlp.e4.down", "l3.mlp.shared.sg", "l0.mlp.correction"):
        less = {k: v for k, v in t.items() if k != bad}
        with pytest.raises(ValueError, match=bad):
            load_ffn_weights(_cfg("mixed"), kc.write_checkpoint(tmp_path / bad, kc.CASES["mixed"], less), "cpu", torch.float32)
    with pytest.raises(ValueError, match="e5"):
        load_ffn_weights(_cfg("mixed"), kc.write_checkpoint(tmp_path / "more", kc.CASES["mixed"], {**t, "l0.mlp.e5.gate": t["l0.mlp.e4.gate"].clone()}), "cpu",
                         torch.float32)


def test_gelu_is_the_gated_activation_with_a_cubic_term():
    from crosspool_b200.models.config import GELU_ALPHA, GELU_CUBIC

    z = _r(100, seed=3) * 3
    assert torch.allclose(z * torch.sigmoid(GELU_ALPHA * z * (1 + GELU_CUBIC * z * z)), oracle.gelu_tanh(z))


# ------------------------------------------------------------------ weight layout

@pytest.mark.parametrize("name", list(kc.CASES))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_fused_projection_holds_every_map_at_its_offset(tmp_path, name, dtype):
    from crosspool_b200.models.weights import load_attention_from_safetensors

    c, t = kc.CASES[name], kc.tensors(name)
    w = load_attention_from_safetensors(_cfg(name), kc.write_checkpoint(tmp_path, c, t), "cpu", dtype)
    assert torch.equal(w.embed, t["embed"].to(dtype)) and torch.equal(w.final_norm.weight, t["final.norm"].float())
    assert ("side_embed" in w.extra) == bool(c.get("token_side"))
    for i, (lw, l) in enumerate(zip(w.layers, c["layers"])):
        mix = {k.split(".mix.")[1]: v.to(dtype) for k, v in t.items() if k.startswith(f"l{i}.mix.")}
        if l["type"] == "mlstm":
            names = "qkvgif"
            assert lw.fp32_from == lw.offs["i"] and torch.equal(lw.mix["norm"], t[f"l{i}.mix.norm"].float())
            bias = torch.zeros_like(lw.proj_bias)
            for n in "if":
                bias[lw.offs[n]:lw.offs[n] + l["mixer"]["heads"]] = t[f"l{i}.mix.{n}.b"].float()
            assert torch.equal(lw.proj_bias, bias)
        else:
            names = "qkvg" if l["mixer"].get("kv_from") is None else "qg"
            assert lw.fp32_from == 0 and lw.proj_bias is None
            if l["mixer"].get("conv"):
                assert torch.equal(lw.mix["conv"], torch.cat([t[f"l{i}.mix.{n}.conv"] for n in names[:-1]]).float().T)
            else:
                assert lw.mix["conv"] is None
        assert set(lw.offs) == {*names, "end"}
        for n in names:
            o = lw.offs[n]
            assert o % 8 == 0 and torch.equal(lw.proj[o:o + mix[n].shape[0]], mix[n])
        assert lw.proj.stride(0) % 8 == 0 and lw.o.stride(0) % 8 == 0 and torch.equal(lw.o, mix["o"])
        assert torch.equal(lw.norm1b.weight, t[f"l{i}.norm1b"].float()) and (lw.norm2b is None) == (l["mlp"] is None)
        if c.get("token_side"):
            assert torch.equal(lw.side_proj, t[f"l{i}.side.proj"].to(dtype)) and lw.side_proj.stride(0) % 8 == 0


def test_weights_of_the_wrong_shape_are_refused(tmp_path):
    from crosspool_b200.models.weights import load_attention_from_safetensors

    for i, key in enumerate(("l1.mix.i", "l0.mix.k.conv", "l2.side.gate", "side.embed")):
        t = kc.tensors("mixed")
        t[key] = t[key][:, :-1]
        d = kc.write_checkpoint(tmp_path / str(i), kc.CASES["mixed"], t)
        with pytest.raises(ValueError, match=key):
            load_attention_from_safetensors(_cfg("mixed"), d, "cpu", torch.float32)


@pytest.mark.parametrize("scaling", [None, (4.0, 1.0, 4.0, 64), (8.0, 1.0, 4.0, 3000), (2.0, 1.0, 1.5, 20)])
def test_rotary_table(scaling):
    from crosspool_b200.models.config import _rotary
    from crosspool_b200.models.layered import rotary_table

    r = {"dims": 24, "base": 5e3, **({"scaling": dict(zip(("factor", "low", "high", "original"), scaling))} if scaling else {})}
    tab = rotary_table(_rotary(r, 32), 3000, "cpu")
    a = torch.arange(3000, dtype=torch.float64)[:, None] * oracle.rotary_frequencies(24, 5e3, r.get("scaling"))
    assert torch.allclose(tab[..., 0].double(), a.cos(), atol=1e-7) and torch.allclose(tab[..., 1].double(), a.sin(), atol=1e-7)


def test_random_models_have_every_part():
    from crosspool_b200.models.weights import random_attention_weights, random_ffn_weights

    c = _cfg("mixed")
    w, f = random_attention_weights(c, 1, "cpu", torch.float32), random_ffn_weights(c, 1, "cpu")
    assert (w.layers[0].norm1.weight == 1).all() and (w.final_norm.weight == 1).all() and (w.layers[0].side_norm.weight == 1).all()
    assert tuple(w.extra["side_embed"].shape) == (211, 64) and w.layers[2].mix["conv"].shape == (2, 144)
    assert f[1] is None and tuple(f[3].shared_gate_up.shape) == (32, 96) and len(f[2].extra["gate_transform"]) == 4


# ------------------------------------------------------------------ cache and states

def test_pages_states_and_convolution_inputs_follow_their_sequences():
    from crosspool_b200.engine.kv_cache import OutOfPages, PagedKvCache

    kv = PagedKvCache.fixed(_cfg("mixed"), 6, 16, "cpu", torch.float32, state_slots=2)
    assert [None if k is None else tuple(k.shape) for k in kv.k] == [(6, 16, 2, 64), None, (6, 16, 2, 64), None]
    assert kv.k[2] is kv.k[0] and kv.v[2] is kv.v[0]
    assert [None if s is None else tuple(s.shape) for s in kv.states] == [None, (2, 3, 988), None, (2, 2, 820)]
    assert [None if s is None else tuple(s.shape) for s in kv.conv] == [(2, 4, 272), None, (2, 2, 144), None]
    assert kv.layout.bytes_per_page_all_layers == 16 * 256 * 4
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


def test_attention_with_convolutions_alone_has_slots():
    from crosspool_b200.models import config as mc

    c = json.loads(json.dumps(kc.CASES["plain"]))
    assert not mc.from_hf_config(c).recurrent
    c["layers"][1]["mixer"]["conv"] = 3
    assert mc.from_hf_config(c).recurrent
