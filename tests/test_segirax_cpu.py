"""Segirax without a GPU: configuration, FFN description, weight layout, cache and state bookkeeping, the replay loop, and
the plain implementation against independent forms of the same equations."""
import io
import json
import math

import pytest
import torch

import segirax_cases as sc
import segirax_oracle as oracle


def _cfg(name):
    from crosspool_b200.models import config as mc

    return mc.from_hf_config(sc.CASES[name], name)


# ------------------------------------------------------------------ the plain implementation itself

def test_oracle_recurrence_equals_its_closed_form():
    g = torch.Generator().manual_seed(0)
    q, k, v = (torch.randn(23, 2, n, generator=g, dtype=torch.float64) for n in (5, 5, 3))
    decay = [0.8, 0.99]
    o, S = oracle.decayed_recurrence(q, k, v, decay)
    for h in range(2):
        i, j = torch.arange(23)[:, None], torch.arange(23)[None, :]
        m = torch.where(j <= i, decay[h] ** (i - j).double(), torch.zeros((), dtype=torch.float64))
        assert torch.allclose(o[:, h], ((q[:, h] @ k[:, h].T) * m) @ v[:, h])
        assert torch.allclose(S[h], sum(decay[h] ** (22 - t) * torch.outer(k[t, h], v[t, h]) for t in range(23)))


def test_oracle_rotation_is_relative_and_leaves_the_rest_alone():
    g = torch.Generator().manual_seed(1)
    a, b = torch.randn(1, 10, generator=g, dtype=torch.float64), torch.randn(1, 10, generator=g, dtype=torch.float64)

    def rot(x, p):
        return oracle.rotate_half(x, torch.tensor([p]), 6, 100.0)

    assert torch.allclose((rot(a, 9) * rot(b, 4)).sum(), (rot(a, 105) * rot(b, 100)).sum())
    assert torch.equal(rot(a, 7)[0, 6:], a[0, 6:])
    # pair (0, 3) turns by the position itself, pair (2, 5) by position * 100 ** (-4 / 6)
    y = rot(a, 2)[0]
    assert torch.allclose(y[0], a[0, 0] * math.cos(2) - a[0, 3] * math.sin(2))
    ang = 2 * 100.0 ** (-4 / 6)
    assert torch.allclose(y[5], a[0, 5] * math.cos(ang) + a[0, 2] * math.sin(ang))


def test_oracle_norms_and_activation():
    x = torch.tensor([[3.0, -4.0]], dtype=torch.float64)
    assert torch.allclose(oracle.rms(x, 0.0), x / math.sqrt(12.5))
    y = oracle.poly_norm(x, torch.tensor([1.0, 2.0, 3.0, 0.5]), 0.0)
    want = x / math.sqrt(12.5) + 2 * x ** 2 / math.sqrt((81 + 256) / 2) + 3 * x ** 3 / math.sqrt((27 ** 2 + 64 ** 2) / 2) + 0.5
    assert torch.allclose(y, want)
    assert torch.allclose(oracle.dynamic_tanh(x, 0.5, torch.tensor([2.0, 1.0]), torch.tensor([0.0, 1.0])),
                          torch.tensor([[2 * math.tanh(1.5), 1 + math.tanh(-2.0)]], dtype=torch.float64))


def test_oracle_is_causal():
    c, t = sc.CASES["mixed"], sc.tensors("mixed")
    ids = sc.prompt(c, 20, 3)
    assert torch.allclose(oracle.forward(c, t, ids)[:12], oracle.forward(c, t, ids[:12]), atol=1e-10)


# ------------------------------------------------------------------ configuration and FFN description

def test_config_reads_every_layer():
    c = _cfg("mixed")
    assert c.layered and c.recurrent and c.gpu_attention_supported and c.num_layers == 4
    assert [s.mixer.kind for s in c.layer_specs] == ["latent_attention", "lightning", "lightning", "latent_attention"]
    assert [s.ff for s in c.layer_specs] == [136, 72, 0, 200]
    m = c.layer_specs[3].mixer
    assert (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.rot.base) == (5, 40, 8, 16, 88, 5e5)
    assert c.kv_bytes_per_token() == 2 * (80 + 96) and c.state_bytes_per_sequence() == 4 * (2 * 48 * 24 + 3 * 16 * 48)
    assert c.rms_norm_eps == 1e-5 and c.logit_scale == 0.7 and c.tie_word_embeddings
    assert not _cfg("heads").recurrent
    assert [s.ff for s in c.with_layers(6).layer_specs] == [136, 72, 0, 200, 136, 72]


def test_attention_parameter_count_matches_the_checkpoint():
    for name in sc.CASES:
        t = sc.tensors(name)
        n = sum(v.numel() for k, v in t.items() if ".mlp." not in k)
        assert _cfg(name).attention_param_bytes() == 2 * n, name


@pytest.mark.parametrize("change", [lambda l: l.update(type="other"), lambda l: l.update(mlp={"kind": "moe", "ff": 8}),
                                    lambda l: l["mixer"]["rot"].update(dims=18), lambda l: l["mixer"]["rot"].update(dims=5)])
def test_config_refuses_what_it_does_not_know(change):
    c = json.loads(json.dumps(sc.CASES["mixed"]))
    change(c["layers"][0])
    from crosspool_b200.models import config as mc

    with pytest.raises(ValueError):
        mc.from_hf_config(c)


def test_config_refuses_a_decay_count_other_than_the_heads():
    c = json.loads(json.dumps(sc.CASES["mixed"]))
    c["layers"][1]["mixer"]["decay"] = [0.5]
    from crosspool_b200.models import config as mc

    with pytest.raises(ValueError, match="decay"):
        mc.from_hf_config(c)


def test_ffn_description_covers_the_checkpoint_and_loads(tmp_path):
    from crosspool_b200.deployment import has_checkpoint, load_ffn_weights

    t = sc.tensors("mixed")
    d = sc.write_checkpoint(tmp_path / "m", sc.CASES["mixed"], t)
    assert has_checkpoint(d) and not has_checkpoint("Qwen/Qwen3-0.6B")
    fw = load_ffn_weights(_cfg("mixed"), d, "cpu", torch.float32)
    assert fw[2] is None
    for i in (0, 1, 3):
        assert torch.equal(fw[i].gate_up, t[f"l{i}.mlp.up"].float()) and torch.equal(fw[i].down, t[f"l{i}.mlp.down"].float())
        coef, eps = fw[i].extra["polynorm"]
        assert torch.equal(coef, t[f"l{i}.mlp.act"].float()) and eps == 1e-5
    t["l2.mlp.up"] = t["l0.mlp.up"].clone()
    with pytest.raises(ValueError, match="l2.mlp.up"):
        load_ffn_weights(_cfg("mixed"), sc.write_checkpoint(tmp_path / "extra", sc.CASES["mixed"], t), "cpu", torch.float32)
    del t["l2.mlp.up"], t["l3.mlp.act"]
    with pytest.raises(ValueError, match="l3.mlp.act"):
        load_ffn_weights(_cfg("mixed"), sc.write_checkpoint(tmp_path / "less", sc.CASES["mixed"], t), "cpu", torch.float32)


# ------------------------------------------------------------------ weight layout

@pytest.mark.parametrize("name", list(sc.CASES))
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_fused_projection_holds_every_map_at_its_offset(tmp_path, name, dtype):
    from crosspool_b200.models.weights import load_attention_from_safetensors

    c, t = sc.CASES[name], sc.tensors(name)
    w = load_attention_from_safetensors(_cfg(name), sc.write_checkpoint(tmp_path, c, t), "cpu", dtype)
    assert torch.equal(w.embed, t["embed"].to(dtype)) and torch.equal(w.lm_head, w.embed)
    for i, (lw, l) in enumerate(zip(w.layers, c["layers"])):
        m, mix = l["mixer"], {k.split(".mix.")[1]: v.to(dtype) for k, v in t.items() if k.startswith(f"l{i}.mix.")}
        names = {"q": "q", "kv": "dkv", "g": "g"} if l["type"] == "latent_attention" else {n: n for n in "qkvg"}
        for sec, key in names.items():
            o = lw.offs[sec]
            assert o % 8 == 0 and torch.equal(lw.proj[o:o + mix[key].shape[0]], mix[key])
        o = lw.offs["rg"]
        assert torch.equal(lw.proj[o:o + c["width"]], t[f"l{i}.rg1"].to(dtype))
        assert torch.equal(lw.proj_bias[o:o + c["width"]], t[f"l{i}.rg1.b"].float()) and lw.proj_bias[:o].abs().sum() == 0
        assert lw.proj.stride(0) % 8 == 0 and lw.o.stride(0) % 8 == 0
        assert (lw.norm2 is None) == (l["mlp"] is None) == (lw.rg2 is None)
        if l["type"] == "lightning":
            assert lw.silu_cols == lw.offs["g"] and torch.allclose(lw.mix["decay_pow"][:, 3], torch.tensor(m["decay"]) ** 3)
            continue
        H, R, d, r, vd = m["heads"], m["kv_rank"], m["dim"], m["rot_dim"], m["vdim"]
        assert torch.equal(lw.mix["uk_t"].reshape(H, R, d).transpose(1, 2).reshape(H * d, R), mix["uk"])
        if "exp_k" in lw.mix:
            # the expanded keys of a (latent, rotary) row: per-head plain keys, then the shared rotary part, then zeros
            row = torch.randn(R + r, generator=torch.Generator().manual_seed(0)).to(dtype)
            k = (lw.mix["exp_k"].float() @ row.float()).view(H, -1)
            assert torch.allclose(k[:, :d].reshape(-1), mix["uk"].float() @ row[:R].float(), atol=1e-4)
            assert torch.equal(k[:, d:d + r], row[R:].float().expand(H, r)) and k[:, d + r:].abs().sum() == 0


def test_weights_of_the_wrong_shape_are_refused(tmp_path):
    from crosspool_b200.models.weights import load_attention_from_safetensors

    t = sc.tensors("mixed")
    t["l0.mix.uk"] = t["l0.mix.uk"][:-1]
    d = sc.write_checkpoint(tmp_path, sc.CASES["mixed"], t)
    with pytest.raises(ValueError, match="l0.mix.uk"):
        load_attention_from_safetensors(_cfg("mixed"), d, "cpu", torch.float32)


# ------------------------------------------------------------------ cache and states

def test_state_slots_follow_their_sequences_and_are_used_again():
    from crosspool_b200.engine.kv_cache import OutOfPages, PagedKvCache

    kv = PagedKvCache.fixed(_cfg("mixed"), 6, 16, "cpu", torch.float32, state_slots=2)
    assert [None if k is None else tuple(k.shape) for k in kv.k] == [(6, 16, 1, 80), None, None, (6, 16, 1, 96)]
    assert [None if s is None else tuple(s.shape) for s in kv.states] == [None, (2, 2, 48, 24), (2, 3, 16, 48), None]
    assert kv.layout.bytes_per_page_all_layers == 16 * (80 + 96) * 4
    kv.ensure(1, 20)
    kv.ensure(2, 5)
    assert {kv.seq_slots[1], kv.seq_slots[2]} == {0, 1} and kv.slots.free_slots == 0
    with pytest.raises(OutOfPages):
        kv.ensure(3, 1)
    assert 3 not in kv.tables and kv.allocator.free_pages == 3
    slot = kv.seq_slots[1]
    kv.release(1)
    kv.ensure(3, 1)
    assert kv.seq_slots[3] == slot
    with pytest.raises(OutOfPages):
        kv.ensure(2, 1000)
    kv.release(2), kv.release(3)
    assert kv.allocator.free_pages == 6 and kv.slots.free_slots == 2


def test_a_model_without_recurrence_needs_no_slots():
    from crosspool_b200.engine.kv_cache import PagedKvCache

    kv = PagedKvCache.fixed(_cfg("heads"), 4, 16, "cpu")
    kv.ensure(1, 30)
    assert kv.slots is None and not kv.seq_slots


def test_elastic_cache_and_ffn_tier_refuse_layered_models():
    from crosspool_b200.ecs import vmm
    from crosspool_b200.models.weights import random_ffn_layer

    with pytest.raises(NotImplementedError):
        vmm.elastic_kv_cache(_cfg("mixed"), 4, 16, "cpu", None, None)
    with pytest.raises(NotImplementedError):
        random_ffn_layer(_cfg("mixed"), 0, tp_size=2)


# ------------------------------------------------------------------ replay loop

class _FakeEngine:
    def __init__(self):
        self.log, self.n = [], 0

    def open_sequence(self):
        self.n += 1
        return f"seq{self.n}"

    def close_sequence(self, s):
        self.log.append(("close", s))

    def run_given(self, portions, want):
        self.log.append(("run", portions, want))
        return torch.arange(3.0 * sum(len(w) for w in want)).view(-1, 3)


def test_replay_keeps_requests_apart_and_writes_only_what_is_wanted(tmp_path, monkeypatch, capsys):
    import numpy as np

    from crosspool_b200.native import build
    from crosspool_b200.runtime import trace_replay as tr

    eng = _FakeEngine()
    eng.warmup = lambda: None
    monkeypatch.setattr(build, "build_kernels", lambda: None)
    monkeypatch.setattr(tr, "build_engine", lambda *a: eng)
    lines = [{"step": 0, "entries": [{"id": "a", "tokens": [1, 2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": [4], "want": [0]}, {"id": "a", "tokens": [3], "want": [0]}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "a", "tokens": [9], "want": []}], "end": ["a", "b"]}]
    monkeypatch.setattr("sys.stdin", io.StringIO("\n".join(json.dumps(l) for l in lines) + "\n\n"))
    assert tr.main(["--model", "m", "--out", str(tmp_path), "--max-tokens", "64"]) == 0
    assert capsys.readouterr().out.split("\n")[:3] == ["done 0", "done 1", "done 2"]
    assert eng.log == [("run", [("seq1", [1, 2])], [[]]), ("run", [("seq2", [4]), ("seq1", [3])], [[0], [0]]), ("close", "seq1"),
                       ("run", [("seq3", [9])], [[]]), ("close", "seq3"), ("close", "seq2")]
    assert [p.name for p in tmp_path.iterdir()] == ["1.f32"]
    assert np.fromfile(tmp_path / "1.f32", "<f4").tolist() == [0, 1, 2, 3, 4, 5]
