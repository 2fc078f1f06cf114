"""Votavik without a GPU: the configuration reader and its validation, the checkpoint loader (names, fused and padded rows, missing and
unexpected tensors), the registry, the states, and closed-form checks of the plain restatement the GPU tests compare with."""
from __future__ import annotations

import copy
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import votavik_oracle as O  # noqa: E402
from test_gpu_votavik import CFG_ODD, CFG_TILES, CFG_WIDE, attention, checkpoint, config, model_of  # noqa: E402

from lit_gpt_b200.config import ClampedGLUSpec, GatedWindowSpec, LinearMixerSpec, VotavikConfig, architectures, load_config, model_class  # noqa: E402


def test_configuration_reads_every_size_and_constant():
    c = VotavikConfig.from_dict(CFG_ODD[0])
    assert (c.vocab_size, c.n_embd, c.side_dim, c.norm_eps, c.n_layer) == (83, 42, 6, 1e-5, 5)
    assert [ly.type for ly in c.layers] == ["gla", "attention", "lightning", "attention", "gla"]
    m = c.layers[1].mixer
    assert isinstance(m, GatedWindowSpec) and (m.heads, m.kv_heads, m.dim, m.vdim, m.window, m.keep, m.scale, m.softcap) == (4, 2, 12, 10, 7, 3, 0.9, 4.0)
    assert (m.rot.dims, m.rot.base, m.rot.interleaved) == (6, 100.0, False) and m.qk_norm and m.sink and m.gate == "head" and not m.bias and not m.distance
    g, li = c.layers[0].mixer, c.layers[2].mixer
    assert isinstance(g, LinearMixerSpec) and (g.heads, g.dim, g.vdim, g.tau, g.decay) == (3, 10, 7, 4.0, None)
    assert (li.heads, li.dim, li.vdim, li.decay) == (2, 14, 9, [0.5, 0.97])
    f = c.layers[0].mlp
    assert isinstance(f, ClampedGLUSpec) and (f.ff, f.limit, f.alpha) == (50, 0.9, 1.702) and c.layers[1].mlp is None
    assert c.schedule() == [(i, i) for i in range(5)]


def test_defaults_of_absent_keys():
    js, _ = config(24, 11, 3, [("attention", dict(heads=3, dim=8, mask=dict(size=4), scale=0.5), None)])
    m = VotavikConfig.from_dict(js).layers[0].mixer
    assert (m.kv_heads, m.vdim, m.keep, m.softcap, m.rot) == (3, 8, 0, 0.0, None)
    js["layers"][0]["mixer"]["rot"] = dict(base=10.0, dims=0)
    assert VotavikConfig.from_dict(js).layers[0].mixer.rot is None


@pytest.mark.parametrize("bad", [
    lambda js: js["layers"][0].__setitem__("type", "gla_2"),
    lambda js: js["layers"][0]["mixer"].__setitem__("tau", 0.0),
    lambda js: js["layers"][1]["mixer"].__setitem__("kv_heads", 3),
    lambda js: js["layers"][1]["mixer"]["rot"].__setitem__("dims", 7),
    lambda js: js["layers"][1]["mixer"]["rot"].__setitem__("dims", 14),
    lambda js: js["layers"][1]["mixer"]["mask"].__setitem__("size", 0),
    lambda js: js["layers"][2]["mixer"].__setitem__("decay", [0.5]),
    lambda js: js["layers"][2]["mixer"].__setitem__("decay", [0.5, 1.5]),
    lambda js: js["layers"][0]["mlp"].__setitem__("kind", "moe"),
    lambda js: js["layers"][0]["mlp"].__setitem__("limit", 0.0),
    lambda js: js["token_side"].__setitem__("dim", 0),
])
def test_configuration_is_validated(bad):
    js = copy.deepcopy(CFG_ODD[0])
    bad(js)
    with pytest.raises(ValueError):
        VotavikConfig.from_dict(js)


def test_registry_and_checkpoint_directory(tmp_path):
    assert "Votavik" in architectures
    (tmp_path / "config.json").write_text(json.dumps(CFG_ODD[0]))
    c = load_config(tmp_path)
    assert isinstance(c, VotavikConfig) and model_class(c).__name__ == "Votavik"


def test_loader_fuses_and_pads_projections():
    w = checkpoint(CFG_ODD, 5)
    model = model_of(CFG_ODD, w, "cpu").to(torch.bfloat16)
    for p in model.parameters():
        p.data.fill_(99.0)
    model.load_tensors(w)
    mx = model.blocks[1].mixer
    rows = torch.cat([w["l1.mix." + n] for n in ("q", "k", "v", "g")])
    assert mx.gate_cols == 4 and torch.equal(mx.w_in[: rows.shape[0]], rows) and mx.w_in.shape[0] % 8 == 0 and not mx.w_in[rows.shape[0] :].any()
    assert torch.equal(mx.q_norm, w["l1.mix.q.norm"]) and torch.equal(mx.k_norm, w["l1.mix.k.norm"]) and torch.equal(mx.sink, w["l1.mix.sink"])
    gx = model.blocks[0].mixer
    rows = torch.cat([w["l0.mix." + n] for n in ("q", "k", "v", "g", "a1")])
    assert gx.channel and gx.spec.decay_rank == 5 and torch.equal(gx.w_in[: rows.shape[0]], rows) and not gx.w_in[rows.shape[0] :].any()
    assert torch.equal(gx.w_in[gx.off_decay : gx.off_decay + 5], w["l0.mix.a1"]) and torch.equal(gx.w_in[gx.off_gate : gx.off_decay], w["l0.mix.g"])
    assert torch.equal(gx.w_decay2, w["l0.mix.a2"]) and torch.equal(gx.decay_bias, w["l0.mix.a2.b"]) and gx.norm.numel() == 7
    lx = model.blocks[2].mixer
    assert not lx.channel and lx.norm.numel() == 18 and torch.allclose(lx.head_decay(torch.device("cpu")), torch.tensor([0.5, 0.97]))
    assert torch.equal(model.blocks[0].mlp.w_up, torch.cat([w["l0.mlp.gate"], w["l0.mlp.up"]])) and model.blocks[1].mlp is None
    assert torch.equal(model.blocks[3].side.w_proj, w["l3.side.proj"]) and model.blocks[3].side.off == 18
    assert torch.equal(model.side_embed, w["side.embed"]) and torch.equal(model.head, w["head"])
    assert not any(bool((p == 99.0).any()) for p in model.parameters())


def test_loader_rejects_missing_and_unexpected_tensors():
    w = checkpoint(CFG_WIDE, 6)
    model = model_of(CFG_WIDE, w, "cpu").to(torch.bfloat16)
    for name in ("l0.mix.sink", "l3.mix.a2.b", "side.embed", "l1.side.norm"):
        with pytest.raises(KeyError):
            model.load_tensors({k: v for k, v in w.items() if k != name})
    with pytest.raises(KeyError):
        model.load_tensors(dict(w, **{"l0.mix.q.b": torch.zeros(144, dtype=torch.bfloat16)}))
    with pytest.raises(ValueError):
        model.load_tensors(dict(w, **{"l1.norm1": torch.zeros(65, dtype=torch.bfloat16)}))
    model.load_tensors(w)


def test_states_have_the_size_of_what_is_kept_and_stay_fp32():
    w = checkpoint(CFG_TILES, 7)
    model = model_of(CFG_TILES, w, "cpu").to(torch.bfloat16)
    model.set_kv_cache(batch_size=3)
    first, second, third = model.states[0], model.states[1], model.states[2]
    assert tuple(first.k_ring.shape) == (3, 44 + 5, 128) and first.k_ring.dtype == torch.bfloat16
    assert tuple(third.v_ring.shape) == (3, 50 + 70, 128)
    assert tuple(second.matrices.shape) == (3, 4 * 32 * 24) and second.matrices.dtype == torch.float32
    model.to(torch.float64)
    assert model.states[1].matrices.dtype == torch.float32
    assert not model.repeatable_steps and model.max_seq_length > 1 << 20
    with pytest.raises(TypeError):
        model.clear_kv_cache()
        model.step([1], [(0, 0, 1)])


# ---- the restatement itself, on cases with a closed form ---------------------------------------------------------------------
def test_oracle_mask_keeps_the_first_tokens_and_the_window():
    mask = dict(size=3, keep_first=2)
    assert O.visible(0, mask) == [0] and O.visible(3, mask) == [0, 1, 2, 3] and O.visible(4, mask) == [0, 1, 2, 3, 4]
    assert O.visible(9, mask) == [0, 1, 7, 8, 9] and O.visible(9, dict(size=1, keep_first=0)) == [9]


def test_oracle_attention_flat_scores_sink_and_cap():
    T, dk, dv = 6, 4, 3
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(T, 1, d, generator=g, dtype=torch.float64) for d in (dk, dk, dv))
    mask = dict(size=2, keep_first=1)
    out = O.capped_attention(q, k, v, None, mask, 0.0, 5.0)
    assert torch.allclose(out[5], v[[0, 4, 5]].mean(0)) and torch.allclose(out[0], v[0])
    out = O.capped_attention(q, k, v, torch.tensor([math.log(3.0)], dtype=torch.float64), mask, 0.0, 5.0)
    assert torch.allclose(out[5], v[[0, 4, 5]].sum(0) / 6.0)            # three keys of weight 1 beside a sink of 3
    big = O.capped_attention(q * 1e6, k, v, None, dict(size=6, keep_first=0), 1.0, 1e-9)
    assert torch.allclose(big[5], v.mean(0), atol=1e-6)                 # a tiny cap makes every score the same


def test_oracle_rotation():
    x = torch.zeros(2, 1, 6, dtype=torch.float64)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 3.0                                   # pair (0, 2) of dims = 4; dimensions 4, 5 pass
    r = O.rotate_half(x, dict(base=100.0, dims=4), 7)
    assert abs(float(r[0, 0, 0]) - math.cos(7.0)) < 1e-12 and abs(float(r[1, 0, 2]) - math.sin(8.0)) < 1e-12 and float(r[0, 0, 5]) == 3.0
    q = torch.randn(3, 1, 4, dtype=torch.float64)
    a, b = O.rotate_half(q, dict(base=10.0, dims=4), 5), O.rotate_half(q, dict(base=10.0, dims=4), 105)
    assert torch.allclose((a[2] * a[0]).sum(), (b[2] * b[0]).sum())     # scores depend on the distance only


def test_oracle_recurrence_and_norms():
    k = torch.ones(4, 1, dtype=torch.float64)
    v = torch.tensor([[1.0], [0.0], [0.0], [2.0]], dtype=torch.float64)
    o = O.decayed_sum(2 * k, k, v, torch.full((4, 1), 0.5, dtype=torch.float64))
    assert torch.allclose(o[:, 0], torch.tensor([2.0, 1.0, 0.5, 4.25], dtype=torch.float64))    # the read-out sees the token's own write
    x = torch.tensor([[1.0, 3.0]], dtype=torch.float64)
    one = torch.ones(2, dtype=torch.float64)
    assert torch.allclose(O.layer_norm(x, one, 0.0), torch.tensor([[-1.0, 1.0]], dtype=torch.float64))
    assert torch.allclose(O.rms(x, one, 4.0), x / 3.0)                   # eps inside the root
    W = {"gate": torch.eye(2, dtype=torch.float64), "up": torch.eye(2, dtype=torch.float64), "down": torch.eye(2, dtype=torch.float64)}
    y = O.clamped_glu(torch.tensor([[5.0, -5.0]], dtype=torch.float64), W, "", dict(limit=1.0))
    assert abs(float(y[0, 0]) - 2.0 / (1.0 + math.exp(-1.702))) < 1e-12 and abs(float(y[0, 1])) < 1e-12


def test_oracle_is_causal_and_uses_every_part():
    cr = config(16, 13, 4, [("attention", attention(2, 1, 4, 6, size=3, keep=1, rot_dims=2, cap=5.0), None)])
    w = checkpoint(cr, 2)
    toks = [1, 5, 2, 7, 7, 3]
    a = O.forward(cr[0], w, toks)
    assert a.shape == (6, 13) and torch.isfinite(a).all() and torch.allclose(O.forward(cr[0], w, toks[:4]), a[:4])
    for name in w:
        changed = dict(w, **{name: w[name] * 1.5 + 0.25})
        assert not torch.allclose(O.forward(cr[0], changed, toks), a), name
