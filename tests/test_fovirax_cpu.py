"""Fovirax without a GPU: the configuration reader and its validation, the order of runs, the frequencies, the checkpoint loader (names, fused
and padded blocks, missing and unexpected tensors), the registry, the states, and closed-form checks of the plain restatement the GPU
tests compare with."""
from __future__ import annotations

import copy
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import fovirax_oracle as O  # noqa: E402
from test_gpu_fovirax import CFG_ODD, CFG_TILES, CFG_WIDE, checkpoint, config, left, model_of, moe, right, tokens_for  # noqa: E402

from lit_gpt_b200.config import FoviraxConfig, GatedWindowSpec, RetentionSpec, RotarySpec, SharedMoESpec, architectures, load_config, model_class  # noqa: E402


def test_configuration_reads_every_size_and_constant():
    c = FoviraxConfig.from_dict(CFG_ODD)
    assert (c.vocab_size, c.n_embd, c.norm_eps, c.residual_mult, c.n_layer) == (83, 42, 1e-5, 0.7, 4)
    assert (c.loop_start, c.loop_stop, c.loop_times) == (1, 3, 3)
    m = c.layers[0].mixer
    assert isinstance(m.left, GatedWindowSpec) and isinstance(m.right, RetentionSpec) and (m.left_scale, m.right_scale) == (0.8, 0.7)
    lf, rt = m.left, m.right
    assert (lf.heads, lf.kv_heads, lf.dim, lf.vdim, lf.window, lf.scale, lf.softcap) == (4, 2, 12, 10, 7, 0.9, 4.0)
    assert (lf.rot.dims, lf.rot.base, lf.rot.factor, lf.rot.low, lf.rot.high, lf.rot.original, lf.rot.interleaved) == (6, 100.0, 3.0, 1.0, 5.0, 40.0, False)
    assert not (lf.gate or lf.qk_norm or lf.sink or lf.keep or lf.bias or lf.distance)
    assert (rt.heads, rt.dim, rt.vdim, rt.decay, rt.rot.dims, rt.rot.base, rt.rot.factor) == (3, 10, 7, [0.5, 0.9, 0.97], 6, 1000.0, None)
    e = c.layers[0].mlp
    assert isinstance(e, SharedMoESpec) and (e.experts, e.top, e.ff, e.shared_ff) == (6, 2, 14, 22)
    assert c.layers[1].mlp is None and c.layers[2].mlp.shared_ff == 0 and c.layers[3].mixer.right.rot is None and c.layers[1].mixer.right_scale == -0.5


def test_runs_of_a_loop_have_states_of_their_own():
    c = FoviraxConfig.from_dict(CFG_ODD)
    assert c.schedule() == [(0, 0), (1, 1), (2, 2), (1, 3), (2, 4), (1, 5), (2, 6), (3, 7)]
    assert [i for i, _ in c.schedule()] == O.run_order(CFG_ODD)
    assert FoviraxConfig.from_dict(CFG_WIDE).schedule() == [(0, 0), (1, 1), (2, 2)]
    assert [i for i, _ in FoviraxConfig.from_dict(CFG_TILES).schedule()] == [0, 1, 0, 1, 2]


def test_defaults_of_absent_keys():
    js = config(24, 11, [(dict(heads=3, dim=8, mask=dict(size=4), scale=0.5), dict(heads=2, dim=6, decay=[0.5, 0.9]), 1.0, 1.0, None)])
    m = FoviraxConfig.from_dict(js).layers[0].mixer
    assert (m.left.kv_heads, m.left.vdim, m.left.softcap, m.left.rot, m.right.vdim, m.right.rot) == (3, 8, 0.0, None, 6, None)
    js["layers"][0]["mixer"]["right"]["rot"] = dict(base=10.0, dims=0)
    assert FoviraxConfig.from_dict(js).layers[0].mixer.right.rot is None
    js["loop"] = None
    assert FoviraxConfig.from_dict(js).schedule() == [(0, 0)]


@pytest.mark.parametrize("bad", [
    lambda js: js["layers"][0].__setitem__("type", "attention"),
    lambda js: js["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 3),
    lambda js: js["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 7),
    lambda js: js["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 10),
    lambda js: js["layers"][1]["mixer"]["right"]["rot"].__setitem__("dims", 16),
    lambda js: js["layers"][1]["mixer"]["left"]["mask"].__setitem__("size", 0),
    lambda js: js["layers"][1]["mixer"]["right"].__setitem__("decay", [0.5]),
    lambda js: js["layers"][1]["mixer"]["right"].__setitem__("decay", [0.5, 1.5]),
    lambda js: js["layers"][0]["mlp"].__setitem__("kind", "dense"),
    lambda js: js["layers"][0]["mlp"]["router"].__setitem__("top", 7),
    lambda js: js["layers"][0]["mlp"]["router"].__setitem__("top", 0),
    lambda js: js["loop"].__setitem__("stop", 5),
    lambda js: js["loop"].__setitem__("times", 0),
])
def test_configuration_is_validated(bad):
    js = copy.deepcopy(CFG_ODD)
    bad(js)
    with pytest.raises(ValueError):
        FoviraxConfig.from_dict(js)


def test_frequencies_blend_by_wavelength():
    """Short wavelengths keep their frequency, long ones are stretched by the factor, those between are blended; YaRN specifications of the
    other designs are what they were."""
    rot = dict(base=500.0, dims=48, scaling=dict(factor=6.0, low=1.0, high=4.0, original=300))
    got = RotarySpec.from_dict(rot, interleaved=False)
    want = [O.frequency(i, rot) for i in range(24)]
    assert all(abs(a - b) < 1e-15 for a, b in zip(got.frequencies(), want)) and got.magnitude == 1.0
    plain = [500.0 ** (-2.0 * i / 48) for i in range(24)]
    kept = [a == b for a, b in zip(want, plain)]
    scaled = [abs(a - b / 6.0) < 1e-15 for a, b in zip(want, plain)]
    assert kept[0] and scaled[-1] and any(not k and not s for k, s in zip(kept, scaled))
    assert kept == sorted(kept, reverse=True) and scaled == sorted(scaled)
    yarn = RotarySpec.from_dict(dict(base=500.0, dims=48, scaling=dict(factor=6.0, original=300, fast=8.0, slow=1.0)))
    assert yarn.magnitude == 0.1 * math.log(6.0) + 1.0 and yarn.frequencies()[0] == 1.0


def test_registry_and_checkpoint_directory(tmp_path):
    assert "Fovirax" in architectures
    (tmp_path / "config.json").write_text(json.dumps(CFG_ODD))
    c = load_config(tmp_path)
    assert isinstance(c, FoviraxConfig) and model_class(c).__name__ == "Fovirax"


def test_loader_fuses_pads_and_stacks():
    w = checkpoint(CFG_ODD, 5)
    model = model_of(CFG_ODD, "cpu").to(torch.bfloat16)
    for p in model.parameters():
        p.data.fill_(99.0)
    model.load_tensors(w)
    mx = model.blocks[0].mixer
    covered = torch.zeros(mx.w_in.shape[0], dtype=torch.bool)
    for at, (name, rows) in zip(mx.offsets, mx.rows):
        assert at % 8 == 0 and torch.equal(mx.w_in[at : at + rows], w["l0.mix." + name])
        covered[at : at + rows] = True
    assert not mx.w_in[~covered].any() and bool((~covered).any())
    assert torch.equal(mx.w_o[:, :40], w["l0.mix.left.o"]) and torch.equal(mx.w_o[:, 40:61], w["l0.mix.right.o"]) and not mx.w_o[:, 61:].any()
    m = model.blocks[0].mlp
    assert torch.equal(m.w_route[:6], w["l0.mlp.router"]) and torch.equal(m.w_route[6:7], w["l0.mlp.shared.sg"]) and not m.w_route[7:].any()
    assert torch.equal(m.w_up[3], torch.cat([w["l0.mlp.e3.gate"], w["l0.mlp.e3.up"]])) and torch.equal(m.w_down[5], w["l0.mlp.e5.down"])
    assert torch.equal(m.shared_up, torch.cat([w["l0.mlp.shared.gate"], w["l0.mlp.shared.up"]])) and torch.equal(m.shared_down, w["l0.mlp.shared.down"])
    assert model.blocks[1].mlp is None and model.blocks[2].mlp.shared_up is None
    assert torch.equal(model.blocks[3].ls2, w["l3.ls2"]) and torch.equal(model.head, w["head"]) and torch.equal(model.final_norm, w["final.norm"])
    assert not any(bool((p == 99.0).any()) for p in model.parameters())


def test_loader_rejects_missing_and_unexpected_tensors():
    w = checkpoint(CFG_WIDE, 6)
    model = model_of(CFG_WIDE, "cpu").to(torch.bfloat16)
    for name in ("l0.mix.right.g", "l2.mlp.e7.up", "l0.mlp.shared.sg", "l1.ls1", "final.norm"):
        with pytest.raises(KeyError):
            model.load_tensors({k: v for k, v in w.items() if k != name})
    with pytest.raises(KeyError):
        model.load_tensors(dict(w, **{"l0.mix.left.q.b": torch.zeros(144, dtype=torch.bfloat16)}))
    with pytest.raises(ValueError):
        model.load_tensors(dict(w, **{"l1.norm1": torch.zeros(65, dtype=torch.bfloat16)}))
    model.load_tensors(dict(w, **{"l1.norm2": torch.zeros(64, dtype=torch.bfloat16)}))     # of a feed-forward the layer does not have


def test_states_have_the_size_of_what_is_kept_and_stay_fp32():
    model = model_of(CFG_TILES, "cpu").to(torch.bfloat16)
    model.set_kv_cache(batch_size=3)
    assert len(model.states) == 5
    first, third = model.states[0], model.states[2]                       # two passes of layer 0
    assert tuple(first.left.k_ring.shape) == (3, 44, 2 * 64) and tuple(first.left.v_ring.shape) == (3, 44, 2 * 128) and first.left.k_ring.dtype == torch.bfloat16
    assert tuple(first.right.matrices.shape) == (3, 4 * 32 * 24) and first.right.matrices.dtype == torch.float32
    assert tuple(third.left.k_ring.shape) == tuple(first.left.k_ring.shape) and third.left.k_ring.data_ptr() != first.left.k_ring.data_ptr()
    assert len(model.state_tensors()) == 15
    model.to(torch.float64)
    assert model.states[1].right.matrices.dtype == torch.float32
    assert not model.repeatable_steps and model.max_seq_length > 1 << 20
    model.clear_kv_cache()
    with pytest.raises(TypeError):
        model.step([1], [(0, 0, 1)])


# ---- the restatement itself, on cases with a closed form ---------------------------------------------------------------------
def test_oracle_attention_flat_scores_and_cap():
    T, dk, dv = 6, 4, 3
    g = torch.Generator().manual_seed(1)
    q, k, v = (torch.randn(T, 1, d, generator=g, dtype=torch.float64) for d in (dk, dk, dv))
    out = O.capped_window_attention(q, k, v, 2, 0.0, 5.0)
    assert torch.allclose(out[5], v[[4, 5]].mean(0)) and torch.allclose(out[0], v[0])
    out = O.capped_window_attention(q * 1e6, k, v, 6, 1.0, 1e-9)
    assert torch.allclose(out[5], v.mean(0), atol=1e-6)                 # a tiny cap makes every score the same
    assert torch.allclose(O.capped_window_attention(q, k, v, 1, 1.0, 2.0), v)


def test_oracle_rotation_recurrence_and_norms():
    x = torch.zeros(2, 1, 6, dtype=torch.float64)
    x[:, 0, 0], x[:, 0, 5] = 1.0, 3.0                                   # pair (0, 2) of dims = 4; dimensions 4, 5 pass
    r = O.rotate_half(x, dict(base=100.0, dims=4), 7)
    assert abs(float(r[0, 0, 0]) - math.cos(7.0)) < 1e-12 and abs(float(r[1, 0, 2]) - math.sin(8.0)) < 1e-12 and float(r[0, 0, 5]) == 3.0
    k = torch.ones(4, 1, 1, dtype=torch.float64)
    v = torch.tensor([1.0, 0.0, 0.0, 2.0], dtype=torch.float64).view(4, 1, 1)
    o = O.retained_sum(2 * k, k, v, torch.tensor([0.5], dtype=torch.float64))
    assert torch.allclose(o.view(-1), torch.tensor([2.0, 1.0, 0.5, 4.25], dtype=torch.float64))    # the read-out sees the token's own write
    y = torch.tensor([[1.0, 3.0]], dtype=torch.float64)
    assert torch.allclose(O.norm(y, torch.zeros(2, dtype=torch.float64), 4.0), y / 3.0)            # eps inside the root, weight around zero


def test_oracle_mixture_weights_and_shared_gate():
    eye = torch.eye(2, dtype=torch.float64)
    W = {"router": torch.tensor([[1.0, 0.0], [0.0, 1.0], [-9.0, -9.0]], dtype=torch.float64), "shared.sg": torch.zeros(1, 2, dtype=torch.float64)}
    for e, s in (("e0.", 1.0), ("e1.", 2.0), ("e2.", 100.0), ("shared.", 4.0)):
        W[e + "gate"], W[e + "up"], W[e + "down"] = eye, eye, s * eye
    h = torch.tensor([[1.0, 1.0]], dtype=torch.float64)
    unit = O.silu(h) * h
    f = dict(router=dict(experts=3, top=2), expert=dict(ff=2), shared=dict(ff=2))
    assert torch.allclose(O.mixture(h, W, "", f), unit * (1.5 + 0.5 * 4.0))
    assert torch.allclose(O.mixture(h, W, "", dict(router=dict(experts=3, top=1), expert=dict(ff=2))), unit)


def test_oracle_is_causal_and_uses_every_part():
    cfg = config(16, 13, [(left(2, 1, 4, 6, 3, 2, 5.0), right(4, 5, 2, [0.5, 0.9]), 0.7, 0.9, moe(3, 2, 6, 5))] * 2, mult=0.8, loop=(0, 1, 2))
    w = checkpoint(cfg, 2)
    toks = tokens_for(cfg, 6, 3)
    a = O.forward(cfg, w, toks)
    assert a.shape == (6, 13) and torch.isfinite(a).all() and torch.allclose(O.forward(cfg, w, toks[:4]), a[:4])
    for name in w:
        changed = dict(w, **{name: w[name] * 1.5 + 0.25})
        if ".e" in name:        # one expert may go unused by these tokens: change the same matrix of all of them
            changed = dict(w, **{n: w[n] * 1.5 + 0.25 for n in w if ".e" in n and n.rsplit(".", 1)[1] == name.rsplit(".", 1)[1]})
        assert not torch.allclose(O.forward(cfg, changed, toks), a), name
    for change in (dict(residual_mult=0.5), dict(loop=dict(start=0, stop=1, times=3)), dict(loop=None)):
        assert not torch.allclose(O.forward(dict(cfg, **change), w, toks), a)
