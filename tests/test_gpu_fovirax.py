"""Fovirax on the GPU: every mechanism alone and whole models through every serving path, against the plain float64 restatement in
``fovirax_oracle.py``.  Configurations and weights are made here; sizes are odd on purpose."""
from __future__ import annotations

import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import fovirax_oracle as O  # noqa: E402

pytestmark = pytest.mark.gpu
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def K():
    from lit_gpt_b200 import kernels

    return kernels


# ---------------------------------------------------------------------------------------------------------
# configurations and random checkpoints
# ---------------------------------------------------------------------------------------------------------
def left(heads, kv_heads, dim, vdim, size, rot_dims, cap, scale=None, base=100.0, scaling=None):
    rot = dict(base=base, dims=rot_dims, **({"scaling": dict(zip(("factor", "low", "high", "original"), scaling))} if scaling else {}))
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=size), rot=rot, softcap=cap, scale=scale if scale is not None else dim ** -0.5)


def right(dim, vdim, rot_dims, decay, base=1000.0):
    return dict(heads=len(decay), dim=dim, vdim=vdim, rot=dict(base=base, dims=rot_dims), decay=decay)


def moe(experts, top, ff, shared=None):
    return dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top), **({"shared": dict(ff=shared)} if shared else {}))


def config(width, vocab, layers, mult=1.0, loop=None, eps=1e-5):
    """layers: (left, right, left scale, right scale, mlp)"""
    cfg = dict(architecture="Fovirax", norm=dict(eps=eps), residual_mult=mult, vocab=vocab, width=width,
               layers=[dict(type="parallel", mixer=dict(left=lf, right=rt, left_scale=ls, right_scale=rs), mlp=mlp) for lf, rt, ls, rs, mlp in layers])
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


# a width no vector access fits, key sizes other than value sizes, partial and whole rotations with every branch of the scaling, a window of
# one, all experts chosen, one chosen, no shared expert, no feed-forward, a negative scale, two looped layers run three times
CFG_ODD = config(42, 83, [
    (left(4, 2, 12, 10, 7, 6, 4.0, scale=0.9, scaling=(3.0, 1.0, 5.0, 40)), right(10, 7, 6, [0.5, 0.9, 0.97]), 0.8, 0.7, moe(6, 2, 14, 22)),
    (left(6, 1, 8, 14, 5, 8, 9.0), right(14, 9, 14, [0.95, 0.6]), 1.2, -0.5, None),
    (left(1, 1, 20, 9, 33, 20, 2.0, base=50.0, scaling=(8.0, 0.5, 2.0, 30)), right(21, 30, 20, [0.99]), 0.4, 0.9, moe(5, 5, 11)),
    (left(2, 2, 6, 6, 1, 2, 30.0), right(6, 6, 0, [0.8, 1.0, 0.0, 0.9]), 1.0, 1.0, moe(4, 1, 20, 13)),
], mult=0.7, loop=(1, 3, 3))
# heads wider than one value chunk of the any-size attention and than the tensor-core tiles take, a window longer than any prompt here, keys
# of 70, 200 and 300 numbers in the recurrence, decays 1 and 0, experts narrow and wide
CFG_WIDE = config(64, 120, [
    (left(2, 2, 72, 136, 21, 72, 15.0), right(70, 40, 34, [1.0, 0.0, 0.9]), 0.9, 0.6, moe(8, 3, 40, 56)),
    (left(3, 1, 24, 264, 300, 8, 3.0, base=1e4, scale=0.35), right(200, 34, 200, [0.999, 0.7]), 0.5, 1.3, None),
    (left(4, 4, 16, 16, 40, 16, 20.0, scaling=(2.0, 1.0, 4.0, 64)), right(300, 12, 150, [0.98]), 1.5, 0.8, moe(16, 4, 24, 16)),
], mult=0.45)
# bf16 prompts on the tensor-core tiles: keys of 64, 40 and 120 beside values of 128, 200 and 160, windows that end inside a key tile and
# beyond one; many-token experts as grouped products
CFG_TILES = config(96, 140, [
    (left(4, 2, 64, 128, 44, 32, 12.0), right(32, 24, 32, [0.9, 0.99, 0.6, 0.999]), 0.7, 0.9, moe(8, 3, 48, 64)),
    (left(2, 1, 40, 200, 70, 40, 25.0, base=1e4, scaling=(4.0, 1.0, 3.0, 100)), right(24, 40, 12, [0.995, 0.5]), 1.1, 0.8, moe(6, 2, 40, 72)),
    (left(6, 3, 120, 160, 130, 60, 6.0), right(64, 128, 64, [0.97, 0.99]), 0.6, 1.0, None),
], mult=0.6, loop=(0, 2, 2))


def checkpoint(cfg, seed, dtype=None):
    """Random bf16 weights of a size that keeps every mechanism alive: caps that bite, norms and scales off their neutral value.  For whole
    models in bf16 the router's logits lie further apart: at a close call between the last expert chosen and the first left out, rounding
    may decide, and the token's state carries that on; the further apart, the less weight the last one has."""
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (mean + torch.randn(*shape, generator=g) * std).to(torch.bfloat16)

    d = cfg["width"]
    w = {"embed": rnd(cfg["vocab"], d), "final.norm": rnd(d, std=0.2), "head": rnd(cfg["vocab"], d, std=d ** -0.5)}
    for i, ly in enumerate(cfg["layers"]):
        p, lf, rt, f = f"l{i}.", ly["mixer"]["left"], ly["mixer"]["right"], ly["mlp"]
        w[p + "norm1"], w[p + "ls1"] = rnd(d, std=0.2), rnd(d, std=0.2, mean=0.8)
        for side, m, G in (("left", lf, lf["kv_heads"]), ("right", rt, rt["heads"])):
            q, H, dk, dv = f"{p}mix.{side}.", m["heads"], m["dim"], m["vdim"]
            for name, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)) + ((("g", H * dv),) if side == "right" else ()):
                w[q + name] = rnd(rows, d, std=1.5 * d ** -0.5)
            w[q + "o"] = rnd(d, H * dv, std=(H * dv) ** -0.5)
        if f is None:
            continue
        w[p + "norm2"], w[p + "ls2"] = rnd(d, std=0.2), rnd(d, std=0.2, mean=0.8)
        m = p + "mlp."
        w[m + "router"] = rnd(f["router"]["experts"], d, std=(9.0 if dtype == torch.bfloat16 else 3.0) * d ** -0.5)
        names = [(f"e{j}.", f["expert"]["ff"]) for j in range(f["router"]["experts"])]
        if f.get("shared"):
            names.append(("shared.", f["shared"]["ff"]))
            w[m + "shared.sg"] = rnd(1, d, std=2.0 * d ** -0.5)
        for name, ff in names:
            w[m + name + "gate"], w[m + name + "up"] = rnd(ff, d, std=1.5 * d ** -0.5), rnd(ff, d, std=1.5 * d ** -0.5)
            w[m + name + "down"] = rnd(d, ff, std=1.5 * ff ** -0.5)
    return w


def model_of(cfg, device="cuda"):
    from lit_gpt_b200.config import FoviraxConfig
    from lit_gpt_b200.fovirax import Fovirax

    return Fovirax(FoviraxConfig.from_dict(cfg)).to(device)


def build(cfg, weights, dtype, slots=2):
    model = model_of(cfg).to(dtype)
    model.load_tensors(weights)
    model.set_kv_cache(batch_size=slots)
    return model.eval()


def tokens_for(cfg, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg["vocab"], (n,), generator=g).tolist()


def rel_err(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).norm() / want.norm().clamp_min(1e-30))


def assert_close(got, want, dtype, what=""):
    """fp32: the whole block within rounding, no row far off.  bf16: a row whose read-out nearly vanishes before its norm, or whose router
    makes a close call, turns rounding into a large difference, in exact arithmetic on rounded inputs just as well; so the typical row must
    be within bf16 rounding and nearly nine in ten close to it.  The fp32 runs of the same tests are the sharp ones."""
    got, want = got.double().cpu(), want.double().cpu()
    rows = (got - want).norm(dim=-1) / want.norm(dim=-1).clamp_min(1e-30)
    if dtype == torch.float32:
        assert rel_err(got, want) < 4e-5 and float(rows.max()) < 3e-4, (what, rel_err(got, want), float(rows.max()), int(rows.argmax()))
    else:
        assert float(rows.median()) < 2.5e-2 and float((rows < 6e-2).double().mean()) >= 0.88, (what, float(rows.median()), rows)


def f64(weights):
    return {k: v.double() for k, v in weights.items()}


def batch_of(seqs):
    from lit_gpt_b200.ragged import state_batch

    return state_batch(seqs, torch.device("cuda"), positions=True)[0]


# ---------------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------------
@BOTH
@pytest.mark.parametrize("d", [42, 64, 1536, 3000, 5000, 9000])
def test_gated_residual_with_the_next_norm(dtype, d):
    """x += mult * scale * (y0 + gate y1) for rows that fill the register chunks partly and wholly, and rows beyond them; y0 dense or the
    weighted sum of gathered rows; norm weights around zero and around one; no norm; no scale."""
    k = K()
    g = torch.Generator().manual_seed(d)
    n, top, eps, mult = 7, 3, 1e-2, -0.37
    x0 = torch.randn(n, d, generator=g)
    y0, y1, table, sc, nw = (torch.randn(*s, generator=g).to(dtype) for s in ((n, d), (n, d), (n * top + 2, d), (d,), (d,)))
    gate, wts = torch.rand(n, generator=g), torch.rand(n, top, generator=g)
    slots = torch.randperm(n * top, generator=g).int().view(n, top)
    tol = 1e-6 if dtype == torch.float32 else 4e-3
    summed = (wts.double()[:, :, None] * table.double()[slots.long()]).sum(1)
    for gathered in (False, True):
        for plus in (False, True):
            base = summed if gathered else y0.double()
            want = x0.double() + mult * sc.double() * (base + gate.double()[:, None] * y1.double())
            x, act = x0.clone().cuda(), torch.empty(n, d, dtype=dtype, device="cuda")
            kw = dict(slot_of=slots.cuda(), wts=wts.cuda()) if gathered else {}
            k.gated_residual(x, (table if gathered else y0).cuda(), eps, y1=y1.cuda(), gate=gate.cuda(), scale=sc.cuda(), mult=mult, norm_w=nw.cuda(),
                             plus_one=plus, act=act, **kw)
            assert rel_err(x, want) < 1e-6
            assert rel_err(act, O.norm(want, nw.double() - (0 if plus else 1), eps)) < tol
    x = x0.clone().cuda()
    k.gated_residual(x, y0.cuda(), eps)
    assert rel_err(x, x0.double() + y0.double()) < 1e-6
    x = x0.clone().cuda()
    k.gated_residual(x, y0.cuda(), eps, y1=y1.cuda(), mult=2.0)          # no gate: the second branch joins as it is
    assert rel_err(x, x0.double() + 2 * (y0.double() + y1.double())) < 1e-6


@BOTH
def test_four_rotations_in_one_launch_some_into_fp32(dtype):
    """Queries and keys of two mixers with frequencies, sizes and head counts of their own, at far positions: two groups in place, two into
    fp32 buffers (unrounded there), everything else untouched."""
    from lit_gpt_b200.config import RotarySpec

    k = K()
    g = torch.Generator().manual_seed(2)
    n, start = 9, 300000
    ra = dict(base=1e4, dims=20, scaling=dict(factor=4.0, low=1.0, high=3.0, original=5000))
    rb = dict(base=1e6, dims=64)
    shapes = [(3, 28, ra), (1, 28, ra), (2, 70, rb), (2, 70, rb)]
    buf0 = torch.randn(n, sum(h * d for h, d, _ in shapes) + 5, generator=g).to(dtype)
    buf, pos = buf0.cuda(), torch.arange(start, start + n, dtype=torch.int32, device="cuda")
    fp = torch.zeros(n, 280, device="cuda")
    segs, wants, at = [], [], 0
    freqs = [torch.tensor(RotarySpec.from_dict(r, interleaved=False).frequencies(), dtype=torch.float64, device="cuda") for r in (ra, rb)]
    dst = [None, None, fp[:, :140], fp[:, 140:]]
    for i, (h, d, rot) in enumerate(shapes):
        src = buf[:, at : at + h * d]
        wants.append(O.rotate_half(buf0.double()[:, at : at + h * d].reshape(n, h, d), rot, start).reshape(n, -1))
        segs.append(k.rope_seg(src, src if dst[i] is None else dst[i], h, d, freq=freqs[i // 2], rot_dims=rot["dims"], interleaved=False))
        at += h * d
    k.head_rope(n, pos, 0.0, *segs, dtype=dtype, device=buf.device)
    at = 3 * 28 + 28
    assert rel_err(buf[:, :84], wants[0]) < (1e-6 if dtype == torch.float32 else 4e-3) and rel_err(buf[:, 84:112], wants[1]) < (1e-6 if dtype == torch.float32 else 4e-3)
    assert rel_err(fp[:, :140], wants[2]) < 1e-6 and rel_err(fp[:, 140:], wants[3]) < 1e-6
    assert torch.equal(buf[:, at:].cpu(), buf0[:, at:])


@pytest.mark.parametrize("vdtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,dk,dv", [(3, 5, 7), (2, 32, 64), (2, 48, 33), (1, 64, 100), (2, 128, 256), (1, 130, 20), (1, 256, 40), (1, 300, 12)])
def test_retained_state_alone(H, dk, dv, vdtype):
    """fp32 queries and keys beside values in the model dtype over every kernel shape: pieces of several sizes, one walk, portions down to
    two tokens, single tokens; a second sequence in the same launch; slots with leftovers; one head with decay 1, one with decay 0."""
    k = K()
    g = torch.Generator().manual_seed(dk + dv)
    n, n2 = 83, 20
    q, kk = torch.randn(n, H * dk, generator=g), torch.randn(n, H * dk, generator=g)
    v = torch.randn(n, H * dv, generator=g).to(vdtype)
    decay = torch.tensor([[0.97], [1.0, 0.5], [0.0, 0.9, 1.0]][H - 1])
    want = O.retained_sum(q.double().view(n, H, dk), kk.double().view(n, H, dk) * dk ** -0.5, v.double().view(n, H, dv), decay.double()).reshape(n, H * dv)
    for what, piece, cuts in [("pieces of 16", 16, [n]), ("pieces of 32", 32, [n]), ("one walk", 1000, [n]), ("portions", 16, [2, 2, 40, 3, 35, 1]),
                              ("single", 0, [1] * n)]:
        old = k.linear_attn_tune(piece)
        try:
            state = torch.full((3, H * dk * dv), 5.0, device="cuda")
            got, other, at = [], [], 0
            for c in cuts:
                extra = at == 0 and c >= n2
                batch = batch_of([(2, at, c)] + ([(0, 0, n2)] if extra else []))
                pack = lambda t: (torch.cat([t[at : at + c], t[:n2]]) if extra else t[at : at + c]).cuda()   # noqa: E731
                o = k.linear_attn(pack(q), pack(kk), pack(v), state, batch.seq_state, batch.max_q_len, H, dk, dv, q_scale=dk ** -0.5, head_decay=decay.cuda())
                got.append(o[:c])
                if extra:
                    other.append(o[c:])
                at += c
        finally:
            k.linear_attn_tune(old)
        assert rel_err(torch.cat(got), want) < 3e-6, (what, rel_err(torch.cat(got), want))
        if other:
            assert rel_err(torch.cat(other), want[:n2]) < 3e-6, what
        assert torch.all(state[1] == 5.0), what       # nobody's slot


def test_a_loud_key_far_back_is_retained():
    """One key hundreds of tokens back, loud and alone in its direction: the query at the end reads its value times decay^distance, in a
    prompt cut into pieces, in portions and in single tokens."""
    k = K()
    n, dk, dv, decay, place = 700, 24, 10, 0.998, 13
    g = torch.Generator().manual_seed(1)
    kk, q, v = (torch.randn(n, m, generator=g) * 0.01 for m in (dk, dk, dv))
    kk[:, 0], q[:, 0] = 0.0, 0.0
    kk[place, 0], q[n - 1, 0] = 30.0, 2.0
    v[place] = torch.linspace(-1, 1, dv)
    for cuts in ([n], [2, 12, 2, n - 18, 2], [500] + [1] * 200):
        state, got, at = torch.full((1, dk * dv), 3.0, device="cuda"), [], 0
        for c in cuts:
            b = batch_of([(0, at, c)])
            s = slice(at, at + c)
            got.append(k.linear_attn(q[s].cuda(), kk[s].cuda(), v[s].cuda(), state, b.seq_state, c, 1, dk, dv, head_decay=torch.tensor([decay], device="cuda")))
            at += c
        last = torch.cat(got)[-1].double().cpu()
        assert rel_err(last, 60.0 * decay ** (n - 1 - place) * v[place].double()) < 1e-3


@BOTH
@pytest.mark.parametrize("H,dv", [(3, 7), (2, 96), (1, 256), (2, 520)])
def test_unweighted_head_norm_with_gate_and_factor_into_a_slice(dtype, H, dv):
    k = K()
    g = torch.Generator().manual_seed(dv)
    n, eps = 6, 1e-3
    o, z = torch.randn(n, H * dv, generator=g) * torch.logspace(-3, 2, n)[:, None], (torch.randn(n, H * dv, generator=g) * 2).to(dtype)
    dst = torch.full((n, H * dv + 16), 4.0, dtype=dtype, device="cuda")
    k.gated_rms_heads(o.cuda(), z.cuda(), None, H, dv, k.GATE_SILU, eps, out_scale=-1.3, out=dst[:, 8 : 8 + H * dv])
    want = -1.3 * O.over_rms(o.double().view(n, H, dv), eps).reshape(n, -1) * O.silu(z.double())
    assert rel_err(dst[:, 8 : 8 + H * dv], want) < (1e-6 if dtype == torch.float32 else 4e-3)
    assert torch.all(dst[:, :8] == 4.0) and torch.all(dst[:, 8 + H * dv :] == 4.0)


def _window(q, kk, v, state, seqs, H, G, dk, dv, size, scale, cap, from_start=False, **kw):
    b = batch_of(seqs)
    return K().window_attn(q.cuda(), kk.cuda(), v.cuda(), state[0], state[1], None, b.seq_state, b.row_seq, b.max_q_len, H, G, dk, dv, size, scale,
                           from_start=from_start, softcap=cap, **kw).float().cpu()


def _rings(slots, rows, G, dk, dv, dtype=torch.float32, fill=9.0):
    return (torch.full((slots, rows, G * dk), fill, device="cuda", dtype=dtype), torch.full((slots, rows, G * dv), fill, device="cuda", dtype=dtype))


@BOTH
def test_loud_key_just_inside_and_just_outside_the_window(dtype):
    """One key is made loud: the query `size - 1` positions later must find it among hundreds of quiet ones, the next must not.  In a prompt
    (bf16: on the tensor cores), in later portions and in single-token steps, on rings that wrap; the output's factor is exact."""
    k = K()
    H, G, dk, dv, size, n, cap, loud, factor = 2, 1, 16, 24, 130, 420, 40.0, 31, 0.25
    g = torch.Generator().manual_seed(9)
    q, kk, v = torch.randn(n, H * dk, generator=g) * 0.3, torch.randn(n, G * dk, generator=g) * 0.1, torch.randn(n, G * dv, generator=g)
    probe = torch.randn(dk, generator=g) * 1.5
    seekers = [loud + size - 1, loud + size, n - 1]
    for i in seekers:
        q[i, :dk] = probe
    kk[loud] = probe * 40.0 / float(probe @ probe)
    q, kk, v = q.to(dtype), kk.to(dtype), v.to(dtype)
    want = factor * O.capped_window_attention(q.double().view(n, H, dk), kk.double().view(n, G, dk), v.double().view(n, G, dv), size, 1.0, cap).reshape(n, H * dv)
    for i in seekers:
        assert bool((want[i, :dv] - factor * v[loud].double()).abs().max() < 1e-3) == (i - loud < size)
    tol = 1e-5 if dtype == torch.float32 else 1.2e-2
    for cuts in ([n], [loud + 2, n - loud - 2], [loud + size - 1, 1, 1, n - loud - size - 1], [2, 200, 2, n - 204], [1] * n):
        for tiled in (False, True):
            if tiled and len(cuts) == n:
                continue
            old = k.window_attn_tune(force_tiled_kernel=tiled)
            try:
                state, got, at = _rings(2, size, G, dk, dv, dtype), [], 0
                for c in cuts:
                    s = slice(at, at + c)
                    got.append(_window(q[s], kk[s], v[s], state, [(1, at, c)], H, G, dk, dv, size, 1.0, cap, from_start=at == 0, out_scale=factor))
                    at += c
            finally:
                k.window_attn_tune(force_tiled_kernel=old)
            got = torch.cat(got)
            assert rel_err(got, want) < tol, (cuts[:4], tiled, rel_err(got, want))
            for i in seekers:
                assert rel_err(got[i], want[i]) < 2 * tol, (cuts[:4], tiled, i)
    for p in range(n - size, n):
        assert torch.equal(state[1][1, p % size].cpu(), v[p])


def test_soft_cap_has_its_exact_size():
    """Two keys with known scores: weights exp(cap tanh(s / cap))."""
    cap, scale = 3.0, 0.5
    q, kk, v = torch.tensor([[0.0, 0.0], [4.0, 2.0]]), torch.tensor([[3.0, 0.0], [0.0, -1.0]]), torch.tensor([[1.0, 0.0], [0.0, 1.0]])
    e = [math.exp(cap * math.tanh(s / cap)) for s in (6.0, -1.0)]
    for cuts in ([2], [1, 1]):
        state, got, at = _rings(1, 5, 1, 2, 2), [], 0
        for c in cuts:
            s = slice(at, at + c)
            got.append(_window(q[s], kk[s], v[s], state, [(0, at, c)], 1, 1, 2, 2, 5, scale, cap))
            at += c
        got = torch.cat(got)
        assert abs(float(got[1, 0]) - e[0] / sum(e)) < 1e-6 and abs(float(got[1, 1]) - e[1] / sum(e)) < 1e-6 and abs(float(got[0, 0]) - 1.0) < 1e-6


@pytest.mark.parametrize("dk,dv,size,cap", [(64, 128, 100, 5.0), (64, 192, 64, 30.0), (128, 256, 150, 12.0), (128, 192, 1, 8.0), (40, 200, 30, 3.0), (8, 256, 1000, 20.0),
                                             (104, 136, 65, 50.0), (48, 64, 129, 10.0)])
def test_prompts_on_the_tensor_cores_with_wide_values(dk, dv, size, cap):
    """bf16 prompts of three unequal sequences in one launch, values wider than keys: windows that end inside a key tile, at its edge, of one
    position and longer than the prompt; loud scores that the cap bends; into a slice with a factor.  Against exact attention on the same
    operands and the any-size kernel; the rings afterwards."""
    k = K()
    H, G = 4, 2
    g = torch.Generator().manual_seed(dk + size)
    lens = [200, 37, 300]
    n = sum(lens)
    q, kk, v = (torch.randn(n, m, generator=g).to(torch.bfloat16) for m in (H * dk, G * dk, G * dv))
    scale, factor = 2.0 * dk ** -0.5, 1.7
    want, at = [], 0
    for ln in lens:
        s = slice(at, at + ln)
        want.append(factor * O.capped_window_attention(q[s].double().view(ln, H, dk), kk[s].double().view(ln, G, dk), v[s].double().view(ln, G, dv), size, scale,
                                                       cap).reshape(ln, H * dv))
        at += ln
    want = torch.cat(want)
    outs = {}
    for mma in (True, False):
        k.WINDOW_PREFILL_MMA = mma
        try:
            state = _rings(3, size, G, dk, dv, torch.bfloat16, 0.0)
            wide = torch.full((n, H * dv + 24), 3.0, dtype=torch.bfloat16, device="cuda")
            _window(q, kk, v, state, [(0, 0, lens[0]), (2, 0, lens[1]), (1, 0, lens[2])], H, G, dk, dv, size, scale, cap, from_start=True, out_scale=factor,
                    out=wide[:, 8 : 8 + H * dv])
            outs[mma] = wide[:, 8 : 8 + H * dv].float().cpu()
        finally:
            k.WINDOW_PREFILL_MMA = True
        assert torch.all(wide[:, :8] == 3.0) and torch.all(wide[:, 8 + H * dv :] == 3.0)
        for slot, first, ln in ((0, 0, lens[0]), (2, lens[0], lens[1]), (1, lens[0] + lens[1], lens[2])):
            for p in range(max(0, ln - size), ln):
                assert torch.equal(state[0][slot, p % size].cpu(), kk[first + p]) and torch.equal(state[1][slot, p % size].cpu(), v[first + p])
    assert rel_err(outs[False], want) < 6e-3
    assert rel_err(outs[True], want) < 1.2e-2
    rows = (outs[True].double() - want).norm(dim=-1) / want.norm(dim=-1).clamp_min(1e-2)
    assert float(rows.max()) < 4e-2


@BOTH
@pytest.mark.parametrize("experts,top", [(5, 1), (16, 2), (7, 7), (64, 8), (100, 32), (300, 3)])
def test_routing_kernel_and_routing_from_logits_agree(dtype, experts, top):
    """The largest logits, softmax among them, and the shared expert's gate: inside the routing kernel and from a matrix product's logits."""
    k = K()
    g = torch.Generator().manual_seed(experts + top)
    n, d = 21, 72
    x = torch.randn(n, d, generator=g).to(dtype)
    w = (torch.randn(experts + 1 + 4, d, generator=g) * 0.5).to(dtype)
    z = x.double() @ w.double().T
    best = z[:, :experts].sort(dim=1, descending=True)
    want_w = torch.softmax(best.values[:, :top], dim=1)
    direct = k.moe_route(x.cuda(), w[:experts].cuda(), None, top, 1, 1, topk_softmax=True, gate_w=w[experts].cuda())
    logits = (x.float() @ w.float().T).cuda()
    given = k.moe_route_logits(logits, experts, top, gate=True)
    for ids, wts, gate in (direct, given):
        assert torch.equal(ids.cpu().long(), best.indices[:, :top])
        assert rel_err(wts, want_w) < 1e-5 and rel_err(gate, torch.sigmoid(z[:, experts])) < 1e-5
    ids, wts = k.moe_route_logits(logits, experts, top)
    assert torch.equal(ids, given[0]) and torch.equal(wts, given[1])
    tie = torch.zeros(3, experts, device="cuda")                 # equal logits: the lowest index first
    ids, wts = k.moe_route_logits(tie, experts, top)
    assert torch.equal(ids.cpu(), torch.arange(top, dtype=torch.int32).expand(3, top)) and torch.allclose(wts, torch.full_like(wts, 1.0 / top))


@BOTH
@pytest.mark.parametrize("width,ml", [(40, moe(6, 2, 24, 40)), (42, moe(5, 1, 13, 7)), (64, moe(4, 4, 16, 200)), (48, moe(7, 3, 24))])
def test_experts_with_gated_shared_expert(dtype, width, ml):
    """One token to many: few-token kernels (up to 8 tokens per pass over the shared weights, and beyond), grouped products, the vendor's and
    this library's; with and without a shared expert."""
    from lit_gpt_b200 import moe as M

    cfg = config(width, 11, [(left(1, 1, 4, 4, 3, 2, 5.0), right(4, 4, 2, [0.5]), 1.0, 1.0, ml)])
    w = checkpoint(cfg, 7)
    model = build(cfg, w, dtype)
    mlp = model.blocks[0].mlp
    g = torch.Generator().manual_seed(3)
    h = torch.randn(150, width, generator=g).to(torch.bfloat16)
    want = O.mixture(h.double(), f64(w), "l0.mlp.", ml)
    for n in (1, 2, 8, 9, 16, 31, 32, 40, 150):
        for vendor in (True, False):
            M.VENDOR_GROUPED_GEMM = vendor
            try:
                t = mlp.terms(h[:n].to(dtype).cuda())
                x = torch.zeros(n, width, device="cuda")
                K().gated_residual(x, t.pop("y0"), 1e-5, **t)
            finally:
                M.VENDOR_GROUPED_GEMM = True
            rows = (x.double().cpu() - want[:n]).norm(dim=-1) / want[:n].norm(dim=-1)
            assert float(rows.max()) < (2e-6 if dtype == torch.float32 else 2.5e-2), (n, vendor, float(rows.max()))


def _drive(mixer, state, h, cuts, slot, dtype):
    """Feed the rows of h to `mixer` in steps of the given sizes for one sequence in `slot`; returns all output rows."""
    out, at = [], 0
    for n in cuts:
        out.append(mixer(h[at : at + n].to(dtype).cuda().contiguous(), batch_of([(slot, at, n)]), state).float().cpu())
        at += n
    assert at == h.shape[0]
    return torch.cat(out)


MIXED = [(left(4, 2, 10, 6, 7, 6, 20.0, scale=2.5, scaling=(3.0, 1.0, 4.0, 50)), right(9, 14, 8, [0.4, 0.9, 0.99])),
         (left(3, 3, 16, 24, 12, 16, 7.0, scale=1.0), right(16, 8, 0, [0.7, 0.95])),
         (left(2, 1, 24, 48, 30, 0, 5.0), right(40, 72, 40, [0.99]))]


@BOTH
@pytest.mark.parametrize("cuts", [[61], [1] * 61, [2, 2, 3, 1, 27, 2, 22, 2], [60, 1]])
@pytest.mark.parametrize("case", range(len(MIXED)))
def test_both_mixers_side_by_side(case, dtype, cuts):
    """In prompts, portions down to two tokens and single tokens, in a slot whose states hold another sequence's leftovers; with rotations of
    both, of one, of neither side."""
    lf, rt = MIXED[case]
    cfg = config(24, 11, [(lf, rt, 0.75, -1.25, None)])
    w = checkpoint(cfg, 3)
    model = build(cfg, w, dtype, slots=3)
    h = torch.randn(61, 24, generator=torch.Generator().manual_seed(5)).to(torch.bfloat16).double()
    want = O.parallel_mixer(h, f64(w), "l0.mix.", cfg["layers"][0]["mixer"], 1e-5)
    for t in model.states[0].tensors():
        t.fill_(7.0)
    got = _drive(model.blocks[0].mixer, model.states[0], h, cuts, slot=1, dtype=dtype)
    assert rel_err(got, want) < (2e-5 if dtype == torch.float32 else 4e-2), rel_err(got, want)


@BOTH
def test_retention_as_a_mixer_of_its_own(dtype):
    """``linear.Retention`` and ``window.GatedWindowAttention`` with projections of their own give the branches of the pair."""
    from lit_gpt_b200.config import FoviraxConfig
    from lit_gpt_b200.linear import Retention

    rt = right(9, 14, 8, [0.4, 0.9, 0.99])
    cfg = config(24, 11, [(left(1, 1, 4, 4, 3, 2, 5.0), rt, 1.0, 1.0, None)])
    w, p = checkpoint(cfg, 3), "l0.mix.right."
    mx = Retention(24, FoviraxConfig.from_dict(cfg).layers[0].mixer.right, 1e-5).cuda().to(dtype)
    mx.w_in.data.zero_()
    rows = torch.cat([w[p + n] for n in "qkvg"])
    mx.w_in.data[: rows.shape[0]].copy_(rows)
    mx.w_o.data.copy_(w[p + "o"])
    h = torch.randn(50, 24, generator=torch.Generator().manual_seed(5)).to(torch.bfloat16).double()
    want = O.retention_branch(h, f64(w), p, rt, 1e-5)
    for cuts in ([50], [2, 3, 40, 1, 4]):
        got = _drive(mx, mx.build_state(2, "cuda"), h, cuts, slot=1, dtype=dtype)
        assert rel_err(got, want) < (2e-5 if dtype == torch.float32 else 4e-2)


def test_padded_projections_take_the_tensor_core_tiles():
    """Head counts whose columns would leave the blocks of the fused product off 16-byte boundaries: the blocks are padded, so a bf16 prompt
    still reaches the tiles."""
    cfg = config(40, 17, [(left(3, 1, 16, 24, 12, 16, 7.0), right(5, 3, 4, [0.5, 0.9, 0.8]), 0.9, 1.1, None)])
    w = checkpoint(cfg, 8)
    model = build(cfg, w, torch.bfloat16)
    mx = model.blocks[0].mixer
    assert all(at % 8 == 0 for at in mx.offsets) and mx.w_in.shape[0] % 8 == 0 and mx.off_right % 8 == 0 and mx.out_cols % 8 == 0
    h = torch.randn(50, 40, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).double()
    lib, called = K().C.load_core(), []
    real = lib.b200_window_attn_tiles
    try:
        lib.b200_window_attn_tiles = lambda *a: called.append(1) or real(*a)
        got = mx(h.to(torch.bfloat16).cuda(), batch_of([(0, 0, 50)]), model.states[0])
    finally:
        lib.b200_window_attn_tiles = real
    assert called and rel_err(got, O.parallel_mixer(h, f64(w), "l0.mix.", cfg["layers"][0]["mixer"], 1e-5)) < 4e-2


# ---------------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------------
ALL = pytest.mark.parametrize("cfg", [CFG_ODD, CFG_WIDE, CFG_TILES], ids=["odd", "wide", "tiles"])


@ALL
@BOTH
def test_prompt_matches_oracle(cfg, dtype):
    w = checkpoint(cfg, 11, dtype)
    toks = tokens_for(cfg, 150, 11)
    model = build(cfg, w, dtype)
    assert_close(model.step(toks, [(1, 0, len(toks))]), O.forward(cfg, w, toks), dtype)


@ALL
def test_layers_follow_the_oracle_one_by_one(cfg):
    """The stream after every layer run in fp32, repeated passes included."""
    w = checkpoint(cfg, 31)
    toks = tokens_for(cfg, 60, 31)
    model = build(cfg, w, torch.float32)
    model.trace = []
    model.step(toks, [(0, 0, len(toks))])
    _, want = O.forward(cfg, w, toks, return_layers=True)
    assert len(model.trace) == len(want) == len(O.run_order(cfg)) == len(model.states)
    for r, (a, b) in enumerate(zip(model.trace, want)):
        assert rel_err(a, b) < 5e-6, (r, rel_err(a, b))


@ALL
@BOTH
def test_decoding_token_by_token_equals_prefill(dtype, cfg):
    w = checkpoint(cfg, 41, dtype)
    toks = tokens_for(cfg, 150, 41)
    model = build(cfg, w, dtype)
    whole = model.step(toks, [(0, 0, len(toks))])
    single = torch.cat([model.step([t], [(1, p, 1)]) for p, t in enumerate(toks)])
    assert_close(single, whole.float(), dtype)
    assert_close(single, O.forward(cfg, w, toks), dtype)


@pytest.mark.parametrize("portions", [[2, 2, 2, 30, 3, 34, 1, 35, 2], [109, 2], [1, 110], [5] * 22 + [1]])
@ALL
def test_prompt_in_portions(portions, cfg):
    """A prompt cut into portions of several sizes, down to two tokens and one, gives the logits of the whole prompt."""
    toks = tokens_for(cfg, sum(portions), 51)
    for dtype in (torch.float32, torch.bfloat16):
        w = checkpoint(cfg, 51, dtype)
        want = O.forward(cfg, w, toks)
        model = build(cfg, w, dtype)
        got, at = [], 0
        for n in portions:
            got.append(model.step(toks[at : at + n], [(1, at, n)]))
            at += n
        assert_close(torch.cat(got), want, dtype)


@BOTH
@pytest.mark.parametrize("cfg", [CFG_ODD, CFG_TILES], ids=["odd", "tiles"])
def test_ragged_batch_equals_each_alone(cfg, dtype):
    """Requests of unequal length in one batch (prefill together, then decoding together with the shorter ones leaving, a new one arriving in
    portions meanwhile) against each alone."""
    from lit_gpt_b200.generate.serve import Session

    w = checkpoint(cfg, 61, dtype)
    model = build(cfg, w, dtype)
    reqs = {"a": tokens_for(cfg, 150, 62), "b": tokens_for(cfg, 9, 63), "c": tokens_for(cfg, 73, 64), "d": tokens_for(cfg, 1, 65), "e": tokens_for(cfg, 60, 66)}
    pre = {"a": 130, "b": 3, "c": 60, "d": 1}
    session = Session(model, slots=2)       # grows while the batch is live
    rows = {rid: [] for rid in reqs}
    out = session.step([(rid, reqs[rid][: pre[rid]], None) for rid in pre], end=["d"])
    at = 0
    for rid in pre:
        rows[rid].append(out[at : at + pre[rid]])
        at += pre[rid]
    pos = dict(pre, e=0)
    while True:
        live = [rid for rid in reqs if pos[rid] < len(reqs[rid])]
        if not live:
            break
        take = {rid: (min(7, len(reqs[rid]) - pos[rid]) if rid == "e" else 1) for rid in live}
        out = session.step([(rid, reqs[rid][pos[rid] : pos[rid] + take[rid]], None) for rid in live],
                           end=[rid for rid in live if pos[rid] + take[rid] == len(reqs[rid])])
        at = 0
        for rid in live:
            rows[rid].append(out[at : at + take[rid]])
            at += take[rid]
            pos[rid] += take[rid]
    assert model.slots.in_use == 0
    want = {rid: O.forward(cfg, w, toks) for rid, toks in reqs.items()}
    assert_close(torch.cat([torch.cat(rows[rid]) for rid in reqs]), torch.cat([want[rid] for rid in reqs]), dtype)
    if dtype == torch.float32:
        for rid in reqs:
            assert_close(torch.cat(rows[rid]), want[rid], dtype, rid)


def test_freed_slots_are_reused_without_leftovers():
    """A request ends, another takes its slot (whose states and rings still hold the first one's), starting with a two-token portion; then a
    third starts with a single token."""
    from lit_gpt_b200.generate.serve import Session

    cfg = CFG_WIDE
    w = checkpoint(cfg, 71)
    model = build(cfg, w, torch.float32, slots=1)
    session = Session(model, slots=1)
    a, b, c = tokens_for(cfg, 80, 72), tokens_for(cfg, 45, 73), tokens_for(cfg, 12, 74)
    session.step([("a", a, [])], end=["a"])
    got = [session.step([("b", b[:2], None)])]
    got.append(session.step([("b", b[2:40], None)]))
    got += [session.step([("b", [t], None)]) for t in b[40:]]
    session.step([], end=["b"])
    single = [session.step([("c", [t], None)]) for t in c]
    assert model.slots.capacity == 1
    assert_close(torch.cat(got), O.forward(cfg, w, b), torch.float32)
    assert_close(torch.cat(single), O.forward(cfg, w, c), torch.float32)


def test_long_decoding_wraps_the_rings_many_times():
    """260 single-token steps behind a prompt: windows of 5 and 7 positions wrap their rings dozens of times, in every pass of the loop."""
    cfg = CFG_ODD
    w = checkpoint(cfg, 81)
    toks = tokens_for(cfg, 300, 81)
    model = build(cfg, w, torch.float32)
    got = [model.step(toks[:40], [(0, 0, 40)])]
    got += [model.step([t], [(0, p, 1)]) for p, t in enumerate(toks[40:], start=40)]
    assert_close(torch.cat(got), O.forward(cfg, w, toks), torch.float32)


@ALL
@BOTH
def test_first_tokens_decode_one_by_one(cfg, dtype):
    w = checkpoint(cfg, 83, dtype)
    toks = tokens_for(cfg, 12, 83)
    model = build(cfg, w, dtype)
    got = torch.cat([model.step([t], [(0, p, 1)]) for p, t in enumerate(toks)])
    assert_close(got, O.forward(cfg, w, toks), dtype)


def test_a_far_token_matters_only_through_the_state():
    """Two prompts differ in one far token only.  With states that forget at once (decay 0), the logits past the window agree to rounding, and
    differ for a token at its edge; with a slow decay they differ however far it lies.  Two layers reach two windows back."""
    def far_difference(decay, place, layers=1):
        cfg = config(32, 40, [(left(2, 1, 8, 8, 20, 4, 30.0), right(8, 8, 4, decay), 1.0, 1.0, None)] * layers)
        w = checkpoint(cfg, 5)
        toks = tokens_for(cfg, 120, 7)
        other = list(toks)
        other[place] = (toks[place] + 1) % 40
        model = build(cfg, w, torch.float32)
        a, b = model.step(toks, [(0, 0, 120)])[-1], model.step(other, [(1, 0, 120)])[-1]
        return rel_err(a, b)

    forget = [0.0, 0.0]
    assert far_difference(forget, 99) < 1e-9 and far_difference(forget, 100) > 1e-5
    assert far_difference(forget, 80, 2) < 1e-9 and far_difference(forget, 81, 2) > 1e-7
    assert far_difference([0.999, 0.995], 10) > 1e-5


@BOTH
def test_generate_entry_points(dtype):
    """Greedy generation through generate() (captured decode graph) and through the batch scheduler give the oracle's tokens."""
    from lit_gpt_b200.generate.base import generate
    from lit_gpt_b200.generate.serve import generate_batch

    cfg = CFG_ODD
    w = checkpoint(cfg, 91, dtype)
    prompt = tokens_for(cfg, 9, 91)
    seq = O.greedy(cfg, w, prompt, 14)
    model = build(cfg, w, dtype, slots=1)
    model.max_seq_length = 64
    y = generate(model, torch.tensor(prompt, device="cuda"), len(seq), temperature=0.0)
    if dtype == torch.float32:
        assert y.tolist() == seq
    again = generate(model, torch.tensor(prompt, device="cuda"), len(seq), temperature=0.0)   # the captured graph once more, over used states
    assert again.tolist() == y.tolist()
    other = tokens_for(cfg, 4, 92)
    model.set_kv_cache(batch_size=2)
    ys = generate_batch(model, [prompt, other], 14)
    assert len(ys[0]) == len(seq) and len(ys[1]) == 4 + 14 and model.slots.in_use == 0
    if dtype == torch.float32:
        assert ys[0] == seq and ys[1] == O.greedy(cfg, w, other, 14)


def test_forward_signature_of_the_other_models():
    """forward(idx, input_pos) with batch rows = slots and shared positions, as GPT.forward: a prompt, then single tokens."""
    cfg = CFG_WIDE
    w = checkpoint(cfg, 95)
    model = build(cfg, w, torch.float32, slots=2)
    a, b = tokens_for(cfg, 12, 96), tokens_for(cfg, 12, 97)
    idx = torch.tensor([a, b], device="cuda")
    out = model(idx[:, :10], torch.arange(10, device="cuda"))
    for p in (10, 11):
        out = torch.cat([out, model(idx[:, p : p + 1], torch.tensor([p], device="cuda"))], dim=1)
    assert out.shape == (2, 12, cfg["vocab"])
    assert rel_err(out[0], O.forward(cfg, w, a)) < 3e-5 and rel_err(out[1], O.forward(cfg, w, b)) < 3e-5


def _write_checkpoint(folder, cfg, weights):
    import json
    import struct

    header, blob = {}, b""
    for name, t in weights.items():
        raw = t.contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    hj = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(hj)) + hj + blob)
    (folder / "config.json").write_text(json.dumps(cfg))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_end_to_end(tmp_path, dtype):
    """The command-line replayer on a checkpoint directory written here: a ragged first step, decoding together, a request that
    ends, a new one in its slot, steps without anything wanted -- the files it writes against the oracle."""
    import json
    import subprocess

    import numpy as np

    cfg = CFG_ODD
    w = checkpoint(cfg, 101, getattr(torch, dtype))
    _write_checkpoint(tmp_path, cfg, w)
    a, b, c = tokens_for(cfg, 40, 102), tokens_for(cfg, 9, 103), tokens_for(cfg, 70, 104)
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:37], "want": [0, 36]}, {"id": "b", "tokens": b[:6], "want": [5]}], "end": []},
        {"step": 1, "entries": [{"id": "a", "tokens": [a[37]], "want": []}, {"id": "b", "tokens": [b[6]], "want": []}], "end": []},
        {"step": 2, "entries": [{"id": "a", "tokens": [a[38]], "want": [0]}, {"id": "b", "tokens": [b[7]], "want": [0]}], "end": ["b"]},
        {"step": 3, "entries": [{"id": "a", "tokens": [a[39]], "want": [0]}], "end": ["a"]},
        {"step": 4, "entries": [{"id": "c", "tokens": c, "want": [0, 1, 63, 64, 69]}], "end": ["c"]},
    ]
    out = tmp_path / "out"
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    res = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(out), "--max-tokens", "120"],
                         input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [ln for ln in res.stdout.splitlines() if ln.startswith("done ")] == [f"done {i}" for i in range(5)]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32", "4.f32"]        # step 1 wanted nothing
    full = {kk: O.forward(cfg, w, t) for kk, t in (("a", a), ("b", b), ("c", c))}
    want = {0: torch.stack([full["a"][0], full["a"][36], full["b"][5]]), 2: torch.stack([full["a"][38], full["b"][7]]),
            3: full["a"][39:40], 4: full["c"][[0, 1, 63, 64, 69]]}
    got = {s: torch.from_numpy(np.fromfile(out / f"{s}.f32", dtype="<f4").reshape(-1, cfg["vocab"])) for s in want}
    assert all(got[s].shape == want[s].shape for s in want)
    assert_close(torch.cat([got[s] for s in want]), torch.cat([want[s] for s in want]), getattr(torch, dtype))


def test_generate_command_line(tmp_path):
    """`python -m lit_gpt_b200.generate.base` on a checkpoint directory without a tokenizer: a prompt of token ids in, the oracle's greedy
    continuation out."""
    import subprocess

    cfg = CFG_WIDE
    w = checkpoint(cfg, 111)
    _write_checkpoint(tmp_path, cfg, w)
    prompt = tokens_for(cfg, 6, 112)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    res = subprocess.run([sys.executable, "-m", "lit_gpt_b200.generate.base", " ".join(str(t) for t in prompt), "--checkpoint_dir", str(tmp_path),
                          "--precision", "32-true", "--temperature", "0", "--max_new_tokens", "9"], cwd=root, capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    printed = [int(t) for t in res.stdout.strip().splitlines()[-1].split()]
    assert printed == O.greedy(cfg, w, prompt, 9)
