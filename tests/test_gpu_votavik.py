"""Votavik on the GPU: every mechanism alone and whole models through every serving path, against the plain float64 restatement in
``votavik_oracle.py``.  Configurations and weights are made here; sizes are odd on purpose."""
from __future__ import annotations

import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import votavik_oracle as O  # noqa: E402

pytestmark = pytest.mark.gpu


def K():
    from lit_gpt_b200 import kernels

    return kernels


# ---------------------------------------------------------------------------------------------------------
# configurations and random checkpoints
# ---------------------------------------------------------------------------------------------------------
def attention(heads, kv_heads, dim, vdim, size, keep, rot_dims, cap, scale=None, base=100.0):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask=dict(size=size, keep_first=keep), rot=dict(base=base, dims=rot_dims),
                softcap=cap, scale=scale if scale is not None else dim ** -0.5)


def gla(heads, dim, vdim, tau, rank):
    return dict(heads=heads, dim=dim, vdim=vdim, tau=tau), rank


def lightning(heads, dim, vdim, decay):
    assert len(decay) == heads
    return dict(heads=heads, dim=dim, vdim=vdim, decay=decay)


def glu(ff, limit):
    return dict(kind="dense", ff=ff, limit=limit)


def config(width, vocab, side, layers, eps=1e-5):
    """layers: (type, mixer, mlp).  The inner size of a gla layer's decay projection rides along for the checkpoint (it is not a key of
    the configuration)."""
    out, ranks = [], {}
    for i, (kind, mixer, mlp) in enumerate(layers):
        if kind == "gla":
            mixer, ranks[i] = mixer
        out.append(dict(type=kind, mixer=mixer, mlp=mlp))
    return dict(architecture="Votavik", layers=out, norm=dict(eps=eps), token_side=dict(dim=side), vocab=vocab, width=width), ranks


# a width no vector access fits, key sizes other than value sizes, grouped heads, kept tokens fewer and more than the window, feed-forwards
# behind every kind of mixer and none behind another
CFG_ODD = config(42, 83, 6, [
    ("gla", gla(3, 10, 7, 4.0, 5), glu(50, 0.9)),
    ("attention", attention(4, 2, 12, 10, size=7, keep=3, rot_dims=6, cap=4.0, scale=0.9), None),
    ("lightning", lightning(2, 14, 9, [0.5, 0.97]), glu(33, 1.4)),
    ("attention", attention(6, 1, 8, 14, size=5, keep=9, rot_dims=8, cap=9.0), glu(20, 2.5)),
    ("gla", gla(1, 21, 30, 1.0, 3), None),
])
# heads wider than one value chunk of the attention tile (> 128), a window of one position, a window longer than any prompt here, no kept
# token, keys of 70 and 200 numbers, one head with decay 1 and one with decay 0
CFG_WIDE = config(64, 120, 24, [
    ("attention", attention(2, 2, 72, 136, size=1, keep=2, rot_dims=72, cap=15.0), glu(96, 1.1)),
    ("lightning", lightning(3, 70, 40, [1.0, 0.0, 0.9]), None),
    ("attention", attention(3, 1, 24, 24, size=300, keep=0, rot_dims=8, cap=2.0, base=1e4, scale=0.35), None),
    ("gla", gla(2, 200, 34, 8.0, 11), glu(40, 0.7)),
])
# bf16 prompts on the tensor-core tiles: heads of 64, 128, 40 / 72 and 120 / 56, windows that end inside a key tile, kept tokens within one
# tile and across two
CFG_TILES = config(96, 140, 16, [
    ("attention", attention(4, 2, 64, 64, size=44, keep=5, rot_dims=32, cap=12.0), glu(72, 1.2)),
    ("lightning", lightning(4, 32, 24, [0.9, 0.99, 0.6, 0.999]), None),
    ("attention", attention(2, 1, 128, 128, size=50, keep=70, rot_dims=128, cap=25.0, base=1e4), None),
    ("gla", gla(4, 24, 40, 16.0, 12), glu(64, 1.6)),
    ("attention", attention(6, 3, 40, 72, size=30, keep=2, rot_dims=10, cap=8.0), None),
    ("attention", attention(2, 2, 120, 56, size=100, keep=1, rot_dims=60, cap=6.0), None),
])


def checkpoint(cfg_ranks, seed):
    """Random bf16 weights of a size that keeps every mechanism alive: caps and clamps that bite, sinks that take probability, decays from
    slow to fast, token inputs that matter."""
    cfg, ranks = cfg_ranks
    g = torch.Generator().manual_seed(seed)

    def rnd(*shape, std=1.0, mean=0.0):
        return (mean + torch.randn(*shape, generator=g) * std).to(torch.bfloat16)

    d, n = cfg["width"], cfg["token_side"]["dim"]
    w = {"embed": rnd(cfg["vocab"], d), "side.embed": rnd(cfg["vocab"], len(cfg["layers"]) * n), "final.norm": rnd(d, std=0.2, mean=1.0),
         "head": rnd(cfg["vocab"], d, std=d ** -0.5)}
    for i, ly in enumerate(cfg["layers"]):
        p, m, f = f"l{i}.", ly["mixer"], ly["mlp"]
        w[p + "norm1"] = rnd(d, std=0.2, mean=1.0)
        H, G, dk, dv = m["heads"], m.get("kv_heads", m["heads"]), m["dim"], m["vdim"]
        q = p + "mix."
        for name, rows in (("q", H * dk), ("k", G * dk), ("v", G * dv)):
            w[q + name] = rnd(rows, d, std=1.5 * d ** -0.5)
        w[q + "o"] = rnd(d, H * dv, std=(H * dv) ** -0.5)
        if ly["type"] == "attention":
            w[q + "q.norm"], w[q + "k.norm"] = rnd(H * dk, std=0.3, mean=1.5), rnd(G * dk, std=0.3, mean=1.5)
            w[q + "sink"], w[q + "g"] = rnd(H, std=1.0, mean=0.5), rnd(H, d, std=2.0 * d ** -0.5)
        else:
            w[q + "g"] = rnd(H * dv, d, std=1.5 * d ** -0.5)
            w[q + "norm"] = rnd(dv if ly["type"] == "gla" else H * dv, std=0.3, mean=1.0)
        if ly["type"] == "gla":
            w[q + "a1"], w[q + "a2"] = rnd(ranks[i], d, std=d ** -0.5), rnd(H * dk, ranks[i], std=2.0 * ranks[i] ** -0.5)
            w[q + "a2.b"] = rnd(H * dk, std=2.0, mean=2.0)
        if f is not None:
            w[p + "norm2"] = rnd(d, std=0.2, mean=1.0)
            w[p + "mlp.gate"], w[p + "mlp.up"] = rnd(f["ff"], d, std=1.5 * d ** -0.5), rnd(f["ff"], d, std=1.5 * d ** -0.5)
            w[p + "mlp.down"] = rnd(d, f["ff"], std=f["ff"] ** -0.5)
        w[p + "side.gate"], w[p + "side.proj"] = rnd(n, d, std=d ** -0.5), rnd(d, n, std=n ** -0.5)
        w[p + "side.norm"] = rnd(d, std=0.2, mean=0.5)
    return w


def model_of(cfg_ranks, weights, device="cuda"):
    from lit_gpt_b200.config import VotavikConfig
    from lit_gpt_b200.votavik import Votavik

    c = VotavikConfig.from_dict(cfg_ranks[0])
    Votavik.complete_config(c, {k: tuple(v.shape) for k, v in weights.items()})
    return Votavik(c).to(device)


def build(cfg_ranks, weights, dtype, slots=2):
    model = model_of(cfg_ranks, weights).to(dtype)
    model.load_tensors(weights)
    model.set_kv_cache(batch_size=slots)
    return model.eval()


def tokens_for(cfg_ranks, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg_ranks[0]["vocab"], (n,), generator=g).tolist()


def rel_err(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return float((got - want).norm() / want.norm().clamp_min(1e-30))


def assert_close(got, want, dtype, what=""):
    """fp32: the whole block within rounding, no row far off.  bf16: a row whose read-out nearly vanishes before its norm (the first token of
    a sequence with q . k near 0, say) turns rounding into a large difference, in exact arithmetic on rounded inputs just as well; so the
    typical row must be within bf16 rounding and nine in ten close to it.  The fp32 runs of the same tests are the sharp ones."""
    got, want = got.double().cpu(), want.double().cpu()
    rows = (got - want).norm(dim=-1) / want.norm(dim=-1).clamp_min(1e-30)
    if dtype == torch.float32:
        assert rel_err(got, want) < 4e-5 and float(rows.max()) < 3e-4, (what, rel_err(got, want), float(rows.max()), int(rows.argmax()))
    else:
        assert float(rows.median()) < 2.5e-2 and float((rows < 6e-2).double().mean()) >= 0.9, (what, float(rows.median()), rows)


def f64(weights):
    return {k: v.double() for k, v in weights.items()}


# ---------------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("d", [42, 64, 1536])
def test_layer_norm_in_the_residual_kernel_and_alone(dtype, d):
    """x += y [normed, weighted]; the copy in the product dtype; the next layer norm -- on rows whose mean is large against their spread,
    where the mean has to come off before the squares are taken."""
    k = K()
    g = torch.Generator().manual_seed(d)
    n, eps = 9, 1e-3
    x0 = torch.randn(n, d, generator=g) + torch.linspace(0, 300, n)[:, None]
    y, post, pre = (torch.randn(*s, generator=g).to(dtype) for s in ((n, d), (d,), (d,)))
    tol = 2e-5 if dtype == torch.float32 else 6e-3
    for normed in (False, True):
        want = x0.double() + (O.rms(y.double(), post.double(), eps) if normed else y.double())
        x, cast, act = x0.clone().cuda(), torch.empty(n, d, dtype=dtype, device="cuda"), torch.empty(n, d, dtype=dtype, device="cuda")
        k.sandwich_residual(x, y.cuda(), post.cuda() if normed else None, eps, pre_w=pre.cuda(), pre_center=True, act=act, cast=cast)
        assert rel_err(x, want) < 1e-6 and rel_err(cast, want) < tol
        assert rel_err(act, O.layer_norm(x.double().cpu(), pre.double(), eps)) < tol
        x2, cast2 = x0.clone().cuda(), torch.empty(n, d, dtype=dtype, device="cuda")
        k.sandwich_residual(x2, y.cuda(), post.cuda() if normed else None, eps, cast=cast2)          # no norm
        assert torch.equal(x2, x) and torch.equal(cast2, cast)
    rows = torch.tensor([8, 0, 3, 3])
    out = torch.empty(4, d, dtype=dtype, device="cuda")
    k.rms_rows(4, eps, k.rms_seg(x, pre.cuda(), out, d, False, in_rows=rows.cuda(), center=True), in_dtype=torch.float32, out_dtype=dtype,
               device=x.device)
    assert rel_err(out, O.layer_norm(x.double().cpu()[rows], pre.double(), eps)) < tol


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_token_gate(dtype):
    k = K()
    g = torch.Generator().manual_seed(4)
    n, cols, layers, vocab = 13, 11, 3, 29
    wide = (torch.randn(n, cols + 5, generator=g) * 3).to(dtype)
    table, toks = torch.randn(vocab, layers * cols, generator=g).to(dtype), torch.randint(0, vocab, (n,), generator=g)
    for i in range(layers):
        got = k.token_gate(wide.cuda()[:, :cols], toks.int().cuda(), table.cuda(), i * cols, k.C.ACT_GELU_TANH)
        want = O.gelu_tanh(wide[:, :cols].double()) * table[toks].double()[:, i * cols : (i + 1) * cols]
        assert rel_err(got, want) < (1e-6 if dtype == torch.float32 else 4e-3)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,rd,base", [(5, 2, 12, 6, 100.0), (4, 4, 64, 64, 1e4), (3, 1, 18, 0, 10.0)])
def test_norm_over_all_heads_then_rotation_in_place(dtype, H, G, dk, rd, base):
    """One norm for all query heads and one for all key heads (heads of very unequal size show a norm taken per head), then half-split
    rotation at far positions; the columns behind stay as they are."""
    k = K()
    g = torch.Generator().manual_seed(H)
    n, eps = 7, 1e-5
    rows = torch.randn(n, (H + G) * dk + 3, generator=g)
    rows[:, :dk] *= 20.0
    rows = rows.to(dtype)
    wq, wk = (torch.randn(m * dk, generator=g).to(dtype) for m in (H, G))
    wq_d, wk_d = wq.cuda(), wk.cuda()
    start = 70000
    pos = torch.arange(start, start + n, dtype=torch.int32)
    rot = dict(base=base, dims=rd)
    want = rows.double().clone()
    for lo, heads, wt in ((0, H, wq), (H * dk, G, wk)):
        part = O.rms(rows.double()[:, lo : lo + heads * dk], wt.double(), eps).view(n, heads, dk)
        want[:, lo : lo + heads * dk] = O.rotate_half(part, rot, start).reshape(n, -1)
    buf = rows.cuda()
    q, kk = buf[:, : H * dk], buf[:, H * dk : (H + G) * dk]
    freq = torch.tensor([base ** (-2.0 * i / rd) for i in range(rd // 2)], dtype=torch.float64, device="cuda") if rd else None
    turn = dict(freq=freq, rot_dims=rd, interleaved=False) if rd else {}
    k.head_rope(n, pos.cuda(), eps, k.rope_seg(q, q, H, dk, norm_w=wq_d, norm_all=True, **turn),
                k.rope_seg(kk, kk, G, dk, norm_w=wk_d, norm_all=True, **turn), dtype=dtype, device=buf.device)
    assert rel_err(buf[:, : (H + G) * dk], want[:, : (H + G) * dk]) < (1e-6 if dtype == torch.float32 else 5e-3)
    assert torch.equal(buf[:, (H + G) * dk :].cpu(), rows[:, (H + G) * dk :])


def _linear_case(kind, H, dk, dv, n, seed, tau=3.0, decay=None):
    g = torch.Generator().manual_seed(seed)
    q, kk, v = (torch.randn(n, H * m, generator=g).to(torch.bfloat16) for m in (dk, dk, dv))
    if kind == "lightning":
        gates = torch.tensor(decay if decay is not None else [0.3 + 0.69 * (j + 1) / H for j in range(H)], dtype=torch.float64)
        per = gates.view(1, H, 1).expand(n, H, dk)
        qd, kd, vd = (O.silu(t.double()) for t in (q, kk, v))
        z = bias = None
    else:
        z, bias = torch.randn(n, H * dk, generator=g) * 3, (torch.randn(H * dk, generator=g) * 2 + 1).to(torch.bfloat16)
        per = (torch.sigmoid(z.double() + bias.double()) ** (1 / tau)).view(n, H, dk)
        qd, kd, vd, gates = q.double() * dk ** -0.5, kk.double(), v.double(), None
    qd, kd, vd = qd.view(n, H, dk), kd.view(n, H, dk), vd.view(n, H, dv)
    want = torch.stack([O.decayed_sum(qd[:, j], kd[:, j], vd[:, j], per[:, j]) for j in range(H)], dim=1).reshape(n, H * dv)
    return q, kk, v, z, bias, gates, want


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("kind", ["gla", "lightning"])
@pytest.mark.parametrize("H,dk,dv", [(3, 5, 7), (2, 32, 64), (2, 48, 33), (1, 64, 100), (2, 128, 128), (1, 130, 20), (1, 256, 40), (1, 300, 12)])
def test_decaying_state_alone(H, dk, dv, kind, dtype):
    """The recurrence over every kernel shape: whole prompts in pieces of several sizes and in one walk, portions down to two tokens, single
    tokens; two sequences in one launch whose slots hold leftovers; the piece borders are where a lost or repeated decay would show."""
    k = K()
    from lit_gpt_b200.ragged import state_batch

    n = 83
    q, kk, v, z, bias, gates, want = _linear_case(kind, H, dk, dv, n, 100 * dk + dv)
    n2 = 20
    dev = lambda t, lo, hi: t[lo:hi].to(dtype).cuda()   # noqa: E731
    runs = [("pieces of 16", 16, [n]), ("pieces of 32", 32, [n]), ("one walk", 1000, [n]), ("portions", 16, [2, 2, 40, 3, 35, 1]), ("single", 0, [1] * n)]
    for what, piece, cuts in runs:
        old = k.linear_attn_tune(piece)
        try:
            state = torch.full((3, H * dk * dv), 5.0, device="cuda")
            got, other, at = [], [], 0
            for c in cuts:
                # slot 2 carries the sequence, slot 0 its first rows once more as a second sequence of the same step
                lo, hi = at, at + c
                extra = at == 0 and c >= n2
                seqs = [(2, at, c)] + ([(0, 0, n2)] if extra else [])
                batch, _ = state_batch(seqs, torch.device("cuda"))
                pack = lambda t: torch.cat([dev(t, lo, hi), dev(t, 0, n2)]) if extra else dev(t, lo, hi)   # noqa: E731
                args = dict(silu=True, head_decay=gates.float().cuda()) if kind == "lightning" else dict(
                    q_scale=dk ** -0.5, decay_in=(torch.cat([z[lo:hi], z[:n2]]) if extra else z[lo:hi]).cuda().contiguous(), decay_bias=bias.to(dtype).cuda(), tau=3.0)
                o = k.linear_attn(pack(q), pack(kk), pack(v), state, batch.seq_state, batch.max_q_len, H, dk, dv, **args)
                got.append(o[:c])
                if extra:
                    other.append(o[c:])
                at += c
        finally:
            k.linear_attn_tune(old)
        tol = 3e-6 if dtype == torch.float32 else 2e-5
        assert rel_err(torch.cat(got), want) < tol, (what, rel_err(torch.cat(got), want))
        if other:
            assert rel_err(torch.cat(other), want[:n2]) < tol, what
        assert torch.all(state[1] == 5.0), what       # nobody's slot


def test_extreme_decays_stay_finite_and_exact():
    """Decays that underflow, decays of exactly 0 and 1, and raw projections far out on both sides, in pieces and walked whole."""
    k = K()
    from lit_gpt_b200.ragged import state_batch

    H, dk, dv, n = 2, 16, 8, 100
    g = torch.Generator().manual_seed(3)
    q, kk, v = (torch.randn(n, H * m, generator=g) for m in (dk, dk, dv))
    z = torch.randn(n, H * dk, generator=g) * 60
    bias = torch.zeros(H * dk)
    batch, _ = state_batch([(0, 0, n)], torch.device("cuda"))
    sig = torch.sigmoid(z.double()).clamp_min(1e-300)
    for tau in (1.0, 16.0):
        per = (sig ** (1 / tau)).view(n, H, dk)
        want = torch.stack([O.decayed_sum(q.double().view(n, H, dk)[:, j], kk.double().view(n, H, dk)[:, j], v.double().view(n, H, dv)[:, j], per[:, j])
                            for j in range(H)], dim=1).reshape(n, H * dv)
        for piece in (16, 1000):
            old = k.linear_attn_tune(piece)
            try:
                got = k.linear_attn(q.cuda(), kk.cuda(), v.cuda(), torch.zeros(1, H * dk * dv, device="cuda"), batch.seq_state, n, H, dk, dv,
                                    decay_in=z.cuda(), decay_bias=bias.cuda(), tau=tau)
            finally:
                k.linear_attn_tune(old)
            assert torch.isfinite(got).all() and rel_err(got, want) < 5e-6
    want = torch.stack([O.decayed_sum(*(O.silu(t.double()).view(n, H, -1)[:, j] for t in (q, kk, v)), torch.full((n, dk), float(j), dtype=torch.float64))
                        for j in range(H)], dim=1).reshape(n, H * dv)
    for piece in (16, 1000):
        old = k.linear_attn_tune(piece)
        try:
            got = k.linear_attn(q.cuda(), kk.cuda(), v.cuda(), torch.zeros(1, H * dk * dv, device="cuda"), batch.seq_state, n, H, dk, dv, silu=True,
                                head_decay=torch.tensor([0.0, 1.0], device="cuda"))
        finally:
            k.linear_attn_tune(old)
        assert rel_err(got, want) < 5e-6


def _drive(mixer, state, h, cuts, slot, dtype):
    """Feed the rows of h to `mixer` in steps of the given sizes for one sequence in `slot`; returns all output rows."""
    from lit_gpt_b200.ragged import state_batch

    out, at = [], 0
    for n in cuts:
        batch, _ = state_batch([(slot, at, n)], torch.device("cuda"), positions=True)
        out.append(mixer(h[at : at + n].to(dtype).cuda().contiguous(), batch, state).float().cpu())
        at += n
    assert at == h.shape[0]
    return torch.cat(out)


MIXERS = {"attention": attention(4, 2, 10, 6, size=7, keep=3, rot_dims=6, cap=20.0, scale=2.5), "gla": gla(3, 10, 6, 5.0, 4),
          "lightning": lightning(3, 9, 14, [0.4, 0.9, 0.99])}


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("cuts", [[61], [1] * 61, [2, 2, 3, 1, 27, 2, 22, 2], [60, 1]])
@pytest.mark.parametrize("kind", sorted(MIXERS))
def test_each_mixer_alone(kind, dtype, cuts):
    """In prompts, portions down to two tokens and single tokens, in a slot whose state holds another sequence's leftovers.  The attention's
    score scale is large, so the softmax is nearly one-hot and a key that is one position off moves the output far beyond rounding."""
    cr = config(24, 11, 4, [(kind, MIXERS[kind], None)])
    w = checkpoint(cr, 3)
    model = build(cr, w, dtype, slots=3)
    g = torch.Generator().manual_seed(5)
    h = torch.randn(61, 24, generator=g).to(torch.bfloat16).double()
    want = O.MIXERS[kind](h, f64(w), "l0.mix.", cr[0]["layers"][0]["mixer"], 1e-5)
    state = model.states[0]
    for t in state.tensors():
        t.fill_(7.0)
    got = _drive(model.blocks[0].mixer, state, h, cuts, slot=1, dtype=dtype)
    assert rel_err(got, want) < (2e-5 if dtype == torch.float32 else 4e-2), rel_err(got, want)


def _window(q, kk, v, state, seqs, H, G, dk, dv, size, keep, scale, cap, sink=None, gate=None, from_start=False):
    from lit_gpt_b200.ragged import state_batch

    batch, _ = state_batch(seqs, torch.device("cuda"))
    return K().window_attn(q.cuda(), kk.cuda(), v.cuda(), state[0], state[1], sink, batch.seq_state, batch.row_seq, batch.max_q_len, H, G, dk, dv, size, scale,
                           from_start=from_start, gate=gate, gate_per_head=True, keep=keep, softcap=cap).float().cpu()


def _rings(slots, rows, G, dk, dv, dtype=torch.float32, fill=9.0):
    return (torch.full((slots, rows, G * dk), fill, device="cuda", dtype=dtype), torch.full((slots, rows, G * dv), fill, device="cuda", dtype=dtype))


@pytest.mark.parametrize("loud,keep", [(31, 4), (3, 4), (4, 4), (0, 1), (1, 1)])
def test_loud_keys_at_the_window_edge_and_among_the_kept_tokens(loud, keep):
    """One key is made loud: the query `size - 1` positions later must find it, hundreds of quiet keys in between.  One position further it
    has left the window -- unless it is among the kept tokens, which every later query finds, however far; the first token that is not
    kept must be gone.  In a prompt, in later portions and in single-token steps, through the tiled and the single-row kernel, on rings
    that wrap."""
    k = K()
    H, G, dk, dv, size, n, cap = 2, 1, 8, 5, 130, 420, 40.0
    g = torch.Generator().manual_seed(9)
    q = torch.randn(n, H * dk, generator=g) * 0.3
    kk = torch.randn(n, G * dk, generator=g) * 0.1
    v = torch.randn(n, G * dv, generator=g)
    probe = torch.randn(dk, generator=g) * 1.5
    seekers = [loud + size - 1, loud + size, loud + 2 * size, n - 1]
    for i in seekers:
        q[i, :dk] = probe
    kk[loud] = probe * 40.0 / float(probe @ probe)
    want = O.capped_attention(q.double().view(n, H, dk), kk.double().view(n, G, dk), v.double().view(n, G, dv), None, dict(size=size, keep_first=keep), 1.0,
                              cap).reshape(n, H * dv)
    for i in seekers:
        found = (want[i, :dv] - v[loud].double()).abs().max() < 1e-3
        assert bool(found) == (i - loud < size or loud < keep)
    for cuts in ([n], [loud + 2, n - loud - 2], [loud + size - 1, 1, 1, n - loud - size - 1], [2, 200, 2, n - 204], [1] * n):
        for tiled in (False, True):
            if tiled and len(cuts) == n:
                continue
            old = k.window_attn_tune(force_tiled_kernel=tiled)
            try:
                state = _rings(2, keep + size, G, dk, dv)
                got, at = [], 0
                for c in cuts:
                    s = slice(at, at + c)
                    got.append(_window(q[s], kk[s], v[s], state, [(1, at, c)], H, G, dk, dv, size, keep, 1.0, cap))
                    at += c
            finally:
                k.window_attn_tune(force_tiled_kernel=old)
            assert rel_err(torch.cat(got), want) < 1e-5, (cuts[:4], tiled)
    # the rows of the cache: kept tokens at their own positions, the window's behind them
    for p in range(keep):
        assert torch.equal(state[0][1, p].cpu(), kk[p])
    for p in range(n - size, n):
        assert torch.equal(state[1][1, keep + (p - keep) % size].cpu(), v[p])


def test_soft_cap_and_sink_have_their_exact_size():
    """Two keys with known scores: weights exp(cap tanh(s / cap)) beside exp(sink), which is neither scaled nor capped and counts once."""
    cap, scale, sink = 3.0, 0.5, 2.0
    q = torch.tensor([[0.0, 0.0], [4.0, 2.0]])
    kk = torch.tensor([[3.0, 0.0], [0.0, -1.0]])
    v = torch.tensor([[1.0, 0.0], [0.0, 1.0]])
    e = [math.exp(cap * math.tanh(s / cap)) for s in (6.0, -1.0)]
    den = sum(e) + math.exp(sink)
    sk = torch.tensor([sink], device="cuda")
    for cuts in ([2], [1, 1]):
        state, got, at = _rings(1, 5, 1, 2, 2), [], 0
        for c in cuts:
            s = slice(at, at + c)
            got.append(_window(q[s], kk[s], v[s], state, [(0, at, c)], 1, 1, 2, 2, 5, 0, scale, cap, sink=sk))
            at += c
        got = torch.cat(got)
        assert abs(float(got[1, 0]) - e[0] / den) < 1e-6 and abs(float(got[1, 1]) - e[1] / den) < 1e-6
        assert abs(float(got[0, 0]) - 1.0 / (1.0 + math.exp(sink))) < 1e-6      # one key with score 0 beside the sink


@pytest.mark.parametrize("dk,dv,size,keep,cap", [(64, 64, 100, 4, 5.0), (64, 80, 64, 64, 30.0), (128, 128, 150, 1, 12.0), (128, 128, 1, 130, 8.0), (40, 24, 30, 0, 3.0),
                                                 (8, 128, 1000, 7, 20.0), (96, 56, 70, 65, 0.0), (120, 104, 65, 200, 50.0)])
def test_prompts_on_the_tensor_cores(dk, dv, size, keep, cap):
    """bf16 prompts of three unequal sequences in one launch: head sizes padded to the tile, key sizes other than value sizes, windows
    that end inside a key tile, at its edge, of one position and longer than the prompt; kept tokens none, within a tile, a whole tile,
    several; loud scores that the cap bends; a sink and a gate per head.  Against exact attention on the same operands and the
    any-size kernel; the cache rows afterwards."""
    k = K()
    H, G = 4, 2
    g = torch.Generator().manual_seed(dk + size)
    lens = [200, 37, 300]
    n = sum(lens)
    q, kk, v = (torch.randn(n, m, generator=g).to(torch.bfloat16) for m in (H * dk, G * dk, G * dv))
    gate, sink = (torch.randn(n, H, generator=g) * 2).to(torch.bfloat16), torch.randn(H, generator=g).to(torch.bfloat16)
    scale = 2.0 * dk ** -0.5
    want, at = [], 0
    for ln in lens:
        s = slice(at, at + ln)
        o = O.capped_attention(q[s].double().view(ln, H, dk), kk[s].double().view(ln, G, dk), v[s].double().view(ln, G, dv), sink.double(),
                               dict(size=size, keep_first=keep), scale, cap)
        want.append((o * torch.sigmoid(gate[s].double())[:, :, None]).reshape(ln, H * dv))
        at += ln
    want = torch.cat(want)
    outs = {}
    for mma in (True, False):
        k.WINDOW_PREFILL_MMA = mma
        try:
            state = _rings(3, keep + size, G, dk, dv, torch.bfloat16, 0.0)
            outs[mma] = _window(q, kk, v, state, [(0, 0, lens[0]), (2, 0, lens[1]), (1, 0, lens[2])], H, G, dk, dv, size, keep, scale, cap, sink=sink.cuda(),
                                gate=gate.cuda(), from_start=True)
        finally:
            k.WINDOW_PREFILL_MMA = True
        for slot, first, ln in ((0, 0, lens[0]), (2, lens[0], lens[1]), (1, lens[0] + lens[1], lens[2])):
            for p in range(ln):
                if p < keep or p >= ln - size:
                    row = p if p < keep else keep + (p - keep) % size
                    assert torch.equal(state[0][slot, row].cpu(), kk[first + p]) and torch.equal(state[1][slot, row].cpu(), v[first + p])
    assert rel_err(outs[False], want) < 6e-3
    assert rel_err(outs[True], want) < 1.2e-2
    rows = (outs[True].double() - want).norm(dim=-1) / want.norm(dim=-1).clamp_min(1e-2)
    assert float(rows.max()) < 4e-2


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_padded_projection_rows_take_the_tensor_core_tiles(dtype):
    """A layer whose gate has fewer rows than a 16-byte access holds: the fused projection is padded, so a bf16 prompt still reaches the
    tiles (the any-size kernel is not called)."""
    cr = config(40, 17, 8, [("attention", attention(3, 1, 16, 24, size=12, keep=2, rot_dims=16, cap=7.0), None)])
    w = checkpoint(cr, 8)
    model = build(cr, w, dtype)
    assert model.blocks[0].mixer.w_in.shape[0] % 8 == 0 and model.blocks[0].mixer.cols >= 3 * 16 + 16 + 24 + 3
    h = torch.randn(50, 40, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16).double()
    lib, called = K().C.load_core(), []
    real = lib.b200_window_attn_tiles
    want = O.attention_mixer(h, f64(w), "l0.mix.", cr[0]["layers"][0]["mixer"], 1e-5)
    try:
        lib.b200_window_attn_tiles = lambda *a: called.append(1) or real(*a)
        from lit_gpt_b200.ragged import state_batch

        batch, _ = state_batch([(0, 0, 50)], torch.device("cuda"), positions=True)
        got = model.blocks[0].mixer(h.to(dtype).cuda(), batch, model.states[0])
    finally:
        lib.b200_window_attn_tiles = real
    assert bool(called) == (dtype == torch.bfloat16)
    assert rel_err(got, want) < (2e-5 if dtype == torch.float32 else 4e-2)


# ---------------------------------------------------------------------------------------------------------
# whole models
# ---------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("cr,seed", [(CFG_ODD, 11), (CFG_WIDE, 12), (CFG_TILES, 13)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_prompt_matches_oracle(cr, seed, dtype):
    w = checkpoint(cr, seed)
    toks = tokens_for(cr, 150, seed)
    model = build(cr, w, dtype)
    assert_close(model.step(toks, [(1, 0, len(toks))]), O.forward(cr[0], w, toks), dtype)


def test_layers_follow_the_oracle_one_by_one():
    """The stream after every layer in fp32."""
    for cr, seed in ((CFG_ODD, 31), (CFG_WIDE, 32), (CFG_TILES, 33)):
        w = checkpoint(cr, seed)
        toks = tokens_for(cr, 60, seed)
        model = build(cr, w, torch.float32)
        model.trace = []
        model.step(toks, [(0, 0, len(toks))])
        _, want = O.forward(cr[0], w, toks, return_layers=True)
        assert len(model.trace) == len(want) == len(cr[0]["layers"])
        for r, (a, b) in enumerate(zip(model.trace, want)):
            assert rel_err(a, b) < 5e-6, (r, rel_err(a, b))


@pytest.mark.parametrize("cr", [CFG_ODD, CFG_WIDE, CFG_TILES])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_decoding_token_by_token_equals_prefill(dtype, cr):
    w = checkpoint(cr, 41)
    toks = tokens_for(cr, 130, 41)
    model = build(cr, w, dtype)
    whole = model.step(toks, [(0, 0, len(toks))])
    single = torch.cat([model.step([t], [(1, p, 1)]) for p, t in enumerate(toks)])
    assert_close(single, whole.float(), dtype)
    assert_close(single, O.forward(cr[0], w, toks), dtype)


@pytest.mark.parametrize("portions", [[2, 2, 2, 30, 3, 34, 1, 35, 2], [109, 2], [1, 110], [5] * 22 + [1]])
@pytest.mark.parametrize("cr", [CFG_ODD, CFG_WIDE, CFG_TILES])
def test_prompt_in_portions(portions, cr):
    """A prompt cut into portions of several sizes, down to two tokens and one, gives the logits of the whole prompt."""
    w = checkpoint(cr, 51)
    toks = tokens_for(cr, sum(portions), 51)
    for dtype in (torch.float32, torch.bfloat16):
        model = build(cr, w, dtype)
        got, at = [], 0
        for n in portions:
            got.append(model.step(toks[at : at + n], [(1, at, n)]))
            at += n
        assert_close(torch.cat(got), O.forward(cr[0], w, toks), dtype)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("cr", [CFG_ODD, CFG_TILES])
def test_ragged_batch_equals_each_alone(cr, dtype):
    """Requests of unequal length in one batch (prefill together, then decoding together with the shorter ones leaving) against each alone."""
    from lit_gpt_b200.generate.serve import Session

    w = checkpoint(cr, 61)
    model = build(cr, w, dtype)
    reqs = {"a": tokens_for(cr, 150, 62), "b": tokens_for(cr, 9, 63), "c": tokens_for(cr, 73, 64), "d": tokens_for(cr, 1, 65)}
    pre = {"a": 130, "b": 3, "c": 60, "d": 1}
    session = Session(model, slots=2)       # grows while the batch is live
    rows = {rid: [] for rid in reqs}
    out = session.step([(rid, reqs[rid][: pre[rid]], None) for rid in reqs], end=["d"])
    at = 0
    for rid in reqs:
        rows[rid].append(out[at : at + pre[rid]])
        at += pre[rid]
    pos = dict(pre)
    while True:
        live = [rid for rid in reqs if pos[rid] < len(reqs[rid])]
        if not live:
            break
        out = session.step([(rid, [reqs[rid][pos[rid]]], None) for rid in live], end=[rid for rid in live if pos[rid] + 1 == len(reqs[rid])])
        for i, rid in enumerate(live):
            rows[rid].append(out[i : i + 1])
            pos[rid] += 1
    assert model.slots.in_use == 0
    want = {rid: O.forward(cr[0], w, toks) for rid, toks in reqs.items()}
    assert_close(torch.cat([torch.cat(rows[rid]) for rid in reqs]), torch.cat([want[rid] for rid in reqs]), dtype)
    if dtype == torch.float32:
        for rid in reqs:
            assert_close(torch.cat(rows[rid]), want[rid], dtype, rid)


def test_freed_slots_are_reused_without_leftovers():
    """A request ends, another takes its slot (whose states and rings still hold the first one's), starting with a two-token portion; then a
    third starts with a single token."""
    from lit_gpt_b200.generate.serve import Session

    cr = CFG_WIDE
    w = checkpoint(cr, 71)
    model = build(cr, w, torch.float32, slots=1)
    session = Session(model, slots=1)
    a, b, c = tokens_for(cr, 80, 72), tokens_for(cr, 45, 73), tokens_for(cr, 12, 74)
    session.step([("a", a, [])], end=["a"])
    got = [session.step([("b", b[:2], None)])]
    got.append(session.step([("b", b[2:40], None)]))
    got += [session.step([("b", [t], None)]) for t in b[40:]]
    session.step([], end=["b"])
    single = [session.step([("c", [t], None)]) for t in c]
    assert model.slots.capacity == 1
    assert_close(torch.cat(got), O.forward(cr[0], w, b), torch.float32)
    assert_close(torch.cat(single), O.forward(cr[0], w, c), torch.float32)


def test_long_decoding_wraps_the_rings_many_times():
    """260 single-token steps behind a prompt: windows of 5 and 7 positions wrap their rings dozens of times, the kept tokens stay."""
    cr = CFG_ODD
    w = checkpoint(cr, 81)
    toks = tokens_for(cr, 300, 81)
    model = build(cr, w, torch.float32)
    got = [model.step(toks[:40], [(0, 0, 40)])]
    got += [model.step([t], [(0, p, 1)]) for p, t in enumerate(toks[40:], start=40)]
    assert_close(torch.cat(got), O.forward(cr[0], w, toks), torch.float32)


def test_first_tokens_decode_one_by_one():
    """The first positions of a sequence, where windows, kept tokens and states fill up, as single-token steps in bf16 and fp32."""
    for cr in (CFG_ODD, CFG_TILES):
        w = checkpoint(cr, 83)
        toks = tokens_for(cr, 12, 83)
        for dtype in (torch.float32, torch.bfloat16):
            model = build(cr, w, dtype)
            got = torch.cat([model.step([t], [(0, p, 1)]) for p, t in enumerate(toks)])
            assert_close(got, O.forward(cr[0], w, toks), dtype)


def test_a_far_needle_survives_only_where_the_design_keeps_it():
    """Two prompts differ in one far token only.  Behind a window without kept tokens the logits far later agree to rounding; when the
    token is among the kept ones, or the layer carries a state, they differ."""
    def far_difference(layer, place):
        cr = config(32, 40, 4, [layer])
        w = checkpoint(cr, 5)
        w["side.embed"] = w["side.embed"] * 0
        toks = tokens_for(cr, 120, 7)
        other = list(toks)
        other[place] = (toks[place] + 1) % 40
        model = build(cr, w, torch.float32)
        a, b = model.step(toks, [(0, 0, 120)])[-1], model.step(other, [(1, 0, 120)])[-1]
        return rel_err(a, b)

    near = ("attention", attention(2, 1, 8, 8, size=20, keep=3, rot_dims=4, cap=30.0), None)
    assert far_difference(near, 3) < 1e-9 and far_difference(near, 99) < 1e-9 and far_difference(near, 2) > 1e-4 and far_difference(near, 100) > 1e-4
    assert far_difference(("lightning", lightning(2, 8, 8, [0.999, 0.995]), None), 10) > 1e-5


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_generate_entry_points(dtype):
    """Greedy generation through generate() (captured decode graph) and through the batch scheduler give the oracle's tokens."""
    from lit_gpt_b200.generate.base import generate
    from lit_gpt_b200.generate.serve import generate_batch

    cr = CFG_ODD
    w = checkpoint(cr, 91)
    prompt = tokens_for(cr, 9, 91)
    seq = O.greedy(cr[0], w, prompt, 14)
    model = build(cr, w, dtype, slots=1)
    model.max_seq_length = 64
    y = generate(model, torch.tensor(prompt, device="cuda"), len(seq), temperature=0.0)
    if dtype == torch.float32:
        assert y.tolist() == seq
    again = generate(model, torch.tensor(prompt, device="cuda"), len(seq), temperature=0.0)   # the captured graph once more, over used states
    assert again.tolist() == y.tolist()
    other = tokens_for(cr, 4, 92)
    model.set_kv_cache(batch_size=2)
    ys = generate_batch(model, [prompt, other], 14)
    assert ys[0] == y.tolist() and len(ys[1]) == 4 + 14 and model.slots.in_use == 0
    if dtype == torch.float32:
        assert ys[1] == O.greedy(cr[0], w, other, 14)


def test_forward_signature_of_the_other_models():
    """forward(idx, input_pos) with batch rows = slots and shared positions, as GPT.forward: a prompt, then single tokens."""
    cr = CFG_WIDE
    w = checkpoint(cr, 95)
    model = build(cr, w, torch.float32, slots=2)
    a, b = tokens_for(cr, 12, 96), tokens_for(cr, 12, 97)
    idx = torch.tensor([a, b], device="cuda")
    out = model(idx[:, :10], torch.arange(10, device="cuda"))
    for p in (10, 11):
        out = torch.cat([out, model(idx[:, p : p + 1], torch.tensor([p], device="cuda"))], dim=1)
    assert out.shape == (2, 12, cr[0]["vocab"])
    assert rel_err(out[0], O.forward(cr[0], w, a)) < 3e-5 and rel_err(out[1], O.forward(cr[0], w, b)) < 3e-5


def _write_checkpoint(folder, cr, weights):
    import json
    import struct

    header, blob = {}, b""
    for name, t in weights.items():
        raw = t.contiguous().view(torch.int16).numpy().tobytes()
        header[name] = {"dtype": "BF16", "shape": list(t.shape), "data_offsets": [len(blob), len(blob) + len(raw)]}
        blob += raw
    hj = json.dumps(header).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(hj)) + hj + blob)
    (folder / "config.json").write_text(json.dumps(cr[0]))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_runner_end_to_end(tmp_path, dtype):
    """The command-line replayer on a checkpoint directory written here: a ragged first step, decoding together, a request that
    ends, a new one in its slot, steps without anything wanted -- the files it writes against the oracle."""
    import json
    import subprocess

    import numpy as np

    cr = CFG_ODD
    w = checkpoint(cr, 101)
    _write_checkpoint(tmp_path, cr, w)
    a, b, c = tokens_for(cr, 40, 102), tokens_for(cr, 9, 103), tokens_for(cr, 70, 104)
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
    full = {kk: O.forward(cr[0], w, t) for kk, t in (("a", a), ("b", b), ("c", c))}
    want = {0: torch.stack([full["a"][0], full["a"][36], full["b"][5]]), 2: torch.stack([full["a"][38], full["b"][7]]),
            3: full["a"][39:40], 4: full["c"][[0, 1, 63, 64, 69]]}
    for step, ref in want.items():
        got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").reshape(-1, cr[0]["vocab"]))
        assert got.shape == ref.shape
        assert_close(got, ref, getattr(torch, dtype), f"step {step}")


def test_generate_command_line(tmp_path):
    """`python -m lit_gpt_b200.generate.base` on a checkpoint directory without a tokenizer: a prompt of token ids in, the oracle's greedy
    continuation out."""
    import subprocess

    cr = CFG_WIDE
    w = checkpoint(cr, 111)
    _write_checkpoint(tmp_path, cr, w)
    prompt = tokens_for(cr, 6, 112)
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    res = subprocess.run([sys.executable, "-m", "lit_gpt_b200.generate.base", " ".join(str(t) for t in prompt), "--checkpoint_dir", str(tmp_path),
                          "--precision", "32-true", "--temperature", "0", "--max_new_tokens", "9"], cwd=root, capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    printed = [int(t) for t in res.stdout.strip().splitlines()[-1].split()]
    assert printed == O.greedy(cr[0], w, prompt, 9)
