"""Fovirax: a decoder-only model of pre-normed blocks over an fp32 residual stream, whose mixer is sliding-window attention and retention
side by side and whose feed-forward is sparse experts beside a gated shared one.

    x = embed[token]                                                                      (fp32)
    per layer run:  x += m * ls1 * mixer(norm_1(x));  x += m * ls2 * ff(norm_2(x))        norm(x) = x / sqrt(mean(x^2) + eps) * (1 + w)
    logits = head . norm_final(x)

Mixer ``parallel`` (``parallel.WindowRetention``): sliding-window attention with rotary positions and capped scores, and linear attention
with a fixed decay per head, each with a scale.  Feed-forward (``moe.SharedSparseExperts``): the experts of the largest router logits and a
shared expert, or none.  A run of consecutive layers may repeat with the same weights; every repetition keeps states of its own.

The residual stream, norms, scores and softmax, router, rotated operands and states of the recurrence and positions are fp32 whatever
the matrix-product dtype is; the products go to the vendor GEMM, everything else is this library's kernels: ``K.gated_residual`` does a
sublayer's scaled residual sum -- with the weighting of the experts -- and the next sublayer's norm in one launch.

Sequences live in slots with a constant-size state per layer run (key / value rings of one window, state matrices), so a sequence can
be any length.  Entry points as the other slot-served models (``ragged.StateServed``).
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch
import torch.nn as nn

from . import kernels as K
from .config import FoviraxConfig, FoviraxLayerSpec
from .moe import SharedSparseExperts
from .parallel import WindowRetention
from .ragged import RaggedBatch, StateServed


class FoviraxBlock(nn.Module):
    def __init__(self, config: FoviraxConfig, spec: FoviraxLayerSpec) -> None:
        super().__init__()
        d, self.eps, self.mult = config.n_embd, config.norm_eps, config.residual_mult
        self.norm_1 = nn.Parameter(torch.zeros(d), requires_grad=False)
        self.mixer = WindowRetention(d, spec.mixer, self.eps)
        self.ls1 = nn.Parameter(torch.ones(d), requires_grad=False)
        has_ff = spec.mlp is not None
        self.mlp: Optional[nn.Module] = SharedSparseExperts(d, spec.mlp) if has_ff else None
        self.norm_2 = nn.Parameter(torch.zeros(d), requires_grad=False) if has_ff else None
        self.ls2 = nn.Parameter(torch.ones(d), requires_grad=False) if has_ff else None

    def forward(self, x: torch.Tensor, act: torch.Tensor, batch: RaggedBatch, state: nn.Module, next_norm: Optional[torch.Tensor]) -> None:
        """x fp32 (n, d) residual, updated in place; act (n, d) = norm_1(x) in the matrix-product dtype on entry, on exit the stream normed
        with `next_norm` (None: unspecified)."""
        y = self.mixer(act, batch, state)
        K.gated_residual(x, y, self.eps, scale=self.ls1, mult=self.mult, norm_w=self.norm_2 if self.mlp is not None else next_norm, plus_one=True, act=act)
        if self.mlp is not None:
            terms = self.mlp.terms(act)
            K.gated_residual(x, terms.pop("y0"), self.eps, scale=self.ls2, mult=self.mult, norm_w=next_norm, plus_one=True, act=act, **terms)


class Fovirax(StateServed, nn.Module):
    repeatable_steps = False   # a step advances recurrent states: repeating it is not idempotent

    def __init__(self, config: FoviraxConfig) -> None:
        super().__init__()
        self.config = config
        d = config.n_embd
        self.embed = nn.Parameter(torch.empty(config.vocab_size, d), requires_grad=False)
        self.blocks = nn.ModuleList(FoviraxBlock(config, spec) for spec in config.layers)
        self.final_norm = nn.Parameter(torch.zeros(d), requires_grad=False)
        self.head = nn.Parameter(torch.empty(config.vocab_size, d), requires_grad=False)
        self.init_serving(config.schedule())
        self.trace: Optional[List[torch.Tensor]] = None     # debugging: set to a list to receive the stream after every layer run

    # ---- weights ----------------------------------------------------------------------------------------------------
    def reset_parameters(self, seed: int = 1234, std: float = 0.02) -> None:
        """Random weights for benchmarks and smoke runs: N(0, std) matrices, norm weights of zero, unit layer scales."""
        gen = torch.Generator(device=self.device).manual_seed(seed)
        for name, p in self.named_parameters():
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("ls1", "ls2"):
                p.data.fill_(1.0)
            elif p.dim() == 1:
                p.data.zero_()
            else:
                p.data.copy_(torch.empty(p.shape, dtype=torch.float32, device=p.device).normal_(0.0, std, generator=gen))

    def load_tensors(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Fill the parameters from the checkpoint's tensors: ``embed``, ``final.norm``, ``head`` and per layer i ``l<i>.norm1|norm2|ls1|ls2``,
        the mixer under ``l<i>.mix.left.`` (``q|k|v|o``) and ``l<i>.mix.right.`` (``q|k|v|g|o``), the feed-forward under ``l<i>.mlp.`` (``router``,
        ``e<j>.gate|up|down``, ``shared.gate|up|down|sg``).  Projections that read the same input are stored fused (zero rows between them
        where their sizes are no multiples of 8), the two output projections side by side, expert weights stacked."""
        used = set()

        def take(name: str) -> torch.Tensor:
            if name not in tensors:
                raise KeyError(f"checkpoint has no tensor {name!r}")
            used.add(name)
            return tensors[name]

        def put(param: torch.Tensor, value: torch.Tensor) -> None:
            if tuple(param.shape) != tuple(value.shape):
                raise ValueError(f"shape mismatch: parameter {tuple(param.shape)} vs checkpoint {tuple(value.shape)}")
            param.data.copy_(value)

        put(self.embed, take("embed"))
        put(self.final_norm, take("final.norm"))
        put(self.head, take("head"))
        for i, block in enumerate(self.blocks):
            p, mx = f"l{i}.", block.mixer
            put(block.norm_1, take(p + "norm1"))
            put(block.ls1, take(p + "ls1"))
            mx.w_in.data.zero_()
            for at, (name, rows) in zip(mx.offsets, mx.rows):
                put(mx.w_in.data[at : at + rows], take(f"{p}mix.{name}"))
            mx.w_o.data.zero_()
            put(mx.w_o.data[:, : mx.left_cols], take(p + "mix.left.o"))
            put(mx.w_o.data[:, mx.off_right : mx.off_right + mx.right_cols], take(p + "mix.right.o"))
            if block.mlp is None:
                used.update(n for n in (p + "norm2", p + "ls2") if n in tensors)   # a layer without feed-forward has no use for them
                continue
            put(block.norm_2, take(p + "norm2"))
            put(block.ls2, take(p + "ls2"))
            m, q = block.mlp, p + "mlp."
            E, ff, ffs = m.spec.experts, m.spec.ff, m.spec.shared_ff
            m.w_route.data.zero_()
            put(m.w_route.data[:E], take(q + "router"))
            for j in range(E):
                put(m.w_up.data[j, :ff], take(f"{q}e{j}.gate"))
                put(m.w_up.data[j, ff:], take(f"{q}e{j}.up"))
                put(m.w_down.data[j], take(f"{q}e{j}.down"))
            if ffs:
                put(m.w_route.data[E : E + 1], take(q + "shared.sg"))
                put(m.shared_up.data[:ffs], take(q + "shared.gate"))
                put(m.shared_up.data[ffs:], take(q + "shared.up"))
                put(m.shared_down, take(q + "shared.down"))
        extra = sorted(set(tensors) - used)
        if extra:
            raise KeyError(f"unexpected tensors in the checkpoint: {extra[:6]}")

    # ---- one step ---------------------------------------------------------------------------------------------------
    def _run(self, tokens: torch.Tensor, batch: RaggedBatch, want_rows: Optional[torch.Tensor]) -> torch.Tensor:
        """tokens int32 (n,) -> fp32 logits (rows wanted or n, vocab)"""
        eps, n, d = self.config.norm_eps, tokens.numel(), self.config.n_embd
        with self._true_fp32():
            x, act = K.embed_pos(tokens, None, self.embed, None, 1.0)
            if self.runs:
                K.rms_rows(n, eps, K.rms_seg(x, self.blocks[self.runs[0][0]].norm_1, act, d, True), in_dtype=torch.float32, out_dtype=self.dtype,
                           device=x.device)
            for r, (layer, state) in enumerate(self.runs):
                nxt = self.blocks[self.runs[r + 1][0]].norm_1 if r + 1 < len(self.runs) else None
                self.blocks[layer](x, act, batch, self.states[state], nxt)
                if self.trace is not None:
                    self.trace.append(x.clone())
            rows = n if want_rows is None else want_rows.numel()
            xn = torch.empty((rows, d), dtype=self.dtype, device=x.device)
            K.rms_rows(rows, eps, K.rms_seg(x, self.final_norm, xn, d, True, in_rows=want_rows), in_dtype=torch.float32, out_dtype=self.dtype, device=x.device)
            return K.mm_f32(xn, self.head)
