"""Votavik: a decoder-only model of pre-normed blocks over an fp32 residual stream, every layer of which has an input of its own from a
second embedding table.

    x = embed[token]                                                                      (fp32)
    per layer i:  x += mixer(ln1(x));  x += ff(ln2(x))                                     ln(x) = (x - mean) / sqrt(var + eps) * w
                  x += norm(W_p (gelu_tanh(W_g x) * side_embed[token][part i])) * w_s       norm(y) = y / sqrt(mean(y^2) + eps)
    logits = head . ln_final(x)

Mixers: ``attention`` -- sliding-window attention with kept first tokens, norms over all query and all key heads, rotary positions on
half-split pairs, capped scores, a sink and a gate per head (``window.GatedWindowAttention``); ``gla`` and ``lightning`` -- linear
attention with a decay per channel or a fixed one per head (``linear.DecayLinearAttention``).  Feed-forwards: gated with clamped
branches (``moe.ClampedGLU``), or none.

The residual stream, norms, scores, softmax, decays, recurrent states and positions are fp32 whatever the matrix-product dtype is; the
products go to the vendor GEMM, everything else is this library's kernels: ``K.sandwich_residual`` does a sublayer's (normed) residual
sum and the next sublayer's norm -- or the copy of the stream that the layer's own input is gated by -- in one launch.

Sequences live in slots with a constant-size state per layer (key / value rings of one window with the kept tokens ahead of them, or
state matrices), so a sequence can be any length.  Entry points as the other slot-served models (``ragged.StateServed``).
"""
from __future__ import annotations

from typing import Dict, List, Optional, Tuple

import torch
import torch.nn as nn
import torch.nn.functional as F

from . import kernels as K
from .config import VotavikConfig, VotavikLayerSpec
from .linear import DecayLinearAttention
from .moe import ClampedGLU
from .ragged import RaggedBatch, StateServed
from .window import GatedWindowAttention


class TokenInput(nn.Module):
    """W_proj (gelu_tanh(W_gate x) * e) with e the token's part of a second embedding table; its norm and the sum are the caller's."""

    def __init__(self, width: int, dim: int, off: int) -> None:
        super().__init__()
        self.off = off
        self.w_gate = nn.Parameter(torch.empty(dim, width), requires_grad=False)
        self.w_proj = nn.Parameter(torch.empty(width, dim), requires_grad=False)
        self.norm = nn.Parameter(torch.ones(width), requires_grad=False)

    def forward(self, x: torch.Tensor, tokens: torch.Tensor, table: torch.Tensor) -> torch.Tensor:
        return F.linear(K.token_gate(F.linear(x, self.w_gate), tokens, table, self.off, K.ACT_GELU_TANH), self.w_proj)


class VotavikBlock(nn.Module):
    def __init__(self, config: VotavikConfig, spec: VotavikLayerSpec, index: int) -> None:
        super().__init__()
        d, self.eps = config.n_embd, config.norm_eps
        self.norm_1 = nn.Parameter(torch.ones(d), requires_grad=False)
        if spec.type == "attention":
            self.mixer: nn.Module = GatedWindowAttention(d, spec.mixer, self.eps, align=8)
        else:
            self.mixer = DecayLinearAttention(d, spec.mixer, self.eps)
        self.mlp: Optional[nn.Module] = ClampedGLU(d, spec.mlp.ff, spec.mlp.limit, spec.mlp.alpha) if spec.mlp is not None else None
        self.norm_2 = nn.Parameter(torch.ones(d), requires_grad=False) if spec.mlp is not None else None
        self.side = TokenInput(d, config.side_dim, index * config.side_dim)

    def forward(self, x: torch.Tensor, act: torch.Tensor, tokens: torch.Tensor, side_embed: torch.Tensor, batch: RaggedBatch, state: nn.Module,
                next_norm: Optional[torch.Tensor]) -> None:
        """x fp32 (n, d) residual, updated in place; act (n, d) = this block's first norm of x in the matrix-product dtype on entry, on
        exit the stream normed with `next_norm` (None: unspecified)."""
        y = self.mixer(act, batch, state)
        if self.mlp is not None:
            K.sandwich_residual(x, y, None, self.eps, pre_w=self.norm_2, pre_center=True, act=act)
            y = self.mlp(act)
        K.sandwich_residual(x, y, None, self.eps, cast=act)
        K.sandwich_residual(x, self.side(act, tokens, side_embed), self.side.norm, self.eps, pre_w=next_norm, pre_center=True, act=act)


class Votavik(StateServed, nn.Module):
    repeatable_steps = False   # a step advances recurrent states: repeating it is not idempotent

    def __init__(self, config: VotavikConfig) -> None:
        super().__init__()
        self.config = config
        d = config.n_embd
        self.embed = nn.Parameter(torch.empty(config.vocab_size, d), requires_grad=False)
        self.side_embed = nn.Parameter(torch.empty(config.vocab_size, config.n_layer * config.side_dim), requires_grad=False)
        self.blocks = nn.ModuleList(VotavikBlock(config, spec, i) for i, spec in enumerate(config.layers))
        self.final_norm = nn.Parameter(torch.ones(d), requires_grad=False)
        self.head = nn.Parameter(torch.empty(config.vocab_size, d), requires_grad=False)
        self.init_serving(config.schedule())
        self.trace: Optional[List[torch.Tensor]] = None     # debugging: set to a list to receive the stream after every layer

    # ---- weights ----------------------------------------------------------------------------------------------------
    def reset_parameters(self, seed: int = 1234, std: float = 0.02) -> None:
        """Random weights for benchmarks and smoke runs: N(0, std) matrices, unit norms, zero sinks, decay biases of 3 (slow decays)."""
        gen = torch.Generator(device=self.device).manual_seed(seed)
        for name, p in self.named_parameters():
            leaf = name.rsplit(".", 1)[-1]
            if "norm" in leaf:
                p.data.fill_(1.0)
            elif leaf == "decay_bias":
                p.data.fill_(3.0)
            elif p.dim() == 1:
                p.data.zero_()
            else:
                p.data.copy_(torch.empty(p.shape, dtype=torch.float32, device=p.device).normal_(0.0, std, generator=gen))

    @staticmethod
    def complete_config(config: VotavikConfig, shapes: Dict[str, Tuple[int, ...]]) -> None:
        """The size the configuration file leaves to the weights: the inner size of the low-rank decay projections."""
        for i, layer in enumerate(config.layers):
            if layer.type == "gla":
                layer.mixer.decay_rank = int(shapes[f"l{i}.mix.a1"][0])

    def load_tensors(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Fill the parameters from the checkpoint's tensors: ``embed``, ``side.embed``, ``final.norm``, ``head`` and per layer i
        ``l<i>.norm1|norm2``, the mixer under ``l<i>.mix.`` (``q|k|v|g|o`` with ``q.norm|k.norm|sink`` for attention, ``norm`` for linear
        attention and ``a1|a2|a2.b`` for per-channel decays), the feed-forward under ``l<i>.mlp.`` (``gate|up|down``) and the token input
        under ``l<i>.side.`` (``gate|proj|norm``).  Projections that read the same input are stored fused."""
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

        def put_rows(param: nn.Parameter, sizes: List[Tuple[str, int]]) -> None:
            """Named blocks of rows one below the other; what is left of the parameter is padding."""
            at = 0
            for name, rows in sizes:
                put(param.data[at : at + rows], take(name))
                at += rows
            param.data[at:].zero_()

        put(self.embed, take("embed"))
        put(self.side_embed, take("side.embed"))
        put(self.final_norm, take("final.norm"))
        put(self.head, take("head"))
        for i, block in enumerate(self.blocks):
            p, mx = f"l{i}.", block.mixer
            s, q = mx.spec, f"l{i}.mix."
            put(block.norm_1, take(p + "norm1"))
            if isinstance(mx, GatedWindowAttention):
                put_rows(mx.w_in, [(q + "q", s.heads * s.dim), (q + "k", s.kv_heads * s.dim), (q + "v", s.kv_heads * s.vdim), (q + "g", mx.gate_cols)])
                put(mx.q_norm, take(q + "q.norm"))
                put(mx.k_norm, take(q + "k.norm"))
                put(mx.sink, take(q + "sink"))
            else:
                rows = [(q + "q", s.heads * s.dim), (q + "k", s.heads * s.dim), (q + "v", s.heads * s.vdim), (q + "g", s.heads * s.vdim)]
                put_rows(mx.w_in, rows + ([(q + "a1", s.decay_rank)] if mx.channel else []))
                if mx.channel:
                    put(mx.w_decay2, take(q + "a2"))
                    put(mx.decay_bias, take(q + "a2.b"))
                put(mx.norm, take(q + "norm"))
            put(mx.w_o, take(q + "o"))
            put(block.side.w_gate, take(p + "side.gate"))
            put(block.side.w_proj, take(p + "side.proj"))
            put(block.side.norm, take(p + "side.norm"))
            if block.mlp is None:
                used.update(n for n in (p + "norm2",) if n in tensors)   # a layer without feed-forward has no use for it
                continue
            put(block.norm_2, take(p + "norm2"))
            ff = block.mlp.w_down.shape[1]
            put_rows(block.mlp.w_up, [(p + "mlp.gate", ff), (p + "mlp.up", ff)])
            put(block.mlp.w_down, take(p + "mlp.down"))
        extra = sorted(set(tensors) - used)
        if extra:
            raise KeyError(f"unexpected tensors in the checkpoint: {extra[:6]}")

    # ---- one step ---------------------------------------------------------------------------------------------------
    def _run(self, tokens: torch.Tensor, batch: RaggedBatch, want_rows: Optional[torch.Tensor]) -> torch.Tensor:
        """tokens int32 (n,) -> fp32 logits (rows wanted or n, vocab)"""
        c, eps = self.config, self.config.norm_eps
        n, d = tokens.numel(), c.n_embd
        with self._true_fp32():
            x, act = K.embed_pos(tokens, None, self.embed, None, 1.0)
            if self.runs:
                K.rms_rows(n, eps, K.rms_seg(x, self.blocks[self.runs[0][0]].norm_1, act, d, False, center=True), in_dtype=torch.float32,
                           out_dtype=self.dtype, device=x.device)
            for r, (layer, state) in enumerate(self.runs):
                nxt = self.blocks[self.runs[r + 1][0]].norm_1 if r + 1 < len(self.runs) else None
                self.blocks[layer](x, act, tokens, self.side_embed, batch, self.states[state], nxt)
                if self.trace is not None:
                    self.trace.append(x.clone())
            rows = n if want_rows is None else want_rows.numel()
            xn = torch.empty((rows, d), dtype=self.dtype, device=x.device)
            K.rms_rows(rows, eps, K.rms_seg(x, self.final_norm, xn, d, False, in_rows=want_rows, center=True), in_dtype=torch.float32,
                       out_dtype=self.dtype, device=x.device)
            return K.mm_f32(xn, self.head)
