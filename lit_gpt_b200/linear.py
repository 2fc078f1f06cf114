"""Linear attention with decaying states: a recurrent mixer whose state is one dim x vdim matrix per head, kept in fp32.

    per head and token:  S <- diag(g) S + k v^T;   o = S^T q           (the read-out sees the token's own write)

``LinearMixerSpec.decay`` given (one fixed decay per head):
    q, k, v = silu(W_q h), silu(W_k h), silu(W_v h);  g = decay_h;
    out = W_o (concat_h(o) / sqrt(mean(.^2) + eps) * w_norm * sigmoid(W_g h))          (the heads normed together)
else (one decay per head and key channel):
    q, k, v = dim^-1/2 W_q h, W_k h, W_v h;  g = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau);
    out = W_o (concat_h(o_h / sqrt(mean(o_h^2) + eps) * w_norm) * silu(W_g h))         (each head normed alone, one weight for all)

All projections that read h run as ONE matrix product (rows q | k | v | gate | decay-in); activations, scaling, decays and the
recurrence are one kernel (``K.linear_attn``; a long prompt runs in pieces side by side), norm and gate another.  What a sequence keeps
between steps (``LinearState``): the state matrices.

``Retention`` is the same recurrence with a fixed decay per head and rotary positions on q and k instead of an activation:

    q, k = rot(W_q h), rot(W_k h) dim^-1/2;  v = W_v h;  g = decay_h;
    out  = W_o (concat_h(o_h / sqrt(mean(o_h^2) + eps)) * silu(W_g h))

q and k leave the rotation in fp32 (they enter the recurrence), and the factor dim^-1/2 goes to q, where it does the same.
"""
from __future__ import annotations

from typing import List, Optional, Tuple, Union

import torch
import torch.nn as nn
import torch.nn.functional as F

from . import kernels as K
from .config import LinearMixerSpec, RetentionSpec
from .ragged import RaggedBatch


class LinearState(nn.Module):
    """Per slot: the fp32 state matrices of all heads, [head][dim][vdim]."""

    def __init__(self, slots: int, spec: Union[LinearMixerSpec, RetentionSpec], device=None) -> None:
        super().__init__()
        self.register_buffer("matrices", torch.zeros((slots, spec.heads * spec.dim * spec.vdim), device=device, dtype=torch.float32), persistent=False)

    def tensors(self):
        return [self.matrices]


class DecayLinearAttention(nn.Module):
    def __init__(self, width: int, spec: LinearMixerSpec, eps: float) -> None:
        super().__init__()
        self.spec, self.eps, self.width = spec, eps, width
        H, dk, dv = spec.heads, spec.dim, spec.vdim
        self.channel = spec.decay is None
        if self.channel and spec.decay_rank <= 0:
            raise ValueError("per-channel decays need the inner size of their low-rank projection")
        self.off_v, self.off_gate, self.off_decay = 2 * H * dk, 2 * H * dk + H * dv, 2 * H * dk + 2 * H * dv
        cols = self.off_decay + (spec.decay_rank if self.channel else 0)
        # rows q | k | v | gate (| decay-in), then zero rows up to a multiple of 8: rows of the product start on 16-byte boundaries
        self.w_in = nn.Parameter(torch.empty(cols + -cols % 8, width), requires_grad=False)
        self.w_decay2 = nn.Parameter(torch.empty(H * dk, spec.decay_rank), requires_grad=False) if self.channel else None
        self.decay_bias = nn.Parameter(torch.zeros(H * dk), requires_grad=False) if self.channel else None
        self.norm = nn.Parameter(torch.ones(dv if self.channel else H * dv), requires_grad=False)
        self.w_o = nn.Parameter(torch.empty(width, H * dv), requires_grad=False)
        self._decay_cache: dict = {}

    def head_decay(self, device: torch.device) -> torch.Tensor:
        """The fixed decays on `device`, fp32 (made from the specification, so no cast of the module touches them)."""
        t = self._decay_cache.get(device)
        if t is None:
            t = self._decay_cache[device] = torch.tensor(self.spec.decay, dtype=torch.float32, device=device)
        return t

    def build_state(self, slots: int, device=None, dtype=None) -> LinearState:
        return LinearState(slots, self.spec, device)

    def forward(self, h: torch.Tensor, batch: RaggedBatch, state: LinearState) -> torch.Tensor:
        """h (n, width) in the matrix-product dtype -> (n, width)"""
        s = self.spec
        H, dk, dv = s.heads, s.dim, s.vdim
        proj = F.linear(h, self.w_in)
        q, k, v = proj[:, : H * dk], proj[:, H * dk : self.off_v], proj[:, self.off_v : self.off_gate]
        gate = proj[:, self.off_gate : self.off_decay]
        if self.channel:
            z = K.mm_f32(proj[:, self.off_decay : self.off_decay + s.decay_rank], self.w_decay2)
            o = K.linear_attn(q, k, v, state.matrices, batch.seq_state, batch.max_q_len, H, dk, dv, q_scale=dk ** -0.5, decay_in=z,
                              decay_bias=self.decay_bias, tau=s.tau)
            y = K.gated_rms_heads(o, gate, self.norm, H, dv, K.GATE_SILU, self.eps)
        else:
            o = K.linear_attn(q, k, v, state.matrices, batch.seq_state, batch.max_q_len, H, dk, dv, silu=True, head_decay=self.head_decay(h.device))
            y = K.gated_rms_heads(o, gate, self.norm, 1, H * dv, K.GATE_SIGMOID, self.eps)
        return F.linear(y, self.w_o)


class Retention(nn.Module):
    def __init__(self, width: int, spec: RetentionSpec, eps: float, projections: bool = True) -> None:
        """projections=False: the input and output projections belong to whoever runs this mixer beside another one (``parallel``), through
        ``turned`` and ``read_out``."""
        super().__init__()
        self.spec, self.eps, self.width = spec, eps, width
        H, dk, dv = spec.heads, spec.dim, spec.vdim
        self.off_v, self.off_gate, cols = 2 * H * dk, 2 * H * dk + H * dv, 2 * H * dk + 2 * H * dv
        # rows q | k | v | gate, then zero rows up to a multiple of 8
        self.w_in = nn.Parameter(torch.empty(cols + -cols % 8, width), requires_grad=False) if projections else None
        self.w_o = nn.Parameter(torch.empty(width, H * dv), requires_grad=False) if projections else None
        self._cache: dict = {}

    def constants(self, device: torch.device) -> Tuple[torch.Tensor, Optional[torch.Tensor]]:
        """Decays (fp32) and angular frequencies (fp64, None without rotation) on `device`, made from the specification, so no cast of the
        module touches them."""
        t = self._cache.get(device)
        if t is None:
            s = self.spec
            turns = s.rot is not None and s.rot.dims > 0
            t = self._cache[device] = (torch.tensor(s.decay, dtype=torch.float32, device=device),
                                       torch.tensor(s.rot.frequencies(), dtype=torch.float64, device=device) if turns else None)
        return t

    def build_state(self, slots: int, device=None, dtype=None) -> LinearState:
        return LinearState(slots, self.spec, device)

    def turned(self, q: torch.Tensor, k: torch.Tensor) -> Tuple[torch.Tensor, torch.Tensor, List]:
        """(q, k) as the recurrence reads them once the returned groups have gone through ``K.head_rope``."""
        s, fr = self.spec, self.constants(q.device)[1]
        if fr is None:
            return q, k, []
        n, cols = q.shape
        both = torch.empty((n, 2 * cols), dtype=torch.float32, device=q.device)
        tq, tk = both[:, :cols], both[:, cols:]
        turn = dict(freq=fr, rot_dims=s.rot.dims, interleaved=s.rot.interleaved, mag=s.rot.magnitude)
        return tq, tk, [K.rope_seg(q, tq, s.heads, s.dim, **turn), K.rope_seg(k, tk, s.heads, s.dim, **turn)]

    def read_out(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: torch.Tensor, batch: RaggedBatch, state: LinearState, *,
                 out_scale: float = 1.0, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Recurrence, norm and gate -> (n, heads * vdim) in the gate's dtype, times out_scale, in `out` if given."""
        s = self.spec
        o = K.linear_attn(q, k, v, state.matrices, batch.seq_state, batch.max_q_len, s.heads, s.dim, s.vdim, q_scale=s.dim ** -0.5,
                          head_decay=self.constants(q.device)[0])
        return K.gated_rms_heads(o, gate, None, s.heads, s.vdim, K.GATE_SILU, self.eps, out_scale=out_scale, out=out)

    def forward(self, h: torch.Tensor, batch: RaggedBatch, state: LinearState) -> torch.Tensor:
        """h (n, width) in the matrix-product dtype -> (n, width)"""
        s = self.spec
        H, dk, dv = s.heads, s.dim, s.vdim
        proj = F.linear(h, self.w_in)
        q, k, segs = self.turned(proj[:, : H * dk], proj[:, H * dk : self.off_v])
        if segs:
            K.head_rope(h.shape[0], batch.row_pos, self.eps, *segs, dtype=h.dtype, device=h.device)
        y = self.read_out(q, k, proj[:, self.off_v : self.off_gate], proj[:, self.off_gate : self.off_gate + H * dv], batch, state)
        return F.linear(y, self.w_o)
