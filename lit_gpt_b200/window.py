"""Sliding-window attention with an attention sink, over a ring of cached keys and values.

    q, k, v = W h + b;  each channel then passes a short causal convolution over time (``K.short_conv``);
    q, k    : rotary positions on the first rot.dims dimensions (interleaved pairs), then x / sqrt(mean(x^2) + eps) per head;
    p_ij    = exp(s_ij) / (exp(sink_h) + sum_j' exp(s_ij')),  s_ij = scale * q_i . k_j,  over 0 <= i - j < window;
    out     = W_o concat_h(sum_j p_ij v_j) + b_o.

What a sequence keeps between steps (``WindowState``, one slot per live sequence): the last conv - 1 projected rows (the
convolution's tail) and the keys and values of its last `ring` >= window positions, position p in ring row p % ring.  The
projections are vendor matrix products; convolution, rotation, norm (one kernel), attention and the ring update are this
library's kernels.

``GatedWindowAttention`` is the same attention over the same rings (``RingState``) without convolution, norm or sink, and with

    s_ij   -= r1_h ln(1 + r2_h (i - j))                      (optional distance bias, two learned numbers per head)
    out     = W_o (concat_h(sum_j p_ij v_j) * sigmoid(W_g h))  (gate per output number, or one per head)

optional biases on q, k, v, optional rotary positions on half-split pairs (``K.head_rope``), and further options of
``GatedWindowSpec``: RMS norms over all query heads and over all key heads before the rotation (same launch), capped scores
s <- c tanh(s / c), the sink above, and kept first tokens: positions j < keep stay visible whatever the window, in cache rows of their
own ahead of the ring's.
"""
from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn
import torch.nn.functional as F

from . import kernels as K
from .config import GatedWindowSpec, WindowMixerSpec
from .ragged import RaggedBatch


class WindowState(nn.Module):
    """Per slot: conv tail (conv - 1, columns of q | k | v) and key / value rings (ring, kv_heads * dim | vdim)."""

    def __init__(self, slots: int, spec: WindowMixerSpec, device=None, dtype=None) -> None:
        super().__init__()
        cols = spec.heads * spec.dim + spec.kv_heads * (spec.dim + spec.vdim)
        self.ring = spec.window
        self.register_buffer("tail", torch.zeros((slots, max(spec.conv - 1, 1), cols), device=device, dtype=dtype), persistent=False)
        self.register_buffer("k_ring", torch.zeros((slots, self.ring, spec.kv_heads * spec.dim), device=device, dtype=dtype), persistent=False)
        self.register_buffer("v_ring", torch.zeros((slots, self.ring, spec.kv_heads * spec.vdim), device=device, dtype=dtype), persistent=False)

    def tensors(self):
        return [self.tail, self.k_ring, self.v_ring]


class WindowAttention(nn.Module):
    def __init__(self, width: int, spec: WindowMixerSpec, eps: float) -> None:
        super().__init__()
        self.spec, self.eps, self.width = spec, eps, width
        H, G, dk, dv = spec.heads, spec.kv_heads, spec.dim, spec.vdim
        self.cols = H * dk + G * dk + G * dv
        # fused projection: rows [0, H dk) queries, then G dk keys, then G dv values; the convolution weights follow the same order
        self.w_qkv = nn.Parameter(torch.empty(self.cols, width), requires_grad=False)
        self.b_qkv = nn.Parameter(torch.zeros(self.cols), requires_grad=False)
        self.conv = nn.Parameter(torch.empty(self.cols, spec.conv), requires_grad=False)
        self.sink = nn.Parameter(torch.zeros(H), requires_grad=False)
        self.w_o = nn.Parameter(torch.empty(width, H * dv), requires_grad=False)
        self.b_o = nn.Parameter(torch.zeros(width), requires_grad=False)
        self._freq_cache: dict = {}

    def inv_freq(self, device: torch.device) -> Optional[torch.Tensor]:
        """Angular frequencies of the rotated pairs on `device`, in double precision (the kernel reduces position * frequency
        before the fp32 sine); made from the specification, so no cast or move of the module touches them."""
        rot = self.spec.rot
        if rot is None or rot.dims == 0:
            return None
        t = self._freq_cache.get(device)
        if t is None:
            t = self._freq_cache[device] = torch.tensor(rot.frequencies(), dtype=torch.float64, device=device)
        return t

    def build_state(self, slots: int, device=None, dtype=None) -> WindowState:
        return WindowState(slots, self.spec, device, dtype)

    def forward(self, h: torch.Tensor, batch: RaggedBatch, state: WindowState) -> torch.Tensor:
        """h (n, width) in the matrix-product dtype -> (n, width)"""
        s, n = self.spec, h.shape[0]
        H, G, dk, dv = s.heads, s.kv_heads, s.dim, s.vdim
        qkv = F.linear(h, self.w_qkv, self.b_qkv)
        out = torch.empty((n, self.cols), dtype=h.dtype, device=h.device)
        q, k, v = out[:, : H * dk], out[:, H * dk : (H + G) * dk], out[:, (H + G) * dk :]
        rot = s.rot
        rd = rot.dims if rot is not None else 0
        mag = rot.magnitude if rot is not None else 1.0
        cw, fr = self.conv, self.inv_freq(h.device)
        groups = [
            K.conv_group(cw[: H * dk], q, 0, H, dk, post=1, rot_dims=rd, inv_freq=fr, rot_mscale=mag, eps=self.eps),
            K.conv_group(cw[H * dk : (H + G) * dk], k, H * dk, G, dk, post=1, rot_dims=rd, inv_freq=fr, rot_mscale=mag, eps=self.eps),
            K.conv_group(cw[(H + G) * dk :], v, (H + G) * dk, G, dv),
        ]
        K.short_conv(qkv, groups, s.conv, state.tail, batch.seq_state, batch.row_seq)
        y = K.window_attn(q, k, v, state.k_ring, state.v_ring, self.sink, batch.seq_state, batch.row_seq, batch.max_q_len, H, G, dk, dv,
                          s.window, s.scale, from_start=batch.identity_ctx)
        return F.linear(y, self.w_o, self.b_o)


class RingState(nn.Module):
    """Per slot: keys and values (keep + ring, kv_heads * dim | vdim) of a sequence's first `keep` and last `ring` positions."""

    def __init__(self, slots: int, ring: int, k_cols: int, v_cols: int, device=None, dtype=None, keep: int = 0) -> None:
        super().__init__()
        self.ring, self.keep = ring, keep
        self.register_buffer("k_ring", torch.zeros((slots, keep + ring, k_cols), device=device, dtype=dtype), persistent=False)
        self.register_buffer("v_ring", torch.zeros((slots, keep + ring, v_cols), device=device, dtype=dtype), persistent=False)

    def tensors(self):
        return [self.k_ring, self.v_ring]


class GatedWindowAttention(nn.Module):
    def __init__(self, width: int, spec: GatedWindowSpec, eps: float = 0.0, align: int = 1, projections: bool = True) -> None:
        """align: the fused projection gets zero rows at its end up to a multiple of `align` (rows of its result then start on 16-byte
        boundaries whatever the number of heads).  projections=False: the input and output projections belong to whoever runs this
        attention beside another mixer (``parallel``), through ``rope_segs`` and ``attend``."""
        super().__init__()
        self.spec, self.eps, self.width = spec, eps, width
        H, G, dk, dv = spec.heads, spec.kv_heads, spec.dim, spec.vdim
        self.gate_cols = 0 if spec.gate is None else (H if spec.gate == "head" else H * dv)
        self.cols = H * dk + G * dk + G * dv + self.gate_cols
        self.cols += -self.cols % align
        # fused projection: rows [0, H dk) queries, then G dk keys, G dv values, then the gate's rows (and padding)
        self.w_in = nn.Parameter(torch.empty(self.cols, width), requires_grad=False) if projections else None
        self.b_in = nn.Parameter(torch.zeros(self.cols), requires_grad=False) if spec.bias and projections else None
        self.r1 = nn.Parameter(torch.zeros(H), requires_grad=False) if spec.distance else None
        self.r2 = nn.Parameter(torch.zeros(H), requires_grad=False) if spec.distance else None
        self.q_norm = nn.Parameter(torch.ones(H * dk), requires_grad=False) if spec.qk_norm else None
        self.k_norm = nn.Parameter(torch.ones(G * dk), requires_grad=False) if spec.qk_norm else None
        self.sink = nn.Parameter(torch.zeros(H), requires_grad=False) if spec.sink else None
        self.w_o = nn.Parameter(torch.empty(width, H * dv), requires_grad=False) if projections else None
        self._freq_cache: dict = {}

    def freq(self, device: torch.device) -> Optional[torch.Tensor]:
        """Angular frequencies of the rotated pairs on `device` (fp64: the kernel reduces position * frequency before the fp32 sine; made from
        the specification, so no cast of the module touches them)."""
        rot = self.spec.rot
        if rot is None or rot.dims == 0:
            return None
        t = self._freq_cache.get(device)
        if t is None:
            t = self._freq_cache[device] = torch.tensor(rot.frequencies(), dtype=torch.float64, device=device)
        return t

    def build_state(self, slots: int, device=None, dtype=None) -> RingState:
        s = self.spec
        return RingState(slots, s.window, s.kv_heads * s.dim, s.kv_heads * s.vdim, device, dtype, keep=s.keep)

    def rope_segs(self, q: torch.Tensor, k: torch.Tensor) -> list:
        """Norms and rotations of the projected q and k, in place, as groups for ``K.head_rope`` (none where there is nothing to do)."""
        s, fr = self.spec, self.freq(q.device)
        if fr is None and not s.qk_norm:
            return []
        turn = dict(freq=fr, rot_dims=s.rot.dims, interleaved=s.rot.interleaved, mag=s.rot.magnitude) if fr is not None else {}
        return [K.rope_seg(q, q, s.heads, s.dim, norm_w=self.q_norm, norm_all=s.qk_norm, **turn),
                K.rope_seg(k, k, s.kv_heads, s.dim, norm_w=self.k_norm, norm_all=s.qk_norm, **turn)]

    def attend(self, q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, gate: Optional[torch.Tensor], batch: RaggedBatch, state: RingState, *,
               out_scale: float = 1.0, out: Optional[torch.Tensor] = None) -> torch.Tensor:
        """Attention over the step's rows and the rings, which the rows then enter -> (n, heads * vdim), times out_scale, in `out` if given."""
        s = self.spec
        return K.window_attn(q, k, v, state.k_ring, state.v_ring, self.sink, batch.seq_state, batch.row_seq, batch.max_q_len, s.heads, s.kv_heads, s.dim,
                             s.vdim, s.window, s.scale, from_start=batch.identity_ctx, dist=(self.r1, self.r2) if s.distance else None, gate=gate,
                             gate_per_head=s.gate == "head", keep=s.keep, softcap=s.softcap, out_scale=out_scale, out=out)

    def forward(self, h: torch.Tensor, batch: RaggedBatch, state: RingState) -> torch.Tensor:
        """h (n, width) in the matrix-product dtype -> (n, width)"""
        s, n = self.spec, h.shape[0]
        H, G, dk, dv = s.heads, s.kv_heads, s.dim, s.vdim
        proj = F.linear(h, self.w_in, self.b_in)
        q, k, v = proj[:, : H * dk], proj[:, H * dk : (H + G) * dk], proj[:, (H + G) * dk : (H + G) * dk + G * dv]
        off = (H + G) * dk + G * dv
        gate = proj[:, off : off + self.gate_cols] if self.gate_cols else None
        segs = self.rope_segs(q, k)
        if segs:   # both norms and both rotations in place, one launch
            K.head_rope(n, batch.row_pos, self.eps, *segs, dtype=h.dtype, device=h.device)
        return F.linear(self.attend(q, k, v, gate, batch, state), self.w_o)
