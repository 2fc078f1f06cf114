"""Two mixers side by side on the same input.

``ParallelState`` keeps the states of both.  ``WindowRetention`` is sliding-window attention (``window.GatedWindowAttention``) beside
retention (``linear.Retention``),

    out = left_scale * W_lo attend(h) + right_scale * W_ro retain(h)

with ONE matrix product for everything that reads h (rows left q | k | v | right q | k | v | gate), ONE launch for the four rotations,
and ONE matrix product for both output projections: the two scales are taken before the results are rounded to the matrix-product dtype, side by side in
one buffer, and [W_lo | W_ro] is stored as one weight.
"""
from __future__ import annotations

from typing import List

import torch
import torch.nn as nn
import torch.nn.functional as F

from . import kernels as K
from .config import WindowRetentionSpec
from .linear import Retention
from .ragged import RaggedBatch
from .window import GatedWindowAttention


class ParallelState(nn.Module):
    def __init__(self, left: nn.Module, right: nn.Module) -> None:
        super().__init__()
        self.left, self.right = left, right

    def tensors(self) -> List[torch.Tensor]:
        return self.left.tensors() + self.right.tensors()


class WindowRetention(nn.Module):
    def __init__(self, width: int, spec: WindowRetentionSpec, eps: float) -> None:
        super().__init__()
        self.spec, self.eps, self.width = spec, eps, width
        lf, rt = spec.left, spec.right
        self.left = GatedWindowAttention(width, lf, eps, projections=False)
        self.right = Retention(width, rt, eps, projections=False)
        # every block of rows starts at a multiple of 8 (zero rows between): its columns of the product start on 16-byte boundaries
        self.rows = [("left.q", lf.heads * lf.dim), ("left.k", lf.kv_heads * lf.dim), ("left.v", lf.kv_heads * lf.vdim), ("right.q", rt.heads * rt.dim),
                     ("right.k", rt.heads * rt.dim), ("right.v", rt.heads * rt.vdim), ("right.g", rt.heads * rt.vdim)]
        self.offsets, at = [], 0
        for _, rows in self.rows:
            self.offsets.append(at)
            at += rows + -rows % 8
        self.w_in = nn.Parameter(torch.empty(at, width), requires_grad=False)
        # columns of the results, each padded the same way: [left | right]
        self.left_cols, self.right_cols = lf.heads * lf.vdim, rt.heads * rt.vdim
        self.off_right = self.left_cols + -self.left_cols % 8
        self.out_cols = self.off_right + self.right_cols + -self.right_cols % 8
        self.w_o = nn.Parameter(torch.empty(width, self.out_cols), requires_grad=False)

    def build_state(self, slots: int, device=None, dtype=None) -> ParallelState:
        return ParallelState(self.left.build_state(slots, device, dtype), self.right.build_state(slots, device, dtype))

    def forward(self, h: torch.Tensor, batch: RaggedBatch, state: ParallelState) -> torch.Tensor:
        """h (n, width) in the matrix-product dtype -> (n, width)"""
        s, n = self.spec, h.shape[0]
        proj = F.linear(h, self.w_in)
        lq, lk, lv, rq, rk, rv, rg = (proj[:, at : at + rows] for at, (_, rows) in zip(self.offsets, self.rows))
        rq, rk, segs = self.right.turned(rq, rk)
        segs = self.left.rope_segs(lq, lk) + segs
        if segs:
            K.head_rope(n, batch.row_pos, self.eps, *segs, dtype=h.dtype, device=h.device)
        pads = self.out_cols != self.left_cols + self.right_cols
        y = (torch.zeros if pads else torch.empty)((n, self.out_cols), dtype=h.dtype, device=h.device)
        self.left.attend(lq, lk, lv, None, batch, state.left, out_scale=s.left_scale, out=y[:, : self.left_cols])
        self.right.read_out(rq, rk, rv, rg, batch, state.right, out_scale=s.right_scale, out=y[:, self.off_right : self.off_right + self.right_cols])
        return F.linear(y, self.w_o)
