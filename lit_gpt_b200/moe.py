"""Sparse mixtures of experts.

``GroupLimitedRouter``: scores s = sigmoid(W x) in fp32.  Experts are CHOSEN by s + correction (a per-expert selection bias
that does not enter the output), among the experts of the ``keep`` best of ``groups`` equal groups of neighbouring experts --
a group is ranked by the sum of its two largest corrected scores -- and the chosen experts are WEIGHTED by s itself, without
renormalisation.  ``SparseExperts``: out = sum_k weight_k * W_down[e_k] relu(W_up[e_k] x)^2 over stacked expert weights, as a
grouped matrix product for many tokens (the vendor's grouped GEMM for bf16, this library's any-size fp32-accumulating kernel
otherwise) and as weight-streaming GEMVs for a few (``K.moe_experts``).

``GroupLimitedRouter(softmax=True, group_max=True)`` scores with a softmax over all experts and ranks a group by its largest
score; ``GatedSparseExperts`` uses it with gated experts, out = sum_k s_k * W_down[e_k] (silu(W_gate[e_k] x) * (W_up[e_k] x)), gate
and up rows stacked into one (experts, 2 ff, width) tensor so that both are one (grouped) product.

``ClampedSparseExperts``: the router adds a bias to its logits, takes the `top` largest and weights them by a softmax among
those few; experts are gated with clamped branches, W_down (g sigmoid(alpha g) (u + 1)), g = min(W_gate x, limit), u = clamp(W_up x,
-limit, limit); ``ClampedGLU`` is one such expert for every token (a shared expert).

``SharedSparseExperts``: the `top` largest logits weighted by a softmax among them, plain gated experts W_down (silu(W_gate x) * (W_up x)),
and a shared expert of that form times the sigmoid of one projected number per token.  The router's rows and that number's row are
one weight and one matrix product with fp32 results.  ``terms`` hands the parts of the result to the residual kernel, which weights
and sums them (``K.gated_residual``).
"""
from __future__ import annotations

from typing import Dict

import torch
import torch.nn as nn

from . import kernels as K
from .config import ClampedMoESpec, GatedMoESpec, MoESpec, SharedMoESpec


VENDOR_GROUPED_GEMM = True   # tests switch it off to run the library's own grouped kernel on the same input


class GroupLimitedRouter(nn.Module):
    def __init__(self, width: int, experts: int, top: int, groups: int = 1, keep: int = 1, *, softmax: bool = False, group_max: bool = False,
                 correction: bool = True, topk_softmax: bool = False, bias: bool = False) -> None:
        """topk_softmax: raw logits choose, weights = softmax among those few; bias: `correction` is a bias inside the logit."""
        super().__init__()
        self.top, self.groups, self.keep, self.softmax, self.group_max = top, groups, keep, softmax, group_max
        self.topk_softmax, self.bias = topk_softmax, bias
        self.weight = nn.Parameter(torch.empty(experts, width), requires_grad=False)
        self.correction = nn.Parameter(torch.zeros(experts), requires_grad=False) if correction else None

    def forward(self, x: torch.Tensor):
        """x (n, width) -> (expert ids int32 (n, top), weights fp32 (n, top))"""
        return K.moe_route(x, self.weight, self.correction, self.top, self.groups, self.keep, softmax=self.softmax, group_max=self.group_max,
                           topk_softmax=self.topk_softmax, bias=self.bias)


class SparseExperts(nn.Module):
    def __init__(self, width: int, spec: MoESpec) -> None:
        super().__init__()
        self.spec = spec
        self.router = GroupLimitedRouter(width, spec.experts, spec.top, spec.groups, spec.keep)
        self.w_up = nn.Parameter(torch.empty(spec.experts, spec.ff, width), requires_grad=False)
        self.w_down = nn.Parameter(torch.empty(spec.experts, width, spec.ff), requires_grad=False)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        ids, weights = self.router(x)
        n, d = x.shape
        if (n * self.spec.top <= K.MOE_GEMV_MAX_PAIRS or x.dtype != torch.bfloat16 or d % 8 or self.spec.ff % 8
                or not VENDOR_GROUPED_GEMM or not hasattr(torch, "_grouped_mm")):
            return K.moe_experts(x, ids, weights, self.w_up, self.w_down)   # this library's kernels only (always so in fp32)
        # many bf16 tokens: the two products go to the vendor's grouped GEMM (as the dense products go to its GEMM), over the
        # rows this library sorted by expert on the device -- no host round trip for the per-expert counts
        plan = K.moe_plan(ids, self.spec.experts)
        ends = plan.expert_off[1:]
        hidden = torch._grouped_mm(K.gather_rows(x, plan.slot_token), self.w_up.transpose(1, 2), offs=ends)
        y = torch._grouped_mm(K.sqrelu_(hidden), self.w_down.transpose(1, 2), offs=ends)
        return K.moe_combine(y, plan, weights)


class GatedSparseExperts(nn.Module):
    def __init__(self, width: int, spec: GatedMoESpec) -> None:
        super().__init__()
        self.spec = spec
        self.router = GroupLimitedRouter(width, spec.experts, spec.top, spec.groups, spec.keep, softmax=True, group_max=True, correction=False)
        self.w_up = nn.Parameter(torch.empty(spec.experts, 2 * spec.ff, width), requires_grad=False)   # per expert: ff gate rows, then ff up rows
        self.w_down = nn.Parameter(torch.empty(spec.experts, width, spec.ff), requires_grad=False)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        ids, weights = self.router(x)
        n, d = x.shape
        if (n * self.spec.top <= K.MOE_GEMV_MAX_PAIRS or x.dtype != torch.bfloat16 or d % 8 or self.spec.ff % 8
                or not VENDOR_GROUPED_GEMM or not hasattr(torch, "_grouped_mm")):
            return K.moe_experts(x, ids, weights, self.w_up, self.w_down, gated=True)
        plan = K.moe_plan(ids, self.spec.experts)
        ends = plan.expert_off[1:]
        both = torch._grouped_mm(K.gather_rows(x, plan.slot_token), self.w_up.transpose(1, 2), offs=ends)
        y = torch._grouped_mm(K.glu(both, K.ACT_SILU), self.w_down.transpose(1, 2), offs=ends)
        return K.moe_combine(y, plan, weights)


class ClampedGLU(nn.Module):
    """W_down (g sigmoid(alpha g) (u + 1)) with g = min(W_gate x, limit), u = clamp(W_up x, -limit, limit); gate and up rows stacked."""

    def __init__(self, width: int, ff: int, limit: float, alpha: float) -> None:
        super().__init__()
        self.limit, self.alpha = limit, alpha
        self.w_up = nn.Parameter(torch.empty(2 * ff, width), requires_grad=False)   # ff gate rows, then ff up rows
        self.w_down = nn.Parameter(torch.empty(width, ff), requires_grad=False)

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return torch.nn.functional.linear(K.glu_clamped(torch.nn.functional.linear(x, self.w_up), self.limit, self.alpha), self.w_down)


class ClampedSparseExperts(nn.Module):
    def __init__(self, width: int, spec: ClampedMoESpec) -> None:
        super().__init__()
        self.spec = spec
        self.router = GroupLimitedRouter(width, spec.experts, spec.top, softmax=False, topk_softmax=True, bias=True)
        self.w_up = nn.Parameter(torch.empty(spec.experts, 2 * spec.ff, width), requires_grad=False)   # per expert: ff gate rows, then ff up rows
        self.w_down = nn.Parameter(torch.empty(spec.experts, width, spec.ff), requires_grad=False)
        self.shared = ClampedGLU(width, spec.shared_ff, spec.shared_limit, spec.alpha) if spec.shared_ff else None

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        """The routed experts' weighted sum; the shared expert is the caller's to add (``self.shared(x)``)."""
        ids, weights = self.router(x)
        n, d = x.shape
        sp = self.spec
        if (n * sp.top <= K.MOE_GEMV_MAX_PAIRS or x.dtype != torch.bfloat16 or d % 8 or sp.ff % 8
                or not VENDOR_GROUPED_GEMM or not hasattr(torch, "_grouped_mm")):
            return K.moe_experts(x, ids, weights, self.w_up, self.w_down, gated=True, limit=sp.limit, alpha=sp.alpha)
        plan = K.moe_plan(ids, sp.experts)
        ends = plan.expert_off[1:]
        both = torch._grouped_mm(K.gather_rows(x, plan.slot_token), self.w_up.transpose(1, 2), offs=ends)
        y = torch._grouped_mm(K.glu_clamped(both, sp.limit, sp.alpha), self.w_down.transpose(1, 2), offs=ends)
        return K.moe_combine(y, plan, weights)


class SharedSparseExperts(nn.Module):
    def __init__(self, width: int, spec: SharedMoESpec) -> None:
        super().__init__()
        self.spec = spec
        E, ff, ffs = spec.experts, spec.ff, spec.shared_ff
        route_rows = E + (1 if ffs else 0)
        # the router's rows, then the row of the shared expert's gate, then zero rows up to a multiple of 8
        self.w_route = nn.Parameter(torch.empty(route_rows + -route_rows % 8, width), requires_grad=False)
        self.w_up = nn.Parameter(torch.empty(E, 2 * ff, width), requires_grad=False)   # per expert: ff gate rows, then ff up rows
        self.w_down = nn.Parameter(torch.empty(E, width, ff), requires_grad=False)
        self.shared_up = nn.Parameter(torch.empty(2 * ffs, width), requires_grad=False) if ffs else None
        self.shared_down = nn.Parameter(torch.empty(width, ffs), requires_grad=False) if ffs else None

    def route(self, x: torch.Tensor):
        """-> expert ids int32 (n, top), their weights fp32 (n, top), the shared expert's gate fp32 (n,) or None"""
        sp, shared = self.spec, self.shared_up is not None
        if sp.top <= 32 and sp.experts <= 3072:
            res = K.moe_route_logits(K.mm_f32(x, self.w_route), sp.experts, sp.top, gate=shared)
        else:
            res = K.moe_route(x, self.w_route[: sp.experts], None, sp.top, 1, 1, topk_softmax=True, gate_w=self.w_route[sp.experts] if shared else None)
        return res if shared else (*res, None)

    def terms(self, x: torch.Tensor) -> Dict[str, torch.Tensor]:
        """The parts of the feed-forward's result as keyword arguments of ``K.gated_residual``."""
        sp, (n, d) = self.spec, x.shape
        ids, weights, gate = self.route(x)
        few = n * sp.top <= K.MOE_GEMV_MAX_PAIRS
        if few and self.shared_up is not None:
            y0, y1 = K.moe_experts_shared(x, ids, weights, self.w_up, self.w_down, self.shared_up, self.shared_down)
            return dict(y0=y0, y1=y1, gate=gate)
        res: Dict[str, torch.Tensor] = {}
        if few or x.dtype != torch.bfloat16 or d % 8 or sp.ff % 8 or not VENDOR_GROUPED_GEMM or not hasattr(torch, "_grouped_mm"):
            res["y0"] = K.moe_experts(x, ids, weights, self.w_up, self.w_down, gated=True)
        else:
            plan = K.moe_plan(ids, sp.experts)
            ends = plan.expert_off[1:]
            both = torch._grouped_mm(K.gather_rows(x, plan.slot_token), self.w_up.transpose(1, 2), offs=ends)
            res["y0"] = torch._grouped_mm(K.glu(both, K.ACT_SILU), self.w_down.transpose(1, 2), offs=ends)
            res["slot_of"], res["wts"] = plan.slot_of, weights
        if self.shared_up is not None:
            hidden = K.glu(torch.nn.functional.linear(x, self.shared_up), K.ACT_SILU)
            res["y1"], res["gate"] = torch.nn.functional.linear(hidden, self.shared_down), gate
        return res


class DenseMLP(nn.Module):
    """W_down act(W_up x), act = the exact (erf) gelu unless another of ``K.ACT_*`` is named, or xIELU with its two learned numbers
    (``xielu=True``); the products are vendor GEMMs, the activation this library's kernel."""

    def __init__(self, width: int, ff: int, activation: int = K.ACT_GELU, xielu: bool = False) -> None:
        super().__init__()
        self.activation = activation
        self.w_up = nn.Parameter(torch.empty(ff, width), requires_grad=False)
        self.w_down = nn.Parameter(torch.empty(width, ff), requires_grad=False)
        self.act = nn.Parameter(torch.zeros(2), requires_grad=False) if xielu else None

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        hidden = torch.nn.functional.linear(x, self.w_up)
        hidden = K.xielu_(hidden, self.act) if self.act is not None else K.activation_(hidden, self.activation)
        return torch.nn.functional.linear(hidden, self.w_down)
