"""Plain, slow restatement of the Fovirax design in torch, one function per mechanism, for the tests to compare the framework
against.  It shares no code with the package: it takes the parsed ``config.json`` dictionary and a ``{tensor name: tensor}``
dictionary and recomputes every position from the whole token list (no state, no batch).

Everything runs in float64 on the CPU: the comparison tolerances of the tests are what the framework's bfloat16 / float32
arithmetic may lose against exact arithmetic.

Notation: ``T`` tokens, ``d`` width, ``H`` heads, ``G`` key / value heads, ``dk`` / ``dv`` per-head key / value sizes.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


def over_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """A weight of zero leaves the normed row as it is."""
    return over_rms(x, eps) * (1 + w)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def frequency(i: int, rot: dict) -> float:
    """Angular frequency of pair i; with a scaling, long wavelengths are stretched by its factor, short ones kept, those between
    blended by where original / wavelength lies between the two bounds."""
    f = rot["base"] ** (-2.0 * i / rot["dims"])
    sc = rot.get("scaling")
    if not sc:
        return f
    turns = sc["original"] * f / (2 * math.pi)          # original / wavelength
    if turns > sc["high"]:
        return f
    if turns < sc["low"]:
        return f / sc["factor"]
    s = (turns - sc["low"]) / (sc["high"] - sc["low"])
    return (1 - s) * f / sc["factor"] + s * f


def rotate_half(x: torch.Tensor, rot: Optional[dict], first_position: int = 0) -> torch.Tensor:
    """x (T, heads, dk): dimensions (i, i + n / 2) of the first n = rot.dims turned by position * frequency(i)."""
    if not rot or rot["dims"] == 0:
        return x
    n = rot["dims"]
    out = x.clone()
    pos = torch.arange(first_position, first_position + x.shape[0], dtype=F64)
    for i in range(n // 2):
        a = (pos * frequency(i, rot))[:, None]
        u, v = x[:, :, i], x[:, :, i + n // 2]
        out[:, :, i] = u * torch.cos(a) - v * torch.sin(a)
        out[:, :, i + n // 2] = v * torch.cos(a) + u * torch.sin(a)
    return out


def capped_window_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, window: int, scale: float, cap: float) -> torch.Tensor:
    """q (T, H, dk), k (T, G, dk), v (T, G, dv) -> (T, H, dv)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        lo = max(0, i - window + 1)
        for g in range(G):
            hs = slice(g * (H // G), (g + 1) * (H // G))
            s = q[i, hs] @ k[lo : i + 1, g].T * scale
            if cap:
                s = cap * torch.tanh(s / cap)
            out[i, hs] = torch.softmax(s, dim=-1) @ v[lo : i + 1, g]
    return out


def attention_branch(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate_half((h @ W[p + "q"].T).view(T, H, dk), m.get("rot"))
    k = rotate_half((h @ W[p + "k"].T).view(T, G, dk), m.get("rot"))
    v = (h @ W[p + "v"].T).view(T, G, dv)
    o = capped_window_attention(q, k, v, m["mask"]["size"], m["scale"], m.get("softcap") or 0.0)
    return o.reshape(T, H * dv) @ W[p + "o"].T


def retained_sum(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor) -> torch.Tensor:
    """q, k (T, H, dk), v (T, H, dv), decay (H): per token and head S <- decay S + k v^T, then o = S^T q."""
    T, H, dk = k.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=F64)
    o = torch.zeros(T, H, v.shape[2], dtype=F64)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = (S * q[t][:, :, None]).sum(dim=1)
    return o


def retention_branch(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate_half((h @ W[p + "q"].T).view(T, H, dk), m.get("rot"))
    k = rotate_half((h @ W[p + "k"].T).view(T, H, dk), m.get("rot")) / math.sqrt(dk)
    v = (h @ W[p + "v"].T).view(T, H, dv)
    o = over_rms(retained_sum(q, k, v, torch.tensor(m["decay"], dtype=F64)), eps).reshape(T, H * dv)
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def parallel_mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    return m["left_scale"] * attention_branch(h, W, p + "left.", m["left"]) + m["right_scale"] * retention_branch(h, W, p + "right.", m["right"], eps)


def expert(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def mixture(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, f: dict) -> torch.Tensor:
    """The `top` experts of largest router logits, weighted by a softmax among those logits, and the gated shared expert."""
    z = h @ W[p + "router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        best = sorted(range(f["router"]["experts"]), key=lambda e: (-z[t, e].item(), e))[: f["router"]["top"]]
        for e, w in zip(best, torch.softmax(z[t, best], dim=0)):
            out[t] += w * expert(h[t], W, f"{p}e{e}.")
    if f.get("shared"):
        out = out + torch.sigmoid(h @ W[p + "shared.sg"].T) * expert(h, W, p + "shared.")
    return out


def run_order(cfg: dict) -> List[int]:
    loop, n = cfg.get("loop"), len(cfg["layers"])
    if not loop:
        return list(range(n))
    return list(range(loop["start"])) + list(range(loop["start"], loop["stop"])) * loop["times"] + list(range(loop["stop"], n))


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], return_layers: bool = False):
    """-> logits (T, vocab) in float64 (and the residual stream after every layer run)."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    seen = []
    for i in run_order(cfg):
        layer, p = cfg["layers"][i], f"l{i}."
        x = x + mult * W[p + "ls1"] * parallel_mixer(norm(x, W[p + "norm1"], eps), W, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + mult * W[p + "ls2"] * mixture(norm(x, W[p + "norm2"], eps), W, p + "mlp.", layer["mlp"])
        seen.append(x.clone())
    logits = norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, seen) if return_layers else logits


def greedy(cfg: dict, weights: Dict[str, torch.Tensor], prompt: List[int], new_tokens: int) -> List[int]:
    """prompt + greedily chosen continuation, recomputing everything for every token."""
    seq = list(prompt)
    for _ in range(new_tokens):
        seq.append(int(forward(cfg, weights, seq)[-1].argmax()))
    return seq
