"""Plain, slow restatement of the Votavik design in torch, one function per mechanism, for the tests to compare the framework
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
GLU_SLOPE = 1.702


def rms(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w


def layer_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    c = x - x.mean(dim=-1, keepdim=True)
    return c / torch.sqrt((c * c).mean(dim=-1, keepdim=True) + eps) * w


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def rotate_half(x: torch.Tensor, rot: Optional[dict], first_position: int = 0) -> torch.Tensor:
    """x (T, heads, dk): dimensions (i, i + n / 2) of the first n = rot.dims turned by position * base^(-2 i / n)."""
    if not rot or rot["dims"] == 0:
        return x
    n = rot["dims"]
    out = x.clone()
    for i in range(n // 2):
        f = rot["base"] ** (-2.0 * i / n)
        for t in range(x.shape[0]):
            a = (first_position + t) * f
            u, v = x[t, :, i], x[t, :, i + n // 2]
            out[t, :, i] = u * math.cos(a) - v * math.sin(a)
            out[t, :, i + n // 2] = v * math.cos(a) + u * math.sin(a)
    return out


def visible(i: int, mask: dict) -> List[int]:
    """Positions that position i sees: the window that ends at i, and the first tokens of the sequence."""
    return [j for j in range(i + 1) if i - j < mask["size"] or j < mask["keep_first"]]


def capped_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, sink: Optional[torch.Tensor], mask: dict, scale: float,
                     cap: float) -> torch.Tensor:
    """q (T, H, dk), k (T, G, dk), v (T, G, dv) -> (T, H, dv)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=F64)
    for i in range(T):
        js = torch.tensor(visible(i, mask))
        for h in range(H):
            g = h // (H // G)
            s = (k[js, g] @ q[i, h]) * scale
            if cap:
                s = cap * torch.tanh(s / cap)
            top = s.max()
            e = torch.exp(s - top)
            den = e.sum() + (torch.exp(sink[h] - top) if sink is not None else 0.0)
            out[i, h] = (e / den) @ v[js, g]
    return out


def attention_mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, dk, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ W[p + "q"].T, W[p + "q.norm"], eps).view(T, H, dk)      # one norm over all heads at once
    k = rms(h @ W[p + "k"].T, W[p + "k.norm"], eps).view(T, G, dk)
    v = (h @ W[p + "v"].T).view(T, G, dv)
    q, k = rotate_half(q, m.get("rot")), rotate_half(k, m.get("rot"))
    o = capped_attention(q, k, v, W[p + "sink"], m["mask"], m["scale"], m["softcap"])
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ W[p + "o"].T


def decayed_sum(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, decay: torch.Tensor) -> torch.Tensor:
    """One head.  q, k (T, dk), v (T, dv), decay (T, dk): per token S <- diag(decay) S + k v^T, then o = S^T q."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=F64)
    o = torch.zeros(k.shape[0], v.shape[1], dtype=F64)
    for t in range(k.shape[0]):
        S = decay[t][:, None] * S + torch.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o


def gla_mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, dk) / math.sqrt(dk)
    k = (h @ W[p + "k"].T).view(T, H, dk)
    v = (h @ W[p + "v"].T).view(T, H, dv)
    z = ((h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]).view(T, H, dk)
    decay = torch.sigmoid(z) ** (1.0 / m["tau"])
    o = torch.stack([decayed_sum(q[:, j], k[:, j], v[:, j], decay[:, j]) for j in range(H)], dim=1)
    o = rms(o, W[p + "norm"], eps).reshape(T, H * dv)                   # per head, one weight for all heads
    return (o * silu(h @ W[p + "g"].T)) @ W[p + "o"].T


def lightning_mixer(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = silu(h @ W[p + "q"].T).view(T, H, dk)
    k = silu(h @ W[p + "k"].T).view(T, H, dk)
    v = silu(h @ W[p + "v"].T).view(T, H, dv)
    o = torch.stack([decayed_sum(q[:, j], k[:, j], v[:, j], torch.full((T, dk), m["decay"][j], dtype=F64)) for j in range(H)], dim=1)
    o = rms(o.reshape(T, H * dv), W[p + "norm"], eps)                   # all heads together
    return (o * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def clamped_glu(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, f: dict) -> torch.Tensor:
    g = (h @ W[p + "gate"].T).clamp(max=f["limit"])
    u = (h @ W[p + "up"].T).clamp(min=-f["limit"], max=f["limit"])
    return (g * torch.sigmoid(GLU_SLOPE * g) * (u + 1)) @ W[p + "down"].T


def token_input(x: torch.Tensor, e: torch.Tensor, W: Dict[str, torch.Tensor], p: str, eps: float) -> torch.Tensor:
    """What a layer's own token embedding e (T, n), gated by the stream x (T, d), adds to the stream."""
    return rms((gelu_tanh(x @ W[p + "gate"].T) * e) @ W[p + "proj"].T, W[p + "norm"], eps)


MIXERS = {"attention": attention_mixer, "gla": gla_mixer, "lightning": lightning_mixer}


def forward(cfg: dict, weights: Dict[str, torch.Tensor], tokens: List[int], return_layers: bool = False):
    """-> logits (T, vocab) in float64 (and the residual stream after every layer)."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps, n = cfg["norm"]["eps"], cfg["token_side"]["dim"]
    ids = torch.tensor(tokens, dtype=torch.long)
    x, side = W["embed"][ids], W["side.embed"][ids]
    seen = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](layer_norm(x, W[p + "norm1"], eps), W, p + "mix.", layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + clamped_glu(layer_norm(x, W[p + "norm2"], eps), W, p + "mlp.", layer["mlp"])
        x = x + token_input(x, side[:, i * n : (i + 1) * n], W, p + "side.", eps)
        seen.append(x.clone())
    logits = layer_norm(x, W["final.norm"], eps) @ W["head"].T
    return (logits, seen) if return_layers else logits


def greedy(cfg: dict, weights: Dict[str, torch.Tensor], prompt: List[int], new_tokens: int) -> List[int]:
    """prompt + greedily chosen continuation, recomputing everything for every token."""
    seq = list(prompt)
    for _ in range(new_tokens):
        seq.append(int(forward(cfg, weights, seq)[-1].argmax()))
    return seq
