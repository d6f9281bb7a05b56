"""Munevik restated on the CPU in float64, one function per mechanism, token loops where the design has a recurrence.

Test infrastructure only: nothing here is imported by the product, and nothing of the product is imported here. The functions take
plain tensors (a checkpoint's state dict under its own names) and the config.json dictionary.

Notation: T tokens of ONE sequence at positions 0..T-1, C the width, rows are tokens.
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

F64 = torch.float64


# ------------------------------------------------------------------------------------------------------------ small pieces
def lin(x: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    y = x @ w.to(F64).T
    return y if b is None else y + b.to(F64)


def layer_norm(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor, eps: float) -> torch.Tensor:
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w.to(F64) + b.to(F64)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps) * w.to(F64)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def shift_conv(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """y_t = b + sum_j w[:, j] u_(t - taps + 1 + j) per channel, zeros before the start. u [T, ch], w [ch, taps]."""
    T, taps = u.shape[0], w.shape[1]
    y = b.to(F64).expand(T, -1).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            y[back:] += w[:, j].to(F64) * u[:T - back]
    return y


def rotate_pairs(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, ..., d]: the pair (2i, 2i + 1), i < dims / 2, turns by pos * base^(-2i / dims); the other dimensions pass."""
    out = x.clone()
    view = (-1,) + (1,) * (x.dim() - 2)
    for i in range(dims // 2):
        a = pos.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).view(view), torch.sin(a).view(view)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def window_mask(T: int, size: Optional[int]) -> torch.Tensor:
    """bool [T, T]: row i may see column j."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    ok = d >= 0
    return ok if size is None else ok & (d < size)


# ------------------------------------------------------------------------------------------------------------------ mixers
def latent_rows(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float):
    """What a layer with a down-projection caches per token: the normed latent [T, r] and the rotated key part [T, dr]."""
    z = lin(h, W[p + "dkv"])
    r = m["kv_rank"]
    c = rms_norm(z[:, :r], W[p + "dkv.norm"], eps)
    return c, rotate_pairs(z[:, r:], torch.arange(h.shape[0]), m["rot"]["dims"], m["rot"]["base"])


def latent_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, c: torch.Tensor, k_rot: torch.Tensor) -> torch.Tensor:
    T = h.shape[0]
    H, dn, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = lin(h, W[p + "q"]).view(T, H, dn + dr)
    qn, qr = q[..., :dn], rotate_pairs(q[..., dn:], torch.arange(T), m["rot"]["dims"], m["rot"]["base"])
    k = lin(c, W[p + "uk"]).view(T, H, dn)
    v = lin(c, W[p + "uv"]).view(T, H, dv)
    ok = window_mask(T, (m.get("mask") or {}).get("size"))
    gate = torch.sigmoid(lin(h, W[p + "g"]))                                   # [T, H]
    out = torch.zeros(T, H, dv, dtype=F64)
    for i in range(H):
        s = (qn[:, i] @ k[:, i].T + qr[:, i] @ k_rot.T) * m["scale"]
        out[:, i] = torch.softmax(s.masked_fill(~ok, -math.inf), dim=-1) @ v[:, i] * gate[:, i:i + 1]
    return lin(out.reshape(T, H * dv), W[p + "o"])


def rglru_recurrence(u: torch.Tensor, r: torch.Tensor, i: torch.Tensor, lam: torch.Tensor) -> torch.Tensor:
    """u, r, i [T, width] -> the states after every token [T, width], from a zero state."""
    log_a = -8.0 * r * softplus(lam.to(F64))
    a, mult = torch.exp(log_a), torch.sqrt(-torch.expm1(2.0 * log_a))
    S, out = torch.zeros(u.shape[1], dtype=F64), torch.zeros_like(u)
    for t in range(u.shape[0]):
        S = a[t] * S + mult[t] * i[t] * u[t]
        out[t] = S
    return out


def block_gate(u: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """w [blocks, n, n] ([out, in]), b [blocks, n]: every part of u passes a matrix of its own, then a sigmoid."""
    n = w.shape[1]
    return torch.cat([torch.sigmoid(lin(u[:, j * n:(j + 1) * n], w[j], b[j])) for j in range(w.shape[0])], dim=1)


def rglru(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
    y = gelu_tanh(lin(h, W[p + "y"], W[p + "y.b"]))
    u = shift_conv(lin(h, W[p + "x"], W[p + "x.b"]), W[p + "conv"], W[p + "conv.b"])
    S = rglru_recurrence(u, block_gate(u, W[p + "ra"], W[p + "ra.b"]), block_gate(u, W[p + "ri"], W[p + "ri.b"]), W[p + "lam"])
    return lin(S * y, W[p + "o"])


# ------------------------------------------------------------------------------------------------------------ feed-forward
def clamped_mlp(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
    lim = m["limit"]
    g = torch.clamp(lin(h, W[p + "gate"]), max=lim)
    u = torch.clamp(lin(h, W[p + "up"]), min=-lim, max=lim)
    return lin(g * torch.sigmoid(1.702 * g) * (u + 1.0), W[p + "down"])


def silu_expert(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(silu(lin(h, W[p + "gate"])) * lin(h, W[p + "up"]), W[p + "down"])


def group_limited_choice(s: List[float], top: int, groups: Optional[dict]) -> List[int]:
    """Scores of one token -> the chosen experts, best first; ties go to the lower index."""
    E = len(s)
    allowed = list(range(E))
    if groups:
        n = E // groups["count"]
        gs = [sum(sorted(s[g * n:(g + 1) * n], reverse=True)[:2]) for g in range(groups["count"])]
        kept = set(sorted(range(groups["count"]), key=lambda g: (-gs[g], g))[:groups["keep"]])
        allowed = [e for e in range(E) if e // n in kept]
    return sorted(allowed, key=lambda e: (-s[e], e))[:top]


def moe(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict) -> torch.Tensor:
    r = m["router"]
    s = torch.sigmoid(lin(h, W[p + "router"]))
    out = silu_expert(h, W, p + "shared.") if m.get("shared") else torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e in group_limited_choice(s[t].tolist(), r["top"], r.get("groups")):
            out[t] += r.get("scale", 1.0) * s[t, e] * silu_expert(h[t:t + 1], W, f"{p}e{e}.")[0]
    return out


# ------------------------------------------------------------------------------------------------------------------- model
def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int], collect: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one sequence. collect: receives the stream after every layer."""
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = W["embed"].to(F64)[torch.tensor(tokens, dtype=torch.long)]
    cached = {}
    for i, layer in enumerate(cfg["layers"]):
        n, m, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
        if layer["type"] == "latent_attention":
            src = m["kv_from"] if m.get("kv_from") is not None else i
            if src == i:
                cached[i] = latent_rows(x, W, n + "mix.", m, eps)
            y = latent_attention(x, W, n + "mix.", m, *cached[src])
        elif layer["type"] == "rglru":
            y = rglru(x, W, n + "mix.", m)
        else:
            raise ValueError(layer["type"])
        x = layer_norm(alpha * x + y, W[n + "norm1"], W[n + "norm1.b"], eps)
        if mlp:
            y = clamped_mlp(x, W, n + "mlp.", mlp) if mlp["kind"] == "dense" else moe(x, W, n + "mlp.", mlp)
            x = layer_norm(alpha * x + y, W[n + "norm2"], W[n + "norm2.b"], eps)
        if collect is not None:
            collect.append(x)
    return lin(layer_norm(x, W["final.norm"], W["final.norm.b"], eps), W["embed"])
