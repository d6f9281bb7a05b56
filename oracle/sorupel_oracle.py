"""Sorupel restated on the CPU in float64, one function per mechanism, token loops where the design has a recurrence.

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
def lin(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    return x @ w.to(F64).T


def unit_rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    return unit_rms(x, eps) * w.to(F64)


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


def rotate_halves(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x [T, ..., d]: dimensions i and i + dims / 2, i < dims / 2, turn by pos * base^(-2i / dims); those from dims on pass."""
    out = x.clone()
    view = (-1,) + (1,) * (x.dim() - 2)
    h = dims // 2
    for i in range(h):
        a = pos.to(F64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).view(view), torch.sin(a).view(view)
        u, v = x[..., i], x[..., i + h]
        out[..., i] = u * c - v * s
        out[..., i + h] = v * c + u * s
    return out


def causal_mask(T: int, chunk: Optional[int] = None) -> torch.Tensor:
    """bool [T, T]: row i may see column j (with chunks: of its own chunk only)."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    ok = j <= i
    return ok if chunk is None else ok & (i // chunk == j // chunk)


def sink_softmax(s: torch.Tensor, ok: torch.Tensor, sink: float) -> torch.Tensor:
    """Weights of the visible columns when one more term exp(sink) stands in the denominator."""
    s = s.masked_fill(~ok, -math.inf)
    full = torch.cat([s, torch.full((s.shape[0], 1), float(sink), dtype=F64)], dim=1)
    return torch.softmax(full, dim=1)[:, :-1]


# --------------------------------------------------------------------------------------------------------------- embedding
def bigram_rows(tokens: List[int], buckets: int, mul_prev: int, mul_cur: int) -> List[int]:
    return [buckets] + [(p * mul_prev + c * mul_cur) % buckets for p, c in zip(tokens[:-1], tokens[1:])]


def embedding(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int]) -> torch.Tensor:
    x = W["embed"].to(F64)[torch.tensor(tokens, dtype=torch.long)]
    b = (cfg.get("embedding") or {}).get("bigram")
    if b:
        x = x + W["bigram"].to(F64)[torch.tensor(bigram_rows(tokens, b["buckets"], b["mul_prev"], b["mul_cur"]))]
    return x


# ------------------------------------------------------------------------------------------------------------------ mixers
def latent_rows(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float):
    """What a layer with a down-projection caches per token: the normed latent [T, r] and the rotated key part [T, dr]."""
    z = lin(h, W[p + "dkv"])
    r = m["kv_rank"]
    c = rms_norm(z[:, :r], W[p + "dkv.norm"], eps)
    return c, rotate_halves(z[:, r:], torch.arange(h.shape[0]), m["rot"]["dims"], m["rot"]["base"])


def latent_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, c: torch.Tensor, k_rot: torch.Tensor) -> torch.Tensor:
    T = h.shape[0]
    H, dn, dr, dv = m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = lin(h, W[p + "q"]).view(T, H, dn + dr)
    qn, qr = q[..., :dn], rotate_halves(q[..., dn:], torch.arange(T), m["rot"]["dims"], m["rot"]["base"])
    k = lin(c, W[p + "uk"]).view(T, H, dn)
    v = lin(c, W[p + "uv"]).view(T, H, dv)
    ok = causal_mask(T)
    out = torch.zeros(T, H, dv, dtype=F64)
    for i in range(H):
        s = (qn[:, i] @ k[:, i].T + qr[:, i] @ k_rot.T) * m["scale"]
        out[:, i] = sink_softmax(s, ok, float(W[p + "sink"][i])) @ v[:, i]
    return lin(out.reshape(T, H * dv) * torch.sigmoid(lin(h, W[p + "g"])), W[p + "o"])


def chunk_attention(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q, k = lin(h, W[p + "q"]), lin(h, W[p + "k"])
    v = k.view(T, G, d)
    pos, rot = torch.arange(T), m["rot"]
    q = rotate_halves(rms_norm(q, W[p + "q.norm"], eps).view(T, H, d), pos, rot["dims"], rot["base"])
    k = rotate_halves(rms_norm(k, W[p + "k.norm"], eps).view(T, G, d), pos, rot["dims"], rot["base"])
    gate = torch.sigmoid(lin(h, W[p + "g"]))
    ok = causal_mask(T, (m.get("mask") or {}).get("size"))
    out = torch.zeros(T, H, d, dtype=F64)
    for i in range(H):
        g = i // (H // G)
        s = (q[:, i] @ k[:, g].T) * m["scale"]
        if m.get("softcap"):
            s = m["softcap"] * torch.tanh(s / m["softcap"])
        out[:, i] = sink_softmax(s, ok, 0.0) @ v[:, g] * gate[:, i:i + 1]
    return lin(out.reshape(T, H * d), W[p + "o"])


def ssd_recurrence(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, A_log: torch.Tensor, D: torch.Tensor) -> torch.Tensor:
    """x [T, H, P], B / C [T, G, N], dt [T, H] (after softplus) -> y [T, H, P]; the state starts at zero."""
    T, H, P = x.shape
    G, N = B.shape[1:]
    y = torch.zeros_like(x)
    grp = torch.tensor([h // (H // G) for h in range(H)])
    S = torch.zeros(H, N, P, dtype=F64)
    A = torch.exp(A_log.to(F64))
    for t in range(T):
        S = torch.exp(-A * dt[t])[:, None, None] * S + dt[t][:, None, None] * B[t, grp][:, :, None] * x[t][:, None, :]
        y[t] = (S * C[t, grp][:, :, None]).sum(1) + D.to(F64)[:, None] * x[t]
    return y


def mamba2(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(lin(h, W[p + "in"]), [inner, inner + 2 * G * N, H], dim=1)
    xbc = silu(shift_conv(xbc, W[p + "conv"], W[p + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    dt = softplus(dt + W[p + "dt_bias"].to(F64))
    y = ssd_recurrence(x.view(T, H, P), B.view(T, G, N), C.view(T, G, N), dt, W[p + "A_log"], W[p + "D"]).reshape(T, inner)
    y = unit_rms((y * silu(z)).view(T, m["norm_groups"], -1), eps).reshape(T, inner) * W[p + "norm"].to(F64)
    return lin(y, W[p + "o"])


# ------------------------------------------------------------------------------------------------------------ feed-forward
def gated_mlp(h: torch.Tensor, W: Dict[str, torch.Tensor], p: str) -> torch.Tensor:
    return lin(gelu_tanh(lin(h, W[p + "gate"])) * lin(h, W[p + "up"]), W[p + "down"])


# ------------------------------------------------------------------------------------------------------------------- model
def forward(cfg: dict, W: Dict[str, torch.Tensor], tokens: List[int], collect: Optional[list] = None) -> torch.Tensor:
    """Logits [T, vocab] (float64) of one sequence. collect: receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = embedding(cfg, W, tokens)
    cached = {}
    for i, layer in enumerate(cfg["layers"]):
        n, m = f"l{i}.", layer["mixer"]
        h = rms_norm(x, W[n + "norm1"], eps)
        if layer["type"] == "latent_attention":
            src = m["kv_from"] if m.get("kv_from") is not None else i
            if src == i:
                cached[i] = latent_rows(h, W, n + "mix.", m, eps)
            y = latent_attention(h, W, n + "mix.", m, *cached[src])
        elif layer["type"] == "mamba2":
            y = mamba2(h, W, n + "mix.", m, eps)
        elif layer["type"] == "attention":
            y = chunk_attention(h, W, n + "mix.", m, eps)
        else:
            raise ValueError(layer["type"])
        x = x + y
        if layer.get("mlp"):
            x = x + gated_mlp(rms_norm(x, W[n + "norm2"], eps), W, n + "mlp.")
        if collect is not None:
            collect.append(x)
    return lin(rms_norm(x, W["final.norm"], eps), W["head"])
