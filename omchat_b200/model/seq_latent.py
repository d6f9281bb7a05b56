"""Latent attention of the sequence-step decoders, host side: rotary tables, the work lists of the tensor-core kernel, and which kernel
attends (csrc/latent_attention.cu). Projections, norms and what is cached stay with the model.
"""
from __future__ import annotations

import json
from typing import Dict, List, Optional

import torch

from .. import seqlib
from ..config import RotarySpec


class RotaryTables:
    """fp32 (cos, sin) [positions, dims / 2, 2] per rotation, shared by the layers that turn alike; angles and functions are evaluated in
    double precision on the host. A table that grows leaves its predecessor alive: captured graphs hold its address."""

    def __init__(self, device):
        self.device = device
        self._tables: Dict[tuple, torch.Tensor] = {}
        self._outgrown: List[torch.Tensor] = []

    def get(self, rot: RotarySpec, positions: int) -> torch.Tensor:
        key = (rot.dims, rot.base, json.dumps(rot.scaling, sort_keys=True) if rot.scaling else None)
        t = self._tables.get(key)
        if t is None or t.shape[0] < positions:
            if t is not None:
                self._outgrown.append(t)
            n = max(positions, 1024)
            f, mult = rot.frequencies()
            ang = torch.arange(n, dtype=torch.float64)[:, None] * torch.tensor(f, dtype=torch.float64)[None, :]
            t = (torch.stack([ang.cos(), ang.sin()], dim=-1) * mult).to(torch.float32).contiguous().to(self.device)
            if t.numel() == 0:   # no rotated dimensions: the kernels still want a valid pointer
                t = torch.zeros(n, 1, 2, device=self.device)
            self._tables[key] = t
        return t


class LatentAttention:
    """Chooses the kernel and keeps the work lists. `plans` describes one step and collects its lists: {"portions": [...]} as the host
    knows the batch, {"decode_parts": n} or {"decode_keys": n} for a step of one row per request (the lists are then written on the
    device, in buffers that live as long as this object, so that a captured graph may use them), or None: the plain kernel."""

    def __init__(self, device, dtype: torch.dtype):
        self.device, self.dtype = device, dtype
        self.rotary = RotaryTables(device)
        self.tensor_attention = True    # False: the plain attention kernel for every shape (A/B, tests)
        self._decode_plans = {}         # (rows, heads, parts, window) -> seqlib.DecodeAttnPlan

    def _plan(self, plans: dict, T: int, H: int, window: int, pos, slot):
        plan = plans.get((H, window))
        if plan is None:
            if "portions" in plans:
                plan = seqlib.LatentAttnPlan(plans["portions"], H, self.device, window=window)
            else:
                parts = plans["decode_parts"] if "decode_parts" in plans else self._decode_parts(T, min(window, plans["decode_keys"]))
                key = (T, H, parts, window)
                plan = self._decode_plans.get(key)
                if plan is None:
                    plan = self._decode_plans[key] = seqlib.DecodeAttnPlan(T, H, parts, self.device, window=window)
                plan.fill(pos, slot)
            plans[(H, window)] = plan
        return plan

    @staticmethod
    def _decode_parts(T: int, keys: int) -> int:
        """Key ranges per row of a decode-only step: of 128 keys or more, of 64 where a short window would leave SMs without a CTA."""
        parts = seqlib.DecodeAttnPlan.parts_for(T, keys)
        return parts if T * parts >= 148 else seqlib.DecodeAttnPlan.parts_for(T, keys, min_keys=64)

    def attend(self, qcat: torch.Tensor, r: int, dr: int, pool: torch.Tensor, cache, pos, slot, plans: Optional[dict], scale: float, *,
               sink: Optional[torch.Tensor] = None, window: Optional[int] = None, gate: Optional[torch.Tensor] = None) -> torch.Tensor:
        """qcat [T, H, r + dr] (absorbed query | rotated query) -> [T, H, r], the weighted sums of cached latents, times
        sigmoid(gate [T, H]) with a gate."""
        T, H = qcat.shape[0], qcat.shape[1]
        window = seqlib.WINDOW_ALL if window is None else min(window, seqlib.WINDOW_ALL)
        if plans is not None and self.tensor_attention and seqlib.latent_attn_mma_ok(H, r, dr, self.dtype):
            out = torch.empty(T, H, r, device=qcat.device, dtype=self.dtype)
            return seqlib.latent_attn_mma(qcat, r, dr, pool, cache.block_table, cache.page_size, self._plan(plans, T, H, window, pos, slot), sink, scale,
                                          out, window=window, gate=gate)
        out = torch.empty(T, H, r, device=qcat.device, dtype=torch.float32)
        return seqlib.latent_attn(qcat, r, dr, pool, cache.block_table, cache.page_size, pos, slot, sink, scale, out, window=window, gate=gate)
