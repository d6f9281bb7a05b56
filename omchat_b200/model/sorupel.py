"""Sorupel: a decoder-only language model of latent-attention layers (some of which attend to another layer's cached rows), state-space
layers with one step size per head, and chunked attention whose values are its keys, each with a dense gated feed-forward or none, over
an embedding that a second row chosen by the pair (previous token, token) is added to.

A sublayer reads an RMS norm of the stream: x <- x + mixer(N1(x)); x <- x + ff(N2(x)). The stream is fp32 on the device; the norm that a
sublayer reads is formed in the launch that adds the sublayer before it.

Mixers. Latent attention (config.LatentAttentionSpec, model/seq_latent.py): keys / values are up-projections of a cached latent plus one
rotated key part, absorbed into the query and the output; a sink in the softmax, a sigmoid gate per element of the concatenated heads; a
layer with kv_from attends to that layer's rows and caches nothing. State space (config.StateSpaceSpec): [z | x | B | C | dt] from one
projection, a causal convolution + silu over x, B, C, the recurrence, silu(z) and an RMS norm in equal parts. Chunked attention
(config.ChunkAttentionSpec): queries and keys normed over their whole projection and rotated, keys as projected for values, a soft cap,
one added to the softmax denominator, a sigmoid gate per head.

Like the other sequence-step decoders the model owns no cache and no loop: `step()` runs ONE packed batch of rows - portions of prompts
beside single decoded tokens, each row addressed by (slot, position) - against a PagedStateCache that the caller
(serving.StepScheduler) manages: pages of latents and of keys and values, per-slot fp32 states and convolution rings, the last token.
`generate()` goes through that scheduler; decode-only steps replay from a CUDA graph (seq_model.py).

Kernels: omc_embed_bigram (rows + first norm), omc_latent_rope_store, omc_latent_attn / omc_latent_attn_mma with sink, omc_linear_gate,
omc_causal_conv (bias + silu), omc_linear_state_scan (step sizes), omc_gate_rms_rows, omc_qk_norm_kv_store with rotation, omc_window_attn /
omc_window_attn_mma with chunks, sink and head gate, omc_glu_mul, omc_rms_residual.

Compute dtype bfloat16: bf16 matrix operands with fp32 accumulation, bf16 cache rows; angles, scores and softmax, norms, stream, states and
everything that enters the recurrence in fp32. Compute dtype float32: everything in fp32 on the FMA pipe.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence

import torch

from .. import lib, seqlib
from ..config import ChunkAttentionSpec, LatentAttentionSpec, SorupelConfig, StateSpaceSpec
from .paged_cache import PagedStateCache
from .seq_latent import LatentAttention
from .seq_linear import NARROW_GEMM_MIN_WEIGHT, dense_linear, stack_rows
from .seq_model import GraphedDecodeMixin, SequenceStepLM, portion_starts


# ------------------------------------------------------------------------------------------------------------------- weights
@dataclass
class LatentW:
    w_in: torch.Tensor             # [q | output gate | dkv (own rows only) | zero rows, C]
    nq: int                        # rows of q: H * (dim + rot_dim)
    ng: int                        # rows of the gate: H * vdim
    dkv_norm: Optional[torch.Tensor]
    uk_t: torch.Tensor             # [H, kv_rank, dim]: per head W_uk^T, the absorbing projection of the unrotated query
    uv: torch.Tensor               # [H * vdim, kv_rank]
    sink: torch.Tensor             # fp32 [H]
    o: torch.Tensor                # [C, H * vdim]


@dataclass
class StateSpaceW:
    w_in: torch.Tensor             # [z | x | B | C | dt | zero rows, C]
    conv: torch.Tensor             # [inner + 2 groups state, taps]
    conv_b: torch.Tensor
    dt_bias: torch.Tensor          # fp32 [heads]
    A_log: torch.Tensor            # fp32 [heads]
    D: torch.Tensor                # fp32 [heads]
    norm: torch.Tensor             # [inner]
    o: torch.Tensor                # [C, inner]


@dataclass
class ChunkAttentionW:
    w_in: torch.Tensor             # [q | k | head gate | zero rows, C]
    cols: Dict[str, slice]         # 'q', 'k', 'g': columns of w_in's output
    q_norm: torch.Tensor           # [H * dim]
    k_norm: torch.Tensor           # [G * dim]
    one: torch.Tensor              # fp32 [H] of zeros: the sink whose term in the denominator is 1
    o: torch.Tensor                # [C, H * dim]


@dataclass
class DenseMlpW:
    gate_up: torch.Tensor          # [2 ff, C]
    down: torch.Tensor             # [C, ff]


@dataclass
class SorupelLayerW:
    norm1: torch.Tensor
    norm2: Optional[torch.Tensor]
    mix: object
    mlp: Optional[DenseMlpW]


@dataclass
class SorupelW:
    embed: torch.Tensor
    bigram: Optional[torch.Tensor]
    final_norm: torch.Tensor
    head: torch.Tensor
    layers: List[SorupelLayerW]


def weights_from_state_dict(sd: Dict[str, torch.Tensor], cfg: SorupelConfig, device, dtype: torch.dtype) -> SorupelW:
    """Checkpoint names: 'embed', 'bigram', 'final.norm', 'head', per layer i 'l<i>.norm1|norm2', 'l<i>.mix.*', 'l<i>.mlp.*'; linear weights
    [out, in]. Load-time re-layouts: one stacked input projection per mixer, W_uk transposed per head, gate and up stacked. Shapes are
    checked against the config."""
    f32 = torch.float32

    def g(name, shape, dt=dtype):
        if name not in sd:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        if tuple(sd[name].shape) != tuple(shape):
            raise ValueError(f"{name} has shape {tuple(sd[name].shape)}, the config says {tuple(shape)}")
        return sd[name].to(device=device, dtype=dt).contiguous()

    C = cfg.hidden_size
    layers = []
    for i, spec in enumerate(cfg.layers):
        m, p = spec.mixer, f"l{i}.mix."
        if isinstance(m, LatentAttentionSpec):
            H, dn, r, nq, ng = m.heads, m.dim, m.kv_rank, m.heads * (m.dim + m.rot_dim), m.heads * m.vdim
            own = m.kv_from is None
            parts = [("q", g(p + "q", (nq, C))), ("g", g(p + "g", (ng, C)))]
            if own:
                parts.append(("dkv", g(p + "dkv", (r + m.rot_dim, C))))
            mix = LatentW(w_in=stack_rows(parts)[0], nq=nq, ng=ng, dkv_norm=g(p + "dkv.norm", (r,)) if own else None,
                          uk_t=g(p + "uk", (H * dn, r)).view(H, dn, r).transpose(1, 2).contiguous(), uv=g(p + "uv", (ng, r)),
                          sink=g(p + "sink", (H,), f32), o=g(p + "o", (C, ng)))
        elif isinstance(m, StateSpaceSpec):
            ch = m.conv_channels
            w_in, _ = stack_rows([("in", g(p + "in", (m.inner + ch + m.heads, C)))])
            mix = StateSpaceW(w_in=w_in, conv=g(p + "conv", (ch, m.conv)), conv_b=g(p + "conv.b", (ch,)), dt_bias=g(p + "dt_bias", (m.heads,), f32),
                              A_log=g(p + "A_log", (m.heads,), f32), D=g(p + "D", (m.heads,), f32), norm=g(p + "norm", (m.inner,)),
                              o=g(p + "o", (C, m.inner)))
        else:
            assert isinstance(m, ChunkAttentionSpec)
            nq, nk = m.heads * m.dim, m.kv_heads * m.dim
            w_in, cols = stack_rows([("q", g(p + "q", (nq, C))), ("k", g(p + "k", (nk, C))), ("g", g(p + "g", (m.heads, C)))])
            mix = ChunkAttentionW(w_in=w_in, cols=cols, q_norm=g(p + "q.norm", (nq,)), k_norm=g(p + "k.norm", (nk,)),
                                  one=torch.zeros(m.heads, device=device, dtype=f32), o=g(p + "o", (C, nq)))
        s, q, mlp = spec.mlp, f"l{i}.mlp.", None
        if s is not None:
            mlp = DenseMlpW(gate_up=torch.cat([g(q + "gate", (s.ff, C)), g(q + "up", (s.ff, C))], dim=0), down=g(q + "down", (C, s.ff)))
        layers.append(SorupelLayerW(norm1=g(f"l{i}.norm1", (C,)), norm2=g(f"l{i}.norm2", (C,)) if s is not None else None, mix=mix, mlp=mlp))
    return SorupelW(embed=g("embed", (cfg.vocab_size, C)), bigram=g("bigram", (cfg.bigram.buckets + 1, C)) if cfg.bigram is not None else None,
                    final_norm=g("final.norm", (C,)), head=g("head", (cfg.vocab_size, C)), layers=layers)


def random_state_dict(cfg: SorupelConfig, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16 weights under the checkpoint names (benchmarks, tests)."""
    gen = torch.Generator().manual_seed(seed)

    def rn(*shape, s=1.0, mean=0.0):
        return (torch.randn(shape, generator=gen) * s + mean).to(torch.bfloat16)

    C, sd = cfg.hidden_size, {}
    sd["embed"], sd["head"], sd["final.norm"] = rn(cfg.vocab_size, C), rn(cfg.vocab_size, C, s=C ** -0.5), rn(C, s=0.2, mean=1.0)
    if cfg.bigram is not None:
        sd["bigram"] = rn(cfg.bigram.buckets + 1, C, s=0.7)
    for i, spec in enumerate(cfg.layers):
        m, p = spec.mixer, f"l{i}.mix."
        sd[f"l{i}.norm1"] = rn(C, s=0.2, mean=1.0)
        if isinstance(m, LatentAttentionSpec):
            sd[p + "q"], sd[p + "g"] = rn(m.heads * (m.dim + m.rot_dim), C, s=1.5 * C ** -0.5), rn(m.heads * m.vdim, C, s=C ** -0.5)
            if m.kv_from is None:
                sd[p + "dkv"], sd[p + "dkv.norm"] = rn(m.kv_rank + m.rot_dim, C, s=C ** -0.5), rn(m.kv_rank, s=0.2, mean=1.0)
            sd[p + "uk"], sd[p + "uv"] = rn(m.heads * m.dim, m.kv_rank, s=1.5 * m.kv_rank ** -0.5), rn(m.heads * m.vdim, m.kv_rank, s=m.kv_rank ** -0.5)
            sd[p + "sink"], sd[p + "o"] = rn(m.heads, s=1.5, mean=1.0), rn(C, m.heads * m.vdim, s=2.0 * (m.heads * m.vdim) ** -0.5)
        elif isinstance(m, StateSpaceSpec):
            sd[p + "in"] = rn(m.inner + m.conv_channels + m.heads, C, s=C ** -0.5)
            sd[p + "conv"], sd[p + "conv.b"] = rn(m.conv_channels, m.conv, s=m.conv ** -0.5), rn(m.conv_channels, s=0.1)
            sd[p + "dt_bias"], sd[p + "A_log"] = rn(m.heads, s=1.5, mean=-3.0), rn(m.heads, s=1.0)   # decays from a few tokens to hundreds
            sd[p + "D"], sd[p + "norm"], sd[p + "o"] = rn(m.heads, mean=1.0), rn(m.inner, s=0.2, mean=1.0), rn(C, m.inner, s=m.inner ** -0.5)
        else:
            nq, nk = m.heads * m.dim, m.kv_heads * m.dim
            sd[p + "q"], sd[p + "k"], sd[p + "g"] = rn(nq, C, s=C ** -0.5), rn(nk, C, s=C ** -0.5), rn(m.heads, C, s=C ** -0.5)
            sd[p + "q.norm"], sd[p + "k.norm"], sd[p + "o"] = rn(nq, s=0.3, mean=1.3), rn(nk, s=0.3, mean=1.3), rn(C, nq, s=2.0 * nq ** -0.5)
        s, q = spec.mlp, f"l{i}.mlp."
        if s is not None:
            sd[f"l{i}.norm2"] = rn(C, s=0.2, mean=1.0)
            sd[q + "gate"], sd[q + "up"], sd[q + "down"] = rn(s.ff, C, s=C ** -0.5), rn(s.ff, C, s=C ** -0.5), rn(C, s.ff, s=s.ff ** -0.5)
    return sd


# ------------------------------------------------------------------------------------------------------------------- decoder
class SorupelDecoder(GraphedDecodeMixin):
    def __init__(self, cfg: SorupelConfig, w: SorupelW, dtype: torch.dtype):
        self.cfg, self.w, self.dtype = cfg, w, dtype
        self.device = w.embed.device
        self.C = cfg.hidden_size
        self.eps = cfg.norm_eps
        self.tensor_gemm = dtype == torch.bfloat16
        self.latent = LatentAttention(self.device, dtype)
        self._arange = None
        self._init_graphs()

    @property
    def tensor_attention(self) -> bool:
        return self.latent.tensor_attention

    @tensor_attention.setter
    def tensor_attention(self, on: bool):    # False: the plain attention kernels for every shape (A/B, tests)
        self.latent.tensor_attention = on

    # ---- cache
    def cache_widths(self) -> List[int]:
        """Cached numbers per token and layer: the latent and the rotated key part of layers with a down-projection of their own, keys and
        values of chunked attentions."""
        def width(m):
            if isinstance(m, LatentAttentionSpec):
                return m.kv_rank + m.rot_dim if m.kv_from is None else 0
            return 2 * m.kv_heads * m.dim if isinstance(m, ChunkAttentionSpec) else 0
        return [width(l.mixer) for l in self.cfg.layers]

    def state_shapes(self) -> List[dict]:
        """Per layer: the recurrence's states and the ring of its convolution's last inputs; behind the layers, with a bigram embedding, the
        last token."""
        out = []
        for l in self.cfg.layers:
            s, m = {}, l.mixer
            if isinstance(m, StateSpaceSpec):
                s["S"] = (m.heads, m.state, m.vdim)
                if m.conv > 1:
                    s["conv"] = (m.conv - 1, m.conv_channels)
            out.append(s)
        if self.cfg.bigram is not None:
            out.append({"token": ((), torch.int32)})
        return out

    def new_cache(self, n_pages: int, n_slots: int, max_pages_per_slot: int = 0) -> PagedStateCache:
        cache = PagedStateCache(self.cache_widths(), self.state_shapes(), n_pages, n_slots, self.cfg.kv_page_size, self.dtype, self.device,
                                max_pages_per_slot)
        for l in self.cfg.layers:   # tables are made here: a step may be under graph capture
            if not isinstance(l.mixer, StateSpaceSpec):
                self.latent.rotary.get(l.mixer.rot, cache.capacity)
        return cache

    def decode_shape(self, B: int, max_keys: int) -> dict:
        """The longest context, rounded up to a power of two: how many key ranges the latent attention of a decode-only step is cut into."""
        if not any(isinstance(l.mixer, LatentAttentionSpec) for l in self.cfg.layers):
            return {}
        return {"decode_keys": 1 << max(max_keys - 1, 0).bit_length()}

    def _linear(self, x, w, out_dtype, narrow: bool = False):
        """narrow: outputs that are few beside K (latents): on long steps the tensor-core GEMM takes such a product from a much smaller matrix
        on than the general rule says."""
        return dense_linear(x, w, out_dtype, tensor_gemm=self.tensor_gemm, min_weight=NARROW_GEMM_MIN_WEIGHT if narrow else None)

    def _one_product(self, T: int) -> bool:
        """Short steps pay per launch: one fp32 product over all rows of a stacked matrix. Long steps pay per byte: what feeds another
        product or a gate leaves in the compute dtype, from a product of its own over a slice of the same matrix."""
        return self.dtype == torch.float32 or T <= lib.SKINNY_MAX_M

    # ---- mixers: normed compute-dtype rows xb [T, C] -> fp32 [T, C]
    def _latent(self, li: int, m: LatentAttentionSpec, mw: LatentW, xb, ctx) -> torch.Tensor:
        cache, pos, slot = ctx["cache"], ctx["pos"], ctx["slot"]
        T, dev, f32 = xb.shape[0], xb.device, torch.float32
        H, dn, dr, dv, r, nqg = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, mw.nq + mw.ng
        own, qn, dkv = m.kv_from is None, None, None
        if self._one_product(T):
            zq = z = self._linear(xb, mw.w_in, f32)
            if own:
                dkv = z[:, nqg:nqg + r + dr]
            if self.dtype != f32:   # the unrotated queries are operands of the absorbing product
                qn = torch.empty(T, H * dn, device=dev, dtype=self.dtype)
        else:
            zq = self._linear(xb, mw.w_in[:nqg], self.dtype)
            if own:
                dkv = self._linear(xb, mw.w_in[nqg:], f32, narrow=True)[:, :r + dr]
        q, gate = zq[:, :mw.nq], zq[:, mw.nq:nqg]
        pool = cache.pools[li if own else m.kv_from]
        qcat = torch.empty(T, H, r + dr, device=dev, dtype=self.dtype)
        # latent norm + key rotation + cache append + query rotation in one launch
        seqlib.latent_rope_store(dkv, r, dr, mw.dkv_norm, self.eps, self.latent.rotary.get(m.rot, cache.capacity), m.rot.dims, pos, slot,
                                 cache.block_table, cache.page_size, pool, q, H, dn, qcat, qn=qn, rot_halves=m.rot.halves)
        # absorbed keys: qcat[t, h, :r] = q[t, h, :dn] @ W_uk,h  (one problem per head, column slices of both buffers)
        qa, sx = (q, dn + dr) if qn is None else (qn, dn)
        seqlib.linear(qa, mw.uk_t, qcat, M=T, N=r, K=dn, ldx=qa.stride(0), sx=sx, ldw=dn, sw=r * dn, ldy=H * (r + dr), sy=r + dr, batch=H)
        olat = self.latent.attend(qcat, r, dr, pool, cache, pos, slot, ctx["plans"], m.scale, sink=mw.sink)
        # values and output gate: att[t, h*dv:(h+1)*dv] = (W_uv,h @ olat[t, h]) * sigmoid(gate[t, h*dv:(h+1)*dv])
        att = torch.empty(T, H * dv, device=dev, dtype=self.dtype)
        seqlib.linear(olat, mw.uv, att, M=T, N=dv, K=r, ldx=H * r, sx=r, ldw=r, sw=dv * r, ldy=H * dv, sy=dv, batch=H, gate=gate)
        return self._linear(att, mw.o, f32)

    def _state_space(self, li: int, m: StateSpaceSpec, mw: StateSpaceW, xb, ctx) -> torch.Tensor:
        cache, pos, slot = ctx["cache"], ctx["pos"], ctx["slot"]
        T, dev, f32, st = xb.shape[0], xb.device, torch.float32, cache.states[li]
        inner, ch, gn = m.inner, m.conv_channels, m.groups * m.state
        if self._one_product(T):
            zall = self._linear(xb, mw.w_in, f32)
            z, zx = zall[:, :inner], zall[:, inner:]
        else:
            z, zx = self._linear(xb, mw.w_in[:inner], self.dtype), self._linear(xb, mw.w_in[inner:], f32)
        u = torch.empty(T, ch, device=dev, dtype=f32)
        seqlib.causal_conv_silu(zx[:, :ch], mw.conv, pos, slot, st.get("conv"), u, single_rows=ctx["single"], bias=mw.conv_b)
        y = torch.empty(T, inner, device=dev, dtype=f32)
        seqlib.linear_state_scan(u[:, inner + gn:], u[:, inner:inner + gn], u[:, :inner], st["S"], y, ctx["row_begin"], ctx["n_portions"], pos, slot,
                                 m.heads, m.groups, m.state, m.vdim, step_size=True, a=zx[:, ch:ch + m.heads], A_log=mw.A_log, dt_bias=mw.dt_bias, D=mw.D)
        yn = torch.empty(T, inner, device=dev, dtype=self.dtype)
        seqlib.gate_rms_rows(y, m.norm_groups, mw.norm, self.eps, z, seqlib.GATE_SILU, yn)
        return self._linear(yn, mw.o, f32)

    def _chunk_attention(self, li: int, m: ChunkAttentionSpec, mw: ChunkAttentionW, xb, ctx) -> torch.Tensor:
        cache, pos, slot, c = ctx["cache"], ctx["pos"], ctx["slot"], mw.cols
        T, dev = xb.shape[0], xb.device
        H, G, d, pool = m.heads, m.kv_heads, m.dim, cache.pools[li]
        z = self._linear(xb, mw.w_in, torch.float32)
        q = torch.empty(T, H * d, device=dev, dtype=self.dtype)
        # norms + rotation + cache append of [rotated keys | keys as projected] in one launch
        seqlib.qk_norm_kv_store(z[:, c["q"]], mw.q_norm, z[:, c["k"]], mw.k_norm, z[:, c["k"]], self.eps, pos, slot, cache.block_table, cache.page_size,
                                pool, q, cs=self.latent.rotary.get(m.rot, cache.capacity), head=d, rot_dims=m.rot.dims, rot_halves=m.rot.halves)
        att = torch.empty(T, H * d, device=dev, dtype=self.dtype)
        chunk, plans = min(m.chunk or seqlib.WINDOW_ALL, seqlib.WINDOW_ALL), ctx["plans"]
        kw = dict(sink=mw.one, gate=z[:, c["g"]], gate_act=seqlib.GATE_SIGMOID, gate_heads=True, chunk=chunk)
        if plans is not None and self.tensor_attention and seqlib.window_attn_mma_ok(H, G, d, d, self.dtype):
            items = None
            if "portions" in plans:   # else one row per request: the kernel reads positions and slots itself
                key = ("items", H // G, chunk)
                items = plans.get(key)
                if items is None:
                    items = plans[key] = seqlib.window_attn_items(plans["portions"], H // G, dev, chunk)
            seqlib.window_attn_mma(q, H, G, d, d, pool, cache.block_table, cache.page_size, items, pos, slot, seqlib.WINDOW_ALL, m.scale, m.softcap, None,
                                   att, **kw)
        else:
            seqlib.window_attn(q, H, G, d, d, pool, cache.block_table, cache.page_size, pos, slot, seqlib.WINDOW_ALL, m.scale, m.softcap, None, att, **kw)
        return self._linear(att, mw.o, torch.float32)

    def _mlp(self, ff: int, mw: DenseMlpW, xb) -> torch.Tensor:
        z = self._linear(xb, mw.gate_up, self.dtype)
        act = torch.empty(xb.shape[0], ff, device=xb.device, dtype=self.dtype)
        seqlib.glu_mul(z, ff, seqlib.ACT_GELU_TANH, act)
        return self._linear(act, mw.down, torch.float32)

    # ---- the step
    @torch.no_grad()
    def step(self, tokens: torch.Tensor, pos: torch.Tensor, slot: torch.Tensor, cache: PagedStateCache,
             want_rows: Optional[torch.Tensor] = None, collect: Optional[list] = None, portions: Optional[Sequence] = None,
             one_row_each: bool = False, decode_keys: Optional[int] = None) -> Optional[torch.Tensor]:
        """tokens / pos / slot: int32 [T] on the device - row t is token tokens[t] at position pos[t] of the request in slot slot[t];
        rows of one request are consecutive and ascending in position, and a request's rows continue where its previous step
        ended. Appends every row to the cache, advances the states and returns fp32 logits [len(want_rows), vocab] (None when no
        row is asked for). collect: receives the stream after every layer. portions: the same batch as the host knows it,
        [(first_row, n_rows, slot, first_pos)] per request. one_row_each: every row is a request of its own; decode_keys: no row of
        it sees more keys than this."""
        T, dev, C, w = tokens.numel(), self.device, self.C, self.w
        if one_row_each:
            portions = None
        row_begin, n_portions = portion_starts(self, T, slot, portions, one_row_each)
        plans = None   # without the host's view of the batch the plain attention kernels run
        if one_row_each and (decode_keys is not None or not self.decode_shape(T, 1)):
            plans = {"decode_keys": decode_keys}
        elif portions is not None:
            plans = {"portions": list(portions)}
        ctx = {"cache": cache, "pos": pos, "slot": slot, "row_begin": row_begin, "n_portions": n_portions, "single": n_portions == T, "plans": plans}
        h32 = torch.empty(T, C, device=dev, dtype=torch.float32)
        xb = torch.empty(T, C, device=dev, dtype=self.dtype)
        first = w.layers[0].norm1 if w.layers else w.final_norm
        if w.bigram is not None:
            b = self.cfg.bigram
            seqlib.embed_bigram(tokens, pos, slot, w.embed, w.bigram, b.mul_prev, b.mul_cur, cache.states[-1]["token"], h32, nw=first, eps=self.eps, xb=xb,
                                single_rows=ctx["single"])
        else:
            seqlib.embed_scale(tokens, w.embed, 1.0, h32, None)
            seqlib.rms_residual(h32, first, self.eps, xb=xb)
        mixers = {LatentAttentionSpec: self._latent, StateSpaceSpec: self._state_space, ChunkAttentionSpec: self._chunk_attention}
        for li, lw in enumerate(w.layers):
            spec = self.cfg.layers[li]
            after = w.layers[li + 1].norm1 if li + 1 < len(w.layers) else w.final_norm   # what stands in front of the next sublayer
            y = mixers[type(spec.mixer)](li, spec.mixer, lw.mix, xb, ctx)
            seqlib.rms_residual(h32, lw.norm2 if lw.mlp is not None else after, self.eps, y=y, x_out=h32, xb=xb)
            if lw.mlp is not None:
                y = self._mlp(spec.mlp.ff, lw.mlp, xb)
                seqlib.rms_residual(h32, after, self.eps, y=y, x_out=h32, xb=xb)
            if collect is not None:
                collect.append(h32.clone())
        if want_rows is None or want_rows.numel() == 0:
            return None
        return self._linear(xb.index_select(0, want_rows), w.head, torch.float32)


# ------------------------------------------------------------------------------------------------------------------- model
class SorupelForCausalLM(SequenceStepLM):
    """Entry point: from_pretrained / from_state_dict, step() for serving loops, generate() for greedy generation."""
    config_class = SorupelConfig
    decoder_class = SorupelDecoder
    weights_from_state_dict = staticmethod(weights_from_state_dict)
