"""Munevik: a decoder-only language model of gated linear recurrent layers and sliding-window latent-attention layers, some of which
attend to another layer's cached rows, with dense clamped feed-forwards or group-limited sigmoid-routed experts.

A sublayer reads the stream x itself and the norm stands after the sum: x <- LN1(alpha x + mixer(x)); x <- LN2(alpha x + ff(x)) with
layer norms (weight and bias). The stream is fp32 on the device; sublayers read its rounding to the compute dtype.

Mixers. Latent attention (config.LatentAttentionSpec, model/seq_latent.py): keys / values are up-projections of a cached latent plus
one rotated key part, absorbed into the query and the output; a window limits what a row sees, every head's output passes a sigmoid
gate, and a layer with kv_from attends to that layer's rows (it caches nothing). Gated linear recurrent unit (config.GatedLruSpec):
a gelu branch times the states of a per-channel recurrence whose input passes a causal convolution and whose gates are block-diagonal
products. The output head is the embedding matrix.

Like the other sequence-step decoders the model owns no cache and no loop: `step()` runs ONE packed batch of rows - portions of prompts
beside single decoded tokens, each row addressed by (slot, position) - against a PagedStateCache that the caller
(serving.StepScheduler) manages: pages of latents for the attentions, per-slot fp32 states and convolution rings for the recurrences.
`generate()` goes through that scheduler; decode-only steps replay from a CUDA graph (seq_model.py).

Kernels: omc_latent_rope_store, omc_latent_attn / omc_latent_attn_mma with window and head gate, omc_causal_conv (bias),
omc_rglru_scan, omc_router_topk (sigmoid scores, groups), the expert-sorted products of seq_moe.py, omc_glu_mul, omc_ln_residual
(residual sum, experts' combine, layer norm).

Compute dtype bfloat16: bf16 matrix operands with fp32 accumulation, bf16 latents; angles, scores and softmax, norms, router, stream,
recurrent states and gates in fp32. Compute dtype float32: everything in fp32 on the FMA pipe.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence

import torch

from .. import lib, seqlib
from ..config import ClampedMlpSpec, GatedLruSpec, GroupedMoeSpec, LatentAttentionSpec, MunevikConfig
from .paged_cache import PagedStateCache
from .seq_latent import LatentAttention
from .seq_linear import NARROW_GEMM_MIN_WEIGHT, dense_linear, stack_rows
from .seq_model import GraphedDecodeMixin, SequenceStepLM, portion_starts
from .seq_moe import expert_workspace, grouped_tensor_gemm_ok, run_sorted_experts


# ------------------------------------------------------------------------------------------------------------------- weights
@dataclass
class LayerNormW:
    w: torch.Tensor                # [C]
    b: torch.Tensor                # [C]


@dataclass
class LatentW:
    w_in: torch.Tensor             # [q | dkv (own rows only) | head gate | zero rows, C]
    nq: int                        # rows of q: H * (dim + rot_dim)
    cols: Dict[str, slice]         # 'q', 'dkv', 'g': columns of w_in's output
    dkv_norm: Optional[torch.Tensor]
    uk_t: torch.Tensor             # [H, kv_rank, dim]: per head W_uk^T, the absorbing projection of the unrotated query
    uv: torch.Tensor               # [H * vdim, kv_rank]
    o: torch.Tensor                # [C, H * vdim]


@dataclass
class LruW:
    w_in: torch.Tensor             # [y | x, C]
    b_in: torch.Tensor             # [2 * width]
    conv: torch.Tensor             # [width, taps]
    conv_b: torch.Tensor           # [width]
    gates: torch.Tensor            # [blocks, 2 n, n]: recurrence gate over input gate of every block
    gates_b: torch.Tensor          # fp32 [2 * width], in the order of the gates' outputs
    lam: torch.Tensor              # fp32 [width]
    o: torch.Tensor                # [C, width]


@dataclass
class DenseMlpW:
    gate_up: torch.Tensor          # [2 ff, C]
    down: torch.Tensor             # [C, ff]


@dataclass
class GroupedMoeW:
    w_in: torch.Tensor             # [router | zero rows | shared gate | shared up, C]
    n_router: int                  # rows of the router with its zero rows
    gate_up: torch.Tensor          # [E, 2 ff, C]
    down: torch.Tensor             # [E, C, ff]
    shared_down: Optional[torch.Tensor]   # [C, shared ff]


@dataclass
class MunevikLayerW:
    norm1: LayerNormW
    norm2: Optional[LayerNormW]
    mix: object
    mlp: object


@dataclass
class MunevikW:
    embed: torch.Tensor
    final_norm: LayerNormW
    layers: List[MunevikLayerW]


def weights_from_state_dict(sd: Dict[str, torch.Tensor], cfg: MunevikConfig, device, dtype: torch.dtype) -> MunevikW:
    """Checkpoint names: 'embed', 'final.norm' (+ '.b'), per layer i 'l<i>.norm1|norm2' (+ '.b'), 'l<i>.mix.*', 'l<i>.mlp.*'; linear
    weights [out, in]. Load-time re-layouts: one stacked input projection per mixer, W_uk transposed per head, the two gates of a
    recurrence block stacked, gate and up of every expert stacked and the experts in one tensor, the shared expert's gate and up
    behind the router. Shapes are checked against the config."""
    f32 = torch.float32

    def g(name, shape, dt=dtype):
        if name not in sd:
            raise KeyError(f"checkpoint has no tensor {name!r}")
        if tuple(sd[name].shape) != tuple(shape):
            raise ValueError(f"{name} has shape {tuple(sd[name].shape)}, the config says {tuple(shape)}")
        return sd[name].to(device=device, dtype=dt).contiguous()

    def norm(name) -> LayerNormW:
        return LayerNormW(w=g(name, (C,)), b=g(name + ".b", (C,)))

    def gate_up(p: str, ff: int):
        return torch.cat([g(p + "gate", (ff, C)), g(p + "up", (ff, C))], dim=0)

    C = cfg.hidden_size
    layers = []
    for i, spec in enumerate(cfg.layers):
        m, p = spec.mixer, f"l{i}.mix."
        if isinstance(m, LatentAttentionSpec):
            H, dn, r, nq = m.heads, m.dim, m.kv_rank, m.heads * (m.dim + m.rot_dim)
            parts = [("q", g(p + "q", (nq, C)))]
            if m.kv_from is None:
                parts.append(("dkv", g(p + "dkv", (r + m.rot_dim, C))))
            parts.append(("g", g(p + "g", (H, C))))
            w_in, cols = stack_rows(parts)
            mix = LatentW(w_in=w_in, nq=nq, cols=cols, dkv_norm=g(p + "dkv.norm", (r,)) if m.kv_from is None else None,
                          uk_t=g(p + "uk", (H * dn, r)).view(H, dn, r).transpose(1, 2).contiguous(), uv=g(p + "uv", (H * m.vdim, r)),
                          o=g(p + "o", (C, H * m.vdim)))
        else:
            assert isinstance(m, GatedLruSpec)
            W, nb = m.width, m.blocks
            n = W // nb
            mix = LruW(w_in=torch.cat([g(p + "y", (W, C)), g(p + "x", (W, C))], dim=0), b_in=torch.cat([g(p + "y.b", (W,)), g(p + "x.b", (W,))]),
                       conv=g(p + "conv", (W, m.conv)), conv_b=g(p + "conv.b", (W,)),
                       gates=torch.cat([g(p + "ra", (nb, n, n)), g(p + "ri", (nb, n, n))], dim=1).contiguous(),
                       gates_b=torch.cat([g(p + "ra.b", (nb, n), f32), g(p + "ri.b", (nb, n), f32)], dim=1).reshape(-1).contiguous(),
                       lam=g(p + "lam", (W,), f32), o=g(p + "o", (C, W)))
        s, q, mlp = spec.mlp, f"l{i}.mlp.", None
        if isinstance(s, ClampedMlpSpec):
            mlp = DenseMlpW(gate_up=gate_up(q, s.ff), down=g(q + "down", (C, s.ff)))
        elif isinstance(s, GroupedMoeSpec):
            w_in, _ = stack_rows([("r", g(q + "router", (s.experts, C)))])
            n_router = w_in.shape[0]
            if s.shared_ff:
                w_in = torch.cat([w_in, gate_up(q + "shared.", s.shared_ff)], dim=0).contiguous()
            mlp = GroupedMoeW(w_in=w_in, n_router=n_router, gate_up=torch.stack([gate_up(f"{q}e{e}.", s.expert_ff) for e in range(s.experts)]).contiguous(),
                              down=torch.stack([g(f"{q}e{e}.down", (C, s.expert_ff)) for e in range(s.experts)]).contiguous(),
                              shared_down=g(q + "shared.down", (C, s.shared_ff)) if s.shared_ff else None)
        layers.append(MunevikLayerW(norm1=norm(f"l{i}.norm1"), norm2=norm(f"l{i}.norm2") if s is not None else None, mix=mix, mlp=mlp))
    return MunevikW(embed=g("embed", (cfg.vocab_size, C)), final_norm=norm("final.norm"), layers=layers)


def random_state_dict(cfg: MunevikConfig, seed: int = 0) -> Dict[str, torch.Tensor]:
    """Random bf16 weights under the checkpoint names (benchmarks, tests)."""
    gen = torch.Generator().manual_seed(seed)

    def rn(*shape, s=1.0, mean=0.0):
        return (torch.randn(shape, generator=gen) * s + mean).to(torch.bfloat16)

    def norm(name):
        sd[name], sd[name + ".b"] = rn(C, s=0.2, mean=1.0), rn(C, s=0.1)

    def mlp(p: str, ff: int):
        sd[p + "gate"], sd[p + "up"], sd[p + "down"] = rn(ff, C, s=1.5 * C ** -0.5), rn(ff, C, s=1.5 * C ** -0.5), rn(C, ff, s=ff ** -0.5)

    C, sd = cfg.hidden_size, {}
    sd["embed"] = rn(cfg.vocab_size, C, s=C ** -0.5)
    norm("final.norm")
    for i, spec in enumerate(cfg.layers):
        m, p = spec.mixer, f"l{i}.mix."
        norm(f"l{i}.norm1")
        if isinstance(m, LatentAttentionSpec):
            sd[p + "q"] = rn(m.heads * (m.dim + m.rot_dim), C, s=1.5 * C ** -0.5)
            if m.kv_from is None:
                sd[p + "dkv"], sd[p + "dkv.norm"] = rn(m.kv_rank + m.rot_dim, C, s=C ** -0.5), rn(m.kv_rank, s=0.2, mean=1.0)
            sd[p + "uk"], sd[p + "uv"] = rn(m.heads * m.dim, m.kv_rank, s=1.5 * m.kv_rank ** -0.5), rn(m.heads * m.vdim, m.kv_rank, s=m.kv_rank ** -0.5)
            sd[p + "g"], sd[p + "o"] = rn(m.heads, C, s=C ** -0.5), rn(C, m.heads * m.vdim, s=2.0 * (m.heads * m.vdim) ** -0.5)
        else:
            W, nb = m.width, m.blocks
            n = W // nb
            sd[p + "y"], sd[p + "y.b"] = rn(W, C, s=C ** -0.5), rn(W, s=0.2, mean=0.3)
            sd[p + "x"], sd[p + "x.b"] = rn(W, C, s=C ** -0.5), rn(W, s=0.2)
            sd[p + "conv"], sd[p + "conv.b"] = rn(W, m.conv, s=m.conv ** -0.5), rn(W, s=0.1)
            sd[p + "ra"], sd[p + "ra.b"] = rn(nb, n, n, s=n ** -0.5), rn(nb, n, s=0.5)
            sd[p + "ri"], sd[p + "ri.b"] = rn(nb, n, n, s=n ** -0.5), rn(nb, n, s=0.5)
            sd[p + "lam"], sd[p + "o"] = rn(W, s=1.5, mean=-5.0), rn(C, W, s=2.0 * W ** -0.5)   # decays from a few tokens to thousands
        s, q = spec.mlp, f"l{i}.mlp."
        if s is not None:
            norm(f"l{i}.norm2")
        if isinstance(s, ClampedMlpSpec):
            mlp(q, s.ff)
        elif isinstance(s, GroupedMoeSpec):
            sd[q + "router"] = rn(s.experts, C, s=2.0 * C ** -0.5)
            for e in range(s.experts):
                mlp(f"{q}e{e}.", s.expert_ff)
            if s.shared_ff:
                mlp(q + "shared.", s.shared_ff)
    return sd


# ------------------------------------------------------------------------------------------------------------------- decoder
class MunevikDecoder(GraphedDecodeMixin):
    def __init__(self, cfg: MunevikConfig, w: MunevikW, dtype: torch.dtype):
        self.cfg, self.w, self.dtype = cfg, w, dtype
        self.device = w.embed.device
        self.C = cfg.hidden_size
        self.eps = cfg.norm_eps
        self.tensor_gemm = dtype == torch.bfloat16
        self.latent = LatentAttention(self.device, dtype)
        self._moe_ws = {}
        self._arange = None
        self._init_graphs()

    # ---- cache
    def cache_widths(self) -> List[int]:
        """Cached numbers per token and layer: the latent and the rotated key part of layers with a down-projection of their own."""
        return [l.mixer.kv_rank + l.mixer.rot_dim if isinstance(l.mixer, LatentAttentionSpec) and l.mixer.kv_from is None else 0
                for l in self.cfg.layers]

    def state_shapes(self) -> List[dict]:
        """Per layer: the recurrence's states and the ring of its convolution's last inputs."""
        out = []
        for l in self.cfg.layers:
            s, m = {}, l.mixer
            if isinstance(m, GatedLruSpec):
                s["S"] = (m.width,)
                if m.conv > 1:
                    s["conv"] = (m.conv - 1, m.width)
            out.append(s)
        return out

    def new_cache(self, n_pages: int, n_slots: int, max_pages_per_slot: int = 0) -> PagedStateCache:
        cache = PagedStateCache(self.cache_widths(), self.state_shapes(), n_pages, n_slots, self.cfg.kv_page_size, self.dtype, self.device,
                                max_pages_per_slot)
        for l in self.cfg.layers:   # tables are made here: a step may be under graph capture
            if isinstance(l.mixer, LatentAttentionSpec):
                self.latent.rotary.get(l.mixer.rot, cache.capacity)
        return cache

    def decode_shape(self, B: int, max_keys: int) -> dict:
        """The longest window or the longest context, whichever is shorter, rounded up to a power of two: how many key ranges the
        attention of a decode-only step is cut into."""
        wins = [l.mixer.window or seqlib.WINDOW_ALL for l in self.cfg.layers if isinstance(l.mixer, LatentAttentionSpec)]
        return {"decode_keys": 1 << max(min(max(wins, default=1), max_keys) - 1, 0).bit_length()}

    def _linear(self, x, w, out_dtype, bias=None, narrow: bool = False):
        """narrow: few outputs over a long K (router, head gates): on long steps the tensor-core GEMM takes it from a much smaller
        matrix on than the general rule says."""
        return dense_linear(x, w, out_dtype, tensor_gemm=self.tensor_gemm, bias=bias, min_weight=NARROW_GEMM_MIN_WEIGHT if narrow else None)

    def _one_product(self, T: int) -> bool:
        """Short steps pay per launch: one fp32 product over all rows of a stacked matrix. Long steps pay per byte: what feeds another
        product leaves in the compute dtype, from a product of its own over a slice of the same matrix."""
        return self.dtype == torch.float32 or T <= lib.SKINNY_MAX_M

    # ---- mixers: compute-dtype rows xb [T, C] -> fp32 [T, C]
    def _attention(self, li: int, m: LatentAttentionSpec, mw: LatentW, xb, ctx) -> torch.Tensor:
        cache, pos, slot = ctx["cache"], ctx["pos"], ctx["slot"]
        T, dev, f32 = xb.shape[0], xb.device, torch.float32
        H, dn, dr, dv, r = m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
        own = m.kv_from is None
        qn = None
        if self._one_product(T):
            z, off = self._linear(xb, mw.w_in, f32), 0
            q = z[:, :mw.nq]
            if self.dtype != f32:   # the unrotated queries are operands of the absorbing product
                qn = torch.empty(T, H * dn, device=dev, dtype=self.dtype)
        else:
            q, z, off = self._linear(xb, mw.w_in[:mw.nq], self.dtype), self._linear(xb, mw.w_in[mw.nq:], f32, narrow=True), mw.nq
        gate = z[:, mw.cols["g"].start - off:mw.cols["g"].stop - off]
        dkv = z[:, mw.cols["dkv"].start - off:mw.cols["dkv"].stop - off] if own else None
        pool = cache.pools[li if own else m.kv_from]
        qcat = torch.empty(T, H, r + dr, device=dev, dtype=self.dtype)
        # latent norm + key rotation + cache append + query rotation in one launch
        seqlib.latent_rope_store(dkv, r, dr, mw.dkv_norm, self.eps, self.latent.rotary.get(m.rot, cache.capacity), m.rot.dims, pos, slot,
                                 cache.block_table, cache.page_size, pool, q, H, dn, qcat, qn=qn)
        # absorbed keys: qcat[t, h, :r] = q[t, h, :dn] @ W_uk,h  (one problem per head, column slices of both buffers)
        qa, sx = (q, dn + dr) if qn is None else (qn, dn)
        seqlib.linear(qa, mw.uk_t, qcat, M=T, N=r, K=dn, ldx=qa.stride(0), sx=sx, ldw=dn, sw=r * dn, ldy=H * (r + dr), sy=r + dr, batch=H)
        olat = self.latent.attend(qcat, r, dr, pool, cache, pos, slot, ctx["plans"], m.scale, window=m.window, gate=gate)
        # values: att[t, h*dv:(h+1)*dv] = W_uv,h @ olat[t, h]; the head's gate is already on olat
        att = torch.empty(T, H * dv, device=dev, dtype=self.dtype)
        seqlib.linear(olat, mw.uv, att, M=T, N=dv, K=r, ldx=H * r, sx=r, ldw=r, sw=dv * r, ldy=H * dv, sy=dv, batch=H)
        return self._linear(att, mw.o, f32)

    def _lru(self, li: int, m: GatedLruSpec, mw: LruW, xb, ctx) -> torch.Tensor:
        cache, pos, slot = ctx["cache"], ctx["pos"], ctx["slot"]
        T, dev, f32, st = xb.shape[0], xb.device, torch.float32, cache.states[li]
        W, n = m.width, m.width // m.blocks
        z = self._linear(xb, mw.w_in, f32, bias=mw.b_in)     # [T, y | x]
        u = torch.empty(T, W, device=dev, dtype=self.dtype)
        seqlib.causal_conv_silu(z[:, W:], mw.conv, pos, slot, st.get("conv"), u, single_rows=ctx["single"], act=seqlib.CONV_LINEAR, bias=mw.conv_b)
        g = torch.empty(T, 2 * W, device=dev, dtype=f32)
        seqlib.linear(u, mw.gates, g, M=T, N=2 * n, K=n, ldx=u.stride(0), sx=n, ldw=n, sw=2 * n * n, ldy=2 * W, sy=2 * n, batch=m.blocks)
        s = torch.empty(T, W, device=dev, dtype=self.dtype)
        seqlib.rglru_scan(u, g, mw.gates_b, mw.lam, z[:, :W], st["S"], s, ctx["row_begin"], ctx["n_portions"], pos, slot, m.blocks, m.decay_scale)
        return self._linear(s, mw.o, f32)

    # ---- feed-forwards: update h32 (and xb) in place, the layer norm included
    def _dense_mlp(self, s: ClampedMlpSpec, mw: DenseMlpW, xb, h32, xb_out, norm: LayerNormW):
        z = self._linear(xb, mw.gate_up, self.dtype)
        act = torch.empty(xb.shape[0], s.ff, device=xb.device, dtype=self.dtype)
        seqlib.glu_mul(z, s.ff, seqlib.ACT_CLAMP_SWISH, act, limit=s.limit, slope=MunevikConfig.SWISH_SLOPE, shift=MunevikConfig.UP_SHIFT)
        y = self._linear(act, mw.down, torch.float32)
        seqlib.ln_residual(h32, self.cfg.postln_alpha, norm.w, norm.b, self.eps, y=y, x_out=h32, xb=xb_out)

    def _moe(self, s: GroupedMoeSpec, mw: GroupedMoeW, xb, h32, xb_out, norm: LayerNormW):
        T, f32 = xb.shape[0], torch.float32
        grouped = grouped_tensor_gemm_ok(self.tensor_gemm, s.expert_ff, self.C)
        tile = 128 if grouped else seqlib.LINEAR_TILE
        ws = expert_workspace(self._moe_ws, T, s.experts, s.top, s.expert_ff, tile, self.C, self.dtype, self.device)
        if self._one_product(T) or not s.shared_ff:
            z = self._linear(xb, mw.w_in, f32, narrow=True)
            zs = z[:, mw.n_router:]
        else:
            z, zs = self._linear(xb, mw.w_in[:mw.n_router], f32, narrow=True), self._linear(xb, mw.w_in[mw.n_router:], self.dtype)
        seqlib.router_topk(z, s.experts, s.experts, s.top, None, False, ws.ids, ws.w, None, ws.counts, score=seqlib.ROUTER_SIGMOID, groups=s.groups,
                           keep=s.keep, scale=s.scale)
        run_sorted_experts(ws, xb, s.experts, s.top, s.expert_ff, tile, mw.gate_up, mw.down, seqlib.ACT_SILU, grouped=grouped)
        y = None
        if s.shared_ff:
            act = torch.empty(T, s.shared_ff, device=xb.device, dtype=self.dtype)
            seqlib.glu_mul(zs, s.shared_ff, seqlib.ACT_SILU, act)
            y = self._linear(act, mw.shared_down, f32)
        seqlib.ln_residual(h32, self.cfg.postln_alpha, norm.w, norm.b, self.eps, y=y, ys=ws.ys, slot_of=ws.slot_of, w=ws.w, top=s.top, x_out=h32,
                           xb=xb_out)

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
        T, dev, f32, C, alpha = tokens.numel(), self.device, torch.float32, self.C, self.cfg.postln_alpha
        if one_row_each:
            portions = None
        row_begin, n_portions = portion_starts(self, T, slot, portions, one_row_each)
        plans = None   # without the host's view of the batch the plain attention kernel runs
        if one_row_each and decode_keys is not None:
            plans = {"decode_keys": decode_keys}
        elif portions is not None:
            plans = {"portions": list(portions)}
        ctx = {"cache": cache, "pos": pos, "slot": slot, "row_begin": row_begin, "n_portions": n_portions, "single": n_portions == T, "plans": plans}
        h32 = torch.empty(T, C, device=dev, dtype=f32)
        xb_out = torch.empty(T, C, device=dev, dtype=self.dtype) if self.dtype != f32 else None   # fp32: sublayers read the stream itself
        xb = xb_out if xb_out is not None else h32
        seqlib.embed_scale(tokens, self.w.embed, 1.0, h32, xb_out)
        for li, lw in enumerate(self.w.layers):
            spec = self.cfg.layers[li]
            mixer = self._attention if isinstance(spec.mixer, LatentAttentionSpec) else self._lru
            y = mixer(li, spec.mixer, lw.mix, xb, ctx)
            seqlib.ln_residual(h32, alpha, lw.norm1.w, lw.norm1.b, self.eps, y=y, x_out=h32, xb=xb_out)
            if spec.mlp is not None:
                ff = self._dense_mlp if isinstance(spec.mlp, ClampedMlpSpec) else self._moe
                ff(spec.mlp, lw.mlp, xb, h32, xb_out, lw.norm2)
            if collect is not None:
                collect.append(h32.clone())
        if want_rows is None or want_rows.numel() == 0:
            return None
        hw, fn = h32.index_select(0, want_rows), self.w.final_norm
        xf = seqlib.ln_residual(hw, 1.0, fn.w, fn.b, self.eps, xb=torch.empty(hw.shape[0], C, device=dev, dtype=self.dtype))
        return self._linear(xf, self.w.embed, f32)


# ------------------------------------------------------------------------------------------------------------------- model
class MunevikForCausalLM(SequenceStepLM):
    """Entry point: from_pretrained / from_state_dict, step() for serving loops, generate() for greedy generation."""
    config_class = MunevikConfig
    decoder_class = MunevikDecoder
    weights_from_state_dict = staticmethod(weights_from_state_dict)
