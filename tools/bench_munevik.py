#!/usr/bin/env python
"""Munevik decoder at sizes that resemble a real model's layers (random weights), beside the framework's closest existing model, the
Voduzen decoder (model/voduzen.py: latent attention over a paged cache, a router over experts, a shared expert, an fp32 residual
stream), at equal width, depth, heads, head widths, latent width, experts, top-k and vocabulary. Voduzen's feed-forwards have two
matrices where Munevik's have three, so theirs are 1.5 times as wide: equal parameters per expert; it has an attention layer wherever
Munevik has a recurrent one.

Per size: prefill of `--prefill` x 1024-token prompts as ONE packed step through serving.StepScheduler (tokens/s), decode steps at
batch B and context ctx through the same scheduler (ms/step, tokens/s), and the new kernels timed alone on one layer's shapes against
their rooflines, each beside the like kernel of an existing path:
  omc_rglru_scan           bytes of its rows (decode: and states) against the copy bandwidth; like: omc_selective_scan (Vefunex) with
                           16 states per channel over as many channels
  omc_causal_conv          bias, no activation, bf16 out: bytes; like: bias + silu (Vefunex)
  block-diagonal gates     omc_linear over blocks: FLOPs against the measured bf16 peak; like: the absorbing product of Voduzen
  omc_latent_attn_mma      with window and head gate: FLOPs = visible keys x heads x 2 (2 r + dr), decode: bytes of the visible rows;
                           like: the same entry without window and gate over contexts of the same length (Voduzen)
  omc_latent_rope_store, omc_ln_residual (with and without the experts' combine), omc_router_topk (sigmoid, groups), omc_glu_mul
                           (clamped swish, silu): bytes read + written; like kernels: the Voduzen form, omc_norm_residual,
                           omc_moe_combine_norm, omc_router_topk (softmax), omc_glu_mul (gelu)
python tools/bench_munevik.py --size s --size m
"""
import argparse
import json
import math
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

import torch  # noqa: E402

from omchat_b200 import seqlib  # noqa: E402
from omchat_b200.config import MunevikConfig, VoduzenConfig  # noqa: E402
from omchat_b200.model import munevik, voduzen  # noqa: E402
from omchat_b200.model.seq_latent import LatentAttention  # noqa: E402
from tools.bench_fofisun import serve  # noqa: E402
from tools.bench_voduzen import peaks, timed  # noqa: E402

# width, recurrence channels / blocks / taps, heads, key (unrotated, rotated) and value widths, latent width, window, experts / groups /
# kept groups / top / expert ff / shared ff, dense ff, vocab
SIZES = {
    "s": dict(C=2048, W=2560, nb=10, conv=4, H=16, dn=128, dr=64, dv=128, r=512, win=1024, E=32, G=4, keep=2, top=4, eff=1024, sff=2048, ff=6144, V=32768),
    "m": dict(C=4096, W=4096, nb=16, conv=4, H=32, dn=128, dr=64, dv=128, r=512, win=1024, E=32, G=4, keep=2, top=4, eff=2048, sff=4096, ff=12288, V=65536),
}
ORDER = (("lru", "dense"), ("own", "moe"), ("shared", "moe"), ("lru", "moe"), ("lru", "moe"), ("own", "moe"))


def config_dict(z):
    moe = {"expert": {"ff": z["eff"]}, "kind": "moe", "router": {"experts": z["E"], "groups": {"count": z["G"], "keep": z["keep"]}, "scale": 2.5, "top": z["top"]},
           "shared": {"ff": z["sff"]}}
    att = {"dim": z["dn"], "heads": z["H"], "kv_rank": z["r"], "mask": {"size": z["win"]}, "rot": {"base": 1e6, "dims": z["dr"]}, "rot_dim": z["dr"],
           "scale": (z["dn"] + z["dr"]) ** -0.5, "vdim": z["dv"]}
    layers = []
    for mix, ff in ORDER:
        mlp = moe if ff == "moe" else {"ff": z["ff"], "kind": "dense", "limit": 7.0}
        if mix == "lru":
            layers.append({"type": "rglru", "mixer": {"blocks": z["nb"], "conv": z["conv"], "width": z["W"]}, "mlp": mlp})
        else:
            layers.append({"type": "latent_attention", "mixer": dict(att, kv_from=1) if mix == "shared" else att, "mlp": mlp})
    return {"architecture": "Munevik", "vocab": z["V"], "width": z["C"], "norm": {"eps": 1e-6}, "postln_alpha": 2.0, "layers": layers}


def voduzen_dict(z):
    """The equal-size neighbour (see the module docstring)."""
    mixer = {"dim": z["dn"], "heads": z["H"], "kv_rank": z["r"], "rot_dim": z["dr"], "vdim": z["dv"], "scale": 1.0 / math.sqrt(z["dn"] + z["dr"]),
             "rot": {"base": 1e6, "dims": z["dr"]}}
    mlp = {"kind": "moe", "expert": {"ff": z["eff"] * 3 // 2}, "router": {"experts": z["E"], "identity": 0, "top": z["top"]}, "shared": {"ff": z["sff"] * 3 // 2}}
    return {"architecture": "Voduzen", "vocab": z["V"], "width": z["C"], "embedding": {"scale": math.sqrt(z["C"])}, "logit_scale": 1.0, "norm": {"eps": 1e-6},
            "layers": [{"type": "latent_attention", "mixer": mixer, "mlp": mlp} for _ in ORDER]}


def kernels(z, n_seq, L, B, ctx):
    """The new kernels alone on one layer's shapes, each beside its like kernel."""
    hbm, tf = peaks()
    dev, bf, f32, i32 = "cuda", torch.bfloat16, torch.float32, torch.int32
    C, W, H, r, dr, dn = z["C"], z["W"], z["H"], z["r"], z["dr"], z["dn"]
    D, page, out, T = r + dr, 64, {}, n_seq * L
    pos = torch.arange(L, dtype=i32, device=dev).repeat(n_seq)
    slot = torch.arange(n_seq, dtype=i32, device=dev).repeat_interleave(L)
    rb = (torch.arange(n_seq + 1, dtype=i32, device=dev) * L).contiguous()
    posd = torch.full((B,), ctx, dtype=i32, device=dev)
    slotd = torch.arange(B, dtype=i32, device=dev)
    rbd = torch.arange(B + 1, dtype=i32, device=dev)
    S_ = max(n_seq, B)

    def rate(ms, nbytes=None, flops=None, **extra):
        rec = {"ms": ms, **extra}
        if nbytes is not None:
            rec.update(gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm)
        if flops is not None:
            rec.update(tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tf)
        return rec

    # ---- recurrence, its convolution and its gates
    n = W // z["nb"]
    zz = torch.randn(T, 2 * W, device=dev)
    u = torch.empty(T, W, device=dev, dtype=bf)
    cw, cb = (torch.randn(W, z["conv"], device=dev) * 0.4).to(bf), torch.zeros(W, device=dev, dtype=bf)
    ring = torch.zeros(S_, z["conv"] - 1, W, device=dev)
    ms = timed(lambda: seqlib.causal_conv_silu(zz[:, W:], cw, pos, slot, ring, u, act=seqlib.CONV_LINEAR, bias=cb))
    out["causal_conv_bias"] = rate(ms, T * W * 6)
    ms = timed(lambda: seqlib.causal_conv_silu(zz[:, W:], cw, pos, slot, ring, u, bias=cb))
    out["vefunex_causal_conv_bias_silu"] = rate(ms, T * W * 6)
    gw = (torch.randn(z["nb"], 2 * n, n, device=dev) * n ** -0.5).to(bf)
    g = torch.empty(T, 2 * W, device=dev)
    ms = timed(lambda: seqlib.linear(u, gw, g, M=T, N=2 * n, K=n, ldx=W, sx=n, ldw=n, sw=2 * n * n, ldy=2 * W, sy=2 * n, batch=z["nb"]))
    out["block_gates"] = rate(ms, T * W * 10, flops=T * 2 * W * n * 2.0)
    gb, lam = torch.zeros(2 * W, device=dev), torch.randn(W, device=dev) - 5.0
    S, so = torch.zeros(S_, W, device=dev), torch.empty(T, W, device=dev, dtype=bf)
    ms = timed(lambda: seqlib.rglru_scan(u, g, gb, lam, zz[:, :W], S, so, rb, n_seq, pos, slot, z["nb"], 8.0))
    out["rglru_scan_prefill"] = rate(ms, T * W * 16)
    ms = timed(lambda: seqlib.rglru_scan(u[:B], g[:B], gb, lam, zz[:B, :W], S, so[:B], rbd, B, posd, slotd, z["nb"], 8.0))
    out["rglru_scan_decode"] = rate(ms, B * W * 24, batch=B)
    N = 16
    pj, A_log = torch.randn(T, 2 * N, device=dev), torch.randn(W, N, device=dev) * 0.5
    dtb, Dv, S2 = torch.full((W,), -2.0, device=dev), torch.ones(W, device=dev), torch.zeros(S_, W, N, device=dev)
    ms = timed(lambda: seqlib.selective_scan(u, zz[:, :W], dtb, pj[:, :N], pj[:, N:], A_log, Dv, zz[:, W:], S2, so, rb, n_seq, pos, slot))
    out["vefunex_selective_scan_prefill"] = rate(ms, T * W * 12 + T * 2 * N * 4)
    ms = timed(lambda: seqlib.selective_scan(u[:B], zz[:B, :W], dtb, pj[:B, :N], pj[:B, N:], A_log, Dv, zz[:B, W:], S2, so[:B], rbd, B, posd, slotd))
    out["vefunex_selective_scan_decode"] = rate(ms, B * W * N * 8 + B * W * 12, batch=B)
    del zz, u, g, so, S2
    # ---- residual sum + layer norm, alone and with the experts' combine
    x, y = torch.randn(T, C, device=dev), torch.randn(T, C, device=dev)
    xb = torch.empty(T, C, device=dev, dtype=bf)
    nw, nbias = torch.ones(C, device=dev, dtype=bf), torch.zeros(C, device=dev, dtype=bf)
    top = z["top"]
    ys = torch.randn(T * top, C, device=dev)
    slot_of = torch.randperm(T * top, device=dev).view(T, top).to(i32)
    wts, gate1 = torch.rand(T, top, device=dev), torch.rand(T, device=dev)
    ms = timed(lambda: seqlib.ln_residual(x, 2.0, nw, nbias, 1e-6, y=y, x_out=x, xb=xb))
    out["ln_residual"] = rate(ms, T * C * 14)
    ms = timed(lambda: seqlib.norm_residual(y, nw, 1e-6, x, xb))
    out["voduzen_norm_residual"] = rate(ms, T * C * 14)
    ms = timed(lambda: seqlib.ln_residual(x, 2.0, nw, nbias, 1e-6, y=y, ys=ys, slot_of=slot_of, w=wts, top=top, x_out=x, xb=xb))
    out["ln_residual_combine"] = rate(ms, T * C * (14 + 4 * top))
    ms = timed(lambda: seqlib.moe_combine_norm(ys, slot_of, wts, top, gate1, y, nw, 1e-6, x, xb))
    out["voduzen_moe_combine_norm"] = rate(ms, T * C * (14 + 4 * top))
    ms = timed(lambda: seqlib.ln_residual(x[:B], 2.0, nw, nbias, 1e-6, y=y[:B], ys=ys, slot_of=slot_of[:B], w=wts, top=top, x_out=x[:B], xb=xb[:B]))
    out["ln_residual_combine_decode"] = rate(ms, B * C * (14 + 4 * top), batch=B)
    ms = timed(lambda: seqlib.moe_combine_norm(ys, slot_of[:B], wts, top, gate1, y[:B], nw, 1e-6, x[:B], xb[:B]))
    out["voduzen_moe_combine_norm_decode"] = rate(ms, B * C * (14 + 4 * top), batch=B)
    del x, y, xb, ys
    # ---- router
    E = z["E"]
    zr = torch.randn(T, E, device=dev)
    ids, w_, counts = torch.empty(T, top, device=dev, dtype=i32), torch.empty(T, top, device=dev), torch.zeros(E, device=dev, dtype=i32)
    ms = timed(lambda: seqlib.router_topk(zr, E, E, top, None, False, ids, w_, None, counts, score=seqlib.ROUTER_SIGMOID, groups=z["G"], keep=z["keep"], scale=2.5))
    out["router_topk_sigmoid_groups"] = rate(ms, T * (E * 4 + top * 8))
    cor = torch.zeros(E, device=dev)
    ms = timed(lambda: seqlib.router_topk(zr, E, E, top, cor, False, ids, w_, None, counts))
    out["voduzen_router_topk_softmax"] = rate(ms, T * (E * 4 + top * 8))
    # ---- gate * up halves
    for name, act, ff, kw in (("glu_mul_clamp_swish", seqlib.ACT_CLAMP_SWISH, z["ff"], dict(limit=7.0, slope=1.702, shift=1.0)),
                              ("glu_mul_silu", seqlib.ACT_SILU, z["eff"] * top, {}), ("tifisun_glu_mul_gelu", seqlib.ACT_GELU_TANH, z["ff"], {})):
        gu, act_o = (torch.randn(T, 2 * ff, device=dev) * 2.0).to(bf), torch.empty(T, ff, device=dev, dtype=bf)
        ms = timed(lambda: seqlib.glu_mul(gu, ff, act, act_o, **kw))
        out[name] = rate(ms, T * ff * 6)
        del gu, act_o
    # ---- latent attention and what stands in front of it
    pages_per = L // page
    pool = (torch.randn(n_seq * pages_per + 1, page, D, device=dev) * 0.3).to(bf)
    table = (torch.arange(n_seq * pages_per, dtype=i32, device=dev) + 1).view(n_seq, pages_per).contiguous()
    dkv, qb = torch.randn(T, D, device=dev), torch.randn(T, H * (dn + dr), device=dev).to(bf)
    lw, cs = torch.ones(r, device=dev, dtype=bf), torch.randn(ctx + L, dr // 2, 2, device=dev)
    q = torch.empty(T, H, D, device=dev, dtype=bf)
    ms = timed(lambda: seqlib.latent_rope_store(dkv, r, dr, lw, 1e-6, cs, dr, pos, slot, table, page, pool, qb, H, dn, q))
    out["voduzen_latent_rope_store"] = rate(ms, T * (D * 6 + H * dr * 4))
    ms = timed(lambda: seqlib.latent_rope_store(None, r, dr, None, 1e-6, cs, dr, pos, slot, table, page, pool, qb, H, dn, q))
    out["latent_rope_queries_only"] = rate(ms, T * H * dr * 4)
    uk = torch.randn(H, r, dn, device=dev).to(bf)
    ms = timed(lambda: seqlib.linear(qb, uk, q, M=T, N=r, K=dn, ldx=qb.stride(0), sx=dn + dr, ldw=dn, sw=r * dn, ldy=H * D, sy=D, batch=H))
    out["voduzen_absorb_product"] = rate(ms, T * H * (dn + r) * 2, flops=T * H * dn * r * 2.0)
    q.normal_(std=0.3)
    o, gate = torch.empty(T, H, r, device=dev, dtype=bf), torch.randn(T, H, device=dev)
    portions = [(s * L, L, s, 0) for s in range(n_seq)]
    for name, win, gt in (("voduzen_latent_attn_prefill", seqlib.WINDOW_ALL, None), ("latent_attn_window_gate_prefill", z["win"], gate),
                          ("latent_attn_window256_gate_prefill", 256, gate)):
        plan = seqlib.LatentAttnPlan(portions, H, dev, window=win)
        ms = timed(lambda: seqlib.latent_attn_mma(q, r, dr, pool, table, page, plan, None, 0.07, o, window=win, gate=gt))
        vis = n_seq * sum(min(i + 1, win) for i in range(L))
        out[name] = rate(ms, flops=vis * H * 2.0 * (2 * r + dr), ctas=plan.n_items)
    del pool, q, o, qb
    pages_d = -(-(ctx + 1) // page)
    pool = (torch.randn(B * pages_d + 1, page, D, device=dev) * 0.3).to(bf)
    table = (torch.arange(B * pages_d, dtype=i32, device=dev) + 1).view(B, pages_d).contiguous()
    q = (torch.randn(B, H, D, device=dev) * 0.3).to(bf)
    o = torch.empty(B, H, r, device=dev, dtype=bf)
    for name, win, gt in (("voduzen_latent_attn_decode", seqlib.WINDOW_ALL, None), ("latent_attn_window_gate_decode", z["win"], gate[:B]),
                          ("latent_attn_window256_gate_decode", 256, gate[:B])):
        keys = min(win, ctx + 1)
        plan = seqlib.DecodeAttnPlan(B, H, LatentAttention._decode_parts(B, keys), dev, window=win)
        plan.fill(posd, slotd)
        ms = timed(lambda: seqlib.latent_attn_mma(q, r, dr, pool, table, page, plan, None, 0.07, o, window=win, gate=gt))
        out[name] = rate(ms, B * keys * D * 2, batch=B, keys=keys, ctas=plan.n_items)
    q32, qn = torch.randn(B, H * (dn + dr), device=dev), torch.empty(B, H * dn, device=dev, dtype=bf)
    ms = timed(lambda: seqlib.latent_rope_store(dkv[:B], r, dr, lw, 1e-6, cs, dr, posd, slotd, table, page, pool, q32, H, dn, q, qn=qn))
    out["latent_rope_store_fp32_queries_decode"] = rate(ms, B * (D * 6 + H * (dn + dr) * 6), batch=B)
    qb = q32.to(bf)
    ms = timed(lambda: seqlib.latent_rope_store(dkv[:B], r, dr, lw, 1e-6, cs, dr, posd, slotd, table, page, pool, qb, H, dn, q))
    out["voduzen_latent_rope_store_decode"] = rate(ms, B * (D * 6 + H * dr * 4), batch=B)
    return out


def measure(size="s", batches=(1, 32), ctx=1024, steps=32, prefill=4, with_kernels=True, with_voduzen=True):
    z = SIZES[size]
    rec = {"size": size, "dims": z}
    cfg = MunevikConfig.from_dict(config_dict(z))
    model = munevik.MunevikForCausalLM.from_state_dict(munevik.random_state_dict(cfg, seed=0), cfg, device="cuda:0")
    rec["munevik"] = serve(model, z["V"], prefill, batches, ctx, steps)
    del model
    torch.cuda.empty_cache()
    if with_voduzen:
        try:
            cfg = VoduzenConfig.from_dict(voduzen_dict(z))
            model = voduzen.VoduzenForCausalLM.from_state_dict(voduzen.random_state_dict(cfg, seed=0), cfg, device="cuda:0")
            rec["voduzen_equal_size"] = serve(model, z["V"], prefill, batches, ctx, steps)
            del model
            torch.cuda.empty_cache()
        except Exception as e:  # noqa: BLE001
            rec["voduzen_equal_size"] = {"error": f"{type(e).__name__}: {e}"[:300]}
    if with_kernels:
        rec["kernels"] = kernels(z, prefill, 1024, max(batches), ctx)
    return rec


def main():
    ap = argparse.ArgumentParser()
    ap.add_argument("--size", action="append", choices=sorted(SIZES))
    ap.add_argument("--batch", type=int, action="append")
    ap.add_argument("--ctx", type=int, default=1024)
    ap.add_argument("--steps", type=int, default=32)
    ap.add_argument("--prefill", type=int, default=4)
    a = ap.parse_args()
    torch.cuda.set_device(0)
    for s in a.size or ["s"]:
        print(json.dumps(measure(s, tuple(a.batch or [1, 32]), a.ctx, a.steps, a.prefill)), flush=True)


if __name__ == "__main__":
    main()
