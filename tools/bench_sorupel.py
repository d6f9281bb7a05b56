#!/usr/bin/env python
"""Sorupel decoder at sizes that resemble a real model's layers (random weights), beside the framework's closest existing model, the Tifisun
decoder (model/tifisun.py: recurrences with a matrix state per head, grouped attention over the last keys with normed queries and keys
and a soft cap, dense gated gelu feed-forwards, an fp32 residual stream), at equal width, depth, heads, key/value heads, head width,
attention reach, feed-forward width and vocabulary. Its latent attention is compared with the Voduzen form of the same kernels.

Per size: prefill of `--prefill` x 1024-token prompts as ONE packed step through serving.StepScheduler (tokens/s), decode steps at
batch B and context ctx through the same scheduler (ms/step, tokens/s), and the new kernels timed alone on one layer's shapes against
their rooflines, each beside the like kernel of an existing path:
  omc_linear_state_scan    step sizes, D. Prefill: FLOPs = rows x heads x 4 state vdim (decay and update count as one multiply-add each, the
                           read-out as one) on the fp32 FMA pipe (nominal 148 SMs x 128 lanes x 2 x clock) and bytes of its rows;
                           decode: the states read and written. like: one decay per head with and without the delta correction
                           (Tifisun; 6 and 4 state vdim) over as many state elements
  omc_gate_rms_rows, omc_rms_residual, omc_embed_bigram, omc_qk_norm_kv_store with rotation, omc_causal_conv (bias + silu, fp32 out): bytes
                           read + written; like: omc_gated_rms_rows (one group), omc_ln_residual, omc_embed_scale,
                           omc_qk_norm_kv_store without rotation, omc_causal_conv_silu without bias
  omc_window_attn_mma      with chunks, sink and head gates: FLOPs = visible keys x heads x 4 dim, decode: bytes of the visible rows; like:
                           a sliding window of the same reach (Tifisun)
  omc_linear_gate          FLOPs against the measured bf16 peak; like: the same product without a gate
  omc_latent_attn_mma      with a sink; like: without (Voduzen); omc_latent_rope_store with halves; like: with pairs
python tools/bench_sorupel.py --size s --size m
"""
import argparse
import json
import os
import sys

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
sys.path.insert(0, ROOT)

import torch  # noqa: E402

from omchat_b200 import seqlib  # noqa: E402
from omchat_b200.config import SorupelConfig, TifisunConfig  # noqa: E402
from omchat_b200.model import sorupel, tifisun  # noqa: E402
from omchat_b200.model.seq_latent import LatentAttention  # noqa: E402
from tools.bench_fofisun import serve  # noqa: E402
from tools.bench_tifisun import FMA_TFLOPS  # noqa: E402
from tools.bench_tifisun import config_dict as tifisun_dict  # noqa: E402
from tools.bench_voduzen import peaks, timed  # noqa: E402

# width, layers, latent heads / key (unrotated, rotated) and value widths / latent width, attention heads / key-value heads / head width /
# chunk, state-space heads / head width / state / groups / taps, ff, vocab, buckets
SIZES = {
    "s": dict(C=2048, L=6, H=16, dn=128, dr=64, dv=128, r=512, G=4, d=128, chunk=512, sH=64, P=64, N=128, sG=8, conv=4, ff=5632, V=32768, buckets=65536),
    "m": dict(C=4096, L=6, H=32, dn=128, dr=64, dv=128, r=512, G=8, d=128, chunk=512, sH=128, P=64, N=128, sG=8, conv=4, ff=8192, V=65536, buckets=131072),
}


def config_dict(z):
    mlp = {"ff": z["ff"], "kind": "dense"}
    lat = {"dim": z["dn"], "heads": z["H"], "kv_rank": z["r"], "rot": {"base": 1e6, "dims": z["dr"]}, "rot_dim": z["dr"],
           "scale": (z["dn"] + z["dr"]) ** -0.5, "vdim": z["dv"]}
    att = {"dim": z["d"], "heads": z["H"], "kv_heads": z["G"], "mask": {"size": z["chunk"]}, "rot": {"base": 1e5, "dims": z["d"] // 2}, "scale": z["d"] ** -0.5,
           "softcap": 50.0, "vdim": z["d"]}
    ssm = {"conv": z["conv"], "groups": z["sG"], "heads": z["sH"], "norm_groups": z["sG"], "state": z["N"], "vdim": z["P"]}
    kinds = [("mamba2", ssm), ("latent_attention", lat), ("attention", att), ("mamba2", ssm), ("latent_attention", dict(lat, kv_from=1)), ("attention", att)]
    return {"architecture": "Sorupel", "vocab": z["V"], "width": z["C"], "norm": {"eps": 1e-5},
            "embedding": {"bigram": {"buckets": z["buckets"], "mul_cur": 7919, "mul_prev": 104729}},
            "layers": [{"type": kinds[i % 6][0], "mixer": kinds[i % 6][1], "mlp": mlp} for i in range(z["L"])]}


def tifisun_size(z):
    """The equal-size neighbour in the terms of tools/bench_tifisun.py."""
    return dict(C=z["C"], L=z["L"], H=z["H"], G=z["G"], d=z["d"], dv=z["d"], conv=z["conv"], window=z["chunk"], rank=z["C"] // 32, ff=z["ff"], V=z["V"])


def kernels(z, n_seq, L, B, ctx):
    """The new kernels alone on one layer's shapes, each beside its like kernel."""
    hbm, tf = peaks()
    dev, bf, i32 = "cuda", torch.bfloat16, torch.int32
    C, H, r, dr, dn, dv, D = z["C"], z["H"], z["r"], z["dr"], z["dn"], z["dv"], z["r"] + z["dr"]
    page, out, T = 64, {}, n_seq * L
    pos = torch.arange(L, dtype=i32, device=dev).repeat(n_seq)
    slot = torch.arange(n_seq, dtype=i32, device=dev).repeat_interleave(L)
    rb = (torch.arange(n_seq + 1, dtype=i32, device=dev) * L).contiguous()
    posd = torch.full((B,), ctx, dtype=i32, device=dev)
    slotd = torch.arange(B, dtype=i32, device=dev)
    rbd = torch.arange(B + 1, dtype=i32, device=dev)
    S_ = max(n_seq, B)

    def rate(ms, nbytes=None, flops=None, peak=tf, **extra):
        rec = {"ms": ms, **extra}
        if nbytes is not None:
            rec.update(gbs=nbytes / ms / 1e6, frac_hbm=nbytes / ms / 1e6 / hbm)
        if flops is not None:
            rec.update(tflops=flops / ms / 1e9, frac_flops=flops / ms / 1e9 / peak)
        return rec

    # ---- recurrence and what stands around it
    sH, P, N, sG = z["sH"], z["P"], z["N"], z["sG"]
    inner, gn = sH * P, sG * N
    ch = inner + 2 * gn
    zz = torch.randn(T, ch + sH, device=dev)
    u, cw, cb = torch.empty(T, ch, device=dev), (torch.randn(ch, z["conv"], device=dev) * 0.4).to(bf), torch.zeros(ch, device=dev, dtype=bf)
    ring = torch.zeros(S_, z["conv"] - 1, ch, device=dev)
    ms = timed(lambda: seqlib.causal_conv_silu(zz[:, :ch], cw, pos, slot, ring, u, bias=cb))
    out["causal_conv_bias_silu"] = rate(ms, T * ch * 8)
    ms = timed(lambda: seqlib.causal_conv_silu(zz[:, :ch], cw, pos, slot, ring, u))
    out["tifisun_causal_conv_silu"] = rate(ms, T * ch * 8)
    A_log, dtb, Dv = torch.zeros(sH, device=dev), torch.full((sH,), -3.0, device=dev), torch.ones(sH, device=dev)
    state, y = torch.zeros(S_, sH, N, P, device=dev), torch.empty(T, inner, device=dev)
    x_, B_, C_, a = u[:, :inner], u[:, inner:inner + gn], u[:, inner + gn:], zz[:, ch:]
    beta, rows_b = torch.randn(T, sH, device=dev), T * (2 * inner + 2 * gn + sH) * 4 + 2 * n_seq * sH * N * P * 4
    for name, kw, per in (("state_scan_step_sizes", dict(step_size=True, a=a, A_log=A_log, dt_bias=dtb, D=Dv), 6.0),
                          ("tifisun_state_scan_delta", dict(a=a, A_log=A_log, dt_bias=dtb, beta=beta), 8.0),
                          ("tifisun_state_scan_head_decay", dict(a=a, A_log=A_log, dt_bias=dtb), 6.0)):
        ms = timed(lambda: seqlib.linear_state_scan(C_, B_, x_, state, y, rb, n_seq, pos, slot, sH, sG, N, P, **kw))
        out[name + "_prefill"] = rate(ms, rows_b, flops=T * sH * per * N * P, peak=FMA_TFLOPS)
        kwd = {k: (v[:B] if k in ("a", "beta") else v) for k, v in kw.items()}
        ms = timed(lambda: seqlib.linear_state_scan(C_[:B], B_[:B], x_[:B], state, y[:B], rbd, B, posd, slotd, sH, sG, N, P, **kwd))
        out[name + "_decode"] = rate(ms, 2.0 * B * sH * N * P * 4, batch=B)
    nw, yn, zb = torch.ones(inner, device=dev, dtype=bf), torch.empty(T, inner, device=dev, dtype=bf), torch.randn(T, inner, device=dev).to(bf)
    ms = timed(lambda: seqlib.gate_rms_rows(y, sG, nw, 1e-5, zb, seqlib.GATE_SILU, yn))
    out["gate_rms_rows"] = rate(ms, T * inner * 8)
    zf = zb.float()
    ms = timed(lambda: seqlib.gated_rms_rows(y, sG, inner // sG, nw[:inner // sG], 1e-5, zf, seqlib.GATE_SILU, yn))
    out["tifisun_gated_rms_rows"] = rate(ms, T * inner * 10)
    ms = timed(lambda: seqlib.gate_rms_rows(y[:B], sG, nw, 1e-5, zf[:B], seqlib.GATE_SILU, yn[:B]))
    out["gate_rms_rows_decode"] = rate(ms, B * inner * 10, batch=B)
    ms = timed(lambda: seqlib.gated_rms_rows(y[:B], sG, inner // sG, nw[:inner // sG], 1e-5, zf[:B], seqlib.GATE_SILU, yn[:B]))
    out["tifisun_gated_rms_rows_decode"] = rate(ms, B * inner * 10, batch=B)
    del zz, u, state, y, yn, zb, zf, x_, B_, C_, a
    # ---- residual sum + norm, embedding
    x, y = torch.randn(T, C, device=dev), torch.randn(T, C, device=dev)
    xb = torch.empty(T, C, device=dev, dtype=bf)
    nw, nb = torch.ones(C, device=dev, dtype=bf), torch.zeros(C, device=dev, dtype=bf)
    for suffix, n in (("", T), ("_decode", B)):
        ms = timed(lambda: seqlib.rms_residual(x[:n], nw, 1e-5, y=y[:n], x_out=x[:n], xb=xb[:n]))
        out["rms_residual" + suffix] = rate(ms, n * C * 14)
        ms = timed(lambda: seqlib.ln_residual(x[:n], 1.0, nw, nb, 1e-5, y=y[:n], x_out=x[:n], xb=xb[:n]))
        out["munevik_ln_residual" + suffix] = rate(ms, n * C * 14)
        ms = timed(lambda: seqlib.post_norm_residual(y[:n], nw, 1e-5, 1.0, x[:n], nw, xb[:n]))
        out["tifisun_post_norm_residual" + suffix] = rate(ms, n * C * 14)
    table, big, prev = torch.randn(z["V"], C, device=dev).to(bf), torch.randn(z["buckets"] + 1, C, device=dev).to(bf), torch.zeros(S_, device=dev, dtype=i32)
    ids = torch.randint(0, z["V"], (T,), device=dev).to(i32)
    ms = timed(lambda: seqlib.embed_bigram(ids, pos, slot, table, big, 104729, 7919, prev, x, nw=nw, eps=1e-5, xb=xb))
    out["embed_bigram_norm"] = rate(ms, T * C * 10)
    ms = timed(lambda: seqlib.embed_scale(ids, table, 1.0, x, xb))
    out["tifisun_embed_scale"] = rate(ms, T * C * 8)
    del x, y, xb, table, big
    # ---- chunked attention and what stands in front of it
    G, d, chunk = z["G"], z["d"], z["chunk"]
    nq, nk = H * d, G * d
    zq, qo = torch.randn(T, nq + nk + H, device=dev), torch.empty(T, nq, device=dev, dtype=bf)
    pages_per = -(-L // page)
    pool = (torch.randn(n_seq * pages_per + 1, page, 2 * nk, device=dev) * 0.3).to(bf)
    table = (torch.arange(n_seq * pages_per, dtype=i32, device=dev) + 1).view(n_seq, pages_per).contiguous()
    wq, wk, cs = torch.ones(nq, device=dev, dtype=bf), torch.ones(nk, device=dev, dtype=bf), torch.randn(ctx + L, d // 4, 2, device=dev)
    for name, kw in (("qk_norm_rope_store", dict(cs=cs, head=d, rot_dims=d // 2, rot_halves=True)), ("tifisun_qk_norm_store", {})):
        ms = timed(lambda: seqlib.qk_norm_kv_store(zq[:, :nq], wq, zq[:, nq:nq + nk], wk, zq[:, nq:nq + nk], 1e-5, pos, slot, table, page, pool, qo, **kw))
        out[name] = rate(ms, T * (nq * 6 + nk * 8))
        ms = timed(lambda: seqlib.qk_norm_kv_store(zq[:B, :nq], wq, zq[:B, nq:nq + nk], wk, zq[:B, nq:nq + nk], 1e-5, pos, slot, table, page, pool, qo, **kw))
        out[name + "_decode"] = rate(ms, B * (nq * 6 + nk * 8), batch=B)
    qb, att = (torch.randn(T, nq, device=dev) * 0.3).to(bf), torch.empty(T, nq, device=dev, dtype=bf)
    one, gate = torch.zeros(H, device=dev), zq[:, nq + nk:]
    portions = [(s * L, L, s, 0) for s in range(n_seq)]
    forms = (("chunk_attn", seqlib.WINDOW_ALL, dict(chunk=chunk, sink=one, gate=gate, gate_act=seqlib.GATE_SIGMOID, gate_heads=True), sum(i % chunk + 1 for i in range(L))),
             ("tifisun_window_attn", chunk, {}, sum(min(i + 1, chunk) for i in range(L))))
    for name, win, kw, vis in forms:
        items = seqlib.window_attn_items(portions, H // G, dev, kw.get("chunk", seqlib.WINDOW_ALL))
        ms = timed(lambda: seqlib.window_attn_mma(qb, H, G, d, d, pool, table, page, items, pos, slot, win, d ** -0.5, 50.0, None, att, **kw))
        out[name + "_prefill"] = rate(ms, flops=n_seq * vis * H * 4.0 * d, ctas=int(items.shape[0]) * G)
    del pool, zq
    pages_d = -(-(ctx + 1) // page)
    pool = (torch.randn(B * pages_d + 1, page, 2 * nk, device=dev) * 0.3).to(bf)
    tabled = (torch.arange(B * pages_d, dtype=i32, device=dev) + 1).view(B, pages_d).contiguous()
    posc = torch.full((B,), ctx // chunk * chunk - 1, dtype=i32, device=dev)     # the last row of a chunk: as many keys as the window
    for name, win, kw, _ in forms:
        kw = {k: (v[:B] if k == "gate" else v) for k, v in kw.items()}
        ms = timed(lambda: seqlib.window_attn_mma(qb[:B], H, G, d, d, pool, tabled, page, None, posc, slotd, win, d ** -0.5, 50.0, None, att[:B], **kw))
        out[name + "_decode"] = rate(ms, B * chunk * 2 * nk * 2, batch=B, keys=chunk, ctas=B * G)
    del pool, qb, att
    # ---- latent attention, its rotation and its gated values
    lpool = (torch.randn(n_seq * pages_per + 1, page, D, device=dev) * 0.3).to(bf)
    dkv, qb = torch.randn(T, D, device=dev), torch.randn(T, H * (dn + dr), device=dev).to(bf)
    lw, cs, q = torch.ones(r, device=dev, dtype=bf), torch.randn(ctx + L, dr // 2, 2, device=dev), torch.empty(T, H, D, device=dev, dtype=bf)
    for name, hv in (("latent_rope_store_halves", True), ("voduzen_latent_rope_store", False)):
        ms = timed(lambda: seqlib.latent_rope_store(dkv, r, dr, lw, 1e-6, cs, dr, pos, slot, table, page, lpool, qb, H, dn, q, rot_halves=hv))
        out[name] = rate(ms, T * (D * 6 + H * dr * 4))
    q.normal_(std=0.3)
    o, sink = torch.empty(T, H, r, device=dev, dtype=bf), torch.zeros(H, device=dev)
    plan = seqlib.LatentAttnPlan(portions, H, dev)
    for name, sk in (("latent_attn_sink", sink), ("voduzen_latent_attn", None)):
        ms = timed(lambda: seqlib.latent_attn_mma(q, r, dr, lpool, table, page, plan, sk, 0.07, o))
        out[name + "_prefill"] = rate(ms, flops=n_seq * L * (L + 1) / 2 * H * 2.0 * (2 * r + dr), ctas=plan.n_items)
    uv, att, g = torch.randn(H * dv, r, device=dev).to(bf), torch.empty(T, H * dv, device=dev, dtype=bf), torch.randn(T, H * dv, device=dev).to(bf)
    for suffix, n, gt in (("", T, g), ("_decode", B, g.float())):
        for name, gg in (("value_product_gate", gt[:n]), ("voduzen_value_product", None)):
            ms = timed(lambda: seqlib.linear(o[:n], uv, att[:n], M=n, N=dv, K=r, ldx=H * r, sx=r, ldw=r, sw=dv * r, ldy=H * dv, sy=dv, batch=H, gate=gg))
            out[name + suffix] = rate(ms, n * H * (r + 2 * dv) * 2 + H * dv * r * 2, flops=n * H * r * dv * 2.0)
    del lpool, q, o
    lpool = (torch.randn(B * pages_d + 1, page, D, device=dev) * 0.3).to(bf)
    q, o = (torch.randn(B, H, D, device=dev) * 0.3).to(bf), torch.empty(B, H, r, device=dev, dtype=bf)
    plan = seqlib.DecodeAttnPlan(B, H, LatentAttention._decode_parts(B, ctx + 1), dev)
    plan.fill(posd, slotd)
    for name, sk in (("latent_attn_sink", sink), ("voduzen_latent_attn", None)):
        ms = timed(lambda: seqlib.latent_attn_mma(q, r, dr, lpool, tabled, page, plan, sk, 0.07, o))
        out[name + "_decode"] = rate(ms, B * (ctx + 1) * D * 2, batch=B, keys=ctx + 1, ctas=plan.n_items)
    return out


def measure(size="s", batches=(1, 32), ctx=1024, steps=32, prefill=4, with_kernels=True, with_tifisun=True):
    z = SIZES[size]
    rec = {"size": size, "dims": z}
    cfg = SorupelConfig.from_dict(config_dict(z))
    model = sorupel.SorupelForCausalLM.from_state_dict(sorupel.random_state_dict(cfg, seed=0), cfg, device="cuda:0")
    rec["sorupel"] = serve(model, z["V"], prefill, batches, ctx, steps)
    del model
    torch.cuda.empty_cache()
    if with_tifisun:
        try:
            t = tifisun_size(z)
            cfg = TifisunConfig.from_dict(tifisun_dict(t))
            model = tifisun.TifisunForCausalLM.from_state_dict(tifisun.random_state_dict(cfg, seed=0, decay_rank=t["rank"], gate_rank=t["rank"], bias_rows=32), cfg,
                                                               device="cuda:0")
            rec["tifisun_equal_size"] = serve(model, z["V"], prefill, batches, ctx, steps)
            del model
            torch.cuda.empty_cache()
        except Exception as e:  # noqa: BLE001
            rec["tifisun_equal_size"] = {"error": f"{type(e).__name__}: {e}"[:300]}
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
