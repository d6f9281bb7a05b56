"""Small Munevik configurations and helpers shared by the Munevik tests."""
import torch

from oracle import munevik_oracle as O

F64 = torch.float64


def dense(ff, limit):
    return {"ff": ff, "kind": "dense", "limit": limit}


def moe(experts, top, ff, count=1, keep=1, scale=1.0, shared=None):
    return {"expert": {"ff": ff}, "kind": "moe", "router": {"experts": experts, "groups": {"count": count, "keep": keep}, "scale": scale, "top": top},
            "shared": {"ff": shared} if shared else None}


def lru(width, blocks, conv, mlp):
    return {"type": "rglru", "mixer": {"blocks": blocks, "conv": conv, "width": width}, "mlp": mlp}


def latent(heads, dim, rot, vdim, rank, window, mlp, base=3000.0, kv_from=None, scale=None):
    m = {"dim": dim, "heads": heads, "kv_rank": rank, "mask": {"size": window}, "rot": {"base": base, "dims": rot}, "rot_dim": rot,
         "scale": scale if scale is not None else (dim + rot) ** -0.5, "vdim": vdim}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def model_dict(vocab, width, layers, page=16, alpha=1.7, eps=1e-5):
    return {"architecture": "Munevik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "kv_page_size": page, "layers": layers}


def config_a(page=16):
    """Every mechanism, widths that are no multiples of 8 or 32, a shared cache read by two layers with windows, heads and widths of their
    own, an attention layer first, a layer without feed-forward, three kept groups of five."""
    return model_dict(131, 72, [
        latent(3, 10, 6, 14, 20, 25, moe(15, 3, 20, 5, 3, 2.5, 28)),
        lru(60, 5, 4, dense(50, 1.2)),
        latent(5, 12, 6, 8, 20, 7, None, kv_from=0),
        lru(36, 3, 3, moe(6, 2, 24, 3, 2, 0.7)),
        latent(2, 24, 8, 20, 12, 40, dense(33, 0.8), base=77.0),
        latent(4, 8, 6, 12, 20, 300, moe(8, 2, 16, 2, 1, 1.0, 12), kv_from=0)], page=page)


def config_b(page=32):
    """Ones and equal values: one head, one block, one tap, one expert out of one, every expert chosen, groups of one expert, all groups
    kept, a window of one key, alpha 1, an odd width."""
    return model_dict(67, 45, [
        lru(9, 1, 1, moe(1, 1, 24)),
        latent(1, 16, 16, 16, 16, 1, moe(4, 4, 12, 4, 4, 1.0, 45)),
        lru(45, 9, 2, None),
        latent(1, 16, 16, 16, 16, 2, moe(6, 2, 10, 6, 3, 1.5), kv_from=1),
        lru(8, 8, 6, dense(1, 3.0))], page=page, alpha=1.0)


def config_c(page=16):
    """Attention shapes the tensor-core kernel takes (bf16), one of them with three heads (a tile of 64 rows holds 21 tokens)."""
    return model_dict(110, 64, [
        lru(96, 3, 4, dense(80, 1.0)),
        latent(4, 32, 16, 24, 48, 33, moe(8, 2, 32, 4, 2, 1.3, 40)),
        latent(3, 16, 16, 40, 48, 64, moe(8, 3, 32, 2, 1, 1.0, 16), kv_from=1),
        latent(16, 16, 32, 16, 144, 20, None)], page=page, alpha=3.0)


def config_d(page=64):
    """Matrices large enough for the tensor-core GEMMs (skinny decode GEMM, grouped expert GEMM over 128-row tiles)."""
    return model_dict(520, 384, [
        lru(768, 6, 4, moe(8, 2, 768, 4, 2, 2.0, 768)),
        latent(8, 64, 32, 64, 192, 50, dense(1536, 2.0)),
        latent(8, 64, 32, 64, 192, 21, moe(8, 2, 768, 2, 1, 1.0, 384), kv_from=1)], page=page)


CONFIGS = {"a": config_a, "b": config_b, "c": config_c, "d": config_d}


def tokens_for(cfg_dict, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg_dict["vocab"], (n,), generator=g).tolist()


def row_errors(got, want):
    """Per row: RMS difference of mean-free logits relative to the RMS of the reference row."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().clamp_min(1e-9)


def all_experts(cfg_dict):
    """The same model with every group kept and every expert chosen. In bf16 a rounding now and then moves a token to another expert
    (weights are not renormalised, so its row changes visibly); without a choice every row is held to the rounding itself."""
    for l in cfg_dict["layers"]:
        if l["mlp"] and l["mlp"]["kind"] == "moe":
            r = l["mlp"]["router"]
            r["top"], r["groups"]["keep"] = r["experts"], r["groups"]["count"]
    return cfg_dict


def config_for(name, dtype):
    """fp32: the configuration as it is; bf16: without a choice of experts."""
    cd = CONFIGS[name]()
    return cd if dtype == torch.float32 else all_experts(cd)


def close(got, want, dtype):
    """fp32: every row within 2e-4. bf16 (config_for): every row within 0.12 and nine in ten within 4e-2."""
    e = row_errors(got, want)
    if dtype == torch.float32:
        return float(e.max()) < 2e-4
    return float(e.max()) < 0.12 and float(torch.quantile(e, 0.9)) < 4e-2


def rand(*shape, seed=0, s=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64) * s


__all__ = ["O", "F64", "CONFIGS", "tokens_for", "row_errors", "close", "config_for", "rand", "config_a", "config_b", "config_c", "config_d"]
