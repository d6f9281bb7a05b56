"""Small Sorupel configurations and helpers shared by the Sorupel tests."""
import torch

from oracle import sorupel_oracle as O

F64 = torch.float64


def dense(ff):
    return {"ff": ff, "kind": "dense"}


def latent(heads, dim, rot, vdim, rank, mlp, base=3000.0, kv_from=None, scale=None):
    m = {"dim": dim, "heads": heads, "kv_rank": rank, "rot": {"base": base, "dims": rot}, "rot_dim": rot,
         "scale": scale if scale is not None else (dim + rot) ** -0.5, "vdim": vdim}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def ssm(heads, vdim, state, groups, conv, norm_groups, mlp):
    return {"type": "mamba2", "mixer": {"conv": conv, "groups": groups, "heads": heads, "norm_groups": norm_groups, "state": state, "vdim": vdim}, "mlp": mlp}


def attention(heads, kv_heads, dim, rot, chunk, mlp, softcap=9.0, base=500.0, scale=None):
    m = {"dim": dim, "heads": heads, "kv_heads": kv_heads, "rot": {"base": base, "dims": rot}, "scale": scale if scale is not None else dim ** -0.5,
         "softcap": softcap, "vdim": dim}
    if chunk is not None:
        m["mask"] = {"size": chunk}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def model_dict(vocab, width, layers, page=16, eps=1e-5, bigram=(61, 7, 3)):
    emb = {"bigram": {"buckets": bigram[0], "mul_prev": bigram[1], "mul_cur": bigram[2]}} if bigram else {}
    return {"architecture": "Sorupel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": emb, "kv_page_size": page, "layers": layers}


def config_a(page=16):
    """Every mechanism, widths that are no multiples of 8 or 32, rows shared by two layers with heads and widths of their own, an attention
    layer first, a layer without feed-forward, heads that do not divide a tile, key widths that are rotated in part."""
    return model_dict(131, 72, [
        attention(6, 2, 10, 6, 25, dense(50)),
        latent(3, 10, 6, 14, 20, dense(33)),
        ssm(6, 10, 12, 3, 4, 4, dense(40)),
        latent(5, 12, 6, 8, 20, None, kv_from=1),
        ssm(4, 9, 7, 1, 3, 1, None),
        attention(5, 1, 14, 14, 40, dense(21), softcap=2.5, base=77.0),
        latent(2, 24, 8, 20, 12, dense(9), base=77.0),
        latent(4, 8, 6, 12, 20, dense(30), kv_from=1)], page=page)


def config_b(page=32):
    """Ones and equal values: one head, one state, one channel, one tap, one bucket, no rotation, no chunk, no soft cap, a chunk of one key, an
    odd width."""
    return model_dict(67, 45, [
        ssm(1, 1, 1, 1, 1, 1, dense(1)),
        latent(1, 16, 16, 16, 16, dense(45)),
        attention(1, 1, 8, 0, None, None, softcap=0.0),
        ssm(3, 3, 45, 3, 2, 9, dense(24)),
        latent(1, 16, 16, 16, 16, None, kv_from=1),
        attention(4, 4, 6, 6, 1, dense(12), softcap=1.0),
        attention(2, 2, 4, 2, 3, dense(8)),
        latent(2, 7, 0, 5, 9, dense(8)),
        ssm(8, 6, 5, 2, 6, 2, dense(8))], page=page, bigram=(1, 5, 9))


def config_c(page=16):
    """Attention shapes the tensor-core kernels take (bf16): a latent layer with three heads (a tile of 64 rows holds 21 tokens), groups of
    three, five and one query heads, chunks shorter and longer than a tile."""
    return model_dict(110, 64, [
        latent(4, 32, 16, 24, 48, dense(80)),
        attention(6, 2, 32, 16, 33, dense(64)),
        ssm(4, 32, 16, 2, 4, 2, dense(48)),
        latent(3, 16, 16, 40, 48, None, kv_from=0),
        attention(5, 1, 16, 16, 100, dense(32), softcap=20.0),
        attention(2, 2, 48, 32, None, dense(32), softcap=0.0),
        latent(16, 16, 32, 16, 144, dense(32))], page=page, bigram=(97, 31, 5))


def config_d(page=64):
    """Matrices large enough for the tensor-core GEMMs, states as wide as the scan's larger forms."""
    return model_dict(520, 384, [
        latent(8, 64, 32, 64, 192, dense(1536)),
        ssm(12, 64, 128, 4, 4, 3, dense(1536)),
        attention(8, 2, 64, 64, 50, dense(768)),
        latent(8, 64, 32, 64, 192, dense(384), kv_from=0)], page=page, bigram=(1000, 519, 2))


CONFIGS = {"a": config_a, "b": config_b, "c": config_c, "d": config_d}


def config_for(name, dtype):
    """fp32: the configuration as it is. bf16: no state-space layer whose norm runs over a single number - that is its sign, which a rounding
    of a value near zero flips."""
    cd = CONFIGS[name]()
    for l in cd["layers"]:
        m = l["mixer"]
        if dtype != torch.float32 and l["type"] == "mamba2" and m["heads"] * m["vdim"] == m["norm_groups"]:
            m.update(norm_groups=1, vdim=max(m["vdim"], 4))
    return cd


def tokens_for(cfg_dict, n, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, cfg_dict["vocab"], (n,), generator=g).tolist()


def row_errors(got, want):
    """Per row: RMS difference of mean-free logits relative to the RMS of the reference row."""
    d = got.double().cpu() - want.double()
    d = d - d.mean(-1, keepdim=True)
    w = want.double() - want.double().mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt().clamp_min(1e-9)


def close(got, want, dtype):
    """fp32: every row within 1e-4. bf16: every row within 0.1 and nine in ten within 4e-2."""
    e = row_errors(got, want)
    if dtype == torch.float32:
        return float(e.max()) < 1e-4
    return float(e.max()) < 0.1 and float(torch.quantile(e, 0.9)) < 4e-2


def rand(*shape, seed=0, s=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=F64) * s


__all__ = ["O", "F64", "CONFIGS", "tokens_for", "row_errors", "close", "config_for", "rand", "config_a", "config_b", "config_c", "config_d", "latent", "ssm", "attention",
           "dense", "model_dict"]
