"""The mechanisms of the Munevik decoder alone on the GPU, each against the plain restatement in oracle/munevik_oracle.py (float64).

Engineered inputs where random ones would hide a fault: a key whose score stands out just inside and just outside a window, at page
borders and at the first position, in prompt portions and for decoded rows; a state whose decay is nearly one; poisoned slots."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu

if not torch.cuda.is_available():  # collected on the CPU box too
    pytest.skip("needs a CUDA device", allow_module_level=True)

from munevik_cases import F64, O, rand  # noqa: E402
from omchat_b200 import seqlib  # noqa: E402
from omchat_b200.config import RotarySpec  # noqa: E402
from omchat_b200.model.seq_latent import RotaryTables  # noqa: E402

DEV = "cuda:0"


def _dev(t, dt=torch.float32):
    return t.to(device=DEV, dtype=dt).contiguous()


def _i32(x):
    return torch.tensor(x, device=DEV, dtype=torch.int32)


# --------------------------------------------------------------------------------------- residual sum, combine and layer norm
@pytest.mark.parametrize("C", [256, 384, 1000, 2048, 4096, 6000, 45, 1, 9000])
@pytest.mark.parametrize("with_y,top", [(True, 0), (False, 0), (True, 3), (False, 1)])
def test_layer_norm_after_the_residual_sum(C, with_y, top):
    """Also rows far from zero mean: the variance is taken about the mean."""
    T, eps, alpha = 7, 1e-5, 1.7
    x, y = rand(T, C, seed=1) + 30.0, rand(T, C, seed=2)
    nw, nb = rand(C, seed=3), rand(C, seed=4)
    ys, w = rand(T * max(top, 1) + 2, C, seed=5), rand(T, max(top, 1), seed=6)
    slot_of = torch.randperm(T * max(top, 1), generator=torch.Generator().manual_seed(1)).view(T, -1)
    slot_of[2, 0] = -1
    v = alpha * x.float().double()
    if with_y:
        v = v + y.float().double()
    for t in range(T):
        for j in range(top):
            if slot_of[t, j] >= 0:
                v[t] += w[t, j] * ys[slot_of[t, j]]
    want = O.layer_norm(v, nw, nb, eps)
    for dt in (torch.float32, torch.bfloat16):
        xd, xb = _dev(x), torch.full((T, C), float("nan"), device=DEV, dtype=dt)
        kw = dict(ys=_dev(ys), slot_of=_i32(slot_of.tolist()), w=_dev(w), top=top) if top else {}
        seqlib.ln_residual(xd, alpha, _dev(nw), _dev(nb), eps, y=_dev(y) if with_y else None, x_out=xd, xb=xb, **kw)
        assert (xd.double().cpu() - want).abs().max() < 3e-4
        assert torch.equal(xb, xd.to(dt))
    only = torch.empty(T, C, device=DEV, dtype=torch.bfloat16)
    keep = _dev(x)
    seqlib.ln_residual(keep, 1.0, _dev(nw, torch.bfloat16), _dev(nb, torch.bfloat16), eps, xb=only)
    ref = O.layer_norm(x.float().double(), nw.bfloat16(), nb.bfloat16(), eps)
    assert torch.equal(keep, _dev(x)) and (only.double().cpu() - ref).abs().max() < 3e-2 * max(1.0, float(ref.abs().max()))


# ------------------------------------------------------------------------------------------------------------------- router
@pytest.mark.parametrize("E,groups,keep,top", [(15, 5, 3, 3), (16, 4, 3, 4), (6, 6, 3, 2), (8, 2, 1, 4), (64, 8, 4, 6), (120, 40, 7, 5), (1, 1, 1, 1), (12, 3, 3, 5)])
def test_group_limited_sigmoid_router(E, groups, keep, top):
    T, scale = 41, 2.5
    z = rand(T, E, seed=E, s=1.5).float().double()
    z[3] = 0.25                                # ties everywhere: lowest indices
    if groups > 1 and E // groups > 1:
        z[5], z[5, 0] = -3.0, 4.0              # the best expert sits in a group whose second best is poor ...
        z[5, E // groups:] = 1.0               # ... and every other group has a better pair of scores
    ids, w = torch.empty(T, top, device=DEV, dtype=torch.int32), torch.empty(T, top, device=DEV)
    counts = torch.zeros(E, device=DEV, dtype=torch.int32)
    seqlib.router_topk(_dev(z), E, E, top, None, False, ids, w, None, counts, score=seqlib.ROUTER_SIGMOID, groups=groups, keep=keep, scale=scale)
    s = torch.sigmoid(z)
    n = torch.zeros(E, dtype=torch.int64)
    for t in range(T):
        order = O.group_limited_choice(s[t].tolist(), top, {"count": groups, "keep": keep})
        assert ids[t].tolist() == order, t
        assert (w[t].double().cpu() - scale * s[t, order]).abs().max() < 1e-6
        n[order] += 1
    assert torch.equal(counts.cpu().long(), n)


def test_router_refuses_groups_that_do_not_fit():
    z, ids, w, c = torch.zeros(2, 10, device=DEV), torch.empty(2, 4, device=DEV, dtype=torch.int32), torch.empty(2, 4, device=DEV), torch.zeros(10, device=DEV, dtype=torch.int32)
    for kw in (dict(groups=3, keep=1), dict(groups=5, keep=6), dict(groups=5, keep=1), dict(groups=5, keep=0)):
        with pytest.raises(seqlib.OmcError):
            seqlib.router_topk(z, 10, 10, 4, None, False, ids, w, None, c, score=seqlib.ROUTER_SIGMOID, **kw)


def test_clamped_swish_feed_forward_halves():
    z, lim = rand(19, 2 * 36, seed=1, s=3.0), 1.3
    out = seqlib.glu_mul(_dev(z), 36, seqlib.ACT_CLAMP_SWISH, torch.empty(19, 36, device=DEV), limit=lim, slope=1.702, shift=1.0)
    g, u = z[:, :36].clamp(max=lim), z[:, 36:].clamp(-lim, lim)
    assert (out.double().cpu() - g * torch.sigmoid(1.702 * g) * (u + 1.0)).abs().max() < 1e-5


# --------------------------------------------------------------------------------------------------------------- recurrence
def _cut_rows(cuts, step, slots):
    rows = [(r, cuts[r][step], cuts[r][step + 1], sl) for r, sl in enumerate(slots)]
    pos = [p for _, lo, hi, _ in rows for p in range(lo, hi)]
    slot = [sl for _, lo, hi, sl in rows for _ in range(lo, hi)]
    return rows, pos, slot


@pytest.mark.parametrize("taps,ch,dt", [(4, 40, torch.float32), (3, 516, torch.bfloat16), (2, 45, torch.float32), (1, 12, torch.float32), (6, 24, torch.float32)])
@pytest.mark.parametrize("long_step", [False, True])
def test_convolution_with_bias_in_portions_over_poisoned_rings(taps, ch, dt, long_step):
    """Two requests in interleaved portions (1, 2, more tokens); x is a column slice of a wider row, as in the model."""
    n = [300, 290] if long_step else [23, 17]
    cuts = ([0, 1, 3, 4, 260, n[0]], [0, 2, 3, 270, 271, n[1]]) if long_step else ([0, 1, 3, 4, 11, n[0]], [0, 1, 3, 9, 10, n[1]])
    x, w, b = [rand(n[r], ch, seed=r) for r in range(2)], rand(ch, taps, seed=2, s=0.6), rand(ch, seed=3)
    want = [O.shift_conv(x[r], w, b) for r in range(2)]
    ring = torch.full((3, taps - 1, ch), float("nan"), device=DEV) if taps > 1 else None
    for step in range(5):
        rows, pos, slot = _cut_rows(cuts, step, (2, 0))
        wide = torch.randn(len(pos), 2 * ch, device=DEV)
        wide[:, ch:] = _dev(torch.cat([x[r][lo:hi] for r, lo, hi, _ in rows]))
        y = torch.empty(len(pos), ch, device=DEV, dtype=dt)
        seqlib.causal_conv_silu(wide[:, ch:], _dev(w), _i32(pos), _i32(slot), ring, y, act=seqlib.CONV_LINEAR, bias=_dev(b),
                                single_rows=all(hi - lo == 1 for _, lo, hi, _ in rows))
        ref = torch.cat([want[r][lo:hi] for r, lo, hi, _ in rows])
        assert (y.double().cpu() - ref).abs().max() < (2e-5 if dt == torch.float32 else 3e-2), step


@pytest.mark.parametrize("W,blocks,dt", [(40, 4, torch.float32), (9, 1, torch.float32), (33, 3, torch.float32), (130, 130, torch.float32), (96, 2, torch.bfloat16)])
@pytest.mark.parametrize("long_step", [False, True])
def test_gated_linear_recurrent_unit_in_portions_against_the_token_loop(W, blocks, dt, long_step):
    """Two requests over poisoned state slots: portions of 1, 2 and many tokens, so that the kernel spreads them over one, two, eight
    and sixteen runs of tokens, with ends inside a run."""
    n = [700, 410] if long_step else [37, 29]
    cuts = ([0, 1, 3, 133, 390, n[0]], [0, 2, 3, 200, 201, n[1]]) if long_step else ([0, 1, 3, 4, 20, n[0]], [0, 1, 3, 19, 20, n[1]])
    nb = W // blocks
    lam, br, bi = rand(W, seed=1, s=1.5) - 4.0, rand(W, seed=2), rand(W, seed=3)
    order = torch.stack([torch.arange(W).view(blocks, nb), W + torch.arange(W).view(blocks, nb)], dim=1).reshape(-1)   # block by block: r, then i
    gb = torch.cat([br, bi])[order]
    ins, want = [], []
    for r in range(2):
        u, zr, zi, y = rand(n[r], W, seed=10 + r).to(dt).double(), rand(n[r], W, seed=20 + r, s=2.0), rand(n[r], W, seed=30 + r, s=2.0), rand(n[r], W, seed=40 + r)
        ins.append((u, torch.cat([zr, zi], dim=1)[:, order], y))
        want.append(O.rglru_recurrence(u, torch.sigmoid(zr + br), torch.sigmoid(zi + bi), lam) * O.gelu_tanh(y))
    state = torch.full((3, W), float("nan"), device=DEV)
    for step in range(5):
        rows, pos, slot = _cut_rows(cuts, step, (2, 0))
        cat = lambda i: torch.cat([ins[r][i][lo:hi] for r, lo, hi, _ in rows])
        out = torch.empty(len(pos), W, device=DEV, dtype=dt)
        rb = _i32([0, rows[0][2] - rows[0][1], len(pos)])
        seqlib.rglru_scan(_dev(cat(0), dt), _dev(cat(1)), _dev(gb), _dev(lam), _dev(cat(2)), state, out, rb, 2, _i32(pos), _i32(slot), blocks, 8.0)
        ref = torch.cat([want[r][lo:hi] for r, lo, hi, _ in rows])
        assert (out.double().cpu() - ref).abs().max() < (2e-5 if dt == torch.float32 else 2e-2) * max(1.0, float(ref.abs().max())), step


@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16])
def test_a_slow_channel_keeps_the_digits_of_its_decay_for_a_thousand_tokens(dt):
    """lam = -12: a = 1 - 2e-5 at r = 0.4, whose own rounding to fp32 would cost up to 3e-5 of the state over 1000 tokens. Token 0 is
    read back a thousand tokens later, through long portions, short ones and single rows; the gelu branch is off (y absent)."""
    W, n = 5, 1100
    u = torch.zeros(n, W, dtype=F64)
    u[0] = torch.arange(1, W + 1, dtype=F64)
    zr, lam = math.log(0.4 / 0.6), -12.0
    g = torch.full((n, 2 * W), zr, dtype=F64)
    state, got = torch.full((1, W), float("nan"), device=DEV), []
    for lo, hi in ((0, 500), (500, 501), (501, 503), (503, 540), (540, n - 1), (n - 1, n)):
        out = torch.empty(hi - lo, W, device=DEV, dtype=dt)
        seqlib.rglru_scan(_dev(u[lo:hi], dt), _dev(g[lo:hi]), None, torch.full((W,), lam, device=DEV), None, state, out, _i32([0, hi - lo]), 1,
                          _i32(list(range(lo, hi))), _i32([0] * (hi - lo)), 1, 8.0)
        got.append(out.double().cpu())
    la = -8.0 * 0.4 * math.log1p(math.exp(lam))
    want = torch.tensor([[math.exp(la * t) * math.sqrt(-math.expm1(2 * la)) * 0.4 * (c + 1) for c in range(W)] for t in range(n)], dtype=F64)
    tol = 4e-6 if dt == torch.float32 else 5e-3
    assert ((torch.cat(got) - want).abs() / want).max() < tol
    assert ((state[0].double().cpu() - want[-1]).abs() / want[-1]).max() < 4e-6      # the state itself is fp32 either way


def test_block_diagonal_gates_as_one_batched_product():
    for n, blocks, dt in ((12, 5, torch.float32), (16, 3, torch.bfloat16), (80, 4, torch.bfloat16), (1, 7, torch.float32)):
        T, W = 19, n * blocks
        u, w = rand(T, W, seed=1).to(dt), (rand(blocks, 2 * n, n, seed=2) * n ** -0.5).to(dt)
        g = torch.empty(T, 2 * W, device=DEV)
        seqlib.linear(u.to(DEV), w.to(DEV), g, M=T, N=2 * n, K=n, ldx=W, sx=n, ldw=n, sw=2 * n * n, ldy=2 * W, sy=2 * n, batch=blocks)
        want = torch.cat([u[:, j * n:(j + 1) * n].double() @ w[j].double().T for j in range(blocks)], dim=1)
        assert (g.double().cpu() - want).abs().max() < 1e-4


# --------------------------------------------------------------------------------------------------------- latent attention
def _latent_case(n, r, dr, H, dtype, page, seed, q=None, rows=None):
    """A cache of n rows [r + dr] in shuffled pages of slot 1 and absorbed queries for every position."""
    g = torch.Generator().manual_seed(seed)
    rows = torch.randn(n, r + dr, generator=g, dtype=F64) if rows is None else rows
    q = torch.randn(n, H, r + dr, generator=g, dtype=F64) if q is None else q
    rows, q = rows.to(dtype), q.to(dtype)
    n_pages = -(-n // page)
    bt = torch.zeros(2, n_pages + 1, dtype=torch.int32)
    bt[1, :n_pages] = torch.randperm(n_pages, generator=g).to(torch.int32) + 1
    pool = torch.full((n_pages + 2, page, r + dr), float("nan"), dtype=dtype)
    for j in range(n):
        pool[int(bt[1, j // page]), j % page] = rows[j]
    return q, rows, bt.to(DEV), pool.to(DEV)


def _attend(q, r, dr, pool, bt, page, lo, hi, window, scale, gate, kind):
    """Rows lo .. hi - 1 of slot 1 through the plain kernel, the tensor-core kernel with a host work list, or the list a decode-only
    step writes on the device (parts key ranges per row)."""
    T, H = hi - lo, q.shape[1]
    qd, pos, slot = q[lo:hi].to(DEV).contiguous(), _i32(list(range(lo, hi))), _i32([1] * (hi - lo))
    gd = _dev(gate[lo:hi]) if gate is not None else None
    out = torch.empty(T, H, r, device=DEV)
    if kind == "plain":
        return seqlib.latent_attn(qd, r, dr, pool, bt, page, pos, slot, None, scale, out, window=window, gate=gd).double().cpu()
    if kind == "tensor":
        plan = seqlib.LatentAttnPlan([(0, T, 1, lo)], H, DEV, window=window)
    else:
        plan = seqlib.DecodeAttnPlan(T, H, kind, DEV, window=window)
        plan.fill(pos, slot)
    return seqlib.latent_attn_mma(qd, r, dr, pool, bt, page, plan, None, scale, out, window=window, gate=gd).double().cpu()


@pytest.mark.parametrize("H,r,dr", [(3, 20, 6), (4, 48, 16), (1, 16, 16), (16, 144, 32), (6, 64, 0), (5, 272, 16)])
@pytest.mark.parametrize("window", [1, 2, 25, 64, 65, 1000])
def test_windowed_gated_latent_attention_against_the_score_matrix(H, r, dr, window):
    n, page, scale = 150, 16, 0.2
    for dtype in (torch.float32, torch.bfloat16):
        q, rows, bt, pool = _latent_case(n, r, dr, H, dtype, page, seed=window)
        gate = rand(n, H, seed=7, s=2.0)
        s = torch.einsum("thd,jd->htj", q.double(), rows.double()) * scale
        p = torch.softmax(s.masked_fill(~O.window_mask(n, window), -math.inf), dim=-1)
        plain = torch.einsum("htj,jd->thd", p, rows.double()[:, :r])
        kinds = ["plain"] + (["tensor", 1, 3] if seqlib.latent_attn_mma_ok(H, r, dr, dtype) else [])
        for gt in (None, gate):
            want = plain if gt is None else plain * torch.sigmoid(gt.float().double())[:, :, None]
            for kind in kinds:
                tol = 3e-5 if dtype == torch.float32 or kind == "plain" else 3e-2
                for lo, hi in ((0, n), (97, n), (n - 1, n), (0, 2), (64, 65)):
                    if isinstance(kind, int) and hi - lo > 60:
                        continue
                    assert (_attend(q, r, dr, pool, bt, page, lo, hi, window, scale, gt, kind) - want[lo:hi]).abs().max() < tol, (dtype, kind, lo)


@pytest.mark.parametrize("window", [1, 16, 33, 64, 100, 129])
@pytest.mark.parametrize("dtype,kind", [(torch.float32, "plain"), (torch.bfloat16, "plain"), (torch.bfloat16, "tensor"), (torch.bfloat16, 1), (torch.bfloat16, 4)])
def test_one_key_that_stands_out_is_seen_exactly_inside_the_window(window, dtype, kind):
    """One of 400 cached rows has a score far above the rest and a latent along an axis of its own: rows from it to window - 1 behind it
    put nearly all their weight there, the row just outside and every row before it none at all. The mark sits at the first position,
    at page borders and around the tiles of 64 keys; whole prompt, a portion deep in the sequence, portions of two, decoded rows."""
    H, r, dr, n, page = 4, 32, 16, 400, 16
    for mark in (0, 15, 16, 63, 64, 199, 200, 383, 399 - window):
        if mark < 0:
            continue
        rows, q = rand(n, r + dr, seed=mark, s=0.1), rand(n, H, r + dr, seed=mark + 1, s=0.1)
        rows[:, 0], rows[:, r], q[:, :, 0], q[:, :, r] = 0.0, 0.0, 0.0, 1.0
        rows[mark, r], rows[mark, 0] = 30.0, 1.0        # found through the rotated part, recognised in the latent
        qc, _, bt, pool = _latent_case(n, r, dr, H, dtype, page, mark, q=q, rows=rows)

        def seen(lo, hi):
            return _attend(qc, r, dr, pool, bt, page, lo, hi, window, 1.0, None, kind)[:, :, 0]

        def check(lo, hi):
            got = seen(lo, hi)
            for i in range(lo, hi):
                inside = mark <= i < mark + window
                assert (got[i - lo] > 0.99).all() if inside else (got[i - lo] == 0).all(), (mark, i, lo, hi)

        if isinstance(kind, str):
            check(0, n)
            check(210, n)
            check(0, 2)
        for i in (mark - 1, mark, mark + 1, mark + window - 1, mark + window):
            if 0 <= i < n:
                check(i, i + 1)
                if i + 2 <= n:
                    check(i, i + 2)


@pytest.mark.parametrize("H,dn,dr,r,rot", [(3, 10, 6, 20, 6), (4, 32, 16, 48, 16), (9, 8, 8, 24, 4), (1, 5, 0, 7, 0)])
def test_rotation_norm_and_append_with_and_without_rows_of_its_own(H, dn, dr, r, rot):
    """bf16 operands from fp32 and from bf16 queries, the extra copy of the unrotated parts, and a layer that appends nothing."""
    eps, base, page = 1e-5, 50.0, 8
    positions = [0, 1, 7, 8, 63, 64, 200]
    T = len(positions)
    q, dkv, w = rand(T, H * (dn + dr), seed=1), rand(T, r + dr + 3, seed=2), rand(r, seed=3)
    cs = RotaryTables(DEV).get(RotarySpec(dims=rot, base=base), 256)
    bt = torch.zeros(2, 40, dtype=torch.int32)
    bt[1] = torch.randperm(40, generator=torch.Generator().manual_seed(5)).to(torch.int32) + 1
    pos = torch.tensor(positions)
    for dt, qdt in ((torch.float32, torch.float32), (torch.bfloat16, torch.float32), (torch.bfloat16, torch.bfloat16)):
        tol = 1e-5 if dt == torch.float32 else 3e-2
        qq = q.to(qdt).double().view(T, H, dn + dr)
        want_q = O.rotate_pairs(qq[..., dn:], pos, rot, base)
        for own in (True, False):
            pool = torch.full((42, page, r + dr), float("nan"), device=DEV, dtype=dt)
            qcat, qn = torch.zeros(T, H, r + dr, device=DEV, dtype=dt), torch.empty(T, H * dn, device=DEV, dtype=dt)
            seqlib.latent_rope_store(_dev(dkv)[:, :r + dr] if own else None, r, dr, _dev(w, dt) if own else None, eps, cs, rot, _i32(positions), _i32([1] * T),
                                     bt.to(DEV), page, pool, _dev(q, qdt), H, dn, qcat, qn=qn)
            assert (qcat[..., r:].double().cpu() - want_q).abs().max() < tol if dr else True
            assert (qcat[..., :r] == 0).all()
            assert (qn.double().cpu().view(T, H, dn) - qq[..., :dn]).abs().max() < tol
            if not own:
                assert torch.isnan(pool).all()
                continue
            c = O.rms_norm(dkv[:, :r].float().double(), w.to(dt), eps)
            kr = O.rotate_pairs(dkv[:, r:r + dr].float().double(), pos, rot, base)
            for i, p in enumerate(positions):
                row = pool[int(bt[1, p // page]), p % page].double().cpu()
                assert (row - torch.cat([c[i], kr[i]])).abs().max() < 3 * tol
            assert int((~torch.isnan(pool)).any(-1).sum()) == T
