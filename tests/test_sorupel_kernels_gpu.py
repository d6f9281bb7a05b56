"""The mechanisms of the Sorupel decoder alone on the GPU, each against the plain restatement in oracle/sorupel_oracle.py (float64).

Engineered inputs where random ones would hide a fault: a key whose score stands out just inside and just outside a chunk, at page
borders and at the first position, in prompt portions and for decoded rows; a state whose decay is nearly one; poisoned slots."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu

if not torch.cuda.is_available():  # collected on the CPU box too
    pytest.skip("needs a CUDA device", allow_module_level=True)

from omchat_b200 import seqlib  # noqa: E402
from omchat_b200.config import RotarySpec  # noqa: E402
from omchat_b200.model.seq_latent import RotaryTables  # noqa: E402
from sorupel_cases import F64, O, rand  # noqa: E402

DEV = "cuda:0"
BF = torch.bfloat16


def _dev(t, dt=torch.float32):
    return t.to(device=DEV, dtype=dt).contiguous()


def _i32(x):
    return torch.tensor(x, device=DEV, dtype=torch.int32)


def _cut_rows(cuts, step, slots):
    rows = [(r, cuts[r][step], cuts[r][step + 1], sl) for r, sl in enumerate(slots)]
    pos = [p for _, lo, hi, _ in rows for p in range(lo, hi)]
    slot = [sl for _, lo, hi, sl in rows for _ in range(lo, hi)]
    return rows, pos, slot


# ----------------------------------------------------------------------------------------------------- embedding, norms, gates
@pytest.mark.parametrize("C,vocab,buckets,mp,mc", [(45, 30, 7, 5, 3), (320, 500, 211, 1000, 17), (13000, 9, 1, 4, 6), (8, 50000, 65537, 2 ** 31 + 11, 48271)])
def test_bigram_embedding_in_portions_over_poisoned_tokens(C, vocab, buckets, mp, mc):
    """Two requests in interleaved portions (first tokens, single tokens, more); the token before a portion comes from the slot."""
    n, eps = [23, 17], 1e-5
    cuts = ([0, 1, 3, 4, 11, n[0]], [0, 2, 3, 9, 10, n[1]])
    ids = [torch.randint(0, vocab, (k,), generator=torch.Generator().manual_seed(k)).tolist() for k in n]
    table, big, w = rand(vocab, C, seed=1), rand(buckets + 1, C, seed=2), rand(C, seed=3)
    prev = torch.full((4,), -1, device=DEV, dtype=torch.int32)
    for dt in (torch.float32, BF):
        tab, bg = _dev(table, dt), _dev(big, dt)
        want = [tab.double().cpu()[torch.tensor(i)] + bg.double().cpu()[torch.tensor(O.bigram_rows(i, buckets, mp, mc))] for i in ids]
        for step in range(5):
            rows, pos, slot = _cut_rows(cuts, step, (3, 1))
            tok = [t for r, lo, hi, _ in rows for t in ids[r][lo:hi]]
            h, xb = torch.empty(len(pos), C, device=DEV), torch.empty(len(pos), C, device=DEV, dtype=dt)
            seqlib.embed_bigram(_i32(tok), _i32(pos), _i32(slot), tab, bg, mp, mc, prev, h, nw=_dev(w, dt), eps=eps, xb=xb, single_rows=len(pos) == 2)
            at = 0
            for r, lo, hi, sl in rows:
                assert (h[at:at + hi - lo].double().cpu() - want[r][lo:hi]).abs().max() < 1e-5
                normed = O.rms_norm(want[r][lo:hi], w.to(dt), eps)
                assert (xb[at:at + hi - lo].double().cpu() - normed).abs().max() < (2e-5 if dt == torch.float32 else 2e-2) * max(1.0, float(normed.abs().max()))
                assert int(prev[sl]) == ids[r][hi - 1]
                at += hi - lo
        prev.fill_(-1)
    # every row a request of its own, the state read and replaced by the one launch
    prev[:] = _i32([3, 1, 2, 0])
    h = torch.empty(3, C, device=DEV)
    seqlib.embed_bigram(_i32([5, 6, 7]), _i32([4, 0, 9]), _i32([2, 0, 1]), tab, bg, mp, mc, prev, h, single_rows=True)
    b = [(2 * mp + 5 * mc) % buckets, buckets, (1 * mp + 7 * mc) % buckets]
    assert torch.equal(h, tab.float()[[5, 6, 7]] + bg.float()[b]) and prev.tolist() == [6, 7, 5, 0]


@pytest.mark.parametrize("C", [256, 384, 1000, 2048, 4096, 6000, 45, 1, 9000])
@pytest.mark.parametrize("with_y,top", [(True, 0), (False, 0), (True, 3), (False, 1)])
def test_residual_sum_with_the_next_norm(C, with_y, top):
    T, eps = 7, 1e-5
    x, y, nw = rand(T, C, seed=1) + 3.0, rand(T, C, seed=2), rand(C, seed=3)
    ys, w = rand(T * max(top, 1) + 2, C, seed=5), rand(T, max(top, 1), seed=6)
    slot_of = torch.randperm(T * max(top, 1), generator=torch.Generator().manual_seed(1)).view(T, -1)
    slot_of[2, 0] = -1
    v = x.float().double()
    if with_y:
        v = v + y.float().double()
    for t in range(T):
        for j in range(top):
            if slot_of[t, j] >= 0:
                v[t] += w[t, j] * ys[slot_of[t, j]]
    for dt in (torch.float32, BF):
        want = O.rms_norm(v, nw.to(dt), eps)
        kw = dict(ys=_dev(ys), slot_of=_i32(slot_of.tolist()), w=_dev(w), top=top) if top else {}
        xd, xb = _dev(x), torch.full((T, C), float("nan"), device=DEV, dtype=dt)
        seqlib.rms_residual(xd, _dev(nw, dt), eps, y=_dev(y) if with_y else None, x_out=xd, xb=xb, **kw)
        assert (xd.double().cpu() - v).abs().max() < 1e-5
        assert (xb.double().cpu() - want).abs().max() < (2e-5 if dt == torch.float32 else 2e-2) * max(1.0, float(want.abs().max()))
        xs = _dev(x)
        seqlib.rms_residual(xs, None, eps, y=_dev(y) if with_y else None, x_out=xs, **kw)
        assert torch.equal(xs, xd)


@pytest.mark.parametrize("groups,n", [(1, 45), (4, 15), (9, 1), (2, 96), (3, 256), (1, 2048), (2, 9000), (1, 10000), (8, 33)])
@pytest.mark.parametrize("gdt,dt", [(torch.float32, torch.float32), (torch.float32, BF), (BF, BF)])
def test_gate_in_front_of_a_norm_in_equal_parts(groups, n, gdt, dt):
    T, eps = 5, 1e-5
    x, z, w = rand(T, groups * n, seed=1), rand(T, groups * n + 8, seed=2, s=2.0), rand(groups * n, seed=3)
    x[2] *= 1e-3       # eps matters
    zd = _dev(z, gdt)[:, 8:] if n % 4 == 0 else _dev(z, gdt)[:, 3:groups * n + 3]
    for act, f in ((seqlib.GATE_SILU, O.silu), (seqlib.GATE_SIGMOID, torch.sigmoid)):
        want = O.unit_rms((x * f(zd.double().cpu())).view(T, groups, n), eps).reshape(T, -1) * w.to(dt).double()
        got = seqlib.gate_rms_rows(_dev(x), groups, _dev(w, dt), eps, zd, act, torch.empty(T, groups * n, device=DEV, dtype=dt))
        assert (got.double().cpu() - want).abs().max() < (2e-5 if dt == torch.float32 else 2e-2) * max(1.0, float(want.abs().max()))


@pytest.mark.parametrize("M,N,K,batch", [(9, 14, 20, 3), (130, 64, 128, 4), (70, 40, 48, 3), (5, 8, 200, 2), (33, 130, 72, 1), (1, 16, 16, 5)])
@pytest.mark.parametrize("xdt,wdt,gdt,ydt", [(torch.float32, torch.float32, torch.float32, torch.float32), (BF, BF, BF, BF), (BF, BF, torch.float32, BF),
                                             (torch.float32, BF, torch.float32, BF)])
def test_product_with_an_output_gate(M, N, K, batch, xdt, wdt, gdt, ydt):
    """Heads as column slices, the gate a column slice of a wider row; every kernel behind omc_linear."""
    x, w, z = _dev(rand(M, batch * K, seed=1), xdt), _dev(rand(batch * N, K, seed=2, s=K ** -0.5), wdt), _dev(rand(M, batch * N + 9, seed=3, s=2.0), gdt)
    y = torch.empty(M, batch * N, device=DEV, dtype=ydt)
    seqlib.linear(x, w, y, M=M, N=N, K=K, ldx=batch * K, sx=K, ldw=K, sw=N * K, ldy=batch * N, sy=N, batch=batch, gate=z[:, 9:])
    xs, ws = x.double().cpu().view(M, batch, K), w.double().cpu().view(batch, N, K)
    want = torch.einsum("mbk,bnk->mbn", xs, ws).reshape(M, -1) * torch.sigmoid(z[:, 9:].double().cpu())
    assert (y.double().cpu() - want).abs().max() < (2e-5 if ydt == torch.float32 else 2e-2)


# ------------------------------------------------------------------------------------------- rotations in front of the caches
@pytest.mark.parametrize("H,G,d,rot,group", [(6, 2, 10, 6, False), (4, 4, 32, 32, False), (3, 1, 16, 4, True), (5, 1, 7, 0, False), (8, 2, 64, 64, True)])
@pytest.mark.parametrize("halves", [True, False])
def test_norm_rotation_and_append_of_keys_that_are_values(H, G, d, rot, group, halves):
    """Norms over the whole projection (or per head), both pairings, values = the keys as projected."""
    eps, base, page = 1e-5, 50.0, 8
    positions = [0, 1, 7, 8, 63, 64, 200]
    T, nq, nk = len(positions), H * d, G * d
    z, wq, wk = rand(T, nq + nk + 3, seed=1), rand(d if group else nq, seed=2), rand(d if group else nk, seed=3)
    cs = RotaryTables(DEV).get(RotarySpec(dims=rot, base=base), 256)
    bt = torch.zeros(2, 40, dtype=torch.int32)
    bt[1] = torch.randperm(40, generator=torch.Generator().manual_seed(5)).to(torch.int32) + 1
    pos = torch.tensor(positions)
    zd = _dev(z)

    def turned(x, w, heads):
        y = x.float().double()
        y = O.rms_norm(y.view(T, heads, d), w, eps) if group else O.rms_norm(y, w, eps).view(T, heads, d)
        if halves:
            return O.rotate_halves(y, pos, rot, base)
        perm = [2 * i for i in range(rot // 2)] + [2 * i + 1 for i in range(rot // 2)] + list(range(rot, d))
        out = torch.empty_like(y)
        out[..., perm] = O.rotate_halves(y[..., perm], pos, rot, base)
        return out
    for dt in (torch.float32, BF):
        tol = 2e-5 if dt == torch.float32 else 4e-2
        pool, qo = torch.full((42, page, 2 * nk), float("nan"), device=DEV, dtype=dt), torch.empty(T, nq, device=DEV, dtype=dt)
        seqlib.qk_norm_kv_store(zd[:, :nq], _dev(wq, dt), zd[:, nq:nq + nk], _dev(wk, dt), zd[:, nq:nq + nk], eps, _i32(positions), _i32([1] * T), bt.to(DEV), page,
                                pool, qo, group=d if group else 0, cs=cs, head=d, rot_dims=rot, rot_halves=halves)
        assert (qo.double().cpu().view(T, H, d) - turned(z[:, :nq], wq.to(dt), H)).abs().max() < tol
        k = turned(z[:, nq:nq + nk], wk.to(dt), G).reshape(T, nk)
        for i, p in enumerate(positions):
            row = pool[int(bt[1, p // page]), p % page].double().cpu()
            assert (row[:nk] - k[i]).abs().max() < tol and (row[nk:] - z[i, nq:nq + nk]).abs().max() < tol
        assert int((~torch.isnan(pool)).any(-1).sum()) == T


def test_rotation_arguments_are_checked():
    z, w, cs = torch.zeros(1, 24, device=DEV), torch.ones(24, device=DEV), torch.zeros(8, 2, 2, device=DEV)
    pool, bt = torch.zeros(1, 8, 48, device=DEV), torch.zeros(1, 1, device=DEV, dtype=torch.int32)
    for head, rot in ((8, 3), (8, 10), (7, 2), (0, 2)):
        with pytest.raises(seqlib.OmcError):
            seqlib.qk_norm_kv_store(z, w, z, w, z, 1e-5, _i32([0]), _i32([0]), bt, 8, pool, torch.empty(1, 24, device=DEV), cs=cs, head=head, rot_dims=rot)


@pytest.mark.parametrize("H,dn,dr,r,rot", [(3, 10, 6, 20, 6), (4, 32, 16, 48, 16), (9, 8, 8, 24, 4), (1, 5, 0, 7, 0)])
def test_latent_rows_and_queries_turned_in_halves(H, dn, dr, r, rot):
    eps, base, page = 1e-5, 50.0, 8
    positions = [0, 1, 7, 8, 63, 64, 200]
    T = len(positions)
    q, dkv, w = rand(T, H * (dn + dr), seed=1), rand(T, r + dr + 3, seed=2), rand(r, seed=3)
    cs = RotaryTables(DEV).get(RotarySpec(dims=rot, base=base), 256)
    bt = torch.zeros(2, 40, dtype=torch.int32)
    bt[1] = torch.randperm(40, generator=torch.Generator().manual_seed(5)).to(torch.int32) + 1
    pos = torch.tensor(positions)
    for dt, qdt in ((torch.float32, torch.float32), (BF, torch.float32), (BF, BF)):
        tol = 1e-5 if dt == torch.float32 else 3e-2
        qq = q.to(qdt).double().view(T, H, dn + dr)
        pool = torch.full((42, page, r + dr), float("nan"), device=DEV, dtype=dt)
        qcat, qn = torch.zeros(T, H, r + dr, device=DEV, dtype=dt), torch.empty(T, H * dn, device=DEV, dtype=dt)
        seqlib.latent_rope_store(_dev(dkv)[:, :r + dr], r, dr, _dev(w, dt), eps, cs, rot, _i32(positions), _i32([1] * T), bt.to(DEV), page, pool, _dev(q, qdt), H,
                                 dn, qcat, qn=qn, rot_halves=True)
        if dr:
            assert (qcat[..., r:].double().cpu() - O.rotate_halves(qq[..., dn:], pos, rot, base)).abs().max() < tol
        c, kr = O.rms_norm(dkv[:, :r].float().double(), w.to(dt), eps), O.rotate_halves(dkv[:, r:r + dr].float().double(), pos, rot, base)
        for i, p in enumerate(positions):
            row = pool[int(bt[1, p // page]), p % page].double().cpu()
            assert (row - torch.cat([c[i], kr[i]])).abs().max() < 3 * tol


# ------------------------------------------------------------------------------------------------------- chunked attention
def _kv_case(n, H, G, d, dtype, page, seed, q=None, k=None, v=None, slots=2):
    """Queries [n, H, d], keys and values [n, G, d] of one sequence; the rows of slot 1 in scattered pages of a NaN-filled pool."""
    q = (rand(n, H, d, seed=seed) if q is None else q).to(dtype)
    k = (rand(n, G, d, seed=seed + 1) if k is None else k).to(dtype)
    v = (rand(n, G, d, seed=seed + 2) if v is None else v).to(dtype)
    pages = -(-n // page)
    bt = torch.zeros(slots, pages, dtype=torch.int32)
    bt[1] = torch.randperm(pages, generator=torch.Generator().manual_seed(seed)).to(torch.int32) + 1
    pool = torch.full((pages + 1, page, 2 * G * d), float("nan"), dtype=dtype)
    for j in range(n):
        pool[bt[1, j // page], j % page] = torch.cat([k[j].reshape(-1), v[j].reshape(-1)])
    return q, k, v, bt.to(DEV), pool.to(DEV)


def _attend(q, G, pool, bt, page, lo, hi, scale, kind, **kw):
    """Rows lo .. hi - 1 of slot 1: the plain kernel, the tensor-core kernel with the host's tiles, or with every row an item of its own."""
    T, H, d = hi - lo, q.shape[1], q.shape[2]
    qd, pos, slot = q[lo:hi].reshape(T, H * d).to(DEV).contiguous(), _i32(list(range(lo, hi))), _i32([1] * T)
    out = torch.empty(T, H * d, device=DEV)
    window, softcap = kw.pop("window", seqlib.WINDOW_ALL), kw.pop("softcap", 0.0)
    if kind == "plain":
        seqlib.window_attn(qd, H, G, d, d, pool, bt, page, pos, slot, window, scale, softcap, None, out, **kw)
    else:
        items = seqlib.window_attn_items([(0, T, 1, lo)], H // G, DEV, kw.get("chunk", seqlib.WINDOW_ALL)) if kind == "tensor" else None
        seqlib.window_attn_mma(qd, H, G, d, d, pool, bt, page, items, pos, slot, window, scale, softcap, None, out, **kw)
    return out.double().cpu().view(T, H, d)


@pytest.mark.parametrize("H,G,d", [(6, 2, 10), (6, 2, 32), (5, 1, 16), (4, 4, 48), (7, 1, 128), (1, 1, 8)])
@pytest.mark.parametrize("chunk", [1, 3, 25, 64, 65, 100, seqlib.WINDOW_ALL])
def test_chunked_attention_against_the_score_matrix(H, G, d, chunk):
    """With a soft cap, one added to the denominator and one gate per head; whole prompts, portions, decoded rows."""
    n, page, scale, cap = 150, 16, 1.5 * d ** -0.5, 4.0
    for dtype in (torch.float32, BF):
        q, k, v, bt, pool = _kv_case(n, H, G, d, dtype, page, seed=chunk % 1000)
        gate, sink = rand(n, H, seed=7, s=2.0), torch.zeros(H, device=DEV)
        want = torch.zeros(n, H, d, dtype=F64)
        for h in range(H):
            s = cap * torch.tanh((q[:, h].double() @ k[:, h // (H // G)].double().T) * scale / cap)
            want[:, h] = O.sink_softmax(s, O.causal_mask(n, chunk), 0.0) @ v[:, h // (H // G)].double() * torch.sigmoid(gate.float().double()[:, h:h + 1])
        kinds = ["plain"] + (["tensor", "rows"] if seqlib.window_attn_mma_ok(H, G, d, d, dtype) else [])
        for kind in kinds:
            tol = 3e-5 if dtype == torch.float32 or kind == "plain" else 3e-2
            for lo, hi in ((0, n), (97, n), (n - 1, n), (0, 2), (64, 65), (99, 101)):
                got = _attend(q, G, pool, bt, page, lo, hi, scale, kind, softcap=cap, sink=sink, gate=_dev(gate[lo:hi]), gate_act=seqlib.GATE_SIGMOID,
                              gate_heads=True, chunk=chunk)
                assert (got - want[lo:hi]).abs().max() < tol, (dtype, kind, lo)
    assert seqlib.window_attn_mma_ok(9, 3, 48, 48, BF) and seqlib.window_attn_mma_ok(7, 1, 128, 128, BF)


@pytest.mark.parametrize("window,keep", [(20, 0), (33, 3), (seqlib.WINDOW_ALL, 2)])
def test_chunks_beside_a_window_and_kept_first_keys(window, keep):
    """The mechanisms of the kernel combine: a window inside a chunk, and kept keys of the first chunk."""
    H, G, d, n, page, chunk = 4, 2, 32, 140, 16, 50
    dist = torch.arange(n)[:, None] - torch.arange(n)[None, :]
    ok = O.causal_mask(n, chunk) & (dist < window) | (torch.arange(n)[None, :] < keep) & (dist >= 0)
    for dtype in (torch.float32, BF):
        q, k, v, bt, pool = _kv_case(n, H, G, d, dtype, page, seed=window % 997)
        want = torch.stack([torch.softmax((q[:, h].double() @ k[:, h // 2].double().T * 0.3).masked_fill(~ok, -math.inf), -1) @ v[:, h // 2].double() for h in range(H)], 1)
        for kind in ["plain"] + (["tensor", "rows"] if dtype == BF else []):
            for lo, hi in ((0, n), (45, 60), (50, 51), (99, 101)):
                got = _attend(q, G, pool, bt, page, lo, hi, 0.3, kind, window=window, keep_first=keep, chunk=chunk)
                assert (got - want[lo:hi]).abs().max() < (3e-5 if kind == "plain" else 3e-2), (dtype, kind, lo)


@pytest.mark.parametrize("chunk", [16, 33, 64, 100, 129])
@pytest.mark.parametrize("dtype,kind", [(torch.float32, "plain"), (BF, "plain"), (BF, "tensor"), (BF, "rows")])
def test_one_key_that_stands_out_is_seen_exactly_inside_its_chunk(chunk, dtype, kind):
    """One of 400 keys has a score far above the rest and a value of its own: rows from it to its chunk's last put nearly all their weight
    there, the next chunk's first row and every earlier row none. The mark sits at the first position, at chunk, page and tile borders;
    whole prompt, a portion deep in the sequence, portions of two, decoded rows."""
    H, G, d, n, page = 6, 2, 32, 400, 16
    for mark in {0, 15, 16, 63, 64, 199, 200, chunk - 1, chunk, 2 * chunk - 1, 2 * chunk, 399}:
        if mark >= n:
            continue
        k, v, q = rand(n, G, d, seed=mark, s=0.1), rand(n, G, d, seed=mark + 1, s=0.1), rand(n, H, d, seed=mark + 2, s=0.1)
        k[..., 0], v[..., 1], q[..., 0] = 0.0, 0.0, 1.0
        k[mark, :, 0], v[mark, :, 1] = 30.0, 1.0
        qc, _, _, bt, pool = _kv_case(n, H, G, d, dtype, page, mark, q=q, k=k, v=v)
        end = (mark // chunk + 1) * chunk       # first row that does not see it

        def check(lo, hi):
            got = _attend(qc, G, pool, bt, page, lo, hi, 1.0, kind, chunk=chunk, sink=torch.zeros(H, device=DEV))[:, :, 1]
            for i in range(lo, hi):
                assert (got[i - lo] > 0.99).all() if mark <= i < end else (got[i - lo] == 0).all(), (mark, i, lo, hi)

        if kind != "rows":
            check(0, n)
            check(210, n)
            check(0, 2)
        for i in (mark - 1, mark, mark + 1, end - 2, end - 1, end, end + 1):
            if 0 <= i < n:
                check(i, i + 1)
                if i + 2 <= n:
                    check(i, i + 2)


@pytest.mark.parametrize("sink", [-30.0, 0.0, 4.0, 60.0])
def test_a_sink_takes_its_share_of_every_row(sink):
    """Equal scores: a row that sees m keys gives m e^s / (m e^s + e^sink) in total - also for the very first row."""
    H, G, d, n, page, r = 4, 2, 32, 70, 16, 32
    one = torch.ones(n, G, d, dtype=F64)
    q, k, v, bt, pool = _kv_case(n, H, G, d, BF, page, 1, q=torch.ones(n, H, d, dtype=F64), k=one, v=one)
    sk = torch.full((H,), sink, device=DEV)
    m = torch.arange(1, n + 1, dtype=F64)
    want = m * math.exp(2.0) / (m * math.exp(2.0) + math.exp(sink))
    for kind in ("plain", "tensor", "rows"):
        got = _attend(q, G, pool, bt, page, 0, n, 2.0 / d, kind, sink=sk)
        assert (got - want[:, None, None]).abs().max() < 1e-2 * float(want.max()) + 1e-9, kind
    rows = torch.zeros(n, r + 16, dtype=F64)
    rows[:, :r], rows[:, r] = 1.0, 2.0
    lat = torch.full((-(-n // page) + 1, page, r + 16), float("nan"), dtype=BF, device=DEV)
    for j in range(n):
        lat[int(bt[1, j // page]), j % page] = rows[j].to(device=DEV, dtype=BF)
    qc = torch.zeros(n, H, r + 16, device=DEV, dtype=BF)
    qc[..., r] = 1.0
    pos, slot = _i32(list(range(n))), _i32([1] * n)
    out = torch.empty(n, H, r, device=DEV)
    plans = [None, seqlib.LatentAttnPlan([(0, n, 1, 0)], H, DEV)] + [seqlib.DecodeAttnPlan(n, H, p, DEV) for p in (1, 3)]
    for plan in plans:
        if plan is None:
            seqlib.latent_attn(qc, r, 16, lat, bt, page, pos, slot, sk, 1.0, out)
        else:
            if isinstance(plan, seqlib.DecodeAttnPlan):
                plan.fill(pos, slot)
            seqlib.latent_attn_mma(qc, r, 16, lat, bt, page, plan, sk, 1.0, out)
        assert (out.double().cpu() - want[:, None, None]).abs().max() < 1e-2 * float(want.max()) + 1e-9


@pytest.mark.parametrize("kind", ["plain", "tensor", 1, 3, 7])
def test_a_latent_row_far_back_is_found_behind_a_sink(kind):
    """One of 900 cached rows stands out (score 30, the sink has 27): every later row gives it e^3 / (1 + e^3) of its weight, at any
    distance, page and tile border; earlier rows none."""
    H, r, dr, n, page = 4, 32, 16, 900, 16
    for mark in (0, 15, 16, 63, 64, 511, 512, 895):
        rows, q = rand(n, r + dr, seed=mark, s=0.1), rand(n, H, r + dr, seed=mark + 1, s=0.1)
        rows[:, 0], rows[:, r], q[:, :, 0], q[:, :, r] = 0.0, 0.0, 0.0, 1.0
        rows[mark], rows[mark, r], rows[mark, 0] = 0.0, 30.0, 1.0
        bt = torch.zeros(2, 57, dtype=torch.int32)
        bt[1] = torch.randperm(57, generator=torch.Generator().manual_seed(mark)).to(torch.int32) + 1
        pool = torch.full((58, page, r + dr), float("nan"), dtype=BF)
        j = torch.arange(n)
        pool[bt[1].long()[j // page], j % page] = rows.to(BF)
        pool, btd, sink = pool.to(DEV), bt.to(DEV), torch.full((H,), 27.0, device=DEV)
        for lo, hi in ((0, n), (mark, mark + 1), (n - 3, n - 1), (n - 1, n)):
            if isinstance(kind, int) and hi - lo > 60:
                continue
            T, qd = hi - lo, q[lo:hi].to(device=DEV, dtype=BF).contiguous()
            pos, slot, out = _i32(list(range(lo, hi))), _i32([1] * T), torch.empty(T, H, r, device=DEV)
            if kind == "plain":
                seqlib.latent_attn(qd, r, dr, pool, btd, page, pos, slot, sink, 1.0, out)
            else:
                plan = seqlib.LatentAttnPlan([(0, T, 1, lo)], H, DEV) if kind == "tensor" else seqlib.DecodeAttnPlan(T, H, kind, DEV)
                if kind != "tensor":
                    plan.fill(pos, slot)
                seqlib.latent_attn_mma(qd, r, dr, pool, btd, page, plan, sink, 1.0, out)
            got, share = out[:, :, 0].double().cpu(), math.exp(3.0) / (1.0 + math.exp(3.0))
            for i in range(lo, hi):
                assert ((got[i - lo] - (share if i >= mark else 0.0)).abs() < 1e-2).all(), (mark, i)


# --------------------------------------------------------------------------------------------------------------- recurrence
@pytest.mark.parametrize("H,G,N,P", [(6, 3, 12, 10), (4, 1, 7, 9), (1, 1, 1, 1), (8, 2, 64, 64), (4, 4, 128, 32), (2, 1, 200, 70), (3, 3, 32, 33)])
def test_state_space_recurrence_in_portions_over_poisoned_slots(H, G, N, P):
    """Two requests in interleaved portions of 1 to 40 tokens (once one token each); inputs are column slices of one row as in the model."""
    n = [73, 60]
    cuts = ([0, 1, 3, 4, 5, 40, n[0]], [0, 2, 3, 19, 20, 21, n[1]])
    inner, gn = H * P, G * N
    u, dt_raw = [rand(k, inner + 2 * gn, seed=k) for k in n], [rand(k, H, seed=k + 1) for k in n]
    A_log, dt_bias, D = rand(H, seed=1, s=1.5), rand(H, seed=2) - 1.0, rand(H, seed=3)
    state = torch.full((4, H, N, P), float("nan"), device=DEV)
    for use_d in (True, False):
        want = [O.ssd_recurrence(u[r][:, :inner].view(-1, H, P), u[r][:, inner:inner + gn].view(-1, G, N), u[r][:, inner + gn:].view(-1, G, N),
                                 O.softplus(dt_raw[r] + dt_bias), A_log, D if use_d else D * 0).reshape(-1, inner) for r in range(2)]
        for step in range(6):
            rows, pos, slot = _cut_rows(cuts, step, (3, 1))
            ud = _dev(torch.cat([u[r][lo:hi] for r, lo, hi, _ in rows]))
            a = _dev(torch.cat([torch.cat([rand(hi - lo, 5, seed=9), dt_raw[r][lo:hi]], 1) for r, lo, hi, _ in rows]))
            starts = [0, rows[0][2] - rows[0][1], len(pos)]
            y = torch.empty(len(pos), inner, device=DEV)
            seqlib.linear_state_scan(ud[:, inner + gn:], ud[:, inner:inner + gn], ud[:, :inner], state, y, _i32(starts), 2, _i32(pos), _i32(slot), H, G, N, P,
                                     step_size=True, a=a[:, 5:], A_log=_dev(A_log), dt_bias=_dev(dt_bias), D=_dev(D) if use_d else None)
            for i, (r, lo, hi, _) in enumerate(rows):
                w = want[r][lo:hi]
                assert (y[starts[i]:starts[i + 1]].double().cpu() - w).abs().max() < 2e-5 * max(1.0, float(w.abs().max())), (step, r)


def test_a_state_that_hardly_decays_keeps_its_digits():
    """exp(-A dt) = 1 - 2e-5: what the first token left in the state, read 1500 times while nothing else enters, against g^t. (A decay that
    is rounded to fp32 before the state meets it drifts away by more than ten times the bound.)"""
    n, H, N, P = 1500, 1, 4, 4
    dt = math.log1p(math.exp(-4.0))
    A = 2e-5 / dt
    u = torch.ones(n, P + 2 * N, device=DEV)
    u[1:, :P] = 0.0
    state, y = torch.full((1, H, N, P), float("nan"), device=DEV), torch.empty(n, P, device=DEV)
    for lo, hi in ((0, 700), (700, 701), (701, n)):
        seqlib.linear_state_scan(u[lo:hi, P + N:], u[lo:hi, P:P + N], u[lo:hi, :P], state, y[lo:hi], _i32([0, hi - lo]), 1, _i32(list(range(lo, hi))),
                                 _i32([0] * (hi - lo)), H, 1, N, P, step_size=True, a=torch.full((hi - lo, 1), -4.0, device=DEV),
                                 A_log=torch.full((1,), math.log(A), device=DEV), dt_bias=torch.zeros(1, device=DEV))
    want = torch.tensor([N * dt * math.exp(-2e-5 * t) for t in range(n)], dtype=F64)
    assert ((y.double().cpu() - want[:, None]).abs().max(1).values / want).max() < 4e-6


def test_recurrence_arguments_are_checked():
    z, st = torch.zeros(1, 4, device=DEV), torch.zeros(1, 1, 4, 4, device=DEV)
    args = (z, z, z, st, torch.empty(1, 4, device=DEV), _i32([0, 1]), 1, _i32([0]), _i32([0]), 1, 1, 4, 4)
    a, one = torch.zeros(1, 1, device=DEV), torch.zeros(1, device=DEV)
    with pytest.raises(seqlib.OmcError):
        seqlib.linear_state_scan(*args, step_size=True, a=a, A_log=one)
    with pytest.raises(seqlib.OmcError):
        seqlib.linear_state_scan(*args, step_size=True, a=a, A_log=one, dt_bias=one, beta=a)
    with pytest.raises(AssertionError):
        seqlib.linear_state_scan(*args, decay_const=one, D=one)
