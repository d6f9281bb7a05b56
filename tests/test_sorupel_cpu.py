"""Host-side parts of the Sorupel path that need no GPU: configuration parsing and its refusals, the registry, cache and state shapes,
weight names and shapes, the work list of a chunked step, and the plain model's mechanisms against closed forms."""
import math

import pytest
import torch

from omchat_b200 import seqlib
from omchat_b200.config import BigramSpec, ChunkAttentionSpec, LatentAttentionSpec, SorupelConfig, StateSpaceSpec
from omchat_b200.model import registry
from omchat_b200.model.checkpoint import config_from_dict
from omchat_b200.model.paged_cache import PagedStateCache
from sorupel_cases import CONFIGS, F64, O, config_a, config_b, rand, tokens_for


def test_config_is_read_from_the_dictionary_and_round_trips():
    cfg = config_from_dict(config_a())
    assert isinstance(cfg, SorupelConfig) and (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps) == (131, 72, 1e-5) and cfg.bigram == BigramSpec(61, 7, 3)
    att, lat, sp, shared = [l.mixer for l in cfg.layers[:4]]
    assert isinstance(att, ChunkAttentionSpec) and (att.heads, att.kv_heads, att.dim, att.chunk, att.softcap) == (6, 2, 10, 25, 9.0)
    assert (att.rot.dims, att.rot.base, att.rot.halves) == (6, 500.0, True)
    assert isinstance(lat, LatentAttentionSpec) and (lat.heads, lat.dim, lat.rot_dim, lat.vdim, lat.kv_rank) == (3, 10, 6, 14, 20)
    assert lat.sink and lat.out_gate and not lat.head_gate and lat.window is None and lat.kv_from is None and lat.rot.halves
    assert isinstance(sp, StateSpaceSpec) and (sp.heads, sp.vdim, sp.state, sp.groups, sp.conv, sp.norm_groups) == (6, 10, 12, 3, 4, 4)
    assert sp.inner == 60 and sp.conv_channels == 60 + 72
    assert shared.kv_from == 1 and cfg.layers[3].mlp is None and cfg.layers[0].mlp.ff == 50 and not cfg.layers[0].mlp.bias
    for f in CONFIGS.values():
        cfg = SorupelConfig.from_dict(f())
        assert SorupelConfig.from_dict(cfg.to_dict()) == cfg
    assert registry.MODEL_CLASSES[SorupelConfig][1] == "SorupelForCausalLM"
    b = config_from_dict(config_b())
    assert b.layers[2].mixer.chunk is None and b.layers[2].mixer.softcap == 0.0 and b.layers[2].mixer.rot.dims == 0


@pytest.mark.parametrize("breakage", [
    lambda x: x["layers"][0].update(type="something_else"), lambda x: x["layers"][3]["mixer"].update(kv_from=2), lambda x: x["layers"][3]["mixer"].update(kv_from=6),
    lambda x: x["layers"][7]["mixer"].update(kv_from=3), lambda x: x["layers"][3]["mixer"].update(kv_rank=16), lambda x: x["layers"][3]["mixer"]["rot"].update(base=1.5),
    lambda x: x["layers"][0]["mixer"]["mask"].update(size=0), lambda x: x["layers"][0]["mixer"]["rot"].update(dims=5), lambda x: x["layers"][0]["mixer"]["rot"].update(dims=12),
    lambda x: x["layers"][1]["mixer"]["rot"].update(dims=8), lambda x: x["layers"][0]["mixer"].update(kv_heads=4), lambda x: x["layers"][0]["mixer"].update(vdim=8),
    lambda x: x["layers"][2]["mixer"].update(groups=4), lambda x: x["layers"][2]["mixer"].update(conv=0), lambda x: x["layers"][2]["mixer"].update(norm_groups=7),
    lambda x: x["layers"][0]["mlp"].update(kind="moe"), lambda x: x["embedding"]["bigram"].update(buckets=0), lambda x: x["layers"][0]["mixer"].update(softcap=-1.0)])
def test_contradictory_configs_are_refused(breakage):
    bad = config_a()
    breakage(bad)
    with pytest.raises(ValueError):
        config_from_dict(bad)


def test_weights_names_shapes_and_state_layout():
    from omchat_b200.model.sorupel import SorupelDecoder, random_state_dict, weights_from_state_dict
    cfg = config_from_dict(config_a())
    sd = random_state_dict(cfg, seed=1)
    w = weights_from_state_dict(sd, cfg, "cpu", torch.float32)
    att, lat, sp, shared = [l.mix for l in w.layers[:4]]
    assert att.cols == {"q": slice(0, 60), "k": slice(60, 80), "g": slice(80, 86)} and att.w_in.shape == (88, 72) and float(att.one.abs().sum()) == 0
    assert (lat.nq, lat.ng) == (48, 42) and lat.w_in.shape == (120, 72) and torch.equal(lat.w_in[48:90], sd["l1.mix.g"].float())
    assert torch.equal(lat.w_in[90:116], sd["l1.mix.dkv"].float()) and torch.equal(lat.uk_t[1], sd["l1.mix.uk"][10:20].float().T)
    assert shared.w_in.shape == (136, 72) and shared.dkv_norm is None and shared.sink.dtype == torch.float32
    assert sp.w_in.shape == (200, 72) and torch.equal(sp.w_in[:198], sd["l2.mix.in"].float()) and sp.conv.shape == (132, 4)
    assert w.layers[3].mlp is None and w.layers[3].norm2 is None and w.bigram.shape == (62, 72)
    dec = SorupelDecoder.__new__(SorupelDecoder)
    dec.cfg, dec.C = cfg, 72
    assert dec.cache_widths() == [40, 26, 0, 0, 0, 28, 20, 0]
    states = dec.state_shapes()
    assert states[2] == {"S": (6, 12, 10), "conv": (3, 132)} and states[4] == {"S": (4, 7, 9), "conv": (2, 50)} and states[-1] == {"token": ((), torch.int32)}
    assert len(states) == 9 and all(states[i] == {} for i in (0, 1, 3, 5, 6, 7))
    assert dec.decode_shape(2, 50) == {"decode_keys": 64} and dec.decode_shape(2, 64) == {"decode_keys": 64}
    cache = PagedStateCache(dec.cache_widths(), states, 5, 3, 16, torch.float32, "cpu")
    assert cache.states[-1]["token"].shape == (3,) and cache.states[-1]["token"].dtype == torch.int32 and cache.states[2]["S"].dtype == torch.float32
    cache.poison_slot(1)
    assert cache.states[-1]["token"].tolist() == [0, -1, 0] and torch.isnan(cache.states[2]["S"][1]).all()
    assert cache.state_bytes_per_slot() == 4 * (720 + 396 + 252 + 100 + 1)
    for name in ("l0.mix.q", "l1.mix.sink", "l2.mix.in", "l7.mlp.down", "bigram"):
        bad = dict(sd)
        bad[name] = sd[name][:-1]
        with pytest.raises(ValueError):
            weights_from_state_dict(bad, cfg, "cpu", torch.float32)
    del sd["l4.mix.conv.b"]
    with pytest.raises(KeyError):
        weights_from_state_dict(sd, cfg, "cpu", torch.float32)
    plain = config_a()
    plain["embedding"] = {}
    cfg = config_from_dict(plain)
    assert cfg.bigram is None and weights_from_state_dict(random_state_dict(cfg), cfg, "cpu", torch.float32).bigram is None


@pytest.mark.parametrize("chunk", [1, 33, 64, 65, 100, seqlib.WINDOW_ALL])
@pytest.mark.parametrize("rep", [1, 3, 5, 6, 64])
def test_work_list_of_a_chunked_step(chunk, rep):
    """Every row in exactly one tile of at most 64 (token, head) rows; from 64 positions on a tile does not cross a chunk's edge."""
    portions = [(0, 150, 1, 0), (150, 1, 0, 300), (151, 230, 2, 170), (381, 2, 3, 99)]
    items = seqlib.window_attn_items(portions, rep, "cpu", chunk).tolist()
    rows = {}
    for first, n, slot, p0 in items:
        assert 1 <= n <= seqlib.MMA_ROWS // rep
        if 64 <= chunk < seqlib.WINDOW_ALL:
            assert p0 // chunk == (p0 + n - 1) // chunk
        for i in range(n):
            assert first + i not in rows
            rows[first + i] = (slot, p0 + i)
    assert rows == {f + i: (s, p + i) for f, n, s, p in portions for i in range(n)}


# ------------------------------------------------------------------------------------------------- the plain model's mechanisms
def test_plain_recurrence_against_its_closed_form():
    """y_t = sum_s prod_(s < u <= t) exp(-A dt_u) dt_s (B_s . C_t) x_s + D x_t; head h reads group floor(h / (heads / groups))."""
    T, H, P, G, N = 9, 4, 2, 2, 3
    x, B, C = rand(T, H, P, seed=1), rand(T, G, N, seed=2), rand(T, G, N, seed=3)
    dt, A_log, D = rand(T, H, seed=4).abs(), rand(H, seed=5), rand(H, seed=6)
    got = O.ssd_recurrence(x, B, C, dt, A_log, D)
    for h in range(H):
        g = h // 2
        for t in range(T):
            want = float(D[h]) * x[t, h]
            for s in range(t + 1):
                want = want + math.exp(-math.exp(float(A_log[h])) * float(dt[s + 1:t + 1, h].sum())) * float(dt[s, h]) * float(B[s, g] @ C[t, g]) * x[s, h]
            assert (got[t, h] - want).abs().max() < 1e-12


def test_plain_bigram_rows_masks_sink_and_rotation():
    assert O.bigram_rows([5, 2, 9], 7, 3, 4) == [7, (15 + 8) % 7, (6 + 36) % 7] and O.bigram_rows([5], 7, 3, 4) == [7]
    ok = O.causal_mask(7, 3)
    assert [int(r.sum()) for r in ok] == [1, 2, 3, 1, 2, 3, 1] and bool(ok[5, 3]) and not bool(ok[5, 2]) and not bool(ok[2, 3])
    assert bool(O.causal_mask(7)[6, 0]) and not bool(O.causal_mask(7)[0, 1])
    s = torch.tensor([[0.3, -1.0], [2.0, 0.5]], dtype=F64)
    p = O.sink_softmax(s, O.causal_mask(2), 0.7)
    assert abs(float(p[0, 0]) - math.exp(0.3) / (math.exp(0.3) + math.exp(0.7))) < 1e-12 and float(p[0, 1]) == 0.0
    assert abs(float(O.sink_softmax(s, O.causal_mask(2), 0.0)[1].sum()) - (math.exp(2) + math.exp(0.5)) / (1 + math.exp(2) + math.exp(0.5))) < 1e-12
    v = torch.tensor([[1.0, 2.0, 0.0, 0.0, 5.0]], dtype=F64)
    r = O.rotate_halves(v, torch.tensor([3]), 4, 100.0)[0]
    want = [math.cos(3.0), 2 * math.cos(0.3), math.sin(3.0), 2 * math.sin(0.3), 5.0]
    assert all(abs(float(a) - b) < 1e-12 for a, b in zip(r, want))


def test_plain_model_is_causal_and_a_chunk_forgets():
    """Changing the last token changes no earlier logits; in a model of one chunked attention a token of the previous chunk does not matter
    (but the token just before does: through the bigram row)."""
    from omchat_b200.model.sorupel import random_state_dict
    cd = config_a()
    sd = random_state_dict(SorupelConfig.from_dict(cd), seed=3)
    t = tokens_for(cd, 20, 1)
    a, b = O.forward(cd, sd, t), O.forward(cd, sd, t[:-1] + [(t[-1] + 1) % 131])
    assert torch.equal(a[:-1], b[:-1]) and (a[-1] - b[-1]).abs().max() > 1e-3
    one = dict(cd, layers=[cd["layers"][0]])
    one["layers"][0]["mixer"]["mask"]["size"] = 5
    c = O.forward(one, sd, t)
    for at, sees in ((13, range(13, 16)), (14, range(14, 16)), (15, range(15, 20))):
        d = O.forward(one, sd, t[:at] + [(t[at] + 1) % 131] + t[at + 1:])
        changed = {i for i in range(20) if (c[i] - d[i]).abs().max() > 1e-9}
        assert changed >= set(i for i in sees if i // 5 == at // 5) and min(changed) == at
        assert (at + 1) // 5 == at // 5 or at + 1 in changed     # the next chunk's first row: its bigram row
        assert max(changed) <= (at + 1) // 5 * 5 + 4
