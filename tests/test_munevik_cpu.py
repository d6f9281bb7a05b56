"""Host-side parts of the Munevik path that need no GPU: configuration parsing and its refusals, the registry, cache and state shapes,
weight names and shapes, the attention work list of a windowed step, and the plain model's mechanisms against closed forms."""
import math

import pytest
import torch

from munevik_cases import F64, O, config_a, config_b, rand, tokens_for
from omchat_b200 import seqlib
from omchat_b200.config import ClampedMlpSpec, GatedLruSpec, GroupedMoeSpec, LatentAttentionSpec, MunevikConfig
from omchat_b200.model import registry
from omchat_b200.model.checkpoint import config_from_dict


def test_config_is_read_from_the_dictionary_and_round_trips():
    cfg = config_from_dict(config_a())
    assert isinstance(cfg, MunevikConfig) and (cfg.vocab_size, cfg.hidden_size, cfg.norm_eps, cfg.postln_alpha) == (131, 72, 1e-5, 1.7)
    a, b, c = cfg.layers[:3]
    m = a.mixer
    assert isinstance(m, LatentAttentionSpec) and (m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank, m.window) == (3, 10, 6, 14, 20, 25)
    assert (m.rot.dims, m.rot.base) == (6, 3000.0) and m.head_gate and m.kv_from is None and m.q_rank is None and not m.sink
    s = a.mlp
    assert isinstance(s, GroupedMoeSpec) and (s.experts, s.top, s.expert_ff, s.groups, s.keep, s.scale, s.shared_ff) == (15, 3, 20, 5, 3, 2.5, 28)
    assert isinstance(b.mixer, GatedLruSpec) and (b.mixer.width, b.mixer.blocks, b.mixer.conv, b.mixer.decay_scale) == (60, 5, 4, 8.0)
    assert isinstance(b.mlp, ClampedMlpSpec) and (b.mlp.ff, b.mlp.limit) == (50, 1.2)
    assert c.mixer.kv_from == 0 and c.mlp is None and cfg.layers[3].mlp.shared_ff is None
    for d in (config_a(), config_b()):
        cfg = MunevikConfig.from_dict(d)
        assert MunevikConfig.from_dict(cfg.to_dict()) == cfg
    assert registry.MODEL_CLASSES[MunevikConfig][1] == "MunevikForCausalLM"


@pytest.mark.parametrize("breakage", [
    lambda x: x["layers"][0].update(type="something_else"), lambda x: x["layers"][2]["mixer"].update(kv_from=1), lambda x: x["layers"][2]["mixer"].update(kv_from=5),
    lambda x: x["layers"][5]["mixer"].update(kv_from=2), lambda x: x["layers"][2]["mixer"].update(kv_rank=16), lambda x: x["layers"][2]["mixer"]["rot"].update(base=1.5),
    lambda x: x["layers"][0]["mixer"]["mask"].update(size=0), lambda x: x["layers"][0]["mixer"]["rot"].update(dims=5), lambda x: x["layers"][0]["mixer"]["rot"].update(dims=8),
    lambda x: x["layers"][1]["mixer"].update(blocks=7), lambda x: x["layers"][1]["mixer"].update(conv=0), lambda x: x["layers"][0]["mlp"]["router"]["groups"].update(count=4),
    lambda x: x["layers"][0]["mlp"]["router"]["groups"].update(keep=6), lambda x: x["layers"][0]["mlp"]["router"].update(top=10), lambda x: x["layers"][1]["mlp"].update(kind="sparse")])
def test_contradictory_configs_are_refused(breakage):
    bad = config_a()
    breakage(bad)
    with pytest.raises(ValueError):
        config_from_dict(bad)


def test_missing_optional_entries_mean_absent_mechanisms():
    d = config_a()
    del d["layers"][0]["mixer"]["mask"], d["layers"][0]["mlp"]["router"]["groups"], d["layers"][0]["mlp"]["router"]["scale"], d["layers"][0]["mlp"]["shared"]
    cfg = config_from_dict(d)
    s = cfg.layers[0].mlp
    assert cfg.layers[0].mixer.window is None and (s.groups, s.keep, s.scale, s.shared_ff) == (1, 1, 1.0, None)


def test_weights_names_shapes_and_state_layout():
    from omchat_b200.model.munevik import MunevikDecoder, random_state_dict, weights_from_state_dict
    cfg = config_from_dict(config_a())
    sd = random_state_dict(cfg, seed=1)
    w = weights_from_state_dict(sd, cfg, "cpu", torch.float32)
    m0, m2 = w.layers[0].mix, w.layers[2].mix
    assert m0.w_in.shape == (80, 72) and m0.nq == 48 and m0.cols == {"q": slice(0, 48), "dkv": slice(48, 74), "g": slice(74, 77)}   # 77 rows, padded
    assert m2.w_in.shape[0] == 96 and m2.cols == {"q": slice(0, 90), "g": slice(90, 95)} and m2.dkv_norm is None
    assert torch.equal(m0.uk_t[1], sd["l0.mix.uk"][10:20].float().T)
    g = w.layers[1].mix
    assert g.gates.shape == (5, 24, 12) and torch.equal(g.gates[3, :12], sd["l1.mix.ra"][3].float()) and torch.equal(g.gates[3, 12:], sd["l1.mix.ri"][3].float())
    assert torch.equal(g.gates_b.view(5, 2, 12)[2, 1], sd["l1.mix.ri.b"][2].float())
    e = w.layers[0].mlp
    assert e.n_router == 16 and e.w_in.shape == (16 + 56, 72) and e.gate_up.shape == (15, 40, 72) and w.layers[2].mlp is None and w.layers[3].mlp.shared_down is None
    dec = MunevikDecoder.__new__(MunevikDecoder)
    dec.cfg, dec.C = cfg, 72
    assert dec.cache_widths() == [26, 0, 0, 0, 20, 0]
    assert dec.state_shapes() == [{}, {"S": (60,), "conv": (3, 60)}, {}, {"S": (36,), "conv": (2, 36)}, {}, {}]
    assert dec.decode_shape(2, 50) == {"decode_keys": 64} and dec.decode_shape(2, 5000) == {"decode_keys": 512}   # the widest window has 300 keys
    for name in ("l0.mix.q", "l1.mix.ra", "l5.mlp.shared.down"):
        bad = dict(sd)
        bad[name] = sd[name][:-1]
        with pytest.raises(ValueError):
            weights_from_state_dict(bad, cfg, "cpu", torch.float32)
    del sd["l4.norm2.b"]
    with pytest.raises(KeyError):
        weights_from_state_dict(sd, cfg, "cpu", torch.float32)


@pytest.mark.parametrize("window", [1, 5, 64, 200, seqlib.WINDOW_ALL])
def test_work_list_of_a_windowed_step_covers_what_every_row_sees_once(window):
    """Every (row, visible key) pair lies in exactly one item's key range; ranges hold no key that no row of the item sees."""
    H = 3
    portions = [(0, 50, 1, 0), (50, 1, 0, 300), (51, 30, 2, 170)]
    plan = seqlib.LatentAttnPlan(portions, H, "cpu", target_ctas=40, min_keys=32, window=window) if torch.cuda.is_available() else None
    if plan is None:   # the plan pins its host buffer, which needs a CUDA driver: build the list without it
        real, torch.Tensor.pin_memory = torch.Tensor.pin_memory, lambda self: self
        try:
            plan = seqlib.LatentAttnPlan(portions, H, "cpu", target_ctas=40, min_keys=32, window=window)
        finally:
            torch.Tensor.pin_memory = real
    items = plan.items.view(-1, 8).tolist()
    seen = {}
    for first, n, slot, p0, kb, ke, part, _ in items:
        assert n <= seqlib.MMA_ROWS // H and 0 <= kb <= ke
        for i in range(n):
            for k in range(max(kb, p0 + i - window + 1), min(ke, p0 + i + 1)):
                seen[(first + i, k)] = seen.get((first + i, k), 0) + 1
        if ke > kb:
            assert kb >= p0 - window + 1 and ke <= p0 + n
    for first, n, slot, p0 in portions:
        for i in range(n):
            for k in range(max(0, p0 + i - window + 1), p0 + i + 1):
                assert seen.pop((first + i, k), 0) == 1, (first + i, k)
    assert not seen


# ------------------------------------------------------------------------------------------------- the plain model's mechanisms
def test_plain_recurrence_against_its_closed_form():
    """Constant gates: S_t = sum_s a^(t - s) sqrt(1 - a^2) i u_s with a = exp(-8 r softplus(lam))."""
    n, W = 12, 3
    u, lam = rand(n, W, seed=1), torch.tensor([-3.0, 0.5, 40.0], dtype=F64)
    r, i = torch.full((n, W), 0.3, dtype=F64), torch.full((n, W), 0.6, dtype=F64)
    got = O.rglru_recurrence(u, r, i, lam)
    for c in range(W):
        a = math.exp(-8.0 * 0.3 * math.log1p(math.exp(float(lam[c])))) if lam[c] < 30 else math.exp(-8.0 * 0.3 * float(lam[c]))
        for t in range(n):
            want = sum(a ** (t - s) * math.sqrt(1.0 - a * a) * 0.6 * float(u[s, c]) for s in range(t + 1))
            assert abs(float(got[t, c]) - want) < 1e-10


def test_plain_block_gate_is_one_block_diagonal_product():
    u, w, b = rand(5, 12, seed=2), rand(3, 4, 4, seed=3), rand(3, 4, seed=4)
    full = torch.block_diag(*w)
    assert (O.block_gate(u, w, b) - torch.sigmoid(u @ full.T + b.reshape(-1))).abs().max() < 1e-12


def test_plain_group_choice():
    s = [0.9, 0.1, 0.5, 0.6, 0.8, 0.2, 0.7, 0.65]      # groups of two: 1.0, 1.1, 1.0, 1.35
    assert O.group_limited_choice(s, 3, {"count": 4, "keep": 2}) == [6, 7, 3]          # the best single expert is in a dropped group
    assert O.group_limited_choice(s, 3, {"count": 4, "keep": 3}) == [0, 6, 7]          # a tie between groups: the lower index stays
    assert O.group_limited_choice(s, 2, {"count": 8, "keep": 2}) == [0, 4]             # groups of one: their one score
    assert O.group_limited_choice(s, 2, None) == [0, 4]
    assert O.group_limited_choice([0.9, 0.0, 0.0, 0.5, 0.45, 0.0], 2, {"count": 2, "keep": 1}) == [3, 4]   # two best scores, not the best one


def test_plain_window_mask_layer_norm_and_rotation():
    ok = O.window_mask(6, 3)
    assert [int(r.sum()) for r in ok] == [1, 2, 3, 3, 3, 3] and bool(ok[5, 3]) and not bool(ok[5, 2]) and not bool(ok[2, 3])
    assert bool(O.window_mask(6, None)[5, 0])
    x = rand(4, 7, seed=5, s=3.0) + 2.0
    want = torch.nn.functional.layer_norm(x, (7,), rand(7, seed=6), rand(7, seed=7), 1e-5)
    assert (O.layer_norm(x, rand(7, seed=6), rand(7, seed=7), 1e-5) - want).abs().max() < 1e-12
    v = torch.tensor([[1.0, 0.0, 5.0]], dtype=F64)
    r = O.rotate_pairs(v, torch.tensor([3]), 2, 10.0)
    assert abs(float(r[0, 0]) - math.cos(3.0)) < 1e-12 and abs(float(r[0, 1]) - math.sin(3.0)) < 1e-12 and float(r[0, 2]) == 5.0


def test_plain_model_is_causal_and_a_window_forgets():
    """Changing the last token changes no earlier logits; in a model of one window of three keys the token three back does not matter."""
    from omchat_b200.model.munevik import random_state_dict
    cd = config_a()
    sd = random_state_dict(MunevikConfig.from_dict(cd), seed=3)
    t = tokens_for(cd, 20, 1)
    a, b = O.forward(cd, sd, t), O.forward(cd, sd, t[:-1] + [(t[-1] + 1) % 131])
    assert torch.equal(a[:-1], b[:-1]) and (a[-1] - b[-1]).abs().max() > 1e-3
    one = dict(cd, layers=[cd["layers"][0]])
    one["layers"][0]["mixer"]["mask"]["size"] = 3
    c = O.forward(one, sd, t)
    for back, same in ((3, True), (2, False)):
        d = O.forward(one, sd, t[:19 - back] + [(t[19 - back] + 1) % 131] + t[20 - back:])
        assert ((c[19] - d[19]).abs().max() < 1e-12) == same
