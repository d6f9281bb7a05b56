"""Sorupel on the GPU against the plain restatement in oracle/sorupel_oracle.py (float64, whole sequences): whole prompts, decoding,
portions, mixed batches over reused pages and slots (poisoned with NaN), chunk edges through the whole model, long decoding, greedy
generation through the scheduler, trace replay. The kernels alone are in test_sorupel_kernels_gpu.py."""
import json
import os
import subprocess
import sys

import pytest
import torch

pytestmark = pytest.mark.gpu

if not torch.cuda.is_available():  # collected on the CPU box too
    pytest.skip("needs a CUDA device", allow_module_level=True)

from sorupel_cases import CONFIGS, O, attention, close, config_a, config_for, dense, latent, model_dict, row_errors, tokens_for  # noqa: E402
from omchat_b200.config import SorupelConfig  # noqa: E402
from omchat_b200.model.sorupel import SorupelForCausalLM, random_state_dict  # noqa: E402
from omchat_b200.serving import StepScheduler  # noqa: E402

DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def build(cfg_dict, dtype, seed=0, edit=None):
    cfg = SorupelConfig.from_dict(cfg_dict)
    sd = random_state_dict(cfg, seed=seed)
    if edit:
        edit(sd)
    return SorupelForCausalLM.from_state_dict(sd, cfg, device=DEV, dtype=dtype), sd


def poison(sched):
    for s in range(sched.cache.n_slots):
        sched.cache.poison_slot(s)
    for pool in sched.cache.pools:
        if pool is not None:
            pool.fill_(float("nan"))


def run_schedule(model, steps, max_tokens, slots=4):
    """steps: [([(key, tokens, want)], end-keys)] over poisoned slots and pages. Returns {key: logit rows in the order they came}."""
    sched = StepScheduler(model, max_tokens=max_tokens, slots=slots)
    poison(sched)
    out = {}
    for entries, end in steps:
        lg = sched.run_step(entries, end)
        at = 0
        for key, _, want in entries:
            for _ in want:
                out.setdefault(key, []).append(lg[at].float().cpu().clone())
                at += 1
    return {k: torch.stack(v) for k, v in out.items()}


def _i32(x):
    return torch.tensor(x, device=DEV, dtype=torch.int32)


@pytest.mark.parametrize("name", ["a", "b", "c"])
def test_whole_prompt_layer_by_layer_in_fp32(name):
    cd = CONFIGS[name]()
    model, sd = build(cd, torch.float32, seed=1)
    toks, ocol = tokens_for(cd, 61, 2), []
    want = O.forward(cd, sd, toks, ocol)
    cache = model.decoder.new_cache(8, 2)
    cache.set_pages(1, 0, [3, 1, 2, 5, 4][:-(-61 // cd["kv_page_size"])])
    cache.sync()
    for s in range(2):
        cache.poison_slot(s)
    n = len(toks)
    for portions in ([(0, n, 1, 0)], None):
        col = []
        lg = model.step(_i32(toks), _i32(list(range(n))), _i32([1] * n), cache, torch.arange(n, device=DEV), collect=col, portions=portions)
        for i, (a, b) in enumerate(zip(col, ocol)):
            assert (a.double().cpu() - b).abs().max() < 1e-4 * max(1.0, float(b.abs().max())), i
        assert close(lg, want, torch.float32)


@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
@BOTH
def test_logits_of_whole_prompts(name, dtype):
    cd = config_for(name, dtype)
    model, sd = build(cd, dtype, seed=3)
    toks = tokens_for(cd, 140 if name != "d" else 90, 4)
    want = O.forward(cd, sd, toks)
    out = run_schedule(model, [([("r", toks, list(range(len(toks))))], ["r"])], max_tokens=256)
    assert close(out["r"], want, dtype)


@pytest.mark.parametrize("name", ["a", "b", "c", "d"])
@pytest.mark.parametrize("dtype,graph", [(torch.float32, True), (torch.float32, False), (torch.bfloat16, True)])
def test_prefill_against_token_by_token_decoding(name, dtype, graph):
    """From the very first token, and from a prompt: every logit row against the oracle's row of the whole sequence."""
    cd = config_for(name, dtype)
    model, sd = build(cd, dtype, seed=5)
    model.decoder.use_graph = graph
    toks = tokens_for(cd, 70, 6)
    want = O.forward(cd, sd, toks)
    for first in (1, 33):
        steps = [([("r", toks[:first], list(range(first)))], [])] + [([("r", [t], [0])], []) for t in toks[first:]]
        assert close(run_schedule(model, steps, max_tokens=128)["r"], want, dtype), first


@pytest.mark.parametrize("name", ["a", "c"])
@BOTH
def test_portions_of_every_size_down_to_two_tokens(name, dtype):
    cd = CONFIGS[name]()
    model, sd = build(cd, dtype, seed=7)
    toks = tokens_for(cd, 171, 8)
    want = O.forward(cd, sd, toks)
    sizes = [2, 3, 2, 17, 1, 16, 15, 2, 33, 59, 2, 1, 1, 2, 5, 10]
    assert sum(sizes) == len(toks)
    steps, at = [], 0
    for s in sizes:
        steps.append(([("r", toks[at:at + s], list(range(s)))], []))
        at += s
    assert close(run_schedule(model, steps, max_tokens=192)["r"], want, dtype)
    # all in portions of two
    steps = [([("r", toks[i:i + 2], list(range(len(toks[i:i + 2]))))], []) for i in range(0, len(toks), 2)]
    assert close(run_schedule(model, steps, max_tokens=192)["r"], want, dtype)


@pytest.mark.parametrize("name", ["a", "c"])
@BOTH
def test_unequal_requests_in_one_batch_with_reused_pages_and_slots(name, dtype):
    """Five requests over three slots: portions beside single tokens, pauses, requests that end and hand their slot and pages
    (poisoned with NaN) to the next one. Every row equals the request run alone (the oracle)."""
    cd = CONFIGS[name]()
    model, sd = build(cd, dtype, seed=9)
    lens = {"p": 90, "q": 37, "r": 1, "s": 64, "t": 50}
    toks = {k: tokens_for(cd, n, 10 + i) for i, (k, n) in enumerate(lens.items())}
    want = {k: O.forward(cd, sd, v) for k, v in toks.items()}
    at, got = {k: 0 for k in toks}, {k: [] for k in toks}
    sched = StepScheduler(model, max_tokens=3 * 96, slots=3)
    poison(sched)
    plan = [[("p", 40), ("q", 2)], [("p", 1), ("q", 30), ("r", 1)], [("p", 1), ("q", 1)], [("q", 4), ("s", 33)], [("p", 20), ("s", 1)],
            [("p", 1), ("s", 2), ("t", 17)], [("p", 27), ("s", 28), ("t", 1)], [("t", 2)], [("t", 30)]]
    for entries in plan:
        ent = []
        for k, n in entries:
            lo, at[k] = at[k], min(at[k] + n, lens[k])
            ent.append((k, toks[k][lo:at[k]], list(range(at[k] - lo))))
        end = [k for k, _, _ in ent if at[k] == lens[k]]
        held = {k: (sched.live[k].slot, list(sched.live[k].pages)) for k in end if k in sched.live}
        lg, i = sched.run_step(ent, end), 0
        for k, _, w in ent:
            got[k] += [lg[i + j].float().cpu().clone() for j in range(len(w))]
            i += len(w)
        for slot, pages in held.values():      # what a request leaves behind is garbage for the next owner
            sched.cache.poison_slot(slot)
            for pool in sched.cache.pools:
                if pool is not None and pages:
                    pool[torch.tensor(pages, device=DEV)] = float("nan")
    for k in toks:
        assert at[k] == lens[k] and close(torch.stack(got[k]), want[k], dtype), k


@BOTH
def test_long_decoding_of_two_requests(dtype):
    cd = CONFIGS["a"]()
    model, sd = build(cd, dtype, seed=11)
    ta, tb = tokens_for(cd, 340, 12), tokens_for(cd, 335, 13)
    wa, wb = O.forward(cd, sd, ta), O.forward(cd, sd, tb)
    steps = [([("a", ta[:10], list(range(10))), ("b", tb[:5], list(range(5)))], [])]
    steps += [([("a", [ta[10 + i]], [0]), ("b", [tb[5 + i]], [0])], []) for i in range(330)]   # over many chunk edges
    out = run_schedule(model, steps, max_tokens=2 * 352)
    assert close(out["a"], wa, dtype) and close(out["b"], wb, dtype)


def chunk_model(chunk, bigram, tensor):
    d = 32 if tensor else 12
    return model_dict(64, 64, [attention(4, 2, d, 8, chunk, None, softcap=5.0), attention(6, 1, d, d, chunk, dense(40))], bigram=(50, 3, 7) if bigram else None)


@pytest.mark.parametrize("bigram", [False, True])
@pytest.mark.parametrize("chunk,tensor", [(16, True), (33, False), (64, True), (70, True)])
@BOTH
def test_a_changed_token_reaches_exactly_its_chunk(chunk, bigram, tensor, dtype):
    """Two sequences that differ in one token: the rows from it to its chunk's end give different logits, every other row the same ones -
    in a whole prompt, in portions and decoded one by one across the edge. With bigram rows the next token's row differs too: for the
    last token of a chunk that changes the whole next chunk."""
    cd = chunk_model(chunk, bigram, tensor)
    model, sd = build(cd, dtype, seed=21)
    n = 150
    for mark in (chunk // 2, chunk - 1, chunk, 2 * chunk - 1):
        ta = tokens_for(cd, n, 5)
        tb = list(ta)
        tb[mark] = (ta[mark] + 7) % 64
        end = ((mark + 1 if bigram else mark) // chunk + 1) * chunk
        cuts = {"whole": [n], "portions": [mark - 1, 2, max(end - mark - 2, 1), 2, 3], "decoded": [end - 3, 1, 1, 1, 1, 1, 1]}
        for kind, sizes in cuts.items():
            sizes = sizes + ([n - sum(sizes)] if sum(sizes) < n else [])
            rows = []
            for t in (ta, tb):
                steps, at = [], 0
                for s in sizes:
                    if s > 0 and at < n:
                        steps.append(([("r", t[at:at + s], list(range(len(t[at:at + s]))))], []))
                        at += s
                rows.append(run_schedule(model, steps, max_tokens=160)["r"])
            diff = (rows[0] - rows[1]).abs().amax(-1)
            assert (diff[mark:end] > 1e-6).all(), (mark, kind)
            assert (diff[:mark] == 0).all() and (diff[end:] == 0).all(), (mark, kind)


@pytest.mark.parametrize("shared", [False, True])
@BOTH
def test_a_marked_token_far_back_is_found(shared, dtype):
    """Latent attention (or a second layer on the first one's rows) that looks for one token: its latent outshines hundreds of others by far.
    Rows hundreds of positions behind it follow the oracle closely and change when the mark becomes another token."""
    cd = model_dict(64, 64, [latent(4, 32, 16, 24, 48, None)] + ([latent(3, 32, 16, 16, 48, None, kv_from=0)] if shared else []), bigram=None)
    i = 1 if shared else 0

    def edit(sd):
        sd["embed"][:, 60:] = 0.0                                    # four dimensions that only the mark, a plain token and the queries know
        sd["embed"][:, 61] = 2.0
        sd["embed"][7, 60] = 40.0
        for k in range(2 if shared else 1):
            sd[f"l{k}.mix.q"][:, 60:] = 0.0
            sd[f"l{k}.mix.o"][60:] = 0.0
        dkv = sd["l0.mix.dkv"]
        dkv[:, 60:] = 0.0
        dkv[0] = 0.0
        dkv[0, 60] = 3.0                                             # latent column 0: the mark
        uk, H, dn = sd[f"l{i}.mix.uk"], (3 if shared else 4), 32
        uk.view(H, dn, 48)[:, 0] = 0.0
        uk.view(H, dn, 48)[:, 0, 0] = 4.0                            # key dimension 0 reads it
        q = sd[f"l{i}.mix.q"].view(H, 48, 64)
        q[:, 0] = 0.0
        q[:, 0, 61] = 4.0                                            # every query asks for it
    model, sd = build(cd, dtype, seed=31, edit=edit)
    n = 420
    toks = [t if t != 7 else 8 for t in tokens_for(cd, n, 6)]
    for mark in (0, 63, 64):
        ta, tb = list(toks), list(toks)
        ta[mark], tb[mark] = 7, 9
        want, other = O.forward(cd, sd, ta), O.forward(cd, sd, tb)
        assert float(row_errors(other, want)[mark:].min()) > 0.15         # the mark decides every row behind it
        for sizes in ([n], [100, 200, 2, 110, 1, 1, 1, 1, 1, 1, 1, 1]):
            steps, at = [], 0
            for s in sizes:
                steps.append(([("r", ta[at:at + s], list(range(s)))], []))
                at += s
            assert close(run_schedule(model, steps, max_tokens=448)["r"], want, dtype), (mark, sizes)


def test_first_tokens_do_not_see_what_a_slot_held_before():
    """The same request twice in the same slot and pages, the second time over whatever the first left: identical logits."""
    cd = config_a()
    model, sd = build(cd, torch.float32, seed=13)
    toks = tokens_for(cd, 40, 14)
    sched = StepScheduler(model, max_tokens=48, slots=1)
    a = sched.run_step([("x", toks, [0, 1, 2, 3, 39])], ["x"]).clone()
    b = sched.run_step([("y", toks[:3], [0, 1, 2])], []).clone()
    c = sched.run_step([("y", toks[3:], [0, 36])], ["y"])
    assert (a[:3] - b).abs().max() < 1e-4 and (a[3:] - c).abs().max() < 1e-4


def test_tensor_core_and_plain_attention_agree():
    cd = CONFIGS["c"]()
    model, sd = build(cd, torch.bfloat16, seed=17)
    toks, rows = tokens_for(cd, 120, 3), []
    for on in (True, False):
        model.decoder.tensor_attention = on
        rows.append(run_schedule(model, [([("r", toks, list(range(120)))], ["r"])], max_tokens=128)["r"])
    assert close(rows[0], rows[1], torch.bfloat16)


def test_greedy_generation_through_the_scheduler():
    """generate() - StepScheduler with chunked prefill over fewer slots than prompts - against the oracle's argmax."""
    cd = config_a()
    model, sd = build(cd, torch.float32, seed=15)
    prompts = [tokens_for(cd, n, 20 + n) for n in (1, 9, 40, 17, 33, 2)]
    outs = model.generate(prompts, max_new_tokens=12, slots=4, chunk=16)
    for p, o in zip(prompts, outs):
        seq = list(p)
        for _ in range(12):
            lg = O.forward(cd, sd, seq)[-1]
            top2 = torch.topk(lg, 2).values
            nxt = int(lg.argmax())
            if float(top2[0] - top2[1]) < 1e-3:      # a near tie: take what the model took and go on
                nxt = int(o[len(seq)])
            seq.append(nxt)
        assert o.tolist() == seq


def test_trace_replay_as_a_subprocess(tmp_path):
    """bin/trace_run on a saved checkpoint: requests that pause and end, wanted rows, 'done' lines, both compute dtypes."""
    from omchat_b200.model.checkpoint import save_checkpoint
    cd = config_a()
    cfg = SorupelConfig.from_dict(cd)
    sd = random_state_dict(cfg, seed=17)
    save_checkpoint(sd, cfg, str(tmp_path / "model"))
    ta, tb = tokens_for(cd, 30, 18), tokens_for(cd, 12, 19)
    wa, wb = O.forward(cd, sd, ta), O.forward(cd, sd, tb)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": ta[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": tb[:2], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": ta[20:21], "want": [0]}, {"id": "b", "tokens": tb[2:], "want": [9]}], "end": ["b"]},
             {"step": 3, "entries": [{"id": "a", "tokens": ta[21:], "want": [8]}], "end": ["a"]}]
    for dtype, tol in (("float32", 2e-4), ("bfloat16", 0.2)):
        out = tmp_path / dtype
        r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "model"), "--dtype", dtype, "--out", str(out),
                            "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
        assert r.returncode == 0, r.stderr[-2000:]
        assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2", "done 3"]
        assert not (out / "1.f32").exists()
        rd = lambda n: torch.frombuffer(bytearray((out / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cd["vocab"])
        assert float(row_errors(rd(0), wa[[0, 19]]).max()) < tol
        assert float(row_errors(rd(2), torch.stack([wa[20], wb[11]])).max()) < tol
        assert float(row_errors(rd(3), wa[29:30]).max()) < tol
