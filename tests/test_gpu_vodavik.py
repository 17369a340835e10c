"""Vodavik on the B200 against the plain CPU oracle (fp64), through sessions, the scheduler and the entry points."""
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from mdlarc_scale_b200 import generation, registry, weights
from mdlarc_scale_b200.layered import Segment
from oracle import vodavik as vo

from gpu_util import have_b200
from vodavik_util import BIG_HEADS, CONFIGS, attention, config, mlstm, oracle_logits, rel_error, tokens

pytestmark = [pytest.mark.gpu, pytest.mark.skipif(not have_b200(), reason="needs a B200")]
ROOT = Path(__file__).resolve().parent.parent
TOL = {"f32": 3e-5, "f16": 1e-2, "bf16": 6e-2}
STEP_PATHS = dict(fused_proj=False, attn_path="stream", mlstm_path="step")   # plain kernels everywhere


def build(cfg, seed=0, fmt="f32", w=None, **kw):
    w = vo.random_weights(cfg, seed) if w is None else w
    return registry.build_engine(cfg, w, "cuda:0", fmt, **kw), w


def run_portions(eng, toks, sizes, t_max=None, session=None):
    """Logits of all tokens, fed in portions of the given sizes (the rest one by one through the decode step)."""
    s = session or eng.new_session(2, t_max or len(toks), 1, 4096, stop_on_end=False)
    slot, at, rows = s.acquire(), 0, []
    sizes = list(sizes) + [1] * (len(toks) - sum(sizes))
    for n in sizes:
        rows.append(s.step([Segment(slot, toks[at:at + n], list(range(n)))])[0])
        at += n
    s.poll()
    s.release(slot)
    return torch.cat(rows)


@pytest.mark.parametrize("fmt", ["f32", "f16", "bf16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts_and_decoding(name, fmt):
    cfg = CONFIGS[name]
    eng, w = build(cfg, 11, fmt)
    toks = tokens(cfg, 300, 5)
    want = oracle_logits(cfg, w, toks)
    whole = run_portions(eng, toks, [300])
    assert rel_error(whole, want) < TOL[fmt]
    assert rel_error(run_portions(eng, toks, [260]), want) < TOL[fmt]            # 40 decoded tokens
    assert rel_error(run_portions(eng, toks[:40], [1]), want[:40]) < TOL[fmt]    # decoded from the second token on
    if fmt != "f32":
        plain, _ = build(cfg, 11, fmt, **STEP_PATHS)
        assert rel_error(run_portions(plain, toks, [260]), want) < TOL[fmt]


@pytest.mark.parametrize("fmt", ["f32", "f16", "bf16"])
def test_head_sizes_above_128(fmt):
    eng, w = build(BIG_HEADS, 2, fmt)
    toks = tokens(BIG_HEADS, 90, 5)
    assert rel_error(run_portions(eng, toks, [60, 2]), oracle_logits(BIG_HEADS, w, toks)) < TOL[fmt]


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_every_layer(fmt):
    """The residual stream after every layer, so that a fault shows at the layer that makes it."""
    for name in ("mixed", "unequal"):
        cfg = CONFIGS[name]
        eng, w = build(cfg, 4, fmt)
        toks = tokens(cfg, 150, 9)
        seq = vo.Sequence(cfg, w, torch.float64)
        seq.step(toks)
        s = eng.new_session(1, 150, 1, 150, stop_on_end=False)
        _, _, res = s.prefill_segments([Segment(s.acquire(), toks)], residuals=True)
        s.poll()
        for got, want in zip(res, seq.residuals):
            assert float((got.cpu().double() - want).abs().max()) < (2e-4 if fmt == "f32" else 6e-2)
            assert float((got.cpu().double() - want).pow(2).mean().sqrt()) < (1e-5 if fmt == "f32" else 5e-3)


@pytest.mark.parametrize("fmt", ["f32", "f16"])
@pytest.mark.parametrize("sizes", [[2] * 60, [3, 64, 1, 128, 2, 127, 5], [129, 2, 255, 2], [256, 257], [63, 65, 2, 126, 130]])
def test_portions(sizes, fmt):
    cfg = CONFIGS["mixed"]
    eng, w = build(cfg, 21, fmt)
    toks = tokens(cfg, sum(sizes) + 6, 3)
    assert rel_error(run_portions(eng, toks, sizes), oracle_logits(cfg, w, toks)) < TOL[fmt]


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_unequal_batches_and_reused_slots(fmt):
    """Mixed calls of long portions, short portions and single tokens; every request equals itself alone, also
    in a slot that an earlier request has used."""
    cfg = CONFIGS["wide_group"]
    eng, w = build(cfg, 8, fmt)
    lens = [200, 1, 77, 130, 2, 33]
    reqs = [tokens(cfg, n, 40 + i) for i, n in enumerate(lens)]
    want = [oracle_logits(cfg, w, r) for r in reqs]
    s = eng.new_session(3, 256, 1, 300, stop_on_end=False)
    at, slot, got, queue = {}, {}, {i: [] for i in range(len(reqs))}, list(range(len(reqs)))
    rng = np.random.default_rng(0)
    while queue or slot:
        while queue and s.free_slots:
            i = queue.pop(0)
            slot[i], at[i] = s.acquire(), 0
        segs, who = [], []
        for i in list(slot):
            n = int(min(rng.choice([1, 2, 50, 120]), lens[i] - at[i]))
            segs.append(Segment(slot[i], reqs[i][at[i]:at[i] + n], list(range(n))))
            who.append(i)
        for i, seg, rows in zip(who, segs, s.step(segs)):
            got[i].append(rows)
            at[i] += len(seg.tokens)
            if at[i] == lens[i]:
                s.release(slot.pop(i))
    s.poll()
    for i in range(len(reqs)):
        assert rel_error(torch.cat(got[i]), want[i]) < TOL[fmt]


def test_decode_step_holds_other_slots():
    cfg = CONFIGS["mixed"]
    eng, w = build(cfg, 8, "f32")
    a, b = tokens(cfg, 50, 1), tokens(cfg, 60, 2)
    s = eng.new_session(3, 64, 1, 128, stop_on_end=False)
    sa, sb = s.acquire(), s.acquire()
    s.step([Segment(sa, a[:40]), Segment(sb, b[:40])])
    rows = {sa: [], sb: []}
    order = [sa] * 3 + [sb] * 5 + [sa, sb] * 7 + [sb] * 8
    done = {sa: 40, sb: 40}
    for k in order:
        toks = a if k == sa else b
        rows[k].append(s.feed([k], [toks[done[k]]]).clone())
        done[k] += 1
    assert rel_error(torch.cat(rows[sa]), oracle_logits(cfg, w, a)[40:50]) < TOL["f32"]
    assert rel_error(torch.cat(rows[sb]), oracle_logits(cfg, w, b)[40:60]) < TOL["f32"]


def far_key_model(every=1000):
    """One attention layer whose scores are dominated by a matching token far back: the queries and keys of two
    token ids are made large, so dropping or misplacing one key moves the logits."""
    cfg = config(128, 90, [attention(2, 1, 32, 48, every=every)])
    w = vo.random_weights(cfg, 5)
    w["l0.mix.q"] = w["l0.mix.q"] * 0.2
    w["l0.mix.sink"] = torch.tensor([3.0, 4.0])
    probe = w["embed"][1] / w["embed"][1].norm()
    for h in range(2):
        w["l0.mix.q"][h * 32] += 6 * probe
    mark = w["embed"][0] / w["embed"][0].norm()
    w["l0.mix.k"][0] += 1.2 * mark
    w["l0.mix.q.norm"][0] = 5.0
    w["l0.mix.k.norm"][0] = 5.0
    return cfg, {k: v.to(torch.bfloat16).float() for k, v in w.items()}


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_far_keys_at_tile_borders(fmt):
    """A token 0 somewhere in the past is what token 1 asks for; places around the borders of the kernels'
    16-, 32- and 128-row slices and of the 256-row query blocks, asked in a prompt and while decoding."""
    cfg, w = far_key_model()
    eng, _ = build(cfg, fmt=fmt, w=w)
    base = torch.randint(2, 90, (420,), generator=torch.Generator().manual_seed(1)).tolist()
    for far in (0, 1, 15, 16, 31, 32, 127, 128, 129, 255, 256, 257, 383, 384):
        toks = list(base)
        toks[far] = 0
        asks = [p for p in (far + 1, far + 2, 257, 300, 384, 385, 400, 412, 419) if p > far]
        for p in asks:
            toks[p] = 1
        want = oracle_logits(cfg, w, toks)
        blind = list(toks)
        blind[far] = 2
        without = oracle_logits(cfg, w, blind)
        assert all(rel_error(want[p:p + 1], without[p:p + 1]) > 10 * TOL[fmt] for p in asks)   # the key matters
        got = run_portions(eng, toks, [405])          # 412 and 419 are decoded
        assert rel_error(got, want) < 2 * TOL[fmt]


def planted(monkeypatch, name, fn):
    monkeypatch.setattr(vo, name, fn)


MISTAKES = {
    "no sink": ("sink_softmax", lambda s, k: torch.softmax(s, -1)),
    "sink scaled": ("sink_softmax", lambda s, k, f=vo.sink_softmax: f(s, k * 0.5)),
    "gain off by one": ("query_temperature", lambda p, c, e, f=vo.query_temperature: f([x + 1 for x in p], c, e)),
    "no gain": ("query_temperature", lambda p, c, e: torch.ones(len(list(p)), dtype=torch.float64)),
    "rms instead of centred norm": ("layer_norm", lambda x, w, eps: vo.rms_unit(x, eps) * w),
    "uncapped gates": ("mlstm_gates", lambda w, p, cap, h: (vo.linear(h, w, f"{p}.mix.i", True),
                                                             torch.nn.functional.logsigmoid(vo.linear(h, w, f"{p}.mix.f", True)))),
    "gelu": ("feed_forward", lambda w, p, h: vo.linear(torch.nn.functional.gelu(vo.linear(h, w, f"{p}.mlp.up")), w, f"{p}.mlp.down")),
}


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_each_mechanism_shows(mistake, monkeypatch):
    """The comparison sees every mechanism: with a mistake planted in the oracle it no longer agrees."""
    cfg = config(144, 120, [attention(4, 2, 24, 40, ff=96, every=3, coef=0.8), mlstm(3, 24, 40, cap=2.0)])
    w = vo.random_weights(cfg, 13)
    for n in ("i", "f"):
        w[f"l1.mix.{n}.b"] = w[f"l1.mix.{n}.b"] * 2
    eng, _ = build(cfg, fmt="f32", w=w)
    toks = tokens(cfg, 70, 2)
    got = run_portions(eng, toks, [64])
    assert rel_error(got, oracle_logits(cfg, w, toks)) < TOL["f32"]
    planted(monkeypatch, *MISTAKES[mistake])
    assert rel_error(got, oracle_logits(cfg, w, toks)) > 100 * TOL["f32"]


def test_stabiliser_starts_at_zero():
    """Low input gates at the start: the running maximum stays at its start value, which the denominator sees."""
    cfg = config(128, 64, [mlstm(2, 16, 24)])
    w = vo.random_weights(cfg, 3)
    w["l0.mix.i.b"] = torch.tensor([-7.0, -8.0])
    w["l0.mix.f.b"] = torch.tensor([6.0, 5.0])
    for fmt in ("f32", "f16"):
        eng, _ = build(cfg, fmt=fmt, w=w)
        toks = tokens(cfg, 200, 6)
        assert rel_error(run_portions(eng, toks, [1, 2, 150]), oracle_logits(cfg, w, toks)) < TOL[fmt]


@pytest.mark.parametrize("fmt", ["f32", "f16", "bf16"])
def test_extreme_gates(fmt):
    """Forget gates that clear the state, long memory, and input gates that swing over the whole capped range."""
    cfg = config(128, 64, [mlstm(4, 48, 64, cap=15.0), mlstm(4, 64, 48, cap=15.0)])
    w = vo.random_weights(cfg, 3)
    for n in range(2):
        w[f"l{n}.mix.f"] = w[f"l{n}.mix.f"] * torch.tensor([1.0, 6.0, 0.2, 3.0])[:, None]
        w[f"l{n}.mix.f.b"] = torch.tensor([-9.0, 0.0, 9.0, 4.0])
        w[f"l{n}.mix.i"] = w[f"l{n}.mix.i"] * torch.tensor([6.0, 1.0, 3.0, 9.0])[:, None]
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    eng, _ = build(cfg, fmt=fmt, w=w)
    toks = tokens(cfg, 500, 6)
    got, want = run_portions(eng, toks, [131, 2, 300, 60]), oracle_logits(cfg, w, toks)
    if fmt == "f32":
        assert rel_error(got, want) < 10 * TOL[fmt]
    else:       # rows whose normaliser n.q nearly vanishes amplify the operand rounding: most rows, not all
        err = np.array([rel_error(got[i:i + 1], want[i:i + 1]) for i in range(len(toks))])
        assert np.quantile(err, 0.9) < 3 * TOL[fmt]


def test_long_decoding():
    cfg = CONFIGS["plain_heads"]
    for fmt in ("f32", "f16"):
        eng, w = build(cfg, 17, fmt)
        toks = tokens(cfg, 700, 4)
        assert rel_error(run_portions(eng, toks, [5]), oracle_logits(cfg, w, toks)) < TOL[fmt]


def test_portions_and_batches_do_not_change_results_beyond_rounding():
    cfg = CONFIGS["mixed"]
    eng, _ = build(cfg, 6, "f16")
    toks = tokens(cfg, 333, 4)
    a = run_portions(eng, toks, [333])
    assert torch.equal(a, run_portions(eng, toks, [333]))                      # deterministic
    for sizes in ([100, 100, 133], [2] * 166 + [1], [332]):
        assert rel_error(run_portions(eng, toks, sizes), a) < 6e-3


def agree(got, rows, want, tol):
    """Tokens equal the oracle's up to a step whose own top-two margin is below ``tol``."""
    for i, (g, t) in enumerate(zip(got, want)):
        if g != t:
            top = np.sort(rows[i].double().numpy())[-2:]
            return top[1] - top[0] < tol
    return True


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_greedy_generation_with_fewer_slots_than_requests(fmt):
    cfg = CONFIGS["mixed"]
    eng, w = build(cfg, 30, fmt)
    prompts = [tokens(cfg, n, 70 + n) for n in (5, 140, 1, 33, 64, 18, 90)]
    out, logits = generation.generate(eng, prompts, 24, max_batch=3, prefill_tokens=100, return_logits=True)
    for i, p in enumerate(prompts):
        want, rows = vo.greedy(cfg, w, p, 24)
        assert len(out[i]) == 24 and agree(out[i], rows, want, 1e-4 if fmt == "f32" else 2e-2)
        seq = vo.Sequence(cfg, w, torch.float64)
        own = seq.step(p + out[i])[len(p) - 1:-1]
        assert rel_error(logits[i], own) < TOL[fmt]
        assert all(int(r.argmax()) == t for r, t in zip(logits[i].cpu(), out[i]))
    assert out == generation.generate(eng, prompts, 24, max_batch=64)


def test_end_token_stops_a_request():
    cfg = CONFIGS["plain_heads"]
    eng, _ = build(cfg, 3, "f32")
    prompts = [tokens(cfg, n, n) for n in (9, 20, 31, 12)]
    full = generation.generate(eng, prompts, 60)
    end = full[0][7]
    out = generation.generate(eng, prompts, 60, end_token=end, max_batch=2)
    for got, ref in zip(out, full):
        assert got == (ref[:ref.index(end) + 1] if end in ref else ref)


def test_sampling():
    from mdlarc_scale_b200.engine import sample_uniform
    cfg = CONFIGS["single_head"]
    eng, _ = build(cfg, 3, "f32")
    prompts = [tokens(cfg, 12, i) for i in range(5)]
    for top_k, temp in ((None, 0.8), (4, 1.5), (1, 1.0)):
        out, logits = generation.generate(eng, prompts, 10, temperature=temp, top_k=top_k, seed=99, max_batch=2,
                                          return_logits=True)
        assert out == generation.generate(eng, prompts, 10, temperature=temp, top_k=top_k, seed=99)   # slots do not matter
        for i, row in enumerate(out):
            for j, t in enumerate(row):
                lg = logits[i][j].cpu().double()
                order = torch.sort(lg, descending=True, stable=True).indices
                keep = order[:top_k] if top_k else order
                p = torch.zeros_like(lg)
                p[keep] = torch.softmax(lg[keep] / temp, 0)
                cdf, u = torch.cumsum(p, 0), sample_uniform(99, i, j)
                lo = float(cdf[t] - p[t])
                assert lo - 1e-5 <= u <= float(cdf[t]) + 1e-5 and p[t] > 0
    assert generation.generate(eng, prompts, 6, temperature=1.0, top_k=1, seed=1) == generation.generate(eng, prompts, 6)


def test_errors():
    cfg = CONFIGS["mixed"]
    eng, _ = build(cfg, 1, "f16")
    s = eng.new_session(1, 20, 1, 64, stop_on_end=False)
    slot = s.acquire()
    with pytest.raises(RuntimeError):
        s.acquire()
    with pytest.raises(ValueError):
        s.step([Segment(slot, list(range(60)))])        # more positions than the slot has
    with pytest.raises(ValueError):
        generation.generate(eng, [[cfg["vocab"]]], 2)
    with pytest.raises(ValueError):
        generation.generate(eng, [[]], 2)
    bad = json.loads(json.dumps(cfg))
    bad["layers"][1]["mixer"]["kv_heads"] = 4
    with pytest.raises(Exception):
        build(bad)


def test_model_folder_command_line_and_trace(tmp_path):
    cfg = CONFIGS["mixed"]
    w = vo.random_weights(cfg, 42)
    weights.write_model_folder(tmp_path / "m", cfg, {k: v.to(torch.bfloat16) for k, v in w.items()})
    prompts = [tokens(cfg, 30, 1), tokens(cfg, 7, 2)]
    (tmp_path / "p.jsonl").write_text("\n".join(json.dumps(p) for p in prompts))
    run = subprocess.run([sys.executable, "-m", "mdlarc_scale_b200.generation", "--model", str(tmp_path / "m"), "--prompts",
                          str(tmp_path / "p.jsonl"), "--max-new", "8", "--dtype", "float32"], cwd=ROOT, capture_output=True,
                         text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    out = [json.loads(x) for x in run.stdout.splitlines() if x.startswith("[")]
    for p, o in zip(prompts, out):
        want, rows = vo.greedy(cfg, w, p, 8)
        assert agree(o, rows, want, 1e-4)
    a, b = tokens(cfg, 60, 3), tokens(cfg, 25, 4)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [0, 49]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[50:51], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[:20], "want": []}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": a[51:], "want": [8]}, {"id": "b", "tokens": b[20:], "want": [1, 4]}],
              "end": ["a", "b"]}]
    (tmp_path / "out").mkdir()
    run = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", "float32", "--out",
                          str(tmp_path / "out"), "--max-tokens", "90"], input="\n".join(map(json.dumps, steps)) + "\n",
                         capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    assert [x for x in run.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    la, lb = oracle_logits(cfg, w, a), oracle_logits(cfg, w, b)
    for n, want in ((0, la[[0, 49]]), (1, la[50:51]), (3, torch.cat([la[59:60], lb[[21, 24]]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert rel_error(got, want) < TOL["f32"]
    assert not (tmp_path / "out" / "2.f32").exists()
