"""Logesun on the B200 against the plain CPU oracle (fp64), through sessions, the scheduler and the entry points."""
import copy
import json
import subprocess
import sys
from pathlib import Path

import numpy as np
import pytest
import torch

from mdlarc_scale_b200 import generation, registry, weights
from mdlarc_scale_b200.layered import Segment
from oracle import logesun as lo

from gpu_util import have_b200
from logesun_util import BIG, CONFIGS, config, dense, latent, moe, oracle_logits, rel_error, tokens

pytestmark = [pytest.mark.gpu, pytest.mark.skipif(not have_b200(), reason="needs a B200")]
ROOT = Path(__file__).resolve().parent.parent
TOL = {"f32": 3e-5, "f16": 1e-2, "bf16": 7e-2}
PLAIN = [dict(attn_path="stream"), dict(gemm_path="simt", attn_path="stream")]
STRICT = config(168, 120, [latent(4, 40, 16, 48, 88, 56, 45, moe(4, 4, 56, limit=1.2, shared=100, shared_limit=0.8)),
                           latent(6, 64, 64, 64, 128, 128, 300, dense(200))], loop=(0, 2, 2))


def build(cfg, seed=0, fmt="f32", w=None, **kw):
    w = lo.random_weights(cfg, seed) if w is None else w
    return registry.build_engine(cfg, w, "cuda:0", fmt, **kw), w


def close_calls(cfg):
    """A choice among experts that rounding can turn over: a few rows may then differ by a whole expert, and the rows
    that see them by a little."""
    return any(x["mlp"] and x["mlp"]["kind"] == "moe" and x["mlp"]["router"]["top"] < x["mlp"]["router"]["experts"] for x in cfg["layers"])


def check(got, want, cfg, fmt, factor=1.0):
    if fmt == "f32" or not close_calls(cfg):
        assert rel_error(got, want) < factor * TOL[fmt]
    else:
        err = np.array([rel_error(got[i:i + 1], want[i:i + 1]) for i in range(len(want))])
        assert np.quantile(err, 0.5) < 2 * factor * TOL[fmt] and np.quantile(err, 0.85) < 4 * factor * TOL[fmt], np.quantile(err, [.5, .85, 1])
        assert np.median(err[:20]) < factor * TOL[fmt]


def run_portions(eng, toks, sizes, t_max=None, session=None, slots=2):
    """Logits of all tokens, fed in portions of the given sizes (the rest one by one through the decode step)."""
    s = session or eng.new_session(slots, t_max or len(toks), 1, 4096, stop_on_end=False)
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
    check(run_portions(eng, toks, [300]), want, cfg, fmt)
    check(run_portions(eng, toks, [260]), want, cfg, fmt)                        # 40 decoded tokens
    check(run_portions(eng, toks[:40], [1]), want[:40], cfg, fmt)                # decoded from the second token on
    if fmt != "f32":
        for kw in PLAIN:
            plain, _ = build(cfg, 11, fmt, **kw)
            check(run_portions(plain, toks, [260]), want, cfg, fmt)


@pytest.mark.parametrize("fmt", ["f32", "f16", "bf16"])
def test_strict_in_16_bit(fmt):
    """Every expert chosen, so that no rounding turns a choice over: all rows agree."""
    eng, w = build(STRICT, 3, fmt)
    toks = tokens(STRICT, 700, 8)
    want = oracle_logits(STRICT, w, toks)
    for sizes in ([700], [300, 2, 350], [5] * 130 + [40]):
        assert rel_error(run_portions(eng, toks, sizes), want) < TOL[fmt]


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_sizes_beyond_the_tensor_core_attention(fmt):
    eng, w = build(BIG, 2, fmt)
    toks = tokens(BIG, 150, 5)
    want = oracle_logits(BIG, w, toks)
    for sizes in ([150], [100, 2, 30]):
        check(run_portions(eng, toks, sizes), want, BIG, fmt)


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_every_layer_run(fmt):
    """The residual stream after every layer run, so that a fault shows at the run that makes it."""
    for cfg in (STRICT, config(136, 50, [latent(3, 24, 8, 16, 40, 72, 20, dense(72)), latent(2, 16, 24, 40, 24, 30, 64)], loop=(0, 2, 3))):
        eng, w = build(cfg, 4, fmt)
        toks = tokens(cfg, 150, 9)
        seq = lo.Sequence(cfg, w, torch.float64)
        seq.step(toks)
        s = eng.new_session(1, 150, 1, 150, stop_on_end=False)
        _, _, res = s.prefill_segments([Segment(s.acquire(), toks)], residuals=True)
        s.poll()
        assert len(res) == len(seq.residuals) == eng.spec.n_runs
        for got, want in zip(res, seq.residuals):
            assert float((got.cpu().double() - want).abs().max()) < (2e-4 if fmt == "f32" else 8e-2)
            assert float((got.cpu().double() - want).pow(2).mean().sqrt()) < (1e-5 if fmt == "f32" else 6e-3)


@pytest.mark.parametrize("fmt", ["f32", "f16"])
@pytest.mark.parametrize("sizes", [[2] * 60, [3, 64, 1, 128, 2, 127, 5], [129, 2, 255, 2], [256, 257], [63, 65, 2, 126, 130]])
def test_portions(sizes, fmt):
    eng, w = build(STRICT, 21, fmt)
    toks = tokens(STRICT, sum(sizes) + 6, 3)
    assert rel_error(run_portions(eng, toks, sizes), oracle_logits(STRICT, w, toks)) < TOL[fmt]


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_portions_of_other_configurations(fmt):
    for name in ("mixed", "many_heads", "head_blocks"):
        cfg = CONFIGS[name]
        eng, w = build(cfg, 22, fmt)
        sizes = [90, 2, 3, 140, 33]
        toks = tokens(cfg, sum(sizes) + 3, 3)
        check(run_portions(eng, toks, sizes), oracle_logits(cfg, w, toks), cfg, fmt)


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_unequal_batches_and_reused_slots(fmt):
    """Mixed calls of long portions, short portions and single tokens; every request equals itself alone, also
    in a slot that an earlier request has used."""
    cfg = STRICT
    eng, w = build(cfg, 8, fmt)
    lens = [200, 1, 77, 330, 2, 33]
    reqs = [tokens(cfg, n, 40 + i) for i, n in enumerate(lens)]
    want = [oracle_logits(cfg, w, r) for r in reqs]
    s = eng.new_session(3, 340, 1, 300, stop_on_end=False)
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
    done = {sa: 40, sb: 40}
    for k in [sa] * 3 + [sb] * 5 + [sa, sb] * 7 + [sb] * 8:
        toks = a if k == sa else b
        rows[k].append(s.feed([k], [toks[done[k]]]).clone())
        done[k] += 1
    assert rel_error(torch.cat(rows[sa]), oracle_logits(cfg, w, a)[40:50]) < TOL["f32"]
    assert rel_error(torch.cat(rows[sb]), oracle_logits(cfg, w, b)[40:60]) < TOL["f32"]


@pytest.mark.parametrize("fmt", ["f16", "bf16"])
@pytest.mark.parametrize("slots", [1, 40, 170])
def test_decode_batches(slots, fmt):
    """Decode steps of few sequences (rows split over CTAs, partial results merged) and of many (several per CTA),
    at unequal lengths."""
    cfg = config(128, 60, [latent(18, 32, 16, 32, 64, 256, 700), latent(8, 32, 64, 32, 64, 512, 300)])
    eng, w = build(cfg, 5, fmt)
    lens = [int(n) for n in np.random.default_rng(slots).integers(1, 900, slots)]
    if slots == 1:
        lens = [900]
    s = eng.new_session(slots, 920, 1, 4096, stop_on_end=False)
    ids = [s.acquire() for _ in range(slots)]
    base = tokens(cfg, 920, 1)
    for lo_ in range(0, slots, 4):
        s.step([Segment(ids[i], base[i:i + lens[i]]) for i in range(lo_, min(slots, lo_ + 4))])
    for _ in range(2):
        rows = s.feed(ids, [base[i + s.lens[ids[i]]] if i + s.lens[ids[i]] < 920 else 7 for i in range(slots)]).clone()
    s.poll()
    for i in {0, slots // 2, slots - 1, int(np.argmax(lens)), int(np.argmin(lens))}:
        toks = base[i:i + lens[i]]
        for k in range(2):
            at = i + lens[i] + k
            toks = toks + [base[at] if at < 920 else 7]
        want = oracle_logits(cfg, w, toks)[-1:]
        assert rel_error(rows[i:i + 1], want) < TOL[fmt]


def strong_key_model(window, heads=2, kv_rank=40):
    """One layer whose scores are dominated by a matching token: the latent, query and key of two token ids are made
    large, so that dropping, misplacing or adding one key moves the logits."""
    cfg = config(128, 90, [latent(heads, 32, 8, 48, 40, kv_rank, window)])
    w = lo.random_weights(cfg, 5)
    w["l0.mix.uq"] *= 0.2
    w["l0.mix.uk"] *= 0.2
    w["l0.mix.sink"] = torch.linspace(3.0, 4.0, heads)
    mark, probe = (w["embed"][i] / w["embed"][i].norm() for i in (0, 1))
    w["l0.mix.dkv"][0] += 3 * mark
    w["l0.mix.dq"][0] += 3 * probe
    w["l0.mix.dkv.norm"][0] = w["l0.mix.dq.norm"][0] = 4.0
    for h in range(heads):
        w["l0.mix.uk"][h * 32, 0] = 1.0
        w["l0.mix.uq"][h * 40, 0] = 1.0
    return cfg, {k: v.to(torch.bfloat16).float() for k, v in w.items()}


@pytest.mark.parametrize("fmt", ["f32", "f16"])
@pytest.mark.parametrize("window,heads,kv_rank", [(100, 2, 40), (128, 2, 40), (129, 19, 130), (1, 2, 40), (400, 33, 260)])
def test_keys_at_window_edges(window, heads, kv_rank, fmt):
    """Token 1 asks for token 0, placed just inside and just outside of the window of rows in a prompt, around the
    borders of key tiles and query blocks, and of decoded tokens."""
    cfg, w = strong_key_model(window, heads, kv_rank)
    eng, _ = build(cfg, fmt=fmt, w=w)
    base = torch.randint(2, 90, (560,), generator=torch.Generator().manual_seed(1)).tolist()
    session = eng.new_session(2, 560, 1, 1024, stop_on_end=False)
    for ask in (127, 128, 255, 256, 300, 384, 511, 512, 539, 545, 558):
        for dist in (window - 1, window):
            if not 0 < dist <= ask:
                continue
            toks = list(base)
            toks[ask - dist], toks[ask] = 0, 1
            blind = list(toks)
            blind[ask - dist] = 2
            seen, hidden = oracle_logits(cfg, w, toks)[ask:ask + 1], oracle_logits(cfg, w, blind)[ask:ask + 1]
            if dist < window:
                assert rel_error(seen, hidden) > 10 * TOL[fmt]      # the key matters
            else:
                assert rel_error(seen, hidden) < 1e-9
            got = run_portions(eng, toks, [540], session=session)   # 545 and 558 are decoded
            assert rel_error(got[ask:ask + 1], seen) < 2 * TOL[fmt], (ask, dist)
            if ask in (256, 300):
                got = run_portions(eng, toks, [ask - 1, 2, 60], session=session)
                assert rel_error(got[ask:ask + 1], seen) < 2 * TOL[fmt], (ask, dist)


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_far_keys(fmt):
    """The same question over a window that sees everything: keys around slice and tile borders, far back."""
    cfg, w = strong_key_model(5000)
    eng, _ = build(cfg, fmt=fmt, w=w)
    base = torch.randint(2, 90, (420,), generator=torch.Generator().manual_seed(1)).tolist()
    session = eng.new_session(2, 420, 1, 1024, stop_on_end=False)
    for far in (0, 1, 15, 16, 31, 32, 127, 128, 129, 255, 256, 257, 383, 384):
        toks = list(base)
        toks[far] = 0
        asks = [p for p in (far + 1, far + 2, 257, 300, 384, 385, 400, 412, 419) if p > far]
        for p in asks:
            toks[p] = 1
        want = oracle_logits(cfg, w, toks)
        got = run_portions(eng, toks, [405], session=session)       # 412 and 419 are decoded
        assert rel_error(got, want) < 2 * TOL[fmt]


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_rotation_far_into_a_sequence(fmt):
    """Scores that rest on the rotated part alone, at positions where an angle off by little shows."""
    cfg = config(128, 64, [latent(2, 8, 32, 48, 40, 40, 64, base=30.0), latent(2, 8, 64, 48, 40, 40, 90, base=2.0e5)])
    w = lo.random_weights(cfg, 5)
    for n in range(2):
        w[f"l{n}.mix.uk"] *= 0.05
        w[f"l{n}.mix.uq"] *= 2.0
        w[f"l{n}.mix.dkv"][40:] *= 2.0
    w = {k: v.to(torch.bfloat16).float() for k, v in w.items()}
    eng, _ = build(cfg, fmt=fmt, w=w)
    toks = tokens(cfg, 2600, 4)
    want = oracle_logits(cfg, w, toks)
    got = run_portions(eng, toks, [2000, 590])
    assert rel_error(got, want) < 3 * TOL[fmt]


MISTAKES = {
    "no sink": ("sink_softmax", lambda s, k: torch.softmax(s, -1)),
    "sink scaled": ("sink_softmax", lambda s, k, f=lo.sink_softmax: f(s, k * 0.5)),
    "window one short": ("window_mask", lambda p, q, k, n, f=lo.window_mask: f(p, q, k, n - 1)),
    "window one long": ("window_mask", lambda p, q, k, n, f=lo.window_mask: f(p, q, k, n + 1)),
    "position off by one": ("rotate_pairs", lambda x, p, b, d, f=lo.rotate_pairs: f(x, [i + (1 if x.dim() == 3 else 0) for i in p], b, d)),
    "halves instead of pairs": ("rotate_pairs", lambda x, p, b, d, f=lo.rotate_pairs: f(
        torch.stack([x[..., :d // 2], x[..., d // 2:d]], -1).flatten(-2), p, b, d)),
    "weights renormalised": ("route", lambda w, p, t, h, f=lo.route: (lambda c, a: (c, a / a.sum(-1, keepdim=True)))(*f(w, p, t, h))),
    "one expert fewer": ("route", lambda w, p, t, h, f=lo.route: f(w, p, t - 1, h)),
    "unclamped": ("clamped_expert", lambda w, p, n, h, f=lo.clamped_expert: f(w, p, 1e9, h)),
    "weight on the output": ("mixture", lambda w, p, m, h: sum(
        a * lo.clamped_expert(w, f"{p}.mlp.e{e}", m["expert"]["limit"], h) * (c == e)
        for c, a in zip(*[[y[:, i:i + 1] for i in range(m["router"]["top"])] for y in lo.route(w, p, m["router"]["top"], h)])
        for e in range(m["router"]["experts"])) + lo.clamped_expert(w, f"{p}.mlp.shared", m["shared"]["limit"], h)),
    "no shared expert": ("mixture", lambda w, p, m, h, f=lo.mixture: f(w, p, {**m, "shared": None}, h)),
    "gelu": ("gated_silu", lambda w, p, h: lo.linear(torch.nn.functional.gelu(lo.linear(h, w, f"{p}.gate")) * lo.linear(h, w, f"{p}.up"), w, f"{p}.down")),
    "no embedding between passes": ("layer_runs", lambda c, f=lo.layer_runs: [(n, k, False) for n, k, _ in f(c)]),
    "one pass": ("layer_runs", lambda c, f=lo.layer_runs: f({**c, "loop": None})),
    "one cache for all passes": ("layer_runs", lambda c, f=lo.layer_runs: [(n, 0, a) for n, _, a in f(c)]),
    "eps outside the root": ("rms_norm", lambda x, w, e: x / ((x * x).mean(-1, keepdim=True).sqrt() + e) * w.to(x.dtype)),
}


@pytest.mark.parametrize("mistake", list(MISTAKES))
def test_each_mechanism_shows(mistake, monkeypatch):
    """The comparison sees every mechanism: with a mistake planted in the oracle it no longer agrees."""
    cfg = config(144, 120, [latent(4, 24, 16, 40, 48, 40, 12, dense(96)),
                            latent(2, 16, 24, 24, 40, 56, 30, moe(6, 2, 40, limit=0.9, shared=56, shared_limit=0.6))], loop=(0, 2, 2), eps=0.03)
    w = lo.random_weights(cfg, 13)
    eng, _ = build(cfg, fmt="f32", w=w)
    toks = tokens(cfg, 70, 2)
    got = run_portions(eng, toks, [64])
    assert rel_error(got, oracle_logits(cfg, w, toks)) < TOL["f32"]
    monkeypatch.setattr(lo, *MISTAKES[mistake])
    assert rel_error(got, oracle_logits(cfg, w, toks)) > 100 * TOL["f32"]


@pytest.mark.parametrize("fmt", ["f32", "f16"])
@pytest.mark.parametrize("experts,top,rows", [(2, 1, 600), (5, 5, 700), (40, 32, 50), (256, 1, 300), (130, 7, 90)])
def test_expert_counts(experts, top, rows, fmt):
    """Few rows per expert and many (pairs of row tiles), experts nobody chooses, as many per token as a warp has lanes."""
    cfg = config(128, 60, [latent(2, 16, 16, 16, 32, 32, 30, moe(experts, top, 24, limit=1.5))])
    eng, w = build(cfg, 6, fmt)
    toks = tokens(cfg, rows, 4)
    check(run_portions(eng, toks, [rows - 3]), oracle_logits(cfg, w, toks), cfg, fmt)


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_loop_ranges(fmt):
    layers = [latent(2, 16, 16, 16, 32, 32, 20 + 7 * i, dense(40) if i % 2 else None) for i in range(4)]
    for loop in (None, (0, 4, 2), (3, 4, 4), (0, 1, 3), (1, 3, 1)):
        cfg = config(128, 60, layers, loop=loop)
        eng, w = build(cfg, 6, fmt)
        toks = tokens(cfg, 60, 4)
        assert rel_error(run_portions(eng, toks, [30, 25]), oracle_logits(cfg, w, toks)) < TOL[fmt]


def test_long_decoding():
    cfg = CONFIGS["no_loop"]
    for fmt in ("f32", "f16"):
        eng, w = build(cfg, 17, fmt)
        toks = tokens(cfg, 700, 4)
        check(run_portions(eng, toks, [5]), oracle_logits(cfg, w, toks), cfg, fmt)


def test_portions_and_batches_do_not_change_results_beyond_rounding():
    eng, _ = build(STRICT, 6, "f16")
    toks = tokens(STRICT, 333, 4)
    a = run_portions(eng, toks, [333])
    assert torch.equal(a, run_portions(eng, toks, [333]))                      # deterministic
    for sizes in ([100, 100, 133], [2] * 166 + [1], [332]):
        assert rel_error(run_portions(eng, toks, sizes), a) < 8e-3


def agree(got, rows, want, tol):
    """Tokens equal the oracle's up to a step whose own top-two margin is below ``tol``."""
    for i, (g, t) in enumerate(zip(got, want)):
        if g != t:
            top = np.sort(rows[i].double().numpy())[-2:]
            return top[1] - top[0] < tol
    return True


@pytest.mark.parametrize("fmt", ["f32", "f16"])
def test_greedy_generation_with_fewer_slots_than_requests(fmt):
    cfg = STRICT
    eng, w = build(cfg, 30, fmt)
    prompts = [tokens(cfg, n, 70 + n) for n in (5, 140, 1, 33, 64, 18, 90)]
    out, logits = generation.generate(eng, prompts, 24, max_batch=3, prefill_tokens=100, return_logits=True)
    for i, p in enumerate(prompts):
        want, rows = lo.greedy(cfg, w, p, 24)
        assert len(out[i]) == 24 and agree(out[i], rows, want, 1e-4 if fmt == "f32" else 5e-2)
        own = lo.Sequence(cfg, w, torch.float64).step(p + out[i])[len(p) - 1:-1]
        assert rel_error(logits[i], own) < TOL[fmt]
        assert all(int(r.argmax()) == t for r, t in zip(logits[i].cpu(), out[i]))
    if fmt == "f32":
        assert out == generation.generate(eng, prompts, 24, max_batch=64)


def test_end_token_and_sampling():
    cfg = CONFIGS["no_loop"]
    eng, _ = build(cfg, 3, "f32")
    prompts = [tokens(cfg, n, n) for n in (9, 20, 31, 12)]
    full = generation.generate(eng, prompts, 40)
    end = full[0][7]
    for got, ref in zip(generation.generate(eng, prompts, 40, end_token=end, max_batch=2), full):
        assert got == (ref[:ref.index(end) + 1] if end in ref else ref)
    a = generation.generate(eng, prompts, 10, temperature=1.2, top_k=4, seed=9, max_batch=2)
    assert a == generation.generate(eng, prompts, 10, temperature=1.2, top_k=4, seed=9)      # slots do not matter
    assert generation.generate(eng, prompts, 6, temperature=1.0, top_k=1, seed=1) == generation.generate(eng, prompts, 6)


def test_errors():
    cfg = CONFIGS["mixed"]
    eng, _ = build(cfg, 1, "f16")
    s = eng.new_session(1, 20, 1, 64, stop_on_end=False)
    slot = s.acquire()
    with pytest.raises(ValueError):
        s.step([Segment(slot, list(range(60)))])        # more positions than the slot has
    for change in (lambda c: c["layers"][1]["mlp"]["router"].update(top=8), lambda c: c["layers"][0]["mixer"].update(q_rank=0),
                   lambda c: c["loop"].update(stop=9), lambda c: c["loop"].update(times=0), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5)):
        bad = copy.deepcopy(cfg)
        change(bad)
        with pytest.raises(Exception):
            build(bad, w=lo.random_weights(cfg, 1))


def test_attention_window_of_grouped_heads():
    """The window belongs to the framework's attention layers, not to one design: grouped heads with one, in a prompt
    and while decoding, against the same attention cut by hand."""
    from mdlarc_scale_b200.layered import LayeredEngine, LayerSpec, ModelSpec
    from oracle import vodavik as vo
    from vodavik_util import attention, config as vconfig
    cfg = vconfig(128, 60, [attention(4, 2, 64, 64, ff=96)])
    w = vo.random_weights(cfg, 2)
    from mdlarc_scale_b200 import vodavik
    spec = vodavik.model_spec(cfg)
    toks = tokens(cfg, 330, 3)
    for window in (1, 50, 129):
        layer = LayerSpec(**{**spec.layers[0].__dict__, "window": window})
        spec_w = ModelSpec(**{**spec.__dict__, "layers": [layer]})
        tensors = {key: w[name] for key, name in vodavik.tensor_names(spec).items()}

        def cut(q, k, v, scale, sink, first_pos):
            rep = q.shape[1] // k.shape[1]
            s = torch.einsum("thd,shd->hts", q, k.repeat_interleave(rep, 1)) * scale
            s = s.masked_fill(~lo.window_mask(first_pos, q.shape[0], k.shape[0], window)[None], -float("inf"))
            return torch.einsum("hts,shu->thu", lo.sink_softmax(s, sink), v.repeat_interleave(rep, 1))

        with pytest.MonkeyPatch.context() as mp:
            mp.setattr(vo, "causal_sink_attention", cut)
            want = vo.Sequence(cfg, w, torch.float64).step(toks)
        for fmt in ("f32", "f16"):
            eng = LayeredEngine(spec_w, tensors, "cuda:0", fmt)
            assert rel_error(run_portions(eng, toks, [200, 100]), want) < TOL[fmt]


def test_model_folder_command_line_and_trace(tmp_path):
    cfg = CONFIGS["mixed"]
    w = lo.random_weights(cfg, 42)
    weights.write_model_folder(tmp_path / "m", cfg, {k: v.to(torch.bfloat16) for k, v in w.items()})
    prompts = [tokens(cfg, 30, 1), tokens(cfg, 7, 2)]
    (tmp_path / "p.jsonl").write_text("\n".join(json.dumps(p) for p in prompts))
    run = subprocess.run([sys.executable, "-m", "mdlarc_scale_b200.generation", "--model", str(tmp_path / "m"), "--prompts",
                          str(tmp_path / "p.jsonl"), "--max-new", "8", "--dtype", "float32"], cwd=ROOT, capture_output=True,
                         text=True, timeout=300)
    assert run.returncode == 0, run.stderr
    out = [json.loads(x) for x in run.stdout.splitlines() if x.startswith("[")]
    for p, o in zip(prompts, out):
        want, rows = lo.greedy(cfg, w, p, 8)
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
    la, lb = oracle_logits(cfg, w, a), oracle_logits(cfg, w, b)
    for n, want in ((0, la[[0, 49]]), (1, la[50:51]), (3, torch.cat([la[59:60], lb[[21, 24]]]))):
        got = torch.from_numpy(np.fromfile(tmp_path / "out" / f"{n}.f32", dtype="<f4")).view(-1, cfg["vocab"])
        assert rel_error(got, want) < TOL["f32"]
