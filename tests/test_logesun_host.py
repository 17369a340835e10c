"""Logesun without a GPU: the oracle against itself and by hand, configuration reading, expansion planning."""
import copy
import math

import numpy as np
import pytest
import torch

from mdlarc_scale_b200 import logesun, registry
from mdlarc_scale_b200.layered import Segment, pack_segments
from oracle import logesun as lo

from logesun_util import BIG, CONFIGS, oracle_logits, rel_error, tokens


@pytest.mark.parametrize("name", ["mixed", "single_head"])
def test_oracle_does_not_depend_on_portions(name):
    cfg = CONFIGS[name]
    w = lo.random_weights(cfg, 3)
    toks = tokens(cfg, 71, 1)
    whole = oracle_logits(cfg, w, toks)
    seq, rows, at = lo.Sequence(cfg, w, torch.float64), [], 0
    for n in (1, 2, 2, 7, 3, 1, 55):
        rows.append(seq.step(toks[at:at + n]))
        at += n
    assert rel_error(torch.cat(rows), whole) < 1e-12


def test_oracle_mechanisms_by_hand():
    # a window of 3: each row sees itself and two before it
    m = lo.window_mask(4, 2, 6, 3)
    assert m.tolist() == [[False, False, True, True, True, False], [False, False, False, True, True, True]]
    # a sink takes part in the denominator only
    p = lo.sink_softmax(torch.zeros(1, 1, 3), torch.tensor([math.log(5.0)]))
    assert torch.allclose(p, torch.full((1, 1, 3), 1 / 8))
    # neighbouring pairs turn, the first by position x 1, the second by position x base^(-1/2); the rest stays
    x = torch.tensor([[1.0, 0.0, 0.0, 2.0, 7.0]], dtype=torch.float64)
    y = lo.rotate_pairs(x, [3], 100.0, 4)[0]
    want = [math.cos(3), math.sin(3), -2 * math.sin(0.3), 2 * math.cos(0.3), 7.0]
    assert torch.allclose(y, torch.tensor(want, dtype=torch.float64))
    # an expert: the gate is capped from above only, the linear part on both sides and shifted by one
    w = {"e.gate": torch.tensor([[1.0]]), "e.up": torch.tensor([[1.0]]), "e.down": torch.tensor([[1.0]])}
    sig = 1 / (1 + math.exp(-1.702 * 2.0))
    assert float(lo.clamped_expert(w, "e", 2.0, torch.tensor([[5.0]]))) == pytest.approx(2 * sig * 3)
    assert float(lo.clamped_expert(w, "e", 2.0, torch.tensor([[-5.0]]))) == pytest.approx(-5 / (1 + math.exp(1.702 * 5)) * -1, rel=1e-5)
    # routing: the largest sigmoids, as they are
    w = {"p.mlp.router": torch.tensor([[0.1], [2.0], [-3.0], [1.0]])}
    chosen, weight = lo.route(w, "p", 2, torch.ones(1, 1))
    assert chosen.tolist() == [[1, 3]] and torch.allclose(weight, torch.sigmoid(torch.tensor([[2.0, 1.0]])))
    assert lo.layer_runs({"layers": [0] * 4, "loop": {"start": 1, "stop": 3, "times": 2}}) == [
        (0, 0, False), (1, 0, False), (2, 0, False), (1, 1, True), (2, 1, False), (3, 0, False)]
    assert lo.layer_runs({"layers": [0] * 2}) == [(0, 0, False), (1, 0, False)]


def test_spec_reads_every_field():
    cfg = CONFIGS["mixed"]
    spec = logesun.model_spec(cfg)
    assert (spec.width, spec.vocab, spec.norm, spec.norm_eps, spec.norm_place) == (200, 331, "rms", 1e-5, "sandwich")
    assert (spec.loop, spec.n_runs, spec.residual_alpha, spec.logit_scale) == ((1, 3, 3), 7, 1.0, 1.0)
    a, b, c = spec.layers
    assert (a.mixer, a.heads, a.dim, a.rot_dim, a.rot_dims, a.vdim, a.q_rank, a.kv_rank, a.window) == ("latent", 5, 40, 24, 24, 56, 72, 48, 50)
    assert a.sink and a.scale == 64 ** -0.5 and a.rot_base == 10000.0 and (a.mlp, a.glu, a.d_ff) == ("glu", "silu", 300)
    assert (b.mlp, b.glu, b.d_ff, b.glu_limit, b.experts, b.top, b.shared_ff, b.shared_limit) == ("moe", "clamped", 40, 2.0, 7, 3, 72, 1.5)
    assert c.mlp is None and c.window == 130
    for cfg in [*CONFIGS.values(), BIG]:
        names = []
        for v in logesun.tensor_names(logesun.model_spec(cfg)).values():
            names += v if isinstance(v, list) else [v]
        assert len(names) == len(set(names)) and set(names) == set(lo.random_weights(cfg, 0))   # nothing missing, nothing unused
    plain = logesun.model_spec(CONFIGS["no_loop"])
    assert plain.loop == (0, 0, 1) and plain.n_runs == 2 and plain.layers[0].shared_ff == 0


def test_bad_configurations_are_rejected():
    cfg = CONFIGS["mixed"]
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["type"] = "conv"
    with pytest.raises(ValueError, match="unknown mixer"):
        logesun.model_spec(bad)
    bad = copy.deepcopy(cfg)
    bad["layers"][0]["mlp"]["kind"] = "other"
    with pytest.raises(ValueError, match="unknown feed-forward"):
        logesun.model_spec(bad)
    w = lo.random_weights(cfg, 0)
    del w["l1.mlp.e4.up"]
    with pytest.raises(ValueError, match="lacks l1.mlp.e4.up"):
        registry.build_engine(cfg, w)
    assert "Logesun" in registry.architectures()


def packed(segs, pos0, rows, window, pitch):
    p = pack_segments(segs, pos0, (rows, window, pitch))
    arr = p.buf.numpy()
    return p, lambda n: arr[p.at[n][0]:p.at[n][0] + p.at[n][1]]


def test_expansion_groups_cover_every_visible_key():
    rng = np.random.default_rng(0)
    for _ in range(60):
        window = int(rng.integers(1, 600))
        rows = (int(rng.integers(0, 20)) + (window + 256 + 127) // 128 + 1) * 128
        segs = [Segment(int(i), list(range(int(rng.integers(1, 1500))))) for i in rng.permutation(int(rng.integers(1, 6)))]
        p, get = packed(segs, [int(rng.integers(0, 900)) for _ in segs], rows, window, 4096)
        covered = set()
        for k in range(p.n_groups):
            (t0, t1), (q0, q1) = p.group_tile[k:k + 2], p.group_qblock[k:k + 2]
            assert 0 < (t1 - t0) * 128 <= rows
            src = get("tile_src")[t0:t1]
            for b in range(q0, q1):
                first, n = get("qb_row0")[b], get("qb_rows")[b]
                for r in (first, first + n - 1):
                    pos, seq = get("pos")[r], get("seq")[r]
                    for key in {max(0, pos - window + 1), pos}:
                        at = get("qb_kv0")[b] + key
                        assert 0 <= at < (t1 - t0) * 128 and src[at // 128] + at % 128 == seq * 4096 + key
                covered |= set(range(first, first + n))
        assert covered == set(range(p.n_tokens)) and len(get("tile_src")) == p.group_tile[-1] + 1


def test_expansion_scratch_too_small():
    with pytest.raises(ValueError, match="expansion scratch"):
        packed([Segment(0, list(range(300)))], [500], 512, 400, 1024)
