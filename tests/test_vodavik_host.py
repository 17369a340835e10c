"""Vodavik without a GPU: the oracle against itself, configuration reading, model folders, packing."""
import math

import numpy as np
import pytest
import torch

from mdlarc_scale_b200 import registry, vodavik, weights
from mdlarc_scale_b200.layered import Segment, pack_segments
from oracle import vodavik as vo

from vodavik_util import CONFIGS, oracle_logits, rel_error, tokens


@pytest.mark.parametrize("name", ["mixed", "single_head"])
def test_oracle_does_not_depend_on_portions(name):
    cfg = CONFIGS[name]
    w = vo.random_weights(cfg, 3)
    toks = tokens(cfg, 41, 1)
    whole = oracle_logits(cfg, w, toks)
    seq, rows, at = vo.Sequence(cfg, w, torch.float64), [], 0
    for n in (1, 2, 2, 7, 3, 1, 25):
        rows.append(seq.step(toks[at:at + n]))
        at += n
    assert rel_error(torch.cat(rows), whole) < 1e-12


def test_oracle_mechanisms_by_hand():
    # one key, no sink weight to speak of: the value itself; a dominant sink: nothing
    q = torch.ones(1, 2, 3)
    k, v = torch.ones(1, 1, 3), torch.tensor([[[5.0, -2.0]]])
    o = vo.causal_sink_attention(q, k, v, 1.0, torch.tensor([-60.0, 60.0]), 0)
    assert torch.allclose(o[0, 0], torch.tensor([5.0, -2.0])) and float(o[0, 1].abs().max()) < 1e-20
    # query gain steps at multiples of `every`
    g = vo.query_temperature([0, 6, 7, 13, 14], 0.5, 7)
    assert [round(float(x), 6) for x in g] == [round(1 + 0.5 * math.log(n), 6) for n in (1, 2, 2, 3, 3)]
    # the recurrence's stabiliser starts at 0: with a very low input gate the denominator is exp(-m) = 1
    one = torch.ones(1, 1, 1)
    o, (s, n, m) = vo.mlstm_recurrence(one, one, one, torch.full((1, 1), -5.0), torch.full((1, 1), -1e-3), None)
    assert float(m) == pytest.approx(-1e-3) and float(o) == pytest.approx(math.exp(-5 + 1e-3) / (math.exp(1e-3) + 1e-6))
    assert torch.allclose(vo.layer_norm(torch.tensor([[1.0, 3.0]]), torch.tensor([2.0, 3.0]), 0.0), torch.tensor([[-2.0, 3.0]]))


def test_spec_reads_every_field():
    cfg = CONFIGS["mixed"]
    spec = vodavik.model_spec(cfg)
    assert (spec.width, spec.vocab, spec.norm, spec.norm_eps) == (200, 331, "layer", 1e-5)
    assert (spec.residual_alpha, spec.logit_scale) == (1.7, 0.5)
    a, shared, rec = spec.layers[1], spec.layers[2], spec.layers[0]
    assert (a.mixer, a.heads, a.kv_heads, a.dim, a.vdim, a.kv_from, a.mlp, a.d_ff) == ("attention", 6, 2, 40, 72, -1, "relu2", 300)
    assert a.qkv_bias and a.qk_norm and a.sink and a.out_gate and (a.q_temp_coef, a.q_temp_every) == (0.4, 16)
    assert shared.kv_from == 1 and shared.mlp is None
    assert (rec.mixer, rec.heads, rec.dim, rec.vdim, rec.gate_cap, rec.mlp) == ("mlstm", 3, 40, 56, 9.0, None)
    names = vodavik.tensor_names(spec)
    assert set(names.values()) == set(vo.random_weights(cfg, 0))       # nothing missing, nothing unused


def test_bad_configurations_are_rejected():
    cfg = CONFIGS["mixed"]
    with pytest.raises(ValueError, match="unknown mixer"):
        vodavik.layer_spec({"type": "conv", "mixer": {"heads": 1, "dim": 8, "vdim": 8}, "mlp": None})
    with pytest.raises(ValueError, match="whole number"):
        e = {"type": "attention", "mlp": None, "mixer": dict(cfg["layers"][1]["mixer"], q_temp={"coef": 1, "every": 2.5})}
        vodavik.layer_spec(e)
    with pytest.raises(ValueError, match="unknown architecture"):
        registry.build_engine({"architecture": "nope"}, {})
    w = vo.random_weights(cfg, 0)
    del w["l1.mix.sink"]
    with pytest.raises(ValueError, match="lacks l1.mix.sink"):
        registry.build_engine(cfg, w)
    assert {"Vodavik", "TinyTransformer"} <= set(registry.architectures())


def test_model_folder_round_trip(tmp_path):
    t = {"a": torch.randn(3, 5).to(torch.bfloat16), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, 2, 2),
         "odd": torch.tensor([1, 2, 3], dtype=torch.uint8), "d": torch.randn(9).half(), "none": torch.empty(0, 4)}
    weights.write_model_folder(tmp_path / "m", {"architecture": "x"}, t)
    cfg, back = weights.read_model_folder(tmp_path / "m")
    assert cfg == {"architecture": "x"} and set(back) == set(t)
    for k, v in t.items():
        assert back[k].dtype == v.dtype and back[k].shape == v.shape and torch.equal(back[k], v)
    raw = (tmp_path / "m" / "model.safetensors").read_bytes()
    (tmp_path / "m" / "model.safetensors").write_bytes(raw[:-4])
    with pytest.raises(ValueError):
        weights.read_model_folder(tmp_path / "m")


def test_pack_segments():
    segs = [Segment(3, list(range(300)), [0, 299], arm=True), Segment(0, [7], [0]), Segment(5, [1, 2])]
    p = pack_segments(segs, [10, 4, 0])
    arr = p.buf.numpy()
    get = lambda n: arr[p.at[n][0]:p.at[n][0] + p.at[n][1]]  # noqa: E731
    assert (p.n_tokens, p.n_segs, p.n_want, p.n_first) == (303, 3, 3, 1)
    assert all(lo % 4 == 0 for lo, _ in p.at.values())
    assert get("pos")[[0, 299, 300, 301, 302]].tolist() == [10, 309, 4, 0, 1]
    assert np.array_equal(get("count"), get("pos") + 1)
    assert get("seq")[[0, 300, 302]].tolist() == [3, 0, 5]
    assert get("want").tolist() == [0, 299, 300]
    assert get("first_row").tolist() == [299] and get("first_seq").tolist() == [3] and get("first_len").tolist() == [310]
    assert get("seg_pos0").tolist() == [10, 4, 0] and get("seg_row0").tolist() == [0, 300, 301]
    # query blocks of at most 256 rows that cover every row once, most visible keys first
    rows = sorted((r, n) for r, n in zip(get("qb_row0").tolist(), get("qb_rows").tolist()))
    assert rows == [(0, 256), (256, 44), (300, 1), (301, 2)]
    last = [int(get("count")[r + n - 1]) for r, n in zip(get("qb_row0"), get("qb_rows"))]
    assert last == sorted(last, reverse=True)
    with pytest.raises(ValueError):
        pack_segments([Segment(0, [1], [1])], [0])
