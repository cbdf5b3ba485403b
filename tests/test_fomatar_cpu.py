"""Host side of the Fomatar design: configuration, registry, weight container, slots and the serving loop, and the plain
forward pass checked against closed forms."""
import json

import numpy as np
import pytest
import torch

from hf2q_b200 import registry, safetensors
from hf2q_b200.engine import Engine, Entry
from hf2q_b200.fomatar import FomatarConfig, Run
from hf2q_b200.ops import Hf2qError
from hf2q_b200.seqops import DenseWeight
from hf2q_b200.state import StatePool
from oracle import fomatar_forward as F
from tests import fomatar_util as U


def test_runs_follow_the_looped_span():
    cfg = FomatarConfig(U.CFG_A)
    assert [r.layer for r in cfg.runs()] == [0, 1, 2, 1, 2, 1, 2, 3]
    assert [r.begins_pass for r in cfg.runs()] == [None, 0, None, 1, None, 2, None, None]
    assert FomatarConfig(U.CFG_B).runs() == [Run(0, None), Run(1, None), Run(2, None)]
    assert [(r.layer, r.begins_pass) for r in cfg.runs()] == [(i, t if first else None) for i, t, first in F.layer_runs(U.CFG_A)]


def test_unknown_kinds_are_refused():
    for edit in (lambda c: c["layers"][0].update(type="other"), lambda c: c["layers"][1]["mlp"].update(kind="other"), lambda c: c["loop"].update(stop=9)):
        c = json.loads(json.dumps(U.CFG_A))
        edit(c)
        with pytest.raises(Hf2qError):
            FomatarConfig(c)


def test_registry_reads_the_architecture(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(U.CFG_B))
    assert registry.architecture_of(tmp_path) == "Fomatar" and "Fomatar" in registry.ARCHITECTURES
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "nothing"}))
    with pytest.raises(Hf2qError, match="not registered"):
        registry.load_model(None, tmp_path)


def test_safetensors_round_trip(tmp_path):
    t = {"a": torch.randn(3, 5).to(torch.bfloat16), "b": torch.arange(7, dtype=torch.int32), "c": torch.randn(2, 2), "e": torch.empty(0, 4)}
    safetensors.save(tmp_path / "x.safetensors", t)
    f = safetensors.SafetensorsFile(tmp_path / "x.safetensors")
    for k, v in t.items():
        got = f.load_tensor(k)
        assert got.dtype == v.dtype and torch.equal(got, v)
    with pytest.raises(ValueError, match="no tensor"):
        f.load_tensor("d")
    f.close()


def test_dense_weight_pads_with_zeros():
    a, b = torch.randn(5, 11).to(torch.bfloat16), torch.randn(3, 11).to(torch.bfloat16)
    w = DenseWeight([a, b], "cpu")
    assert (w.n, w.k, w.offsets) == (16, 16, [0, 8])
    assert torch.equal(w.w[:5, :11], a) and torch.equal(w.w[8:11, :11], b) and float(w.w.float().abs().sum()) == pytest.approx(
        float(a.float().abs().sum() + b.float().abs().sum()), rel=1e-6)
    assert DenseWeight(a, "cpu").n == 5


def test_a_reused_slot_starts_from_zero():
    p = StatePool(2, "cpu")
    p.recurrent("s", 2, 3)
    p.recurrent("t", 4)
    p.ring("k", (2, 2), torch.bfloat16)
    p.allocate()
    a, b = p.open(), p.open()
    assert {a, b} == {0, 1} and p.n_free == 0
    with pytest.raises(RuntimeError):
        p.open()
    p.views(a)["s"].fill_(3.0)
    p.views(b)["t"].fill_(5.0)
    p.pos[a], p.length[a] = 9, 9
    p.close(a)
    with pytest.raises(RuntimeError):
        p.close(a)
    assert p.open() == a
    assert float(p.views(a)["s"].abs().sum()) == 0.0 and int(p.pos[a, 0]) == 0 and p.length[a] == 0
    assert float(p.views(b)["t"].sum()) == 20.0


class _Sum:
    """Stand-in decoder: the "logits" of a place are the sequence's running sum of token ids."""
    n_slots = 2

    def __init__(self):
        self.free, self.sums, self.tok = [0, 1], {}, torch.zeros(1)

    def open_slot(self):
        s = self.free.pop(0)
        self.sums[s] = 0
        return s

    def close_slot(self, s):
        self.free.append(s)

    def bind(self, s):
        self.slot, self.tok = s, torch.tensor([self.sums[s]])

    def extend(self, s, ids, want):
        c = torch.cumsum(ids, 0) + self.sums[s]
        self.sums[s] = int(c[-1])
        return c[torch.tensor(want, dtype=torch.long)].float()[:, None]

    def generate(self, n):
        return torch.arange(n) + self.sums[self.slot] + 1


def test_engine_keeps_requests_apart_and_orders_the_rows():
    m = _Sum()
    e = Engine(m)
    assert e.step([Entry("a", [1, 2, 3], [2, 0])]).flatten().tolist() == [6, 1]
    assert e.step([Entry("b", [10], [0]), Entry("a", [4], [0])], end=["a"]).flatten().tolist() == [10, 10]
    assert e.step([Entry("c", [5], [])]) is None and len(m.free) == 0
    assert e.step([Entry("c", [5], [0])], end=["b", "c"]).flatten().tolist() == [10]
    assert Engine(_Sum()).generate([[1], [2, 3], [4]], 3) == [[1, 2, 3], [5, 6, 7], [4, 5, 6]]


# ---- the plain forward pass against closed forms ------------------------------------------------------------
def test_window_of_the_plain_attention():
    rng = np.random.default_rng(0)
    q, k, v = rng.standard_normal((9, 1, 4)), rng.standard_normal((9, 1, 4)), np.arange(9.0)[:, None, None]
    zero = np.zeros(1)
    assert np.allclose(F.window_attention(q, k, v, 1, 1.0, zero, zero), v)
    # equal scores: the mean of the window; with r1 = 1, r2 = 1 the weights are 1 / (1 + distance)
    flat = F.window_attention(0 * q, k, v, 3, 1.0, zero, zero)
    assert flat[8, 0, 0] == pytest.approx(7.0) and flat[1, 0, 0] == pytest.approx(0.5)
    far = F.window_attention(0 * q, k, v, 3, 1.0, np.ones(1), np.ones(1))
    assert far[8, 0, 0] == pytest.approx((8 + 7 / 2 + 6 / 3) / (1 + 1 / 2 + 1 / 3))


def test_plain_recurrences_on_constant_input():
    one = np.ones((6, 1, 1))
    # no forgetting, unit gates: numerator and normaliser both grow by one per token
    out = F.mlstm(one, one, 3 * one, np.zeros((6, 1)), np.zeros((6, 1)))
    assert np.allclose(out[:, 0, 0], 3.0 * np.arange(1, 7) / (np.arange(1, 7) + 1e-6))
    # weak input gates against a maximum that starts at 0: the normaliser's floor exp(-m) shows
    out = F.mlstm(one[:1], one[:1], one[:1], np.full((1, 1), -5.0), np.full((1, 1), -1.0))
    assert out[0, 0, 0] == pytest.approx(np.exp(-4.0) / (max(np.exp(-4.0), np.exp(1.0)) + 1e-6))
    # delta rule with beta = 1 stores exactly v for a unit key, whatever was there before
    v = np.arange(6.0)[:, None, None]
    assert np.allclose(F.gated_delta(one, one, v, np.ones((6, 1)), one), v)
    half = F.gated_delta(one, one, one, np.full((6, 1), 0.0), one * 0.5)
    assert np.allclose(half, 0.0)


def test_token_shift_and_bigram_of_the_first_token():
    h = np.arange(6.0).reshape(3, 2)
    assert np.allclose(F.token_shift(h, np.array([0.0, 1.0])), [[0, 0], [2, 1], [4, 3]])
    w = U.as_f64(U.weights(U.CFG_A))
    x = F.embedding(U.CFG_A, w, np.array([4, 9]))
    bg = U.CFG_A["embedding"]["bigram"]
    assert np.allclose(x[0], w["embed"][4] + w["bigram"][bg["buckets"]])
    assert np.allclose(x[1], w["embed"][9] + w["bigram"][(4 * bg["mul_prev"] + 9 * bg["mul_cur"]) % bg["buckets"]])
