"""Host side of the Runopel design: configuration, registry, weight layout, and the plain forward pass checked against
closed forms."""
import copy
import json

import numpy as np
import pytest
import torch

from hf2q_b200 import registry
from hf2q_b200.feedforward import FEED_FORWARDS, ClampedGlu, RoutedExperts
from hf2q_b200.mixers import MIXERS, LatentAttention, Mamba2
from hf2q_b200.ops import Hf2qError
from hf2q_b200.runopel import RunopelConfig
from hf2q_b200.state import StatePool
from oracle import runopel_forward as F
from tests import runopel_util as U


def test_unknown_kinds_are_refused():
    for edit in (lambda c: c["layers"][0].update(type="parallel"), lambda c: c["layers"][0]["mlp"].update(kind="other"), lambda c: c.update(streams=0)):
        c = copy.deepcopy(U.CFG_A)
        edit(c)
        with pytest.raises(Hf2qError):
            RunopelConfig(c)
    assert RunopelConfig(U.CFG_A).streams == 3


def test_registry_knows_the_design(tmp_path):
    (tmp_path / "config.json").write_text(json.dumps(U.CFG_B))
    assert registry.architecture_of(tmp_path) == "Runopel" and "Runopel" in registry.ARCHITECTURES
    assert MIXERS["mamba2"] is Mamba2 and MIXERS["latent_attention"] is LatentAttention
    assert FEED_FORWARDS == {"dense": ClampedGlu, "moe": RoutedExperts}


def getters(w, p):
    return lambda n, *s: w[p + n], lambda n, *s: w[p + n].float()


def test_gate_and_up_rows_alternate():
    w = U.weights(U.CFG_A)
    ff = ClampedGlu(None, U.CFG_A["layers"][0]["mlp"], 72, *getters(w, "l0.mlp."), "cpu", torch.float32)
    assert (ff.gate_up.n, ff.gate_up.k, ff.down.k) == (112, 72, 56)
    assert torch.equal(ff.gate_up.w[0:104:2], w["l0.mlp.gate"]) and torch.equal(ff.gate_up.w[1:104:2], w["l0.mlp.up"])
    assert not ff.gate_up.w[104:].any() and not ff.gate_up_b[104:].any() and torch.equal(ff.gate_up_b[1:104:2], w["l0.mlp.up.b"].float())
    ex = RoutedExperts(None, U.CFG_A["layers"][1]["mlp"], 72, *getters(w, "l1.mlp."), "cpu", torch.float32)
    assert (ex.gate_up.n, ex.down.n, ex.down.k) == (5 * 64, 5 * 72, 32)
    assert torch.equal(ex.gate_up.w[3 * 64 + 1:3 * 64 + 56:2], w["l1.mlp.e3.up"]) and torch.equal(ex.down.w[4 * 72:, :28], w["l1.mlp.e4.down"])


def test_latent_weights_in_both_layouts_and_the_cache():
    w, c = U.weights(U.CFG_B), U.CFG_B["layers"][1]["mixer"]
    m = LatentAttention(None, c, 1e-5, 52, *getters(w, "l1.mix."), "cpu", torch.bfloat16, 1000)
    assert torch.equal(m.uk_t.w[:, :9], w["l1.mix.uk"].T) and torch.equal(m.uv.w[:, :17], w["l1.mix.uv"])
    assert torch.equal(m.ukv.w[:9, :17], w["l1.mix.uk"]) and torch.equal(m.ukv.w[16:27, :17], w["l1.mix.uv"])
    pool = StatePool(2, "cpu")
    m.declare(pool, "r1.", 64, torch.bfloat16)
    pool.allocate()
    assert pool.views(1)["r1.latent"].shape == (5 - 1 + 64, 24 + 8)          # only the latent and the rotated part are kept
    assert LatentAttention(None, c, 1e-5, 52, *getters(w, "l1.mix."), "cpu", torch.bfloat16, 3).window == 3
    bad = copy.deepcopy(c)
    bad["rot"]["dims"] = 4
    with pytest.raises(ValueError):
        LatentAttention(None, bad, 1e-5, 52, *getters(w, "l1.mix."), "cpu", torch.bfloat16, 1000)


def test_mamba_groups_must_divide():
    w, c = U.weights(U.CFG_A), dict(U.CFG_A["layers"][1]["mixer"])
    for bad in ({"groups": 4}, {"norm_groups": 5}):
        with pytest.raises(ValueError):
            Mamba2(None, {**c, **bad}, 1e-5, 72, *getters(w, "l1.mix."), "cpu", torch.float32, 10)


# ---- the plain forward pass against closed forms ------------------------------------------------------------
def test_streams():
    X = np.arange(12.0).reshape(3, 2, 2)
    assert np.allclose(F.read_streams(X, np.array([0.0, 2.0, 0.0])), 2 * X[1])
    mix = np.array([[0, 1.0, 0], [0, 0, 1.0], [1.0, 0, 0]])                   # from -> to: a rotation of the streams
    got = F.write_streams(X, np.ones((2, 2)), mix, np.array([1.0, 0, 0]), 0.5)
    assert np.allclose(got[1], X[0]) and np.allclose(got[2], X[1]) and np.allclose(got[0], X[2] + 0.5)


def test_state_space_on_constant_input():
    one = np.ones((5, 1, 1))
    t = np.arange(1, 6)
    flat = F.state_space(one, one, one, np.ones((5, 1)), np.array([-np.inf]), np.zeros(1))        # no decay: a running sum
    assert np.allclose(flat[:, 0, 0], t)
    half = F.state_space(one, one, one, np.full((5, 1), 2.0), np.log([np.log(2.0) / 2]), np.array([3.0]))
    assert np.allclose(half[:, 0, 0], 2.0 * (2.0 - 0.5 ** (t - 1)) + 3.0)
    two = F.state_space(np.ones((1, 4, 1)), np.array([[[1.0], [5.0]]]), np.ones((1, 2, 1)), np.ones((1, 4)), np.zeros(4), np.zeros(4))
    assert np.allclose(two[0, :, 0], [1, 1, 5, 5])                            # heads of a group share its B and C


def test_short_conv_and_gate_before_norm():
    y = F.short_conv(np.array([[1.0], [2.0], [3.0]]), np.array([[10.0, 1.0]]), np.array([0.5]))
    assert np.allclose(y[:, 0], F.silu(np.array([1.5, 12.5, 23.5])))
    v = F.gated_group_norm(np.array([[3.0, 4.0, 1.0, 1.0]]), np.full((1, 4), 50.0), np.ones(4), 2, 0.0)
    assert np.allclose(v, [[3 / np.sqrt(12.5), 4 / np.sqrt(12.5), 1, 1]])


def test_rotation_and_window():
    x = np.random.default_rng(0).standard_normal((6, 1, 4))
    r = F.rotate(x, 100.0)
    assert np.allclose(r[0], x[0]) and np.allclose((r ** 2).sum(-1), (x ** 2).sum(-1))
    same = np.repeat(x[:1], 6, 0)                                             # scores depend on the distance only
    a = F.rotate(same, 100.0)[:, 0]
    assert np.allclose(a[5] @ a[3], a[2] @ a[0]) and not np.allclose(a[5] @ a[3], a[5] @ a[4])
    assert np.allclose(F.rotate(x[2:], 100.0, first=2), r[2:])
    v = np.arange(6.0)[:, None, None]
    flat = F.window_softmax(0 * x, 0 * x, v, 3, 1.0)
    assert flat[5, 0, 0] == pytest.approx(4.0) and flat[1, 0, 0] == pytest.approx(0.5)
    assert np.allclose(F.window_softmax(x, x, v, 1, 1.0), v)


def test_clamps_and_scaled_expert_inputs():
    eye, z = np.eye(1), np.zeros(1)
    f = lambda g, u: F.clamped_glu(np.ones((1, 1)), g * eye, z, u * eye, z, eye, z, 2.0)[0, 0]
    at = lambda g, u: g * F.sigmoid(1.702 * g) * (u + 1)
    assert f(9.0, 9.0) == pytest.approx(at(2.0, 2.0)) and f(-9.0, -9.0) == pytest.approx(at(-9.0, -2.0))       # the gate has no lower bound
    h, router = np.array([[2.0]]), np.array([[1.0], [3.0], [-1.0]])
    s, ids = F.route(h, router, 2)
    assert ids.tolist() == [[1, 0]] and s[0, 1] == pytest.approx(1 / (1 + np.exp(-6.0)))
    experts = [(np.array([[float(e)]]), np.array([[1.0]]), np.array([[1.0]])) for e in range(3)]
    x1, x0 = s[0, 1] * 2.0, s[0, 0] * 2.0
    assert F.expert_mixture(h, router, experts, 2)[0, 0] == pytest.approx(F.silu(x1) * x1 + F.silu(0.0) * x0)


def test_whole_forward_is_causal_and_counts_its_layers():
    w = U.as_f64(U.weights(U.CFG_A))
    ids, layers = U.tokens(U.CFG_A, 12), []
    full = F.forward(U.CFG_A, w, ids, layers)
    assert len(layers) == 4 and np.allclose(F.forward(U.CFG_A, w, ids[:7]), full[:7])
