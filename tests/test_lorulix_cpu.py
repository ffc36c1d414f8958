"""Lorulix without a GPU: the oracle's mechanisms against direct formulas, configuration reading, the loader's tensor list."""
import copy
import math

import numpy as np
import pytest

from oracle import ref_lorulix as R
from tests.lorulix_cases import CASES, buckets_of


def test_distance_buckets_are_single_near_and_logarithmic_far():
    got = [R.distance_bucket(n, 8, 64) for n in range(80)]
    assert got[:4] == [0, 1, 2, 3]  # the near half
    # 4 .. 64 is 2^4: every doubling is one bucket, the last one takes the rest
    assert got[4:8] == [4] * 4 and got[8:16] == [5] * 8 and got[16:32] == [6] * 16 and got[32:] == [7] * 48
    assert [R.distance_bucket(n, 2, 9) for n in (0, 1, 2, 50)] == [0, 1, 1, 1]
    assert [R.distance_bucket(n, 6, 50) for n in (2, 3, 7, 8, 19, 20)] == [2, 3, 3, 4, 4, 5]


def test_query_temperature_grows_in_steps():
    got = [R.query_temperature(p, 0.5, 4) for p in range(12)]
    np.testing.assert_allclose(got, [1] * 3 + [1 + 0.5 * math.log(2)] * 4 + [1 + 0.5 * math.log(3)] * 4 + [1 + 0.5 * math.log(4)])


def test_convolution_looks_back_and_starts_from_zeros():
    u = np.array([[1.0], [2.0], [4.0], [8.0]])
    np.testing.assert_allclose(R.causal_convolution(u, np.array([[100.0, 10.0, 1.0]]))[:, 0], [1, 12, 124, 248])
    np.testing.assert_allclose(R.causal_convolution(u[:2], np.array([[5.0, 1000.0, 100.0, 10.0, 1.0]]))[:, 0], [1, 12])
    np.testing.assert_allclose(R.input_convolution(u, np.array([[1.0, 0.5]]))[:, 0], [1.5, 4, 8, 16])


def test_delta_rule_writes_what_is_missing():
    k = np.array([[1.0, 0.0], [0.0, 1.0], [1.0, 0.0], [0.6, 0.8]])[:, None]
    v = np.array([[2.0], [5.0], [10.0], [0.0]])[:, None]
    one, zero = np.ones((4, 1)), np.zeros((4, 1))
    got = R.delta_rule(k, k, v, one, zero)[:, 0, 0]
    np.testing.assert_allclose(got, [2, 5, 10, 0], atol=1e-12)  # each key reads its own value back: the old one under it is gone
    got = R.delta_rule(k, k, v, 0.5 * one, zero)[:, 0, 0]
    np.testing.assert_allclose(got[:3], [1, 2.5, 5.5])
    # with decay: the state halves before it is read, S = (0.5, 0) at the second token
    got = R.delta_rule(k, np.repeat(k[:1], 4, 0), v, one, np.log(0.5) * one)[:, 0, 0]
    np.testing.assert_allclose(got, [2, 0, 10, 0], atol=1e-12)


def test_delta_rule_equals_its_triangular_system():
    rng = np.random.default_rng(0)
    t, d, e = 11, 5, 3
    q, k, v = rng.normal(size=(t, 1, d)), R.unit_vectors(rng.normal(size=(t, 1, d))), rng.normal(size=(t, 1, e))
    beta, g = rng.random((t, 1)), -rng.random((t, 1))
    L = np.cumsum(g[:, 0])
    a = np.array([[beta[i, 0] * math.exp(L[i] - L[j]) * (k[i, 0] @ k[j, 0]) if j < i else 0.0 for j in range(t)] for i in range(t)])
    u = np.linalg.solve(np.eye(t) + a, beta * v[:, 0])
    want = np.array([sum(math.exp(L[i] - L[j]) * (q[i, 0] @ k[j, 0]) * u[j] for j in range(i + 1)) for i in range(t)])
    np.testing.assert_allclose(R.delta_rule(q, k, v, beta, g)[:, 0], want, rtol=1e-9, atol=1e-12)


def test_gated_feed_forward_clamps_one_side_of_the_gate_and_both_of_the_other():
    g, u = np.array([3.0, -9.0, 1.0, 1.0]), np.array([0.0, 0.0, 5.0, -5.0])
    s = lambda z: 1 / (1 + math.exp(-1.702 * z))
    np.testing.assert_allclose(R.clamped_gate(g, u, 2.0), [2 * s(2), -9 * s(-9), 3 * s(1), -s(1)])


def test_router_keeps_the_scores_as_they_are():
    z = np.log(np.array([0.1, 0.4, 0.2, 0.3]))
    chosen, w = R.choose_experts(z, {"experts": 4, "top": 2, "scale": 2.5})
    assert chosen.tolist() == [1, 3]
    np.testing.assert_allclose(w, [1.0, 0.75])


@pytest.mark.parametrize("name", CASES)
def test_tokens_behind_a_position_do_not_change_it(name):
    cfg = CASES[name]
    w = R.random_weights(cfg, 3, buckets=buckets_of(name))
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 20)
    whole = R.forward(toks, w, cfg)
    np.testing.assert_allclose(R.forward(toks[:13], w, cfg), whole[:13], rtol=1e-9, atol=1e-9)


@pytest.mark.parametrize("name", CASES)
def test_loader_asks_for_exactly_the_tensors_of_the_configuration(name):
    from dmlx_b200.models import lorulix

    cfg = CASES[name]
    assert sorted({n for _, _, names in lorulix.tensor_names(cfg) for n in names}) == sorted(R.tensor_shapes(cfg))
    for i, (spec, entry) in enumerate(zip(lorulix.layer_specs(cfg, buckets_of(name)), cfg["layers"])):
        m, mlp = entry["mixer"], entry["mlp"]
        assert (spec["n_heads"], spec["n_kv_heads"], spec["key_dim"], spec["value_dim"]) == (m["heads"], m["kv_heads"], m["dim"], m["vdim"])
        assert spec["input_taps"] == cfg["canon"]["taps"]
        if entry["type"] == "delta":
            assert spec["conv_taps"] == m["conv"]
        else:
            assert (spec["scale"], spec["rel_reach"], spec["rel_buckets"], spec["kv_source"]) == (m["scale"], m["bias_max"], buckets_of(name)(i), m.get("kv_from", -1) + 1)
            assert (spec["q_temp_coef"], spec["q_temp_every"]) == (m["q_temp"]["coef"], m["q_temp"]["every"])
        if mlp and mlp["kind"] == "moe":
            assert (spec["n_experts"], spec["top_k"], spec["expert_ffn"], spec["router_scale"], spec["ffn"]) == (
                mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"], mlp["router"]["scale"], mlp.get("shared", {}).get("ff", 0))
        else:
            assert "n_experts" not in spec and spec.get("ffn", 0) == (mlp["ff"] if mlp else 0) and spec.get("ff_limit") == (mlp["limit"] if mlp else None)


def test_unknown_branches_are_refused():
    from dmlx_b200 import models
    from dmlx_b200.models import lorulix

    assert models.architecture_of({"architecture": "Lorulix"}) == "Lorulix"
    changes = [lambda l: l[0].update(type="other"), lambda l: l[0]["mlp"].update(kind="other"), lambda l: l[1]["mixer"].update(kv_from=1),
               lambda l: l[1]["mixer"].update(kv_from=2), lambda l: l[1]["mixer"].update(dim=16), lambda l: l[4]["mixer"].update(kv_from=1),
               lambda l: l[2]["mixer"].update(kv_heads=3), lambda l: l[2]["mixer"].update(bias_max=4)]
    for change in changes:
        cfg = copy.deepcopy(CASES["attention_only"])
        change(cfg["layers"])
        with pytest.raises(models.ConfigError):
            lorulix.layer_specs(cfg, lambda i: 8)
    cfg = copy.deepcopy(CASES["mixed_order"])
    cfg["layers"][3]["mixer"]["kv_from"] = 2  # a layer without pages
    with pytest.raises(models.ConfigError):
        lorulix.layer_specs(cfg, lambda i: 8)
