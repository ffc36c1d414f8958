"""Dovorax without a GPU: the oracle's mechanisms against direct formulas, configuration reading, the loader's tensor list."""
import copy
import math

import numpy as np
import pytest

from oracle import ref_dovorax as R
from tests.dovorax_cases import CASES


def test_yarn_keeps_fast_pairs_slows_slow_ones_and_grows_with_the_factor():
    s = {"factor": 4.0, "original": 1000, "fast": 16.0, "slow": 1.0}
    plain, one = R.yarn_frequencies(64, 10000.0, None)
    got, size = R.yarn_frequencies(64, 10000.0, s)
    assert one == 1.0 and size == pytest.approx(0.1 * math.log(4.0) + 1.0)
    turns = 1000 * plain / (2 * math.pi)  # of each pair over the original length
    np.testing.assert_allclose(got[turns > 25], plain[turns > 25])
    np.testing.assert_allclose(got[turns < 0.6], plain[turns < 0.6] / 4.0)
    between = (turns < 14) & (turns > 1.5)
    assert between.any() and (got[between] < plain[between]).all() and (got[between] > plain[between] / 4).all()


def test_yarn_with_a_ramp_of_no_width():
    got, _ = R.yarn_frequencies(8, 50.0, {"factor": 2.0, "original": 3, "fast": 64.0, "slow": 32.0})  # both ends lie below pair 0
    plain, _ = R.yarn_frequencies(8, 50.0, None)
    np.testing.assert_allclose(got[1:], plain[1:] / 2)


def test_rotation_pairs_the_halves_of_the_first_dimensions():
    x = np.array([[1.0, 2.0, 3.0, 4.0, 9.0]])
    got = R.rotate_halves(x, [2], {"dims": 4, "base": 100.0})[0]
    c0, s0, c1, s1 = np.cos(2), np.sin(2), np.cos(0.2), np.sin(0.2)
    np.testing.assert_allclose(got, [c0 - 3 * s0, 2 * c1 - 4 * s1, 3 * c0 + s0, 4 * c1 + 2 * s1, 9.0])


def test_convolution_looks_back_and_starts_from_zeros():
    u = np.array([[1.0], [2.0], [4.0], [8.0]])
    w = np.array([[100.0, 10.0, 1.0]])
    np.testing.assert_allclose(R.causal_convolution(u, w, 0.5)[:, 0], [1.5, 12.5, 124.5, 248.5])


def test_one_more_in_the_denominator_also_far_out():
    s = np.array([[0.0, math.log(2.0)], [-900.0, -900.0], [900.0, -np.inf]])
    np.testing.assert_allclose(R.softmax(s, True), [[0.25, 0.5], [0.0, 0.0], [1.0, 0.0]], atol=1e-12)


def test_matrix_memory_equals_its_unstabilised_sum():
    rng = np.random.default_rng(0)
    t, h, d, e = 9, 2, 4, 3
    q, k, v = rng.normal(size=(t, h, d)), rng.normal(size=(t, h, d)), rng.normal(size=(t, h, e))
    li, lf = rng.normal(size=(t, h)) * 2, -rng.random((t, h))
    got = R.matrix_memory(q, k, v, li, lf)
    m = np.zeros(h)
    for i in range(t):
        m = np.maximum(lf[i] + m, li[i])
        for head in range(h):
            w = np.array([math.exp(li[j, head] + lf[j + 1:i + 1, head].sum()) * (k[j, head] @ q[i, head]) for j in range(i + 1)])
            den = max(abs(w.sum()), 1.0) / math.exp(m[head])  # e^-m is one before the scaling
            np.testing.assert_allclose(got[i, head], (w @ v[:i + 1, head]) / math.exp(m[head]) / (den + 1e-6), rtol=1e-9)


def test_running_maximum_starts_at_zero():
    one = np.ones((1, 1, 1))
    got = R.matrix_memory(one, one, one, np.array([[-3.0]]), np.array([[-0.5]]))[0, 0, 0]
    w = math.exp(-3.0)  # m = max(-0.5, -3): the denominator is e^0.5 at the scale of e^-m
    assert got == pytest.approx(w * math.exp(0.5) / (math.exp(0.5) + 1e-6))


def test_linear_recurrence_keeps_its_energy():
    la = np.log(np.array([[0.5], [0.8], [0.25]]))
    got = R.gated_linear_unit_recurrence(np.array([[2.0], [1.0], [4.0]]), la, np.array([[1.0], [0.5], [0.25]]))[:, 0]
    a = 2.0 * math.sqrt(0.75)
    b = 0.8 * a + 0.6 * 0.5
    np.testing.assert_allclose(got, [a, b, 0.25 * b + math.sqrt(1 - 0.0625)])


def test_router_takes_the_best_groups_first():
    z = np.log(np.array([0.30, 0.01, 0.20, 0.19, 0.22, 0.08]))
    router = {"experts": 6, "top": 2, "groups": {"count": 3, "keep": 1}}
    chosen, w = R.choose_experts(z, router)
    assert chosen.tolist() == [0, 1]  # group 0 holds the largest score
    np.testing.assert_allclose(w, [0.30 / 0.31, 0.01 / 0.31])
    router["groups"]["keep"] = 2
    assert R.choose_experts(z, router)[0].tolist() == [0, 4]
    assert R.choose_experts(z, {"experts": 6, "top": 3})[0].tolist() == [0, 4, 2]


def test_activations_at_known_points():
    np.testing.assert_allclose(R.gelu(np.array([0.0, 1.0, -1.0])), [0.0, 0.8413447460685429, -0.15865525393145707])
    np.testing.assert_allclose(R.gelu_tanh(np.array([0.0, 1.0, -1.0])), [0.0, 0.8411919906082768, -0.15880800939172324])


@pytest.mark.parametrize("name", CASES)
def test_tokens_behind_a_position_do_not_change_it(name):
    cfg = CASES[name]
    w = R.random_weights(cfg, 3)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 20)
    whole = R.forward(toks, w, cfg)
    np.testing.assert_allclose(R.forward(toks[:13], w, cfg), whole[:13], rtol=1e-9, atol=1e-9)


@pytest.mark.parametrize("name", CASES)
def test_loader_asks_for_exactly_the_tensors_of_the_configuration(name):
    from dmlx_b200.models import dovorax

    cfg = CASES[name]
    assert sorted({n for _, _, names in dovorax.tensor_names(cfg) for n in names}) == sorted(R.tensor_shapes(cfg))
    for i, (spec, entry) in enumerate(zip(dovorax.layer_specs(cfg), cfg["layers"])):
        m, mlp = entry["mixer"], entry["mlp"]
        if entry["type"] == "latent_attention":
            assert (spec["n_heads"], spec["key_dim"], spec["value_dim"], spec["kv_rank"], spec["q_rank"], spec["rot_dim"]) == (
                m["heads"], m["dim"], m["vdim"], m["kv_rank"], m["q_rank"], m["rot_dim"])
            assert spec["window"] == m["mask"]["size"] and spec["scale"] == m["scale"] and spec["kv_source"] == m.get("kv_from", -1) + 1
            assert spec.get("yarn_factor", 0.0) == m["rot"].get("scaling", {}).get("factor", 0.0)
        elif entry["type"] == "parallel":
            a, r = m["left"], m["right"]
            assert (spec["n_heads"], spec["n_kv_heads"], spec["key_dim"], spec["value_dim"], spec["conv_taps"], spec["rot_dim"]) == (
                a["heads"], a["kv_heads"], a["dim"], a["vdim"], a["conv"], a["rot"]["dims"])
            assert (spec["mem_heads"], spec["mem_key_dim"], spec["mem_value_dim"], spec["mem_gate_cap"]) == (r["heads"], r["dim"], r["vdim"], r["gate_cap"])
            assert (spec["mix_scale"], spec["mem_scale"]) == (m["left_scale"], m["right_scale"])
        else:
            assert (spec["n_heads"] * spec["value_dim"], spec["n_heads"], spec["conv_taps"]) == (m["width"], m["blocks"], m["conv"])
        if mlp and mlp["kind"] == "moe":
            groups = mlp["router"].get("groups", {"count": 1, "keep": 1})
            assert (spec["n_experts"], spec["top_k"], spec["expert_ffn"], spec["n_groups"], spec["keep_groups"], spec["ffn"]) == (
                mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"], groups["count"], groups["keep"], mlp.get("shared", {}).get("ff", 0))
        else:
            assert "n_experts" not in spec and spec.get("ffn", 0) == (mlp["ff"] if mlp else 0)


def test_unknown_branches_are_refused():
    from dmlx_b200 import models
    from dmlx_b200.models import dovorax

    assert models.architecture_of({"architecture": "Dovorax"}) == "Dovorax"
    changes = [lambda l: l[0].update(type="other"), lambda l: l[0]["mlp"].update(kind="other"), lambda l: l[0]["mixer"]["rot"].update(dims=4),
               lambda l: l[1]["mixer"].update(kv_from=1), lambda l: l[1]["mixer"].update(kv_from=2), lambda l: l[1]["mixer"].update(kv_rank=64),
               lambda l: l[2]["mixer"].update(kv_from=1, kv_rank=72, rot_dim=16)]
    for change in changes:
        cfg = copy.deepcopy(CASES["latent_only"])
        change(cfg["layers"])
        with pytest.raises(models.ConfigError):
            dovorax.layer_specs(cfg)
