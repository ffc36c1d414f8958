"""Sotavik without a GPU: the oracle's mechanisms against direct formulas, configuration reading, the loader's tensor list."""
import copy

import numpy as np
import pytest

from oracle import ref_sotavik as R
from tests.sotavik_cases import CASES


def test_recurrence_decays_the_rows_of_the_key_channels():
    k = np.array([[[1.0, 2.0]], [[0.0, 0.0]]])
    v = np.array([[[3.0]], [[5.0]]])
    q = np.array([[[0.0, 0.0]], [[1.0, 10.0]]])
    o = R.gated_linear_recurrence(q, k, v, np.log(np.array([[[0.5, 0.5]], [[0.5, 0.25]]])))
    assert o[1, 0, 0] == pytest.approx(0.5 * 3.0 + 10 * 0.25 * 6.0)


def test_recurrence_includes_the_token_itself_undecayed():
    one = np.ones((1, 1, 1))
    assert R.gated_linear_recurrence(one, 2 * one, 3 * one, -50 * one)[0, 0, 0] == 6.0


def test_rotation_turns_neighbouring_pairs():
    x = np.array([[1.0, 0.0, 1.0, 0.0]])
    got = R.rotate_pairs(x, [3], 100.0)[0]
    np.testing.assert_allclose(got, [np.cos(3), np.sin(3), np.cos(0.3), np.sin(0.3)], atol=1e-12)
    q, k = np.random.default_rng(0).normal(size=(2, 1, 6))
    dot = lambda a, b: float((R.rotate_pairs(q, [a], 50.0) * R.rotate_pairs(k, [b], 50.0)).sum())
    assert dot(7, 4) == pytest.approx(dot(103, 100))


def test_latent_scores_add_both_parts_and_the_sink_has_no_value():
    q = np.ones((2, 1, 2))
    out = R.latent_attend(q, 2 * q, np.zeros((2, 1, 2)), np.array([[0.0, 0.0], [1.0, 0.0]]), np.array([[[1.0]], [[0.0]]]), 0.5, np.array([0.7]))
    e = np.exp([0.0, 1.0, 0.7])
    assert out[0, 0, 0] == pytest.approx(1 / (1 + np.exp(0.7)))
    assert out[1, 0, 0] == pytest.approx(e[0] / e.sum())


def test_log_sigmoid_far_out():
    np.testing.assert_allclose(R.log_sigmoid(np.array([-800.0, 0.0, 800.0])), [-800.0, -np.log(2), 0.0])


def test_depth_average_weighs_every_result():
    assert R.depth_average([1.0, -2.0, 0.5], [np.ones(2), np.full(2, 3.0), np.full(2, 4.0)]).tolist() == [-3.0, -3.0]


@pytest.mark.parametrize("name", CASES)
def test_tokens_behind_a_position_do_not_change_it(name):
    cfg = CASES[name]
    w = R.random_weights(cfg, 3)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 20)
    whole = R.forward(toks, w, cfg)
    np.testing.assert_allclose(R.forward(toks[:13], w, cfg), whole[:13], rtol=1e-9, atol=1e-9)


@pytest.mark.parametrize("name", CASES)
def test_loader_asks_for_exactly_the_tensors_of_the_configuration(name):
    from dmlx_b200.models import sotavik

    cfg = CASES[name]
    assert sorted(n for _, _, names in sotavik.tensor_names(cfg) for n in names) == sorted(R.tensor_shapes(cfg))
    for i, (spec, entry) in enumerate(zip(sotavik.layer_specs(cfg, lambda i: 7 + i), cfg["layers"])):
        m, mlp = entry["mixer"], entry["mlp"]
        assert (spec["n_heads"], spec["key_dim"], spec["value_dim"]) == (m["heads"], m["dim"], m["vdim"])
        if entry["type"] == "gla":
            assert spec["decay_rank"] == 7 + i and spec["decay_tau"] == m["tau"]
        else:
            assert (spec["kv_rank"], spec["rot_dim"], spec["rot_base"], spec["scale"]) == (m["kv_rank"], m["rot_dim"], m["rot"]["base"], m["scale"])
        if mlp:
            assert (spec["n_experts"], spec["top_k"], spec["expert_ffn"]) == (mlp["router"]["experts"], mlp["router"]["top"], mlp["expert"]["ff"])
            assert spec["ffn"] == mlp.get("shared", {}).get("ff", 0)
        else:
            assert "n_experts" not in spec and "ffn" not in spec


def test_unknown_branches_are_refused():
    from dmlx_b200 import models
    from dmlx_b200.models import sotavik

    assert models.architecture_of({"architecture": "Sotavik"}) == "Sotavik"
    for change in (lambda l: l.update(type="other"), lambda l: l["mlp"].update(kind="other"), lambda l: l["mixer"]["rot"].update(dims=4)):
        cfg = copy.deepcopy(CASES["latent_only"])
        change(cfg["layers"][0])
        with pytest.raises(models.ConfigError):
            sotavik.layer_specs(cfg, lambda i: 1)
