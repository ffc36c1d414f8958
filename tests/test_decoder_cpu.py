"""Decoder stack without a GPU: the oracle's mechanisms against direct formulas, configuration reading, model folders."""
import json

import numpy as np
import pytest

from oracle import ref_decoder as R
from tests.decoder_cases import CASES


def test_window_mask_keeps_exactly_the_last_tokens():
    m = R.window_mask(3, 7, 2)  # queries at positions 4, 5, 6
    assert m.astype(int).tolist() == [[0, 0, 0, 1, 1, 0, 0], [0, 0, 0, 0, 1, 1, 0], [0, 0, 0, 0, 0, 1, 1]]
    assert R.window_mask(1, 4, 0).all()


def test_sink_takes_weight_without_a_value():
    p = R.sink_softmax(np.array([0.0, 1.0]), 2.0)
    e = np.exp([0.0, 1.0, 2.0])
    np.testing.assert_allclose(p, e[:2] / e.sum(), rtol=1e-12)
    np.testing.assert_allclose(R.sink_softmax(np.array([0.0, 1.0]), None).sum(), 1.0)


def test_distance_slopes_are_a_geometric_series():
    s = R.distance_slopes(8)
    assert s[0] == 0.5 and s[-1] == 2.0 ** -8
    np.testing.assert_allclose(R.distance_slopes(3), [2 ** (-8 / 3), 2 ** (-16 / 3), 2 ** -8])


def test_bias_is_taken_off_the_score_not_the_weight():
    q, k, v = np.zeros((1, 1, 2)), np.zeros((3, 1, 2)), np.arange(3.0).reshape(3, 1, 1)
    got = R.attend(q, k, v, 1.0, slopes=np.array([1.0]))[0, 0, 0]
    w = np.exp([-2.0, -1.0, 0.0])
    assert got == pytest.approx((w * np.arange(3)).sum() / w.sum())


def test_root_mean_square_norm_has_eps_inside_the_root():
    assert R.root_mean_square_norm(np.array([3.0, 4.0]), 0.25)[0] == pytest.approx(3.0 / np.sqrt(12.75))


def test_layer_runs_repeat_the_loop_and_mark_its_passes():
    cfg = CASES["middle_loop"]
    assert R.layer_runs(cfg) == [(0, False), (1, True), (1, True), (2, False)]
    assert R.layer_runs(CASES["odd_sizes"]) == [(0, True), (1, False)] * 3
    assert R.layer_runs(CASES["no_loop"]) == [(0, False), (1, False)]
    assert R.layer_runs(CASES["whole_loop"]) == [(0, True)]


@pytest.mark.parametrize("name", CASES)
def test_tokens_behind_a_position_do_not_change_it(name):
    cfg = CASES[name]
    w = R.random_weights(cfg, 3)
    toks = np.random.default_rng(1).integers(0, cfg["vocab"], 40)
    whole = R.forward(toks, w, cfg)
    np.testing.assert_allclose(R.forward(toks[:25], w, cfg), whole[:25], rtol=1e-9, atol=1e-9)


@pytest.mark.parametrize("name", CASES)
def test_loader_asks_for_exactly_the_tensors_of_the_configuration(name):
    from dmlx_b200.models import tafuvik

    cfg = CASES[name]
    assert sorted(n for _, _, n in tafuvik.tensor_names(cfg)) == sorted(R.tensor_shapes(cfg))
    specs = tafuvik.layer_specs(cfg)
    for spec, entry in zip(specs, cfg["layers"]):
        m = entry["mixer"]
        assert (spec["n_heads"], spec["n_kv_heads"], spec["key_dim"], spec["value_dim"]) == (m["heads"], m["kv_heads"], m["dim"], m["vdim"])
        assert spec["window"] == m["mask"]["size"] and spec["scale"] == m["scale"]
        assert spec["ffn"] == (entry["mlp"]["ff"] if entry["mlp"] else 0)


def test_unknown_designs_and_branches_are_refused(tmp_path):
    from dmlx_b200 import models
    from dmlx_b200.models import tafuvik

    with pytest.raises(models.ConfigError):
        models.architecture_of({"architecture": "Nothing"})
    assert models.architecture_of({"architectures": ["LlamaForCausalLM"]}) == "LlamaForCausalLM"
    cfg = json.loads(json.dumps(CASES["no_loop"]))
    cfg["layers"][0]["type"] = "other"
    with pytest.raises(models.ConfigError):
        tafuvik.layer_specs(cfg)
    cfg = json.loads(json.dumps(CASES["no_loop"]))
    cfg["layers"][0]["mlp"]["kind"] = "other"
    with pytest.raises(models.ConfigError):
        tafuvik.layer_specs(cfg)
    with pytest.raises(models.UnsupportedDtype):
        models.load_model(str(tmp_path), "int4")


def test_safetensors_file_reads_one_tensor_at_a_time_and_rounds_to_bf16(tmp_path):
    from dmlx_b200.safetensors_io import SafetensorsFile, write_safetensors

    path = str(tmp_path / "t.safetensors")
    a = np.array([[1.0, 1.00390625, 1.01171875]], np.float32)  # the last two lie half way between bf16 neighbours
    write_safetensors(path, {"a": ("F32", a), "b": ("BF16", np.array([0x3F80, 0xC000], np.uint16)), "i": ("I32", np.array([7], np.int32))}, {})
    f = SafetensorsFile(path)
    assert sorted(f.names()) == ["a", "b", "i"] and f.shape("a") == (1, 3) and "c" not in f
    assert f.bf16("a").tolist() == [[0x3F80, 0x3F80, 0x3F82]]
    assert f.bf16("b").tolist() == [0x3F80, 0xC000] and f["i"].tolist() == [7]
    with pytest.raises(ValueError):
        f.bf16("i")
