"""Dovorax as a served model, against the oracle: each mechanism, the whole stack, and what must not depend on how tokens reach it
(portions, batches, pages and state slots used again, graphs)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import ref_dovorax as R
from oracle.ref_math import bf16_round
from tests.dovorax_cases import CASES, config, dense, experts, latent, parallel, rglru, rotation
from tests.test_gpu_sotavik import LatentCase

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 3e-5  # relative to the root mean square of what is compared
DTYPES = ["float32", "bfloat16"]


def _bf16(a):
    return bf16_round(np.asarray(a, np.float32)).astype(np.float64)


def _load(tmp_path, cfg, seed, dtype, max_rows=512, slots=4, change=None, decisive=True):
    from dmlx_b200.models import Limits, load_model

    w = R.random_weights(cfg, seed, decisive)
    if change:
        change(w)
        w = {n: _bf16(a) for n, a in w.items()}
    R.write_model(str(tmp_path), cfg, w)
    return load_model(str(tmp_path), dtype, Limits(max_rows, slots, slots)), w


def _error(got, want):
    return np.sqrt(((got - want) ** 2).mean(-1).max() / (want ** 2).mean())


def _close(got, want, tol):
    """Within tol at all positions but one in fifty (or one), and nowhere further off than twenty times.  Where a matrix memory's output is
    next to nothing, the norm behind it makes rounding of its sign: such positions are rare, and as far off in the oracle when it rounds."""
    e = np.sqrt(((got - want) ** 2).mean(-1) / (want ** 2).mean())
    return bool(np.isfinite(got).all() and (e > tol).sum() <= max(1, len(e) // 50) and e.max() <= 20 * tol)


def _tol(dtype, w, cfg, tokens):
    """What rounding alone may cause: in bfloat16 three times the error the oracle makes on these tokens when it rounds every
    matrix operand and result to bf16."""
    if dtype == "float32":
        return F32_TOL
    return 3 * _error(R.forward(tokens, w, cfg, _bf16), R.forward(tokens, w, cfg))


def _tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


def _step(loaded, toks, portions=None, pages=None):
    """Logits of every token, in portions of the given sizes (the last one repeats)."""
    from dmlx_b200.serving import TokenFeeder

    feeder = TokenFeeder(loaded, pages or (len(toks) + 31) // 32)
    portions, out, at = list(portions or [len(toks)]), [], 0
    while at < len(toks):
        n = portions.pop(0) if len(portions) > 1 else portions[0]
        part = toks[at:at + n]
        out.append(feeder.step([("r", part, range(len(part)))]))
        at += len(part)
    return np.concatenate(out)


# ---- the stack -----------------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CASES)
def test_whole_prompt_layer_by_layer_and_logits(tmp_path, name, dtype):
    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 11, dtype)
    toks = _tokens(cfg, 150, 5)
    want, trail = R.forward(toks, w, cfg, want_layers=True)
    loaded.model.record_layers(True)
    got = _step(loaded, toks)
    layers = loaded.model.recorded_layers(len(toks))
    rounded = R.forward(toks, w, cfg, _bf16, want_layers=True)[1]
    for i in range(len(trail)):
        tol = F32_TOL if dtype == "float32" else 3 * _error(rounded[i], trail[i])
        assert _close(layers[i], trail[i], tol), (name, "layer", i)
    assert _close(got, want, _tol(dtype, w, cfg, toks)), name


@pytest.mark.parametrize("name", ["recurrent_only", "latent_only", "parallel_only", "odd_sizes"])
def test_router_over_the_whole_width(tmp_path, name):
    """Router weights without structure: every coordinate of the residual takes part in the choice."""
    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 12, "float32", decisive=False)
    toks = _tokens(cfg, 60, 5)
    assert _close(_step(loaded, toks), R.forward(toks, w, cfg), F32_TOL)


MECHANISMS = ["rotation", "yarn", "yarn_size", "latent_norm", "query_norm", "window", "short_conv", "qk_norm", "sink", "gate_cap", "gate_bias",
              "head_norm", "out_gate", "left", "right", "input_gate", "decay_gate", "out_branch", "groups", "renormalise", "shared",
              "unit_offset", "alpha"]


def test_every_mechanism_shows(tmp_path):
    """The model equals the oracle, and not the oracle without one of the mechanisms."""
    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 21, "float32", decisive=False)
    toks = _tokens(cfg, 70, 9)
    got = _step(loaded, toks)
    assert _error(got, R.forward(toks, w, cfg)) <= F32_TOL
    for mechanism in MECHANISMS:
        assert _error(got, R.forward(toks, w, cfg, without={mechanism})) > 100 * F32_TOL, mechanism


def test_normaliser_of_the_matrix_memory(tmp_path):
    """The output's own norm hides the denominator unless its eps is of the output's size."""
    cfg = config(64, 90, [parallel(2, 1, 16, 16, 3, rotation(8), (3, 24, 20), scales=(0.5, 1.5))], eps=0.2)
    loaded, w = _load(tmp_path, cfg, 22, "float32")
    toks = _tokens(cfg, 70, 9)
    got = _step(loaded, toks)
    assert _error(got, R.forward(toks, w, cfg)) <= F32_TOL
    assert _error(got, R.forward(toks, w, cfg, without={"normaliser"})) > 100 * F32_TOL
    loaded, w = _load(tmp_path / "b", cfg, 22, "bfloat16")
    assert _close(_step(loaded, toks), R.forward(toks, w, cfg), _tol("bfloat16", w, cfg, toks))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CASES)
def test_portions_decoding_batches_and_reused_pages_and_slots(tmp_path, name, dtype):
    """Requests cut into portions of every size down to single tokens, in batches with others, on pages and state slots that
    earlier requests gave back: every logit equals the whole prompt's."""
    from dmlx_b200.serving import TokenFeeder

    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 31, dtype)
    rng = np.random.default_rng(17)
    prompts = {i: _tokens(cfg, n, 100 + i) for i, n in enumerate((131, 97, 64, 3, 33, 1, 120, 66))}
    want = {i: R.forward(p, w, cfg) for i, p in prompts.items()}
    feeder = TokenFeeder(loaded, 14)
    waiting, live, got = list(prompts), [], {i: [] for i in prompts}
    while waiting or live:
        budget = lambda: sum((len(prompts[i]) + 31) // 32 for i in live)
        while waiting and len(live) < 4 and budget() + (len(prompts[waiting[0]]) + 31) // 32 <= 14:
            live.append(waiting.pop(0))
        entries = []
        for i in live:
            at = feeder.length(i)
            if rng.random() < 0.2:
                continue  # left out of this step
            n = min(int(rng.choice([1, 1, 1, 2, 2, 3, 4, 5, 7, 16, 31, 33, 64])), len(prompts[i]) - at)
            entries.append((i, prompts[i][at:at + n], range(n)))
        logits = feeder.step(entries)
        o = 0
        for i, part, _ in entries:
            got[i].append(logits[o:o + len(part)])
            o += len(part)
            if feeder.length(i) == len(prompts[i]):
                feeder.end(i)
                live.remove(i)
    assert feeder.free_pages() == 14
    tol = max(_tol(dtype, w, cfg, prompts[i]) for i in (0, 1, 6))
    for i in prompts:
        assert _close(np.concatenate(got[i]), want[i], max(tol, _tol(dtype, w, cfg, prompts[i]))), (name, i)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [2, 3, 4, 5, 32, 50])
def test_portions_of_one_size_against_token_by_token(tmp_path, portion, dtype):
    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 41, dtype)
    toks = _tokens(cfg, 110, 6)
    cut, single = _step(loaded, toks, [portion]), _step(loaded, toks, [1])
    tol = _tol(dtype, w, cfg, toks)
    assert _close(cut, single, tol)
    assert _close(single, R.forward(toks, w, cfg), tol)


def test_long_decoding_with_graphs(tmp_path):
    """400 decoded tokens through replayed graphs, windows passing over decoded tokens: a state that drifted or a page that was
    missed would show at the end."""
    import torch

    from dmlx_b200.serving import TokenFeeder

    cfg = config(80, 120, [rglru(72, 3, 4, experts(4, 2, 24, (2, 1), 16)), latent(4, 16, 8, 24, 56, 32, 50, experts(3, 2, 16)),
                           parallel(4, 2, 24, 16, 4, rotation(8), (2, 24, 40)), latent(2, 24, 8, 16, 56, 24, 129, dense(40), kv_from=1)])
    for dtype in DTYPES:
        loaded, w = _load(tmp_path / dtype, cfg, 51, dtype, change=lambda w: (w["l2.mix.right.f.b"].__iadd__(3.0), w["l0.mix.lam"].__isub__(3.0)))
        toks = _tokens(cfg, 420, 7)
        want = R.forward(toks, w, cfg)
        feeder = TokenFeeder(loaded, 14)
        with torch.cuda.stream(torch.cuda.Stream()):
            feeder.step([("a", toks[:20], [])])
            got = np.concatenate([feeder.step([("a", [t], [0])]) for t in toks[20:]])
        assert _close(got, want[20:], _tol(dtype, w, cfg, toks))


def test_replayed_graphs_equal_eager_steps(tmp_path):
    import torch

    from dmlx_b200.serving import TokenFeeder

    cfg = CASES["mixed_order"]
    loaded, _ = _load(tmp_path, cfg, 61, "bfloat16")
    toks = {i: _tokens(cfg, 80, 70 + i) for i in range(3)}
    runs = []
    for graphs in (False, True):
        loaded.model.enable_graphs(graphs)
        feeder = TokenFeeder(loaded, 12)
        with torch.cuda.stream(torch.cuda.Stream()):
            feeder.step([(i, t[:30 + 9 * i], []) for i, t in toks.items()])
            runs.append([feeder.step([(i, [t[30 + 9 * i + s]], [0]) for i, t in toks.items()]) for s in range(25)])
    for a, b in zip(*runs):
        np.testing.assert_array_equal(a, b)


@pytest.mark.parametrize("name", ["mixed_order", "wide"])
def test_tensor_core_and_cuda_core_paths_agree_in_the_stack(tmp_path, name):
    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 71, "bfloat16")
    toks = _tokens(cfg, 140, 3)
    out = []
    for mma in (True, False):
        loaded.model.set_attn_mma(mma)
        out.append(_step(loaded, toks, [100, 1]))
    assert _close(out[0], out[1], _tol("bfloat16", w, cfg, toks))


# ---- mechanisms with inputs that make them stand out -------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 4, 7])
def test_convolutions_whose_oldest_tap_is_the_heaviest(tmp_path, taps, dtype):
    """Portions around the number of taps: the inputs before a portion come out of the state."""
    cfg = config(64, 90, [rglru(48, 2, taps), parallel(4, 2, 16, 24, taps, rotation(8), (2, 12, 16))], alpha=0.5)

    def heavy(w):
        for n in w:
            if n.endswith(".conv"):
                w[n][:, 0] += 2.0

    loaded, w = _load(tmp_path, cfg, 13, dtype, change=heavy)
    toks = _tokens(cfg, 40, 2)
    want, tol = R.forward(toks, w, cfg), _tol(dtype, w, cfg, toks)
    for portions in ([40], [1], [2], [3], [5], [1, 2, 1, 3, 1, 6, 7, 1], [39, 1], [taps + 1]):
        assert _close(_step(loaded, toks, portions), want, tol), portions


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_large_step_of_unequal_portions(tmp_path, dtype):
    """More than a thousand rows in one step, portions that start and end anywhere among them, and a second step behind it."""
    from dmlx_b200.serving import TokenFeeder

    cfg = config(64, 90, [parallel(4, 2, 24, 40, 4, rotation(12), (2, 20, 24)), rglru(48, 2, 4),
                          parallel(2, 1, 136, 144, 4, rotation(136), (1, 16, 16), dense(24))], alpha=1.0)
    loaded, w = _load(tmp_path, cfg, 23, dtype, max_rows=1400, slots=8)
    lens = (610, 1, 2, 3, 37, 500, 4)
    prompts = {i: _tokens(cfg, n + 9, 500 + i) for i, n in enumerate(lens)}
    feeder = TokenFeeder(loaded, 60)
    first = feeder.step([(i, p[:-9], range(len(p) - 9)) for i, p in prompts.items()])
    second = feeder.step([(i, p[-9:], range(9)) for i, p in prompts.items()])
    at = 0
    for i, n in enumerate(lens):
        want = R.forward(prompts[i], w, cfg)
        got = np.concatenate([first[at:at + n], second[9 * i:9 * i + 9]])
        assert _close(got, want, _tol(dtype, w, cfg, prompts[i])), n
        at += n


def _special_token(cfg, w, token, coordinate=0, size=6.0):
    """One token id lights up a coordinate that is dark for all others and that no sublayer writes."""
    w["embed"][:, coordinate] = 0.0
    w["embed"][token, coordinate] = size
    for n in w:
        if n.endswith(".o") or n.endswith(".down"):
            w[n][coordinate] = 0.0


@pytest.mark.parametrize("dtype", DTYPES)
def test_matrix_memory_keeps_one_token_among_hundreds(tmp_path, dtype):
    cfg = config(64, 90, [parallel(2, 1, 16, 16, 2, rotation(8), (2, 32, 40), scales=(0.02, 2.0))], alpha=0.7)

    def plant(w):
        _special_token(cfg, w, 7)
        p = "l0.mix.right."
        w[p + "i"][:] = 0.0
        w[p + "i"][:, 0] = 3.0   # the special token's input gate opens, the others' are shut
        w[p + "i.b"][:] = -6.0
        w[p + "f"][:] = 0.0
        w[p + "f.b"][:] = 11.0  # nothing is forgotten

    loaded, w = _load(tmp_path, cfg, 14, dtype, change=plant)
    toks = [t if t != 7 else 8 for t in _tokens(cfg, 330, 2)]
    toks[5] = 7
    want, tol = R.forward(toks, w, cfg), _tol(dtype, w, cfg, toks)
    other = R.forward(toks[:5] + [8] + toks[6:], w, cfg)
    assert _error(want[300:], other[300:]) > 20 * tol
    for portions in ([330], [300, 1], [31, 1, 33, 64, 2], [4, 1, 7]):
        assert _close(_step(loaded, toks, portions), want, tol), portions


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("forget", [-30.0, 0.0, 5.0])
def test_matrix_memory_of_violent_gates(tmp_path, forget, dtype):
    """Input gates that jump by thirty from token to token, with decays that leave nothing and with weak ones: exponents far beyond
    what unstabilised sums hold."""
    cfg = config(64, 90, [parallel(2, 1, 16, 16, 2, rotation(8), (3, 24, 20), scales=(0.1, 1.5), cap=30.0)], alpha=0.7)

    def plant(w):
        w["l0.mix.right.i"][:] *= 12.0
        w["l0.mix.right.f.b"][:] = forget

    loaded, w = _load(tmp_path, cfg, 15, dtype, change=plant)
    toks = _tokens(cfg, 150, 2)
    want, tol = R.forward(toks, w, cfg), _tol(dtype, w, cfg, toks)
    for portions in ([150], [1], [70, 3, 40, 1, 1]):
        got = _step(loaded, toks, portions)
        assert _close(got, want, max(tol, 1e-4)), portions


@pytest.mark.parametrize("dtype", DTYPES)
def test_linear_recurrence_keeps_the_first_tokens(tmp_path, dtype):
    cfg = config(64, 90, [rglru(96, 3, 3)], alpha=0.3)

    def plant(w):
        _special_token(cfg, w, 7)
        w["l0.mix.lam"][:] = -12.0   # next to no decay
        w["l0.mix.lam"][::5] = 4.0   # beside channels that forget at once
        w["l0.mix.x"][:, 0] = 40.0

    loaded, w = _load(tmp_path, cfg, 16, dtype, change=plant)
    toks = [t if t != 7 else 8 for t in _tokens(cfg, 330, 2)]
    toks[0] = 7
    want, tol = R.forward(toks, w, cfg), _tol(dtype, w, cfg, toks)
    assert _error(want[300:], R.forward([8] + toks[1:], w, cfg)[300:]) > 5 * tol
    for portions in ([330], [300, 1], [31, 1, 33, 64, 2], [1, 100]):
        assert _close(_step(loaded, toks, portions), want, tol), portions


@pytest.mark.parametrize("dtype", DTYPES)
def test_sharp_scores_find_single_keys(tmp_path, dtype):
    """Scores so sharp that most queries read one key, near or hundreds of tokens away, over pages and windows' edges."""
    cfg = config(96, 120, [latent(4, 24, 8, 24, 48, 32, 70, scale=1.2, scaling=(2.0, 100, 16.0, 1.0)),
                           parallel(4, 2, 32, 24, 2, rotation(16, scaling=(3.0, 90, 16.0, 1.0)), (2, 16, 16), scales=(1.5, 0.2), scale=1.0)])
    loaded, w = _load(tmp_path, cfg, 17, dtype)
    toks = _tokens(cfg, 360, 4)
    want, tol = R.forward(toks, w, cfg), _tol(dtype, w, cfg, toks)
    for portions in ([360], [280, 1], [64, 33, 2, 100]):
        assert _close(_step(loaded, toks, portions), want, tol), portions


def test_positions_far_out(tmp_path):
    """Rotations thousands of tokens from the start, in f32."""
    cfg = config(48, 64, [latent(2, 16, 16, 16, 24, 24, 40, scale=0.5, scaling=(4.0, 256, 32.0, 1.0)), rglru(32, 2, 2)])
    loaded, w = _load(tmp_path, cfg, 18, "float32", max_rows=2600)
    toks = _tokens(cfg, 2560, 4)
    want = R.forward(toks, w, cfg)
    got = _step(loaded, toks, [2550, 1])
    assert _error(got[2000:], want[2000:]) <= F32_TOL


class WindowCase(LatentCase):
    def run(self, rows, q, scale, window, mma=True):
        t = self.torch
        kd = self.kv.page_shapes(0)[0][2]
        qd = t.zeros((len(rows), self.heads, kd), dtype=self.type, device="cuda")
        qd[:, :, :q.shape[2]] = t.tensor(q, dtype=self.type)
        i32 = lambda a: t.tensor(np.asarray(a), dtype=t.int32, device="cuda")
        out = self.kv.window_attention(0, qd, i32([s for s, _ in rows]), i32([p + 1 for _, p in rows]), scale, window=window, mma=mma)
        return out.float().cpu().numpy()

    def want(self, rows, q, scale, window):
        out = np.zeros((len(rows), self.heads, self.rank))
        for r, (s, p) in enumerate(rows):
            keys = self.keys[s][max(0, p + 1 - window) if window else 0:p + 1]
            out[r] = R.softmax(q[r] @ keys.T * scale, False) @ keys[:, :self.rank]
        return out


@pytest.mark.parametrize("mma", [True, False])
@pytest.mark.parametrize("heads,window", [(4, 1), (4, 31), (16, 32), (3, 33), (20, 64), (4, 65), (33, 100), (2, 250)])
def test_a_key_just_inside_and_just_outside_the_latent_window(heads, window, mma):
    """One key stands out; queries one after the other (a prompt) and single ones, the last that sees it and the first that does not."""
    rank, rot, n = 48, 16, 400
    for at in (0, 31, 32, 95, 140):
        case = WindowCase([n], heads, rank, rot, seed=at)
        case.keys[0] *= 0.05
        case.keys[0][at] = 0
        case.keys[0][at, rank:] = 4.0
        case.keys[0][at, :8] = 3.0
        case.keys[0] = _bf16(case.keys[0])
        case.write()
        last = at + window - 1
        for places in (range(max(last - 5, 0), last + 7), [last], [last + 1], [at], [n - 1]):
            rows = [(0, p) for p in places]
            q = np.zeros((len(rows), heads, rank + rot))
            q[:, :, rank:] = 1.0
            got = case.run(rows, _bf16(q), 1.0, window, mma)[:, :, :8]
            for (_, p), o in zip(rows, got):
                if at <= p <= last:
                    assert np.abs(o - 3.0).max() < 0.1, (at, p)
                else:
                    assert np.abs(o).max() < 1.0, (at, p)


@pytest.mark.parametrize("mma", [True, False])
@pytest.mark.parametrize("heads,rank,rot,window", [(6, 96, 32, 45), (16, 64, 16, 128), (20, 208, 48, 300), (33, 288, 64, 64), (128, 512, 64, 1000)])
def test_latent_windows_over_unequal_contexts(heads, rank, rot, window, mma):
    from dmlx_b200 import device as dev

    case = WindowCase([1500, 70, 1, 33, 900], heads, rank, rot)
    case.write()
    rng = np.random.default_rng(4)
    rows = [(0, p) for p in range(200, 213)] + [(1, 69), (2, 0)] + [(3, p) for p in range(33)] + [(4, 899), (0, 1499)]
    q = _bf16(rng.normal(size=(len(rows), heads, rank + rot)))
    scale = 2.0 * (rank + rot) ** -0.5
    want = case.want(rows, q, scale, window)
    try:
        for pages in (0, 1, 3):
            dev.set_attn_pages_per_chunk(pages)
            assert _error(case.run(rows, q, scale, window, mma), want) <= 4 * _error(_bf16(want), want), pages
    finally:
        dev.set_attn_pages_per_chunk(0)


@pytest.mark.parametrize("experts_, top, groups", [(40, 5, (8, 3)), (130, 16, (2, 1)), (64, 1, (64, 2)), (300, 7, None), (48, 32, None)])
def test_router_of_many_experts(tmp_path, experts_, top, groups):
    cfg = config(64, 90, [rglru(32, 1, 2, experts(experts_, top, 8, groups, 8))])
    loaded, w = _load(tmp_path, cfg, 19, "float32", decisive=False)
    toks = _tokens(cfg, 33, 4)
    assert _close(_step(loaded, toks, [20, 1]), R.forward(toks, w, cfg), F32_TOL)


# ---- state, engine, programs ---------------------------------------------------------------------------------------------------
def test_state_through_fork_extend_rollback_and_release(tmp_path):
    from dmlx_b200 import _lib

    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 93, "float32", slots=4)
    toks = _tokens(cfg, 60, 3)
    want = R.forward(toks, w, cfg)
    kv, other = loaded.new_cache(12, 4), loaded.new_cache(8, 4)
    m = loaded.model

    def go(pool, slot, a, b):
        m.step(pool, [(slot, b - a, a, 0)], toks[a:b])
        return m.logits(0, 1)[0]

    go(kv, 0, 0, 40)
    kv.fork(0, 1, 40)
    with pytest.raises(_lib.B200Error):
        kv.fork(0, 2, 32)
    with pytest.raises(_lib.B200Error):
        kv.rollback(0, 30)
    other.extend(2, kv, 0)
    for pool, slot in ((kv, 0), (kv, 1), (other, 2)):
        assert _error(go(pool, slot, 40, 60), want[59]) <= F32_TOL
    kv.release([0])
    assert _error(go(kv, 0, 0, 60), want[59]) <= F32_TOL


def _greedy(w, cfg, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(R.forward(toks, w, cfg)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["recurrent_only", "latent_only", "parallel_only", "odd_sizes", "mixed_order"])
def test_greedy_generation_through_the_engine(tmp_path, name):
    """More prompts than slots, chunked prefill beside decoding: the tokens are those of each prompt alone."""
    from dmlx_b200.serving import generate

    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 81, "float32", max_rows=96)
    prompts = [_tokens(cfg, n, 200 + n) for n in (40, 1, 55, 9, 33, 64)]
    got = generate(loaded, prompts, 8, prefill_chunk=23)
    for p, g in zip(prompts, got):
        assert g == _greedy(w, cfg, p, 8)


def test_generation_under_page_pressure_and_with_prefix_sharing_asked_for(tmp_path):
    """A pool too small for all requests (deferral, preemption by recomputation: the state starts over), and prefix sharing, which
    a recurrent state does not allow: same tokens."""
    from dmlx_b200.serving import generate

    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 91, "float32", max_rows=256)
    head = _tokens(cfg, 70, 1)
    prompts = [head + _tokens(cfg, n, 300 + n) for n in (5, 9, 2)]
    want = [_greedy(w, cfg, p, 24) for p in prompts]
    assert generate(loaded, prompts, 24, prefill_chunk=32, n_pages=6) == want
    assert generate(loaded, prompts, 24, prefill_chunk=32, prefix_sharing=True) == want


def test_prefix_sharing_of_layers_that_share_their_latents(tmp_path):
    """A stack without state shares prefix pages; a layer without pages of its own reads the shared ones."""
    from dmlx_b200.serving import generate

    cfg = CASES["latent_only"]
    loaded, w = _load(tmp_path, cfg, 92, "float32", max_rows=256)
    assert loaded.model.cache_layers()[1] == (0, 0, 0, 0, 0)
    head = _tokens(cfg, 70, 1)
    prompts = [head + _tokens(cfg, n, 300 + n) for n in (5, 9, 2)]
    assert generate(loaded, prompts, 10, prefill_chunk=32, prefix_sharing=True) == [_greedy(w, cfg, p, 10) for p in prompts]


def test_prefix_pages_of_shared_latents_saved_and_restored(tmp_path):
    from dmlx_b200.prefix_store import PrefixDiskStore

    cfg = CASES["latent_only"]
    loaded, _ = _load(tmp_path / "m", cfg, 96, "bfloat16")
    toks = _tokens(cfg, 100, 8)
    kv = loaded.new_cache(8, 4)
    loaded.model.step(kv, [(0, 96, 0, 0)], toks[:96])
    store = PrefixDiskStore(str(tmp_path / "pages"))
    assert store.save_prefix(kv, 0, toks[:96]) == 3
    fresh = loaded.new_cache(8, 4)
    fresh.set_free_order([5, 2, 7, 0, 1, 3, 4, 6])
    assert store.restore_prefix(fresh, 0, toks[:97]) == 96
    out = []
    for pool in (kv, fresh):
        loaded.model.step(pool, [(0, 4, 96, 0)], toks[96:], [0, 1, 2, 3])
        out.append(loaded.model.logits(1, 4))
    np.testing.assert_array_equal(out[0], out[1])


def test_stop_tokens_and_sampling(tmp_path):
    from dmlx_b200.serving import generate

    cfg = CASES["recurrent_only"]
    loaded, w = _load(tmp_path, cfg, 95, "bfloat16")
    prompt = _tokens(cfg, 12, 4)
    plain = generate(loaded, [prompt], 20)[0]
    assert generate(loaded, [prompt], 20, stop_tokens=[plain[6]])[0] == plain[:plain.index(plain[6]) + 1]
    a = generate(loaded, [prompt], 20, temperature=2.0, top_k=20, seed=5)[0]
    assert a == generate(loaded, [prompt], 20, temperature=2.0, top_k=20, seed=5)[0]
    assert generate(loaded, [prompt], 20, temperature=1.0, top_k=1, seed=9)[0] == plain


def test_missing_or_wrong_tensors_are_named():
    from dmlx_b200 import _lib
    from dmlx_b200 import device as dev
    from dmlx_b200.models import dovorax

    cfg = CASES["odd_sizes"]
    w = R.random_weights(cfg, 1)
    bits = lambda a: (np.asarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)
    drop = {"l1.mix.uk": "key expansion", "l1.mix.dq.norm": "query latent norm", "l0.mix.right.f.b": "forget gate bias", "l0.mix.left.k.conv": "k convolution",
            "l2.mix.lam": "lru lambda", "l0.mlp.router": "router", "l1.mlp.e3.down": "elements"}
    for gone, text in drop.items():
        with pytest.raises(_lib.B200Error, match=text):
            model = dev.DecoderModel(cfg["width"], cfg["vocab"], dovorax.layer_specs(cfg), 1e-5, max_rows=64, max_reqs=1, max_seqs=1,
                                     flags=dev.DEC_SUM_NORM | dev.DEC_NORM_OFFSET, residual_scale=2.0)
            for layer, which, names in dovorax.tensor_names(cfg):
                have = [n for n in names if n != gone]
                if have:
                    model.set_tensor(layer, which, np.concatenate([bits(w[n]).ravel() for n in have]))
            model.finalize()


def test_impossible_layers_are_refused():
    from dmlx_b200 import _lib
    from dmlx_b200 import device as dev
    from dmlx_b200.models import dovorax

    specs = dovorax.layer_specs(CASES["mixed_order"])
    make = lambda layers, **kw: dev.DecoderModel(192, 64, layers, 1e-5, max_rows=64, max_reqs=1, max_seqs=1, **kw)
    make(specs, flags=dev.DEC_SUM_NORM).close()
    changes = [(1, dict(conv_taps=0)), (1, dict(n_groups=4)), (1, dict(top_k=7)), (1, dict(window=8)), (2, dict(rot_dim=34)), (2, dict(mem_gate_cap=0.0)),
               (2, dict(flags=specs[2]["flags"] & ~dev.DEC_QK_NORM)), (3, dict(kv_source=4)), (3, dict(kv_rank=32)), (3, dict(kv_source=2)), (0, dict(mem_heads=2))]
    for i, change in changes:
        layers = [dict(s) for s in specs]
        layers[i].update(change)
        with pytest.raises(_lib.B200Error, match=f"layer {i}"):
            make(layers, flags=dev.DEC_SUM_NORM)
    with pytest.raises(_lib.B200Error):
        make(specs, flags=dev.DEC_SUM_NORM | dev.DEC_DEPTH_AVERAGE)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_program(tmp_path, dtype):
    cfg = CASES["mixed_order"]
    w = R.random_weights(cfg, 97)
    R.write_model(str(tmp_path / "m"), cfg, w)
    a, b, c = (_tokens(cfg, n, n) for n in (70, 40, 90))
    steps = [
        {"step": 0, "entries": [{"id": "a", "tokens": a[:50], "want": [49, 3]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}, {"id": "a", "tokens": a[50:51], "want": []}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "c", "tokens": c[:33], "want": [32]}, {"id": "a", "tokens": a[51:53], "want": [0, 1]}], "end": []},
        {"step": 3, "entries": [{"id": "a", "tokens": a[53:], "want": [16]}], "end": ["a"]},
        {"step": 4, "entries": [{"id": "c", "tokens": c[33:], "want": [0, 56]}], "end": ["c"]},
    ]
    out = tmp_path / "out"
    out.mkdir()
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(out), "--max-tokens", "192"],
                       input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, env=dict(os.environ, PYTHONPATH=""), timeout=280)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(5)]
    fa, fc = R.forward(a, w, cfg), R.forward(c, w, cfg)
    want = {0: fa[[49, 3]], 2: np.stack([fc[32], fa[51], fa[52]]), 3: fa[[69]], 4: fc[[33, 89]]}
    assert sorted(os.listdir(out)) == [f"{s}.f32" for s in want]
    for s, x in want.items():
        got = np.fromfile(out / f"{s}.f32", "<f4").reshape(-1, cfg["vocab"])
        assert got.shape == x.shape and _error(got, x) <= _tol(dtype, w, cfg, a), s


def test_command_line_generates_the_engine_s_tokens(tmp_path):
    cfg = CASES["odd_sizes"]
    w = R.random_weights(cfg, 98)
    R.write_model(str(tmp_path), cfg, w)
    p = _tokens(cfg, 20, 2)
    r = subprocess.run([sys.executable, "-m", "dmlx_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt",
                        ",".join(map(str, p)), "--prompt", str(p[0]), "--max-new-tokens", "6"], capture_output=True, text=True, cwd=ROOT, timeout=280)
    assert r.returncode == 0, r.stderr
    assert [json.loads(l) for l in r.stdout.strip().split("\n")] == [_greedy(w, cfg, p, 6), _greedy(w, cfg, p[:1], 6)]
