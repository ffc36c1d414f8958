"""Lorulix as a served model, against the oracle: each mechanism, the whole stack, and what must not depend on how tokens reach it
(portions, batches, pages and state slots used again, graphs)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import ref_lorulix as R
from oracle.ref_math import bf16_round
from tests.lorulix_cases import CASES, attention, buckets_of, config, delta, dense, experts
from tests.test_gpu_window_attention import Pool

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 3e-5  # relative to the root mean square of what is compared
DTYPES = ["float32", "bfloat16"]


def _bf16(a):
    return bf16_round(np.asarray(a, np.float32)).astype(np.float64)


def _load(tmp_path, cfg, seed, dtype, max_rows=512, slots=4, change=None, decisive=True, buckets=8):
    from dmlx_b200.models import Limits, load_model

    w = R.random_weights(cfg, seed, decisive, buckets)
    if change:
        change(w)
        w = {n: _bf16(a) for n, a in w.items()}
    R.write_model(str(tmp_path), cfg, w)
    return load_model(str(tmp_path), dtype, Limits(max_rows, slots, slots)), w


def _error(got, want):
    return np.sqrt(((got - want) ** 2).mean(-1).max() / (want ** 2).mean())


def _close(got, want, tol):
    """Within tol at all positions but one in fifty (or one), and nowhere further off than twenty times.  Where a head of the delta rule reads next to
    nothing, the norm behind it makes rounding of its sign: such positions are rare, and as far off in the oracle when it rounds."""
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
    loaded, w = _load(tmp_path, cfg, 11, dtype, buckets=buckets_of(name))
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


@pytest.mark.parametrize("name", ["delta_only", "attention_only", "odd_sizes", "wide_heads"])
def test_router_over_the_whole_width(tmp_path, name):
    """Router weights without structure: every coordinate of the residual takes part in the choice."""
    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 12, "float32", decisive=False, buckets=buckets_of(name))
    toks = _tokens(cfg, 60, 5)
    assert _close(_step(loaded, toks), R.forward(toks, w, cfg), F32_TOL)


MECHANISMS = ["positions", "unit_offset", "canon1", "canon2", "gate1", "gate2", "post_norm", "short_conv", "conv_silu", "unit_norm", "beta", "dt_bias", "decay",
              "delta", "head_norm", "out_gate", "qk_norm", "q_temp", "distance", "limit", "router_scale", "shared", "shared_gate"]


def test_every_mechanism_shows(tmp_path):
    """The model equals the oracle, and not the oracle without one of the mechanisms."""
    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 21, "float32", decisive=False, buckets=buckets_of("mixed_order"))
    toks = _tokens(cfg, 70, 9)
    got = _step(loaded, toks)
    assert _error(got, R.forward(toks, w, cfg)) <= F32_TOL
    for mechanism in MECHANISMS:
        assert _error(got, R.forward(toks, w, cfg, without={mechanism})) > 100 * F32_TOL, mechanism


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CASES)
def test_portions_decoding_batches_and_reused_pages_and_slots(tmp_path, name, dtype):
    """Requests cut into portions of every size down to single tokens, in batches with others, on pages and state slots that
    earlier requests gave back: every logit equals the whole prompt's."""
    from dmlx_b200.serving import TokenFeeder

    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 31, dtype, buckets=buckets_of(name))
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
    loaded, w = _load(tmp_path, cfg, 41, dtype, buckets=buckets_of("mixed_order"))
    toks = _tokens(cfg, 110, 6)
    cut, single = _step(loaded, toks, [portion]), _step(loaded, toks, [1])
    tol = _tol(dtype, w, cfg, toks)
    assert _close(cut, single, tol)
    assert _close(single, R.forward(toks, w, cfg), tol)


def test_long_decoding_with_graphs(tmp_path):
    """400 decoded tokens through replayed graphs: a state that drifted, a convolution's input or a page that was missed would show at the end."""
    import torch

    from dmlx_b200.serving import TokenFeeder

    cfg = config(80, 120, [delta(3, 1, 24, 16, 4, experts(4, 2, 24, shared=16)), attention(4, 2, 24, 16, experts(3, 2, 16), bias_max=150, temp=(0.3, 50)),
                           delta(2, 2, 40, 24, 3, dense(40)), attention(2, 2, 24, 16, dense(24), kv_from=1, bias_max=300)])
    for dtype in DTYPES:
        loaded, w = _load(tmp_path / dtype, cfg, 51, dtype, change=lambda w: w["l0.mix.A_log"].__isub__(3.0))
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
    loaded, _ = _load(tmp_path, cfg, 61, "bfloat16", buckets=buckets_of("mixed_order"))
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
    loaded, w = _load(tmp_path, cfg, 71, "bfloat16", buckets=buckets_of(name))
    toks = _tokens(cfg, 140, 3)
    out = []
    for mma in (True, False):
        loaded.model.set_attn_mma(mma)
        out.append(_step(loaded, toks, [100, 1]))
    assert _close(out[0], out[1], _tol("bfloat16", w, cfg, toks))


# ---- mechanisms with inputs that make them stand out -------------------------------------------------------------------------
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
def test_convolutions_whose_oldest_tap_is_the_heaviest(tmp_path, taps, dtype):
    """Portions around the number of taps: the inputs before a portion come out of the state, those of the sublayers' own
    convolutions and of q, k and v alike."""
    cfg = config(64, 90, [delta(4, 2, 16, 24, taps, dense(40)), attention(2, 1, 16, 24, None, bias_max=20)], taps=taps)

    def heavy(w):
        for n in w:
            if n.endswith((".conv", ".canon1", ".canon2")):
                w[n][:, 0] += 1.5

    loaded, w = _load(tmp_path, cfg, 13, dtype, change=heavy)
    toks = _tokens(cfg, 40, 2)
    want, tol = R.forward(toks, w, cfg), _tol(dtype, w, cfg, toks)
    for portions in ([40], [1], [2], [3], [5], [1, 2, 1, 3, 1, 6, 7, 1], [39, 1], [taps + 1]):
        assert _close(_step(loaded, toks, portions), want, tol), portions


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("taps", [2, 3, 4, 5])
def test_a_large_step_of_unequal_portions(tmp_path, taps, dtype):
    """More than a thousand rows in one step, portions that start and end anywhere among them, and a second step behind it."""
    from dmlx_b200.serving import TokenFeeder

    cfg = config(64, 90, [delta(4, 2, 24, 40, 4, dense(24)), attention(4, 2, 24, 40, None, bias_max=300), delta(2, 1, 136, 144, taps, experts(4, 2, 16, shared=8))],
                 taps=taps, positions=700)
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
    w["pos"][:, coordinate] = 0.0
    for n in w:
        if n.endswith(".o") or n.endswith(".down"):
            w[n][coordinate] = 0.0


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_keeps_one_token_among_hundreds(tmp_path, dtype):
    """One token is written once; hundreds behind it neither decay the state nor write to it."""
    cfg = config(64, 90, [delta(2, 1, 32, 40, 2)], taps=1)

    def plant(w):
        _special_token(cfg, w, 7)
        p = "l0.mix."
        w[p + "b"][:] = 0.0
        w[p + "b"][:, 0] = 8.0    # the special token writes with its whole weight, the others (through pos) hardly
        w["l0.norm1"][1] = 3.0
        w["embed"][:, 1] = -2.0
        w["embed"][7, 1] = 0.0
        w["pos"][:, 1] = 0.0
        w[p + "b"][:, 1] = 2.0
        w[p + "A_log"][:] = -9.0  # next to no decay

    loaded, w = _load(tmp_path, cfg, 14, dtype, change=plant)
    toks = [t if t != 7 else 8 for t in _tokens(cfg, 330, 2)]
    toks[5] = 7
    want, tol = R.forward(toks, w, cfg), _tol(dtype, w, cfg, toks)
    other = R.forward(toks[:5] + [8] + toks[6:], w, cfg)
    assert _error(want[300:], other[300:]) > 3 * tol
    for portions in ([330], [300, 1], [31, 1, 33, 64, 2], [4, 1, 7]):
        assert _close(_step(loaded, toks, portions), want, tol), portions


@pytest.mark.parametrize("dtype", DTYPES)
def test_first_tokens_and_positions(tmp_path, dtype):
    """Single tokens at position 0 in used slots, and the same token at different positions."""
    from dmlx_b200.serving import TokenFeeder

    cfg = config(48, 60, [attention(2, 1, 16, 16, bias_max=9), delta(2, 1, 16, 16, 3)], positions=40)
    loaded, w = _load(tmp_path, cfg, 24, dtype)
    feeder = TokenFeeder(loaded, 4, 2)
    for round_ in range(5):
        toks = [3 + round_] * 6
        got = np.concatenate([feeder.step([(round_, toks[:1], [0])]), feeder.step([(round_, toks[1:], range(5))])])
        assert _close(got, R.forward(toks, w, cfg), _tol(dtype, w, cfg, toks))
        feeder.end(round_)


def test_positions_end_where_the_table_does(tmp_path):
    from dmlx_b200 import _lib
    from dmlx_b200.serving import generate

    cfg = config(48, 60, [delta(2, 1, 16, 16, 3), attention(2, 1, 16, 16, bias_max=9)], positions=40)
    loaded, w = _load(tmp_path, cfg, 25, "float32")
    toks = _tokens(cfg, 40, 3)
    assert _close(_step(loaded, toks, pages=2), R.forward(toks, w, cfg), F32_TOL)
    with pytest.raises(_lib.B200Error, match="40"):
        _step(loaded, toks + [1], pages=2)
    assert generate(loaded, [toks[:30]], 10)[0] == _greedy(w, cfg, toks[:30], 10)
    with pytest.raises(_lib.B200Error):
        generate(loaded, [toks], 3)
    with pytest.raises(_lib.B200Error):
        generate(loaded, [toks[:38]], 12)


@pytest.mark.parametrize("dtype", DTYPES)
def test_sharp_scores_find_single_keys(tmp_path, dtype):
    """Scores so sharp that most queries read one key, near or hundreds of tokens away, over pages and the edges of the distance buckets."""
    cfg = config(96, 120, [attention(4, 2, 32, 24, scale=1.0, bias_max=150), attention(4, 2, 32, 24, scale=1.2, bias_max=40, kv_from=0)], positions=400)
    loaded, w = _load(tmp_path, cfg, 17, dtype, change=lambda w: w["l0.mix.rel"].__imul__(3.0))
    toks = _tokens(cfg, 360, 4)
    want, tol = R.forward(toks, w, cfg), _tol(dtype, w, cfg, toks)
    for portions in ([360], [280, 1], [64, 33, 2, 100]):
        assert _close(_step(loaded, toks, portions), want, tol), portions


def test_positions_far_out(tmp_path):
    """Query temperatures and distances thousands of tokens from the start, in f32."""
    cfg = config(48, 64, [attention(2, 1, 16, 16, scale=0.5, bias_max=1500, temp=(0.7, 100)), delta(2, 1, 16, 16, 2)], positions=2560)
    loaded, w = _load(tmp_path, cfg, 18, "float32", max_rows=2600, buckets=32)
    toks = _tokens(cfg, 2560, 4)
    want = R.forward(toks, w, cfg)
    got = _step(loaded, toks, [2550, 1])
    assert _error(got[2000:], want[2000:]) <= F32_TOL


@pytest.mark.parametrize("mma", [True, False])
@pytest.mark.parametrize("shape", [(4, 2, 80, 48), (6, 1, 16, 72), (20, 1, 128, 128), (3, 3, 200, 136)], ids=str)
def test_distance_table_at_every_distance(shape, mma):
    """Scores of nothing but the table, one distance far above the others: the output is the value at that distance, in prompts and in
    single rows, however the keys are cut."""
    from dmlx_b200 import device as dev

    n, reach = 300, 90
    p = Pool(shape, [n], False)
    hq, g, kd, vd = shape
    rng = np.random.default_rng(3)
    v = _bf16(rng.normal(size=(n, g, vd)))
    q, seq, ctx = p.append([(0, 0, n)], np.zeros((n, hq, kd)), np.zeros((n, g, kd)), v)
    for pages in (0, 1, 3):
        dev.set_attn_pages_per_chunk(pages)
        try:
            for at in (0, 1, 30, 31, 32, 33, 63, 64, reach - 2, reach - 1):
                table = 0.1 * rng.normal(size=(hq, reach))
                table[:, at] = 25.0
                want = np.zeros((n, hq, vd))
                dist = np.minimum(np.maximum(np.arange(n)[:, None] - np.arange(n)[None, :], 0), reach - 1)
                for h in range(hq):
                    s = np.where(np.arange(n)[:, None] >= np.arange(n)[None, :], table[h][dist], -np.inf)
                    e = np.exp(s - s.max(-1, keepdims=True))
                    want[:, h] = e / e.sum(-1, keepdims=True) @ v[:, h // (hq // g)]
                whole = p.kv.window_attention(0, q, seq, ctx, 1.0, mma=mma, distances=table).double().cpu().numpy()
                np.testing.assert_allclose(whole, want, atol=2e-2)
                rows = [0, at, min(at + 31, n - 1), 150, n - 1]
                one = p.kv.window_attention(0, q[rows].contiguous(), seq[rows].contiguous(), ctx[rows].contiguous(), 1.0, mma=mma, distances=table)
                np.testing.assert_allclose(one.double().cpu().numpy(), want[rows], atol=2e-2)
        finally:
            dev.set_attn_pages_per_chunk(0)


class DeltaCase:
    def __init__(self, lens, heads, kv_heads, dk, dv, taps=3, dtype="bfloat16", seed=0, rate=0.3, change=None):
        import torch

        from dmlx_b200 import device as dev

        rng = np.random.default_rng(seed)
        self.heads, self.kv_heads, self.dk, self.dv, self.taps, self.torch = heads, kv_heads, dk, dv, taps, torch
        self.channels = 2 * kv_heads * dk + heads * dv
        self.rows = [_bf16(rng.normal(size=(n, self.channels + heads * (dv + 2)))) for n in lens]
        if change:
            self.rows = [_bf16(change(r, self)) for r in self.rows]
        self.conv = _bf16(rng.normal(size=(self.channels, taps)))
        self.rate, self.dt = rate * np.exp(0.5 * rng.normal(size=heads)), rng.normal(size=heads)
        self.norm = 1 + 0.3 * rng.normal(size=dv)
        self.type = torch.float32 if dtype == "float32" else torch.bfloat16
        state = (heads * dk * dv + 3) // 4 * 4 + (taps - 1) * self.channels
        self.kv = dev.LayeredKVCache([(1, 16, 16), (0, 0, 0, 0, (state + 3) // 4 * 4)], 4, len(lens) + 1, 4, heads, max_rows=4096,
                                     kv_dtype=dev.KV_F32 if dtype == "float32" else dev.KV_BF16)

    def step(self, portions, chunked=True):
        """portions: [(sequence, from, to)] of one batch -> outputs per portion.  Sequence i sits in slot i + 1."""
        t = self.torch
        f = lambda a: t.tensor(np.asarray(a), dtype=t.float32, device="cuda")
        i32 = lambda a: t.tensor(np.asarray(a), dtype=t.int32, device="cuda")
        rows = t.tensor(np.concatenate([self.rows[s][a:b] for s, a, b in portions]), dtype=self.type, device="cuda")
        conv = t.tensor(np.ascontiguousarray(self.conv.T), dtype=t.bfloat16, device="cuda")
        cu = np.cumsum([0] + [b - a for _, a, b in portions])
        seq = np.concatenate([[s + 1] * (b - a) for s, a, b in portions])
        req = np.concatenate([[i] * (b - a) for i, (_, a, b) in enumerate(portions)])
        pos = np.concatenate([np.arange(a, b) for _, a, b in portions])
        out = self.kv.delta(1, rows, conv, f(self.rate), f(self.dt), f(self.norm), self.kv_heads, self.dk, 1e-5, i32(cu), i32(req), i32(seq), i32(pos), chunked)
        out = out.float().cpu().numpy()
        return [out[cu[i]:cu[i + 1]] for i in range(len(portions))]

    def want(self, s):
        x, c, h, k = self.rows[s], self.channels, self.heads, self.kv_heads
        y = R.silu(R.causal_convolution(x[:, :c], self.conv))
        t, kd = len(x), k * self.dk
        part = lambda a, n: R.unit_vectors(a.reshape(t, k, self.dk)).repeat(h // k, axis=1) * n
        o = R.delta_rule(part(y[:, :kd], self.dk ** -0.5), part(y[:, kd:2 * kd], 1.0), y[:, 2 * kd:].reshape(t, h, self.dv),
                         R.sigmoid(x[:, c + h * self.dv:c + h * self.dv + h]), -self.rate * R.softplus(x[:, -h:] + self.dt))
        o = R.root_mean_square_norm(o, 1e-5) * self.norm
        return o * R.silu(x[:, c:c + h * self.dv]).reshape(t, h, self.dv)


DELTA_SHAPES = [(4, 2, 48, 40, 3), (3, 1, 32, 64, 4), (2, 2, 128, 128, 4), (6, 2, 19, 13, 2), (1, 1, 256, 128, 4), (2, 1, 256, 264, 1), (2, 1, 40, 300, 5), (1, 1, 24, 1100, 2),
                (1, 1, 33, 1030, 3), (2, 1, 130, 66, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", DELTA_SHAPES, ids=str)
def test_delta_rule_over_chunk_borders(shape, dtype):
    """Portions that end at, before and behind the borders of 32-token chunks, chunk by chunk and token by token, and states handed on."""
    heads, kv, dk, dv, taps = shape
    lens = (1, 31, 32, 33, 64, 65, 130)
    tol = 3e-5 if dtype == "float32" else 8e-3
    for chunked in (True, False):
        case = DeltaCase(lens, heads, kv, dk, dv, taps, dtype)
        for s, got in enumerate(case.step([(s, 0, n) for s, n in enumerate(lens)], chunked)):
            assert _close(got.reshape(len(got), -1), case.want(s).reshape(len(got), -1), tol), (s, chunked)
        case = DeltaCase(lens, heads, kv, dk, dv, taps, dtype)
        want, cuts = case.want(6), (0, 5, 6, 38, 40, 41, 100, 130)
        got = np.concatenate([case.step([(6, a, b)], chunked)[0] for a, b in zip(cuts, cuts[1:])])
        assert _close(got.reshape(130, -1), want.reshape(130, -1), tol), chunked


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rate", [1e-6, 0.02, 3.0, 400.0])
def test_delta_rule_of_weak_and_violent_decays(rate, dtype):
    case = DeltaCase((150,), 3, 3, 32, 48, 2, dtype, rate=rate)
    want = case.want(0).reshape(150, -1)
    for portions in ([(0, 0, 150)], [(0, 0, 70), (0, 70, 73), (0, 73, 149), (0, 149, 150)]):
        got = np.concatenate([case.step([p])[0] for p in portions]).reshape(150, -1)
        assert _close(got, want, 1e-4 if dtype == "float32" else 8e-3), portions


@pytest.mark.parametrize("dtype", DTYPES)
def test_delta_rule_of_keys_that_repeat(dtype):
    """All tokens of a chunk share one key, and write with their whole weight: every write replaces the one before, and the system that
    a chunk solves is as far from the identity as it gets."""

    def same(rows, case):
        kd = case.kv_heads * case.dk
        rows[:, kd:2 * kd] = np.abs(rows[:1, kd:2 * kd]) * 2.0
        rows[:, case.channels + case.heads * case.dv:][:, :case.heads] = 9.0
        return rows

    case = DeltaCase((100,), 2, 1, 32, 24, 1, dtype, rate=1e-4, change=same)
    case.conv = np.abs(case.conv)
    want = case.want(0).reshape(100, -1)
    for portions in ([(0, 0, 100)], [(0, i, i + 1) for i in range(100)], [(0, 0, 40), (0, 40, 100)]):
        got = np.concatenate([case.step([p])[0] for p in portions]).reshape(100, -1)
        assert _close(got, want, 1e-4 if dtype == "float32" else 8e-3), portions


@pytest.mark.parametrize("experts_, top", [(40, 5), (130, 16), (64, 1), (300, 7), (48, 32), (31, 3), (32, 4), (33, 2)])
def test_router_of_many_experts(tmp_path, experts_, top):
    """Also where the gate of the shared expert lies in another group of lanes than the experts' logits."""
    cfg = config(64, 90, [delta(2, 1, 16, 16, 2, experts(experts_, top, 8, 1.7, 8))])
    loaded, w = _load(tmp_path, cfg, 19, "float32", decisive=False)
    toks = _tokens(cfg, 33, 4)
    assert _close(_step(loaded, toks, [20, 1]), R.forward(toks, w, cfg), F32_TOL)


# ---- state, engine, programs ---------------------------------------------------------------------------------------------------
def test_state_through_fork_extend_rollback_and_release(tmp_path):
    from dmlx_b200 import _lib

    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 93, "float32", slots=4, buckets=buckets_of("mixed_order"))
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


@pytest.mark.parametrize("rows", [(10,), (1,)])
def test_a_step_without_pages_leaves_states_alone(tmp_path, rows):
    """A step whose pages do not fit is flagged and changes no state: the same tokens run again on a pool that has been freed."""
    from dmlx_b200 import _lib

    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 94, "float32", buckets=buckets_of("mixed_order"))
    toks = _tokens(cfg, 70, 3)
    kv, m, n = loaded.new_cache(3, 3), loaded.model, rows[0]
    m.step(kv, [(0, 32, 0, 0)], toks[:32])
    m.step(kv, [(1, 33, 0, 0)], toks[:33])
    with pytest.raises(_lib.B200Error):
        m.step(kv, [(0, n, 32, 0)], toks[32:32 + n])
    kv.release([1])
    m.step(kv, [(0, n, 32, 0)], toks[32:32 + n])
    assert _error(m.logits(0, 1)[0], R.forward(toks[:32 + n], w, cfg)[-1]) <= F32_TOL


def _greedy(w, cfg, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(R.forward(toks, w, cfg)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["delta_only", "attention_only", "odd_sizes", "mixed_order", "one_tap"])
def test_greedy_generation_through_the_engine(tmp_path, name):
    """More prompts than slots, chunked prefill beside decoding: the tokens are those of each prompt alone."""
    from dmlx_b200.serving import generate

    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 81, "float32", max_rows=96, buckets=buckets_of(name))
    prompts = [_tokens(cfg, n, 200 + n) for n in (40, 1, 55, 9, 33, 64)]
    got = generate(loaded, prompts, 8, prefill_chunk=23)
    for p, g in zip(prompts, got):
        assert g == _greedy(w, cfg, p, 8)


def test_generation_under_page_pressure_and_with_prefix_sharing_asked_for(tmp_path):
    """A pool too small for all requests (deferral, preemption by recomputation: the state starts over), and prefix sharing, which
    a recurrent state does not allow: same tokens."""
    from dmlx_b200.serving import generate

    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 91, "float32", max_rows=256, buckets=buckets_of("mixed_order"))
    head = _tokens(cfg, 70, 1)
    prompts = [head + _tokens(cfg, n, 300 + n) for n in (5, 9, 2)]
    want = [_greedy(w, cfg, p, 24) for p in prompts]
    assert generate(loaded, prompts, 24, prefill_chunk=32, n_pages=6) == want
    assert generate(loaded, prompts, 24, prefill_chunk=32, prefix_sharing=True) == want


def test_stop_tokens_and_sampling(tmp_path):
    from dmlx_b200.serving import generate

    cfg = CASES["delta_only"]
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
    from dmlx_b200.models import lorulix

    cfg = CASES["odd_sizes"]
    w = R.random_weights(cfg, 1, buckets=buckets_of("odd_sizes"))
    bits = lambda a: (np.asarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)
    drop = {"l1.mix.k.conv": "k convolution", "l1.mix.A_log": "decay rate", "l0.mix.rel": "distance table", "l0.mlp.shared.sg": "shared expert gate", "pos": "positions",
            "l2.canon2": "input convolution 2", "l3.rg1.b": "result gate bias 1", "l2.mix.q.norm": "q norm", "l1.mlp.e3.down": "elements"}
    for gone, text in drop.items():
        with pytest.raises(_lib.B200Error, match=text):
            model = dev.DecoderModel(cfg["width"], cfg["vocab"], lorulix.layer_specs(cfg, buckets_of("odd_sizes")), 1e-5, max_rows=64, max_reqs=1, max_seqs=1,
                                     flags=dev.DEC_NORM_OFFSET, max_positions=cfg["max_positions"])
            for layer, which, names in lorulix.tensor_names(cfg):
                have = [n for n in names if n != gone]
                if have:
                    model.set_tensor(layer, which, np.concatenate([bits(w[n]).ravel() for n in have]))
            model.finalize()


def test_impossible_layers_are_refused():
    from dmlx_b200 import _lib
    from dmlx_b200 import device as dev
    from dmlx_b200.models import lorulix

    specs = lorulix.layer_specs(CASES["mixed_order"], buckets_of("mixed_order"))
    make = lambda layers, **kw: dev.DecoderModel(192, 64, layers, 1e-5, max_rows=64, max_reqs=1, max_seqs=1, **kw)
    make(specs).close()
    flag = lambda i, on, off=0: dict(flags=(specs[i]["flags"] | on) & ~off)
    changes = [(0, dict(conv_taps=0)), (0, dict(n_kv_heads=3)), (0, dict(window=8)), (0, dict(rel_buckets=8, rel_reach=20)), (1, dict(rel_reach=16)), (1, dict(conv_taps=3)),
               (1, dict(top_k=10)), (1, dict(rot_dim=8, rot_base=1e4)), (1, flag(1, dev.DEC_QK_NORM)), (1, flag(1, 0, dev.DEC_ROUTER)), (1, dict(ffn=0)),
               (1, flag(1, dev.DEC_FF_GELU)), (3, dict(kv_source=4)), (3, dict(kv_source=3)), (3, dict(key_dim=24)), (5, dict(kv_source=4)), (0, dict(input_taps=-1)),
               (0, dict(ff_limit=-1.0))]
    for i, change in changes:
        layers = [dict(s) for s in specs]
        layers[i].update(change)
        with pytest.raises(_lib.B200Error, match=f"layer {i}"):
            make(layers)
    with pytest.raises(_lib.B200Error):
        make(specs, flags=dev.DEC_SUM_NORM)


@pytest.mark.parametrize("dtype", DTYPES)
def test_trace_replay_program(tmp_path, dtype):
    cfg = CASES["mixed_order"]
    w = R.random_weights(cfg, 97, buckets=buckets_of("mixed_order"))
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
    w = R.random_weights(cfg, 98, buckets=buckets_of("odd_sizes"))
    R.write_model(str(tmp_path), cfg, w)
    p = _tokens(cfg, 20, 2)
    r = subprocess.run([sys.executable, "-m", "dmlx_b200", "generate", "--model", str(tmp_path), "--dtype", "float32", "--prompt",
                        ",".join(map(str, p)), "--prompt", str(p[0]), "--max-new-tokens", "6"], capture_output=True, text=True, cwd=ROOT, timeout=280)
    assert r.returncode == 0, r.stderr
    assert [json.loads(l) for l in r.stdout.strip().split("\n")] == [_greedy(w, cfg, p, 6), _greedy(w, cfg, p[:1], 6)]
