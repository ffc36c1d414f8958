"""Sotavik as a served model, against the oracle: each mechanism, the whole stack, and what must not depend on how tokens reach it
(portions, batches, pages and state slots used again, graphs)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import ref_sotavik as R
from oracle.ref_math import bf16_round
from tests.sotavik_cases import CASES, config, experts, gla, latent

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 3e-5  # relative to the root mean square of what is compared
DTYPES = ["float32", "bfloat16"]


def _load(tmp_path, cfg, seed, dtype, max_rows=512, slots=4, change=None, rank=7):
    from dmlx_b200.models import Limits, load_model

    w = R.random_weights(cfg, seed, rank)
    if change:
        change(w)
        w = {n: a if n.endswith(".table") else _bf16(a) for n, a in w.items()}
    R.write_model(str(tmp_path), cfg, w)
    return load_model(str(tmp_path), dtype, Limits(max_rows, slots, slots)), w


def _error(got, want):
    return np.sqrt(((got - want) ** 2).mean(-1).max() / (want ** 2).mean())


def _bf16(a):
    return bf16_round(np.asarray(a, np.float32)).astype(np.float64)


def _tol(dtype, w, cfg, tokens):
    """What rounding alone may cause: in bfloat16 three times the error the oracle makes on these tokens when it rounds every
    matrix operand and result to bf16."""
    if dtype == "float32":
        return F32_TOL
    return 3 * _error(R.forward(tokens, w, cfg, _bf16), R.forward(tokens, w, cfg))


def _tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CASES)
def test_whole_prompt_layer_by_layer_and_logits(tmp_path, name, dtype):
    from dmlx_b200.serving import TokenFeeder

    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 11, dtype)
    toks = _tokens(cfg, 150, 5)
    want, trail = R.forward(toks, w, cfg, want_layers=True)
    loaded.model.record_layers(True)
    got = TokenFeeder(loaded, 8).step([("r", toks, range(len(toks)))])
    layers = loaded.model.recorded_layers(len(toks))
    rounded = R.forward(toks, w, cfg, _bf16, want_layers=True)[1]
    for i in range(len(trail)):
        tol = F32_TOL if dtype == "float32" else 3 * _error(rounded[i], trail[i])
        assert _error(layers[i], trail[i]) <= tol, (name, "layer", i)
    assert _error(got, want) <= _tol(dtype, w, cfg, toks), name


@pytest.mark.parametrize("mechanism", ["decay", "tau", "decay_bias", "head_norm", "out_gate", "latent_norm", "rotation", "sink", "shared",
                                       "depth_average"])
def test_every_mechanism_shows(tmp_path, mechanism):
    """The model equals the oracle, and not the oracle without one of the mechanisms."""
    from dmlx_b200.serving import TokenFeeder

    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 21, "float32")
    toks = _tokens(cfg, 60, 9)
    got = TokenFeeder(loaded, 4).step([("r", toks, range(60))])
    assert _error(got, R.forward(toks, w, cfg)) <= F32_TOL
    assert _error(got, R.forward(toks, w, cfg, without={mechanism})) > 100 * F32_TOL


@pytest.mark.parametrize("other", [3, 19])
def test_inner_width_of_the_decay_projection_comes_from_the_tensor(tmp_path, other):
    from dmlx_b200.serving import TokenFeeder

    cfg = CASES["gla_only"]
    loaded, w = _load(tmp_path, cfg, 22, "float32", rank=other)
    toks = _tokens(cfg, 40, 3)
    assert _error(TokenFeeder(loaded, 2).step([("r", toks, range(40))]), R.forward(toks, w, cfg)) <= F32_TOL


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
    for i in prompts:
        assert _error(np.concatenate(got[i]), want[i]) <= max(_tol(dtype, w, cfg, prompts[i]), _tol(dtype, w, cfg, prompts[0])), (name, i)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("portion", [2, 4, 5, 32, 50])
def test_portions_of_one_size_against_token_by_token(tmp_path, portion, dtype):
    from dmlx_b200.serving import TokenFeeder

    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 41, dtype)
    toks = _tokens(cfg, 110, 6)
    feeder = TokenFeeder(loaded, 8)
    cut = np.concatenate([feeder.step([("a", toks[i:i + portion], range(len(toks[i:i + portion])))]) for i in range(0, 110, portion)])
    single = np.concatenate([feeder.step([("b", [t], [0])]) for t in toks])
    tol = _tol(dtype, w, cfg, toks)
    assert _error(cut, single) <= tol
    assert _error(single, R.forward(toks, w, cfg)) <= tol


def test_long_decoding_with_graphs(tmp_path):
    """400 decoded tokens through replayed graphs: a state that drifted or a page that was missed would show at the end."""
    import torch

    from dmlx_b200.serving import TokenFeeder

    cfg = config(80, 120, [gla(2, 24, 40, 16.0, experts(3, 1, 24, 16)), latent(4, 16, 8, 24, 56, experts(3, 2, 16, 8))])
    for dtype in DTYPES:
        loaded, w = _load(tmp_path / dtype, cfg, 51, dtype, change=lambda w: w["l0.mix.a2.b"].__iadd__(4.0))
        toks = _tokens(cfg, 420, 7)
        want = R.forward(toks, w, cfg)
        feeder = TokenFeeder(loaded, 14)
        with torch.cuda.stream(torch.cuda.Stream()):
            feeder.step([("a", toks[:20], [])])
            got = np.concatenate([feeder.step([("a", [t], [0])]) for t in toks[20:]])
        assert _error(got, want[20:]) <= _tol(dtype, w, cfg, toks)


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
    from dmlx_b200.serving import TokenFeeder

    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 71, "bfloat16")
    toks = _tokens(cfg, 140, 3)
    out = []
    for mma in (True, False):
        loaded.model.set_attn_mma(mma)
        feeder = TokenFeeder(loaded, 8)
        out.append(np.concatenate([feeder.step([("a", toks[:100], range(100))])] + [feeder.step([("a", [t], [0])]) for t in toks[100:]]))
    assert _error(out[0], out[1]) <= _tol("bfloat16", w, cfg, toks)


def _greedy(w, cfg, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(R.forward(toks, w, cfg)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["gla_only", "odd_sizes", "mixed_order"])
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


def test_prefix_sharing_of_a_stack_without_state(tmp_path):
    from dmlx_b200.serving import generate

    cfg = CASES["latent_only"]
    loaded, w = _load(tmp_path, cfg, 92, "float32", max_rows=256)
    head = _tokens(cfg, 70, 1)
    prompts = [head + _tokens(cfg, n, 300 + n) for n in (5, 9, 2)]
    assert generate(loaded, prompts, 10, prefill_chunk=32, prefix_sharing=True) == [_greedy(w, cfg, p, 10) for p in prompts]


def test_stop_tokens_and_sampling(tmp_path):
    from dmlx_b200.serving import generate

    cfg = CASES["gla_only"]
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
    from dmlx_b200.models import sotavik

    cfg = CASES["odd_sizes"]
    w = R.random_weights(cfg, 1)
    bits = lambda a: (np.asarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)
    drop = {"l1.mix.uk": "key expansion", "l0.mix.a2.b": "decay bias", "l2.dwa": "depth weights", "l1.mlp.e3.down": "elements", "l0.mlp.table": "table"}
    for gone, text in drop.items():
        with pytest.raises(_lib.B200Error, match=text):
            model = dev.DecoderModel(cfg["width"], cfg["vocab"], sotavik.layer_specs(cfg, lambda i: 7), 1e-5, max_rows=64, max_reqs=1, max_seqs=1,
                                     flags=dev.DEC_SCALAR_NORM | dev.DEC_DEPTH_AVERAGE)
            for layer, which, names in sotavik.tensor_names(cfg):
                have = [n for n in names if n != gone]
                if which == "table":
                    if have:
                        model.set_table(layer, w[names[0]])
                elif have:
                    model.set_tensor(layer, which, np.concatenate([bits(w[n]).ravel() for n in have]))
            model.finalize()
    bad = np.array(w["l0.mlp.table"])
    bad[3, 1] = 5
    with pytest.raises(_lib.B200Error, match="expert 5 of 5"):
        model.set_table(0, bad)


# ---- the kernels on their own ------------------------------------------------------------------------------------------
def _gla_oracle(rows, a2, b, norm, heads, dk, dv, tau, eps):
    t = rows.shape[0]
    cut = np.cumsum([0, heads * dk, heads * dk, heads * dv, heads * dv])
    q, k, v, g = (rows[:, cut[i]:cut[i + 1]].reshape(t, heads, -1) for i in range(4))
    la = R.log_sigmoid(rows[:, cut[4]:] @ a2.T + b) / tau
    o = R.gated_linear_recurrence(q * dk ** -0.5, k, v, la.reshape(t, heads, dk))
    return R.silu_gated(g, R.root_mean_square_norm(o, eps, norm))


class GlaCase:
    def __init__(self, lens, heads, dk, dv, rank=5, tau=4.0, bias=1.0, dtype="bfloat16", seed=0):
        import torch

        from dmlx_b200 import device as dev

        rng = np.random.default_rng(seed)
        self.heads, self.dk, self.dv, self.tau, self.torch = heads, dk, dv, tau, torch
        self.rows = [_bf16(rng.normal(size=(n, 2 * heads * (dk + dv) + rank))) for n in lens]
        self.a2, self.b = 0.5 * rng.normal(size=(heads * dk, rank)), bias + rng.normal(size=heads * dk)
        self.norm = 1 + 0.3 * rng.normal(size=dv)
        self.type = torch.float32 if dtype == "float32" else torch.bfloat16
        self.kv = dev.LayeredKVCache([(1, 16, 16), (0, 0, 0, 0, heads * dk * dv)], 4, len(lens) + 1, 4, heads, max_rows=4096,
                                     kv_dtype=dev.KV_F32 if dtype == "float32" else dev.KV_BF16)

    def step(self, portions, chunked=True):
        """portions: [(sequence, from, to)] of one batch -> outputs per portion.  Sequence i sits in slot i + 1."""
        t = self.torch
        f = lambda a: t.tensor(np.asarray(a), dtype=t.float32, device="cuda")
        i32 = lambda a: t.tensor(np.asarray(a), dtype=t.int32, device="cuda")
        rows = t.tensor(np.concatenate([self.rows[s][a:b] for s, a, b in portions]), dtype=self.type, device="cuda")
        cu = np.cumsum([0] + [b - a for _, a, b in portions])
        seq = np.concatenate([[s + 1] * (b - a) for s, a, b in portions])
        pos = np.concatenate([np.arange(a, b) for _, a, b in portions])
        out = self.kv.gla(1, rows, f(self.a2), f(self.b), f(self.norm), self.heads, self.tau, 1e-5, i32(cu), i32(seq), i32(pos), chunked)
        out = out.float().cpu().numpy()
        return [out[cu[i]:cu[i + 1]] for i in range(len(portions))]

    def want(self, s):
        return _gla_oracle(self.rows[s], self.a2, self.b, self.norm, self.heads, self.dk, self.dv, self.tau, 1e-5)


@pytest.mark.parametrize("heads,dk,dv,tau,bias", [(2, 48, 40, 4.0, 1.0), (3, 32, 64, 16.0, 3.0), (1, 128, 160, 1.0, 0.0), (2, 20, 24, 8.0, 12.0), (1, 256, 70, 2.0, 2.0)])
def test_gla_chunks_equal_single_tokens_and_the_recurrence(heads, dk, dv, tau, bias):
    """Portions around the chunk length, mixed with single tokens; weak decays keep the first tokens alive to the end."""
    case = GlaCase([101, 64, 37, 5], heads, dk, dv, tau=tau, bias=bias)
    parts = [[(0, 0, 40), (1, 0, 1), (2, 0, 5), (3, 0, 5)], [(0, 40, 41), (1, 1, 33), (2, 5, 37)], [(1, 33, 64), (0, 41, 43)], [(0, 43, 101)]]
    for chunked in (True, False):
        got = {i: [] for i in range(4)}
        for p in parts:
            for (s, _, _), o in zip(p, case.step(p, chunked)):
                got[s].append(o)
        for s in range(4):
            want = case.want(s)
            rounding = _error(_bf16(want), want)
            assert _error(np.concatenate(got[s]), want) <= 3 * rounding, (chunked, s)


@pytest.mark.parametrize("bias", [-30.0, -400.0])
def test_gla_strong_decays_take_the_pairwise_route(bias):
    """Decays that leave nothing of a token after one or two more: factored exponentials would overflow."""
    case = GlaCase([96], 2, 32, 24, tau=1.0, bias=0.0)
    case.b[::3] = bias
    case.b[1::7] = 30.0  # beside channels that keep everything
    got = np.concatenate([case.step([(0, 0, 70)])[0], case.step([(0, 70, 96)])[0]])
    want = case.want(0)
    assert np.isfinite(got).all()
    assert _error(got, want) <= 3 * _error(_bf16(want), want)


def test_gla_remembers_one_token_among_hundreds():
    """A single key and query stand out, 300 tokens apart, in prompts and in decoding."""
    case = GlaCase([320], 1, 64, 32, tau=16.0, bias=14.0)
    q, k = case.rows[0][:, :64], case.rows[0][:, 64:128]
    k *= 0.02
    k[7] = 0
    k[7, 5] = 40.0
    q *= 0.05
    q[310:, 5] = 3.0
    for cut in (320, 300, 311):
        got = np.concatenate([case.step([(0, 0, cut)])[0]] + [case.step([(0, i, i + 1)])[0] for i in range(cut, 320)])
        want = case.want(0)
        assert _error(got[310:], want[310:]) <= 3 * _error(_bf16(want), want)
        v7 = case.rows[0][7, 128:160]
        o = want[315, 0] / (case.norm * case.rows[0][315, 160:192] / (1 + np.exp(-case.rows[0][315, 160:192])))
        assert np.corrcoef(o, v7)[0, 1] > 0.99


def test_gla_f32_is_exact_and_a_reused_slot_starts_from_zero():
    case = GlaCase([50, 50], 2, 24, 20, dtype="float32")
    first = case.step([(0, 0, 50)])[0]
    case.rows[0], case.rows[1] = case.rows[1], case.rows[0]
    second = case.step([(0, 0, 50)])[0]  # the same slot, another sequence
    assert _error(second, case.want(0)) <= 1e-5 and _error(first, case.want(1)) <= 1e-5


def test_state_through_fork_extend_rollback_and_release(tmp_path):
    from dmlx_b200 import _lib

    cfg = CASES["mixed_order"]
    loaded, w = _load(tmp_path, cfg, 93, "float32", slots=4)
    toks = _tokens(cfg, 60, 3)
    want = R.forward(toks, w, cfg)
    kv, other = loaded.new_cache(12, 4), loaded.new_cache(8, 4)
    assert kv.state_bytes() == 4 * sum(l["mixer"]["heads"] * l["mixer"]["dim"] * l["mixer"]["vdim"] for l in cfg["layers"] if l["type"] == "gla")
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


class LatentCase:
    """A pool with one latent layer whose pages the test writes itself."""

    def __init__(self, lens, heads, rank, rot, dtype="bfloat16", seed=0, extra_pages=3):
        import torch

        from dmlx_b200 import device as dev

        rng = np.random.default_rng(seed)
        self.torch, self.dev, self.heads, self.rank, self.rot, self.lens = torch, dev, heads, rank, rot, lens
        self.type = torch.float32 if dtype == "float32" else torch.bfloat16
        pages = sum((n + 31) // 32 for n in lens) + extra_pages
        per = max((n + 31) // 32 for n in lens)
        self.kv = dev.LayeredKVCache([(1, rank + rot, rank, 1, 0)], pages, len(lens), per, heads, max_rows=2048,
                                     kv_dtype=dev.KV_F32 if dtype == "float32" else dev.KV_BF16)
        self.kv.set_free_order(rng.permutation(pages).tolist())
        self.keys = [_bf16(rng.normal(size=(n, rank + rot))) for n in lens]
        self.tables = [self.kv.alloc(i, (n + 31) // 32) for i, n in enumerate(lens)]

    def write(self):
        (_, _, kd), vshape = self.kv.page_shapes(0)
        for keys, table in zip(self.keys, self.tables):
            for p, page in enumerate(table):
                block = np.zeros((1, 32, kd), np.float32)
                part = keys[p * 32:(p + 1) * 32]
                block[0, :len(part), :part.shape[1]] = part
                raw = block if self.type == self.torch.float32 else (block.view(np.uint32) >> 16).astype(np.uint16)
                self.kv.page_load(0, page, raw, np.zeros(vshape, raw.dtype), None, None)

    def run(self, rows, q, scale, sink=None, mma=True):
        """rows [(sequence, position)], q [T, heads, rank + rot]."""
        t = self.torch
        kd = self.kv.page_shapes(0)[0][2]
        qd = t.zeros((len(rows), self.heads, kd), dtype=self.type, device="cuda")
        qd[:, :, :q.shape[2]] = t.tensor(q, dtype=self.type)
        i32 = lambda a: t.tensor(np.asarray(a), dtype=t.int32, device="cuda")
        out = self.kv.window_attention(0, qd, i32([s for s, _ in rows]), i32([p + 1 for _, p in rows]), scale, sinks=sink, mma=mma)
        return out.float().cpu().numpy()

    def want(self, rows, q, scale, sink=None):
        out = np.zeros((len(rows), self.heads, self.rank))
        for r, (s, p) in enumerate(rows):
            keys = self.keys[s][:p + 1]
            sc = q[r] @ keys.T * scale
            out[r] = R.sink_softmax(sc, None if sink is None else sink[:, None]) @ keys[:, :self.rank]
        return out


SHAPES = [(6, 96, 32), (16, 64, 16), (20, 208, 48), (5, 50, 6), (33, 288, 64), (128, 512, 64), (1, 16, 0)]


@pytest.mark.parametrize("mma", [True, False])
@pytest.mark.parametrize("heads,rank,rot", SHAPES)
def test_latent_attention_of_prompts_and_decoding(heads, rank, rot, mma):
    case = LatentCase([300, 70, 1, 33, 256], heads, rank, rot)
    case.write()
    rng = np.random.default_rng(4)
    rows = [(0, p) for p in range(200, 213)] + [(1, 69)] + [(2, 0)] + [(3, p) for p in range(33)] + [(4, 255)] + [(0, 299)]
    q = _bf16(rng.normal(size=(len(rows), heads, rank + rot)))
    sink = 2.0 + rng.normal(size=heads)
    scale = 2.0 * (rank + rot) ** -0.5
    for s in (None, sink):
        want = case.want(rows, q, scale, s)
        assert _error(case.run(rows, q, scale, s, mma), want) <= 4 * _error(_bf16(want), want)


def test_latent_attention_f32():
    case = LatentCase([130, 40], 7, 72, 10, "float32")
    case.write()
    rng = np.random.default_rng(4)
    rows = [(0, p) for p in range(100, 130)] + [(1, 39)]
    q = _bf16(rng.normal(size=(len(rows), 7, 82)))
    want = case.want(rows, q, 0.2, np.ones(7))
    assert _error(case.run(rows, q, 0.2, np.ones(7)), want) <= 1e-5


@pytest.mark.parametrize("mma", [True, False])
def test_latent_attention_finds_a_far_key_at_every_border(mma):
    """One key stands out, at page and tile borders, the first token and the query's own place; one position later it is unseen."""
    heads, rank, rot, n = 4, 64, 32, 700
    places = [0, 1, 31, 32, 63, 64, 127, 128, 255, 256, 511, 512, 698, 699]
    for at in places:
        case = LatentCase([n], heads, rank, rot, seed=at)
        case.keys[0] *= 0.1
        case.keys[0][at, :] = 0
        case.keys[0][at, rank:] = 4.0
        case.keys[0][at, :8] = 3.0
        case.keys[0] = _bf16(case.keys[0])
        case.write()
        q = np.zeros((3, heads, rank + rot))
        q[:, :, rank:] = 1.0
        rows = [(0, max(at - 1, 0)), (0, at), (0, n - 1)]
        got = case.run(rows, _bf16(q), 1.0, np.zeros(heads), mma)
        if at > 0:
            assert np.abs(got[0, :, :8]).max() < 1.0, at
        assert np.abs(got[1:, :, :8] - 3.0).max() < 0.05, at


def test_latent_attention_sink_counts_once_however_the_keys_are_cut():
    from dmlx_b200 import device as dev

    case = LatentCase([900], 3, 64, 16)
    case.keys[0][:] = 0
    case.keys[0][:, 0] = 1.0
    case.write()
    q = np.zeros((1, 3, 80))
    sink = np.log(np.array([900.0, 300.0, 0.001]))
    try:
        for pages in (0, 1, 2, 4, 7, 64):
            dev.set_attn_pages_per_chunk(pages)
            got = case.run([(0, 899)], q, 1.0, sink)[0, :, 0]
            np.testing.assert_allclose(got, 900 / (900 + np.exp(sink)), rtol=6e-3)
    finally:
        dev.set_attn_pages_per_chunk(0)


@pytest.mark.parametrize("heads,rank,rot", [(12, 80, 16), (40, 144, 32)])
def test_latent_attention_of_many_unequal_contexts(heads, rank, rot):
    """A decode step whose contexts differ a hundredfold: long ones are cut between workers, short ones share one."""
    rng = np.random.default_rng(8)
    lens = [2900, 1700, 5, 64, 1, 333, 32, 33, 1200] + rng.integers(1, 120, 21).tolist()
    case = LatentCase(lens, heads, rank, rot)
    case.write()
    rows = [(s, n - 1) for s, n in enumerate(lens)]
    q = _bf16(rng.normal(size=(len(rows), heads, rank + rot)))
    sink = rng.normal(size=heads)
    want = case.want(rows, q, 0.15, sink)
    assert _error(case.run(rows, q, 0.15, sink), want) <= 4 * _error(_bf16(want), want)


@pytest.mark.parametrize("mma", [True, False])
def test_latent_attention_of_scores_that_keep_growing(mma):
    """Every page's scores exceed all before by more than the scale of a running sum tolerates, and then fall again."""
    heads, rank, rot, n = 10, 96, 32, 640
    case = LatentCase([n], heads, rank, rot)
    level = np.concatenate([np.linspace(0, 80, 400), np.linspace(80, 20, 240)])
    case.keys[0] *= 0.2
    case.keys[0][:, rank] = level / 4
    case.keys[0] = _bf16(case.keys[0])
    case.write()
    rng = np.random.default_rng(2)
    q = _bf16(0.3 * rng.normal(size=(4, heads, rank + rot)))
    q[:, :, rank] = 4.0
    rows = [(0, 150), (0, 399), (0, 500), (0, 639)]
    want = case.want(rows, q, 1.0, np.zeros(heads))
    got = case.run(rows, q, 1.0, np.zeros(heads), mma)
    assert np.isfinite(got).all()
    assert _error(got, want) <= 4 * _error(_bf16(want), want)


# ---- programs ------------------------------------------------------------------------------------------------------------
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
