"""The decoder stack as a served model, against the oracle: each mechanism alone, the whole stack, and what must not depend
on how tokens reach it (portions, batches, pages and slots used again, graphs)."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

from oracle import ref_decoder as R
from oracle.ref_math import bf16_round
from tests.decoder_cases import CASES, attention, config

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
F32_TOL = 2e-5  # relative to the root mean square of what is compared


def _load(tmp_path, cfg, seed, dtype, max_rows=512, slots=4):
    from dmlx_b200.models import Limits, load_model

    w = R.random_weights(cfg, seed)
    R.write_model(str(tmp_path), cfg, w)
    return load_model(str(tmp_path), dtype, Limits(max_rows, slots, slots)), w


def _error(got, want):
    return np.sqrt(((got - want) ** 2).mean(-1).max() / (want ** 2).mean())


def _bf16(a):
    return bf16_round(a.astype(np.float32)).astype(np.float64)


def _tol(dtype, w, cfg, tokens, **kw):
    """What rounding alone may cause: in bfloat16 three times the error the oracle makes on these tokens when it rounds every
    matrix operand and result to bf16 (deep loops and narrow heads amplify it, so it differs from model to model)."""
    if dtype == "float32":
        return F32_TOL
    return 3 * _error(R.forward(tokens, w, cfg, _bf16, **kw), R.forward(tokens, w, cfg, **kw))


def _tokens(cfg, n, seed):
    return np.random.default_rng(seed).integers(0, cfg["vocab"], n).tolist()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
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
        assert _error(layers[i], trail[i]) <= tol, (name, "layer run", i)
    assert _error(got, want) <= _tol(dtype, w, cfg, toks), name


MECHANISMS = {"bias": "DEC_QKV_BIAS", "qk_norm": "DEC_QK_NORM", "distance": "DEC_DISTANCE_BIAS", "sink": "DEC_SINK",
              "post_norm": "DEC_POST_NORM"}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("has", [(), *[(m,) for m in MECHANISMS]], ids=str)
def test_each_mechanism_alone(has, dtype):
    """Layers with none or one of the mechanisms; leaving it out of the oracle must show."""
    from dmlx_b200 import device as dev
    from dmlx_b200.models import tafuvik

    cfg = config(96, 160, [attention(6, 3, 40, 24, 25, 1.0 if "qk_norm" in has else 0.3, ff=80)] * 2, embed_scale=2.0)
    w = R.random_weights(cfg, 21)
    specs = [dict(s, flags=sum(getattr(dev, MECHANISMS[m]) for m in has)) for s in tafuvik.layer_specs(cfg)]
    model = dev.DecoderModel(96, 160, specs, cfg["norm"]["eps"], 2.0, None, dev.DT_F32 if dtype == "float32" else dev.DT_BF16, 128, 2, 2)
    skip = {n for n, m in (("sink", "sink"), ("q_bias", "bias"), ("k_bias", "bias"), ("v_bias", "bias"), ("postnorm1", "post_norm"),
                           ("postnorm2", "post_norm")) if m not in has}
    bits = lambda a: (a.astype(np.float32).view(np.uint32) >> 16).astype(np.uint16)
    for layer, which, name in tafuvik.tensor_names(cfg):
        if which not in skip:
            model.set_tensor(layer, which, bits(w[name]))
    model.finalize()
    kv = model.make_cache(8, 2, 8)
    toks = _tokens(cfg, 70, 9)
    model.step(kv, [(0, 70, 0, 0)], toks, list(range(70)))
    got = model.logits(1, 70)
    tol = _tol(dtype, w, cfg, toks, has=set(has))
    assert _error(got, R.forward(toks, w, cfg, has=set(has))) <= tol
    if has:
        assert _error(got, R.forward(toks, w, cfg, has=set())) > 2 * tol


def test_missing_or_wrong_tensors_are_named():
    from dmlx_b200 import _lib
    from dmlx_b200 import device as dev
    from dmlx_b200.models import tafuvik

    cfg = CASES["no_loop"]
    w = R.random_weights(cfg, 1)
    bits = lambda a: (a.astype(np.float32).view(np.uint32) >> 16).astype(np.uint16)
    drop = {"l1.mix.sink": "sink", "l0.norm2b": "post-norm 2", "head": "head"}
    for gone, text in drop.items():
        with pytest.raises(_lib.B200Error, match=text):
            model = dev.DecoderModel(cfg["width"], cfg["vocab"], tafuvik.layer_specs(cfg), 1e-5, max_rows=64, max_reqs=1, max_seqs=1)
            for layer, which, name in tafuvik.tensor_names(cfg):
                if name != gone:
                    model.set_tensor(layer, which, bits(w[name]))
            model.finalize()
    with pytest.raises(_lib.B200Error, match="elements"):
        model.set_tensor(0, "q", np.zeros(7, np.uint16))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", CASES)
def test_portions_decoding_batches_and_reused_pages(tmp_path, name, dtype):
    """Requests cut into portions of every size down to single tokens, in batches with others, on pages and slots that earlier
    requests gave back: every logit equals the whole prompt's."""
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
            n = min(int(rng.choice([1, 1, 1, 2, 2, 3, 7, 16, 31, 33, 64])), len(prompts[i]) - at)
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


@pytest.mark.parametrize("portion", [2, 5, 32, 50])
def test_portions_of_one_size_against_token_by_token(tmp_path, portion):
    from dmlx_b200.serving import TokenFeeder

    cfg = CASES["middle_loop"]
    loaded, w = _load(tmp_path, cfg, 41, "float32")
    toks = _tokens(cfg, 110, 6)
    feeder = TokenFeeder(loaded, 8)
    cut = [feeder.step([("a", toks[i:i + portion], range(len(toks[i:i + portion])))]) for i in range(0, 110, portion)]
    single = [feeder.step([("b", [t], [0])]) for t in toks]
    np.testing.assert_allclose(np.concatenate(cut), np.concatenate(single), atol=2e-4, rtol=0)
    assert _error(np.concatenate(single), R.forward(toks, w, cfg)) <= F32_TOL


def test_long_decoding_far_behind_the_window(tmp_path):
    """700 decoded tokens: the window slides over pages written by decoding, graphs replay, logits stay the oracle's."""
    from dmlx_b200.serving import TokenFeeder

    import torch

    cfg = CASES["whole_loop"]
    loaded, w = _load(tmp_path, cfg, 51, "bfloat16")
    toks = _tokens(cfg, 720, 7)
    want = R.forward(toks, w, cfg)
    feeder = TokenFeeder(loaded, 24)
    with torch.cuda.stream(torch.cuda.Stream()):
        feeder.step([("a", toks[:20], [])])
        got = np.concatenate([feeder.step([("a", [t], [0])]) for t in toks[20:]])
    assert _error(got, want[20:]) <= _tol("bfloat16", w, cfg, toks)


def test_replayed_graphs_equal_eager_steps(tmp_path):
    from dmlx_b200.serving import TokenFeeder

    import torch

    cfg = CASES["wide_head"]
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


def test_tensor_core_and_cuda_core_attention_agree_in_the_stack(tmp_path):
    from dmlx_b200.serving import TokenFeeder

    cfg = CASES["middle_loop"]
    loaded, _ = _load(tmp_path, cfg, 71, "bfloat16")
    toks = _tokens(cfg, 140, 3)
    out = []
    for mma in (True, False):
        loaded.model.set_attn_mma(mma)
        feeder = TokenFeeder(loaded, 8)
        out.append(np.concatenate([feeder.step([("a", toks[:100], range(100))])] + [feeder.step([("a", [t], [0])]) for t in toks[100:]]))
    assert _error(out[0], out[1]) <= 2e-2


def _greedy(w, cfg, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(R.forward(toks, w, cfg)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("name", ["middle_loop", "odd_sizes", "no_loop"])
def test_greedy_generation_through_the_engine(tmp_path, name):
    """More prompts than slots, chunked prefill beside decoding: the tokens are those of each prompt alone."""
    from dmlx_b200.serving import generate

    cfg = CASES[name]
    loaded, w = _load(tmp_path, cfg, 81, "float32", max_rows=96)
    prompts = [_tokens(cfg, n, 200 + n) for n in (40, 1, 75, 9, 33, 64)]
    got = generate(loaded, prompts, 14, prefill_chunk=23)
    for p, g in zip(prompts, got):
        assert g == _greedy(w, cfg, p, 14)


def test_generation_under_page_pressure_and_with_shared_prefixes(tmp_path):
    """A pool too small for all requests (deferral, preemption by recomputation), and requests that take over a live request's
    prompt pages: same tokens."""
    from dmlx_b200.serving import generate

    cfg = CASES["middle_loop"]
    loaded, w = _load(tmp_path, cfg, 91, "float32", max_rows=256)
    head = _tokens(cfg, 70, 1)
    prompts = [head + _tokens(cfg, n, 300 + n) for n in (5, 9, 2, 30)]
    want = [_greedy(w, cfg, p, 40) for p in prompts]
    assert generate(loaded, prompts, 40, prefill_chunk=32, n_pages=7) == want
    assert generate(loaded, prompts, 40, prefill_chunk=32, prefix_sharing=True) == want


def test_stop_tokens_and_sampling(tmp_path):
    from dmlx_b200.serving import generate

    cfg = CASES["no_loop"]
    loaded, w = _load(tmp_path, cfg, 95, "bfloat16")
    prompt = _tokens(cfg, 12, 4)
    plain = generate(loaded, [prompt], 20)[0]
    cut = generate(loaded, [prompt], 20, stop_tokens=[plain[6]])[0]
    assert cut == plain[:plain.index(plain[6]) + 1]
    a = generate(loaded, [prompt], 20, temperature=1.0, top_k=20, seed=5)[0]
    assert a == generate(loaded, [prompt], 20, temperature=1.0, top_k=20, seed=5)[0]
    assert a != plain
    assert generate(loaded, [prompt], 20, temperature=1.0, top_k=1, seed=9)[0] == plain
    with pytest.raises(ValueError):
        generate(loaded, [[cfg["vocab"]]], 1)


def test_prefix_pages_saved_and_restored(tmp_path):
    """Pages of a layered pool through the on-disk prefix store: a restored slot continues with the same logits."""
    from dmlx_b200.prefix_store import PrefixDiskStore

    cfg = CASES["wide_head"]
    loaded, _ = _load(tmp_path / "m", cfg, 96, "bfloat16")
    toks = _tokens(cfg, 100, 8)
    kv = loaded.new_cache(8, 4)
    loaded.model.step(kv, [(0, 96, 0, 0)], toks[:96])
    store = PrefixDiskStore(str(tmp_path / "pages"))
    assert store.save_prefix(kv, 0, toks[:96]) == 3
    fresh = loaded.new_cache(8, 4)
    fresh.set_free_order([5, 2, 7, 0, 1, 3, 4, 6])
    n = store.restore_prefix(fresh, 0, toks[:97])
    assert n == 96
    out = []
    for pool in (kv, fresh):
        loaded.model.step(pool, [(0, 4, 96, 0)], toks[96:], [0, 1, 2, 3])
        out.append(loaded.model.logits(1, 4))
    np.testing.assert_array_equal(out[0], out[1])


def _run_replay(folder, out, steps, max_tokens, dtype):
    env = dict(os.environ, PYTHONPATH="")
    return subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(folder), "--dtype", dtype, "--out", str(out), "--max-tokens",
                           str(max_tokens)], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, env=env, timeout=280)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_replay_program(tmp_path, dtype):
    cfg = CASES["whole_loop"]
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
    r = _run_replay(tmp_path / "m", out, steps, 192, dtype)
    assert r.returncode == 0, r.stderr
    assert [l for l in r.stdout.split("\n") if l.startswith("done")] == [f"done {i}" for i in range(5)]
    assert sorted(os.listdir(out)) == ["0.f32", "2.f32", "3.f32", "4.f32"]
    fa, fc = R.forward(a, w, cfg), R.forward(c, w, cfg)
    want = {0: fa[[49, 3]], 2: np.stack([fc[32], fa[51], fa[52]]), 3: fa[[69]], 4: fc[[33, 89]]}
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
