"""Attention over layered pools, and the q/k/v step in front of it, against the oracle: windows, distance bias, sinks,
GQA groups and widths of every kind, on both kernels, in prompts and in decoding.

Faults of a window's edge are made visible by planting: one value row is large and its key fits the query, so a
key that is wrongly seen or wrongly left out moves the output by far more than rounding."""
import numpy as np
import pytest

from oracle import ref_decoder as R
from oracle.ref_math import bf16_round

pytestmark = pytest.mark.gpu

# (query heads, kv heads, key width, value width)
SHAPES = [(4, 2, 80, 48), (6, 2, 64, 128), (5, 1, 128, 64), (4, 4, 24, 40), (16, 2, 200, 136), (20, 1, 16, 72), (3, 1, 33, 17), (2, 1, 272, 40),
          (8, 1, 144, 256)]
WINDOWS = [0, 1, 31, 33, 100]


def _r(a):
    return bf16_round(np.asarray(a, np.float32)).astype(np.float64)


class Pool:
    """One layer, filled through the q/k/v step with given rows (no norm, no bias)."""

    def __init__(self, shape, lens, f32, order_seed=0, n_layers=1):
        import torch

        from dmlx_b200 import device as dev

        self.dev, self.torch = dev, torch
        self.hq, self.g, self.kd, self.vd = shape
        pages = sum((n + 31) // 32 for n in lens) + 3
        self.kv = dev.LayeredKVCache([(self.g, self.kd, self.vd)] * n_layers, pages, len(lens), pages, self.hq, max_rows=2048,
                                     kv_dtype=dev.KV_F32 if f32 else dev.KV_BF16)
        self.kv.set_free_order(np.random.default_rng(order_seed).permutation(pages).tolist())
        self.dtype = torch.float32 if f32 else torch.bfloat16
        self.f32 = f32

    def rows(self, a):
        return self.torch.tensor(np.asarray(a), device="cuda").to(self.dtype)

    def append(self, batch, q, k, v, layer=0, **kw):
        """batch: [(slot, base, count)]; q, k, v: rows of the whole batch.  Returns (q for attention, row_seq, row_ctx)."""
        t = self.torch
        self.kv.reserve(self.dev.pack_desc_array([(s, c, b, 0) for s, b, c in batch]).cuda())
        pos = t.tensor([b + i for _, b, c in batch for i in range(c)], dtype=t.int32, device="cuda")
        seq = t.tensor([s for s, _, c in batch for _ in range(c)], dtype=t.int32, device="cuda")
        rows = np.concatenate([q.reshape(len(q), -1), k.reshape(len(k), -1), v.reshape(len(v), -1)], 1)
        qd = self.kv.qkv(layer, self.rows(rows), self.hq, pos, seq, **{"qk_norm": False, **kw})
        return qd, seq, (pos + 1).to(t.int32)


def _random(rng, lens, shape, t=None):
    hq, g, kd, vd = shape
    n = sum(lens)
    return _r(rng.normal(size=(n, hq, kd))), _r(rng.normal(size=(n, g, kd))), _r(rng.normal(size=(n, g, vd)))


def _check(got, want, f32, what):
    tol = 2e-5 if f32 else 6e-3
    err = np.abs(got - want).max() / np.abs(want).max()
    assert err <= tol, (what, err)


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_prompts_and_decoding_of_unequal_requests(shape, f32):
    """A batch of whole prompts, then a batch that mixes a portion with single tokens, every window, both kernels."""
    rng = np.random.default_rng(sum(shape))
    lens = [65, 1, 150, 32]
    hq, g, kd, vd = shape
    slopes, sinks, scale = R.distance_slopes(hq), rng.normal(size=hq), 1.7 * kd ** -0.5
    p = Pool(shape, [n + 40 for n in lens], f32)
    q, k, v = _random(rng, lens, shape)
    qd, seq, ctx = p.append([(i, 0, n) for i, n in enumerate(lens)], q, k, v)
    more = [1, 37, 1, 2]
    q2, k2, v2 = _random(rng, more, shape)
    off = np.cumsum([0] + lens)
    off2 = np.cumsum([0] + more)
    cases = [("prompt", qd, seq, ctx, [(q[off[i]:off[i + 1]], k[off[i]:off[i + 1]], v[off[i]:off[i + 1]]) for i in range(4)])]
    first = {}
    for window in WINDOWS:
        for mma in ((False,) if f32 else (True, False)):
            first[window, mma] = p.kv.window_attention(0, qd, seq, ctx, scale, window, slopes, sinks, mma).double().cpu().numpy()
    qd2, seq2, ctx2 = p.append([(i, lens[i], more[i]) for i in range(4)], q2, k2, v2)
    for (window, mma), got in first.items():
        parts = [R.attend(*cases[0][4][i], scale, window, slopes, sinks) for i in range(4)]
        _check(got, np.concatenate(parts), f32, ("prompt", window, mma))
        got2 = p.kv.window_attention(0, qd2, seq2, ctx2, scale, window, slopes, sinks, mma).double().cpu().numpy()
        parts = []
        for i in range(4):
            kk = np.concatenate([k[off[i]:off[i + 1]], k2[off2[i]:off2[i + 1]]])
            vv = np.concatenate([v[off[i]:off[i + 1]], v2[off2[i]:off2[i + 1]]])
            parts.append(R.attend(q2[off2[i]:off2[i + 1]], kk, vv, scale, window, slopes, sinks))
        _check(got2, np.concatenate(parts), f32, ("portion", window, mma))
    assert p.kv.error_word() == 0


@pytest.mark.parametrize("shape", [(4, 2, 80, 48), (5, 1, 128, 64), (20, 1, 16, 72), (2, 1, 272, 40)], ids=str)
@pytest.mark.parametrize("window", [1, 2, 31, 32, 33, 64, 95])
def test_window_edges_show_a_key_one_token_off(shape, window):
    """The key just inside the window and the key just outside carry a value that stands out; as a prompt portion and as
    single tokens, at positions around page borders."""
    hq, g, kd, vd = shape
    n = 192
    rng = np.random.default_rng(window)
    for at in (window, 96, 127, 128, 129, 191):
        for inside in (True, False):
            j = at - window + 1 if inside else at - window
            if j < 0 or at >= n:
                continue
            q, k, v = _random(rng, [n], shape)
            v = _r(0.01 * v)
            q[:] = 0.5
            k = _r(-0.2 * np.abs(k))
            k[j] = 1.0
            v[j] = 8.0
            p = Pool(shape, [n], False, order_seed=at)
            qd, seq, ctx = p.append([(0, 0, n)], q, k, v)
            want = R.attend(q, k, v, 0.3, window)
            assert (np.abs(want[at]).max() > 1.0) == inside
            for mma in (True, False):
                whole = p.kv.window_attention(0, qd, seq, ctx, 0.3, window, None, None, mma).double().cpu().numpy()
                rows = slice(max(at - 3, 0), at + 1)
                _check(whole[rows], want[rows], False, ("prompt", at, inside, mma))
                one = p.kv.window_attention(0, qd[at:at + 1].contiguous(), seq[at:at + 1].contiguous(), ctx[at:at + 1].contiguous(), 0.3, window,
                                            None, None, mma).double().cpu().numpy()
                _check(one, want[at:at + 1], False, ("decode", at, inside, mma))


@pytest.mark.parametrize("mma", [True, False])
def test_sink_counts_once_whatever_the_number_of_chunks(mma):
    """Equal scores of zero: the weight of every value is 1 / (n + exp(sink)); forced chunk lengths cut the row differently."""
    from dmlx_b200 import device as dev

    shape, n = (6, 3, 48, 16), 700
    hq, g, kd, vd = shape
    p = Pool(shape, [n], False)
    q, k, v = np.zeros((n, hq, kd)), np.zeros((n, g, kd)), np.ones((n, g, vd))
    qd, seq, ctx = p.append([(0, 0, n)], q, k, v)
    sinks = np.log(np.array([1.0, 10.0, 350.0, 700.0, 7000.0, 1e-3]))
    rows = [0, 1, 31, 32, 255, 699]
    try:
        for chunk in (1, 3, 8, 64, 0):
            dev.set_attn_pages_per_chunk(chunk)
            got = p.kv.window_attention(0, qd[rows].contiguous(), seq[rows].contiguous(), ctx[rows].contiguous(), 1.0, 0, None, sinks, mma).double().cpu().numpy()
            want = np.array([[(r + 1) / (r + 1 + np.exp(s)) for s in sinks] for r in rows])
            np.testing.assert_allclose(got, np.broadcast_to(want[..., None], got.shape), rtol=5e-3)
            full = p.kv.window_attention(0, qd, seq, ctx, 1.0, 0, None, sinks, mma).double().cpu().numpy()
            np.testing.assert_allclose(full[rows], np.broadcast_to(want[..., None], got.shape), rtol=5e-3)
    finally:
        dev.set_attn_pages_per_chunk(0)


def test_distance_bias_is_relative_and_joins_before_the_sink():
    """With a sink, slope * (i - j) and slope * j give different weights: only the first matches."""
    shape, n = (4, 1, 32, 32), 90
    rng = np.random.default_rng(8)
    q, k, v = _random(rng, [n], shape)
    slopes, sinks = R.distance_slopes(4), np.full(4, 1.5)
    p = Pool(shape, [n], True)
    qd, seq, ctx = p.append([(0, 0, n)], q, k, v)
    got = p.kv.window_attention(0, qd, seq, ctx, 0.2, 0, slopes, sinks).double().cpu().numpy()
    _check(got, R.attend(q, k, v, 0.2, 0, slopes, sinks), True, "relative")
    assert np.abs(got - R.attend(q, k, v, 0.2, 0, slopes, None)).max() > 1e-2
    assert np.abs(got - R.attend(q, k, v, 0.2, 0, None, sinks)).max() > 1e-2


def test_far_key_among_thousands_long_context_and_full_scratch():
    """One key 2900 tokens back that outweighs everything between; the scratch holds so few partial sums that the
    plan has to lengthen its chunks."""
    from dmlx_b200 import device as dev

    import torch

    shape, n = (4, 2, 64, 64), 3000
    hq, g, kd, vd = shape
    rng = np.random.default_rng(4)
    q, k, v = _random(rng, [n], shape)
    k[99] = _r(3.0 * q[-1, ::2])  # fits head 0 of each group at the last position
    v[99] = 5.0
    pages = 94
    kv = dev.LayeredKVCache([(g, kd, vd)], pages, 1, pages, hq, max_rows=2048, attn_scratch_chunks=70)
    p = Pool.__new__(Pool)
    p.dev, p.torch, p.kv, p.dtype, p.hq = dev, torch, kv, torch.bfloat16, hq
    qs = []
    for b in range(0, n, 1000):
        qd, seq, ctx = p.append([(0, b, 1000)], q[b:b + 1000], k[b:b + 1000], v[b:b + 1000])
    want = R.attend(q[-40:], k, v, 0.125, 0)
    tail = slice(960, 1000)
    assert want[-1, 0].mean() > 3.0
    for rows in (tail, slice(999, 1000)):
        got = kv.window_attention(0, qd[rows].contiguous(), seq[rows].contiguous(), ctx[rows].contiguous(), 0.125, 0).double().cpu().numpy()
        _check(got, want[-len(got):], False, rows)
    assert kv.error_word() == 0


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("shape", SHAPES, ids=str)
def test_qkv_step_norms_biases_and_pages(shape, f32):
    """Biases are added before the norm, q and k have unit root mean square per head, v is left alone, and every row is in its page."""
    import torch

    hq, g, kd, vd = shape
    rng = np.random.default_rng(hq + kd)
    lens = [3, 40, 33]
    q, k, v = _random(rng, lens, shape)
    bias = rng.normal(size=hq * kd + g * (kd + vd)).astype(np.float32)
    p = Pool(shape, lens, f32)
    qd, _, _ = p.append([(i, 0, n) for i, n in enumerate(lens)], q, k, v, bias=torch.tensor(bias, device="cuda"), qk_norm=True, eps=0.3)
    bq, bk, bv = np.split(bias.astype(np.float64), [hq * kd, hq * kd + g * kd])
    tol = dict(rtol=1e-5, atol=1e-6) if f32 else dict(rtol=1e-2, atol=1e-2)
    np.testing.assert_allclose(qd[..., :kd].double().cpu().numpy(), R.root_mean_square_norm(q + bq.reshape(hq, kd), 0.3), **tol)
    assert not qd[..., kd:].any()
    off = 0
    for i, n in enumerate(lens):
        kk, vv = p.kv.gather(0, i)
        np.testing.assert_allclose(kk.double().cpu().numpy(), R.root_mean_square_norm(k[off:off + n] + bk.reshape(g, kd), 0.3), **tol)
        np.testing.assert_allclose(vv.double().cpu().numpy(), v[off:off + n] + bv.reshape(g, vd), **tol)
        off += n


@pytest.mark.parametrize("f32", [False, True])
def test_layered_pool_pages_fork_extend_and_travel(f32):
    """Copy-on-write after a fork, a copy into another pool, and page bytes out and back in, in layers of different shape."""
    import torch

    from dmlx_b200 import device as dev

    layers = [(2, 48, 24), (1, 16, 80)]
    dt = dev.KV_F32 if f32 else dev.KV_BF16
    rng = np.random.default_rng(2)
    kv = dev.LayeredKVCache(layers, 12, 3, 6, 4, max_rows=256, kv_dtype=dt)
    element = torch.float32 if f32 else torch.bfloat16
    held = {0: [], 1: []}

    def feed(slot, base, n):
        kv.reserve(dev.pack_desc_array([(slot, n, base, 0)]).cuda())
        pos = torch.arange(base, base + n, dtype=torch.int32, device="cuda")
        seq = torch.full((n,), slot, dtype=torch.int32, device="cuda")
        out = []
        for l, (g, kd, vd) in enumerate(layers):
            rows = torch.tensor(_r(rng.normal(size=(n, 4 * kd + g * (kd + vd)))), device="cuda").to(element)
            kv.qkv(l, rows, 4, pos, seq, qk_norm=False)
            out.append(rows[:, 4 * kd:].float().cpu().numpy())
        return out

    def view(pool, l, slot):
        k, v = pool.gather(l, slot)
        return np.concatenate([k.float().cpu().numpy().reshape(len(k), -1), v.float().cpu().numpy().reshape(len(v), -1)], 1)

    base = feed(0, 0, 45)
    kv.fork(0, 1, 45)
    a, b = feed(0, 45, 2), feed(1, 45, 3)  # slot 0 writes into the shared page first and gets its own copy
    for l in range(2):
        np.testing.assert_array_equal(view(kv, l, 0), np.concatenate([base[l], a[l]]))
        np.testing.assert_array_equal(view(kv, l, 1), np.concatenate([base[l], b[l]]))
    other = dev.LayeredKVCache(layers, 7, 2, 4, 4, max_rows=64, kv_dtype=dt)
    other.extend(1, kv, 1)
    for l in range(2):
        np.testing.assert_array_equal(view(other, l, 1), view(kv, l, 1))
    pages = other.alloc(0, 2)
    for l in range(2):
        for src, dst in zip(kv.block_table(0), pages):
            k, v, _, _ = kv.page_raw(l, src)
            assert k.shape == other.page_shapes(l)[0] and v.shape == other.page_shapes(l)[1]
            other.page_load(l, dst, k, v)
    other.set_len(0, 47)
    for l in range(2):
        np.testing.assert_array_equal(view(other, l, 0), view(kv, l, 0))
    with pytest.raises(Exception):
        dev.LayeredKVCache([(2, 48, 24), (1, 16, 64)], 7, 2, 4, 4, kv_dtype=dt).extend(0, kv, 0)
