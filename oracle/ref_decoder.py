"""Plain numpy restatement of the configurable decoder stack (the Tafuvik design): one function per
mechanism, every request on its own, no cache, no batching, f64 unless a rounding hook is given.

Configurations are the dictionaries that a model folder's config.json holds; weights are
name -> array.  `rnd` is applied wherever a 16-bit implementation may round (matmul operands and results,
cached keys and values); the default keeps full precision.
"""
from __future__ import annotations

import numpy as np


def ident(a):
    return a


# ---- mechanisms --------------------------------------------------------------------------------------
def root_mean_square_norm(x, eps, weight=None):
    y = x / np.sqrt((x * x).mean(-1, keepdims=True) + eps)
    return y if weight is None else y * weight


def linear(x, weight, bias=None):
    y = x @ weight.T
    return y if bias is None else y + bias


def silu_gated(gate, up):
    return gate / (1.0 + np.exp(-gate)) * up


def distance_slopes(n_heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / n_heads) for h in range(n_heads)])


def window_mask(n_query, n_key, window):
    """[n_query, n_key] booleans; query row r stands at position n_key - n_query + r."""
    i = np.arange(n_key - n_query, n_key)[:, None]
    j = np.arange(n_key)[None, :]
    keep = j <= i
    return keep if not window else keep & (i - j < window)


def sink_softmax(scores, sink):
    """Softmax over the last axis whose denominator also holds exp(sink); scores may be -inf where masked."""
    m = scores.max(-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(scores - m)
    total = e.sum(-1, keepdims=True)
    if sink is not None:
        total = total + np.exp(sink - m)
    return e / total


def attend(q, k, v, scale, window=0, slopes=None, sink=None):
    """q [T, H, D], k [S, G, D], v [S, G, E] (the T queries are the last T positions) -> [T, H, E]."""
    t, h, _ = q.shape
    s, g, _ = k.shape
    mask = window_mask(t, s, window)
    dist = np.arange(s - t, s)[:, None] - np.arange(s)[None, :]
    out = np.zeros((t, h, v.shape[2]), q.dtype)
    for head in range(h):
        kv = head // (h // g)
        sc = (q[:, head] @ k[:, kv].T) * scale
        if slopes is not None:
            sc = sc - slopes[head] * dist
        sc = np.where(mask, sc, -np.inf)
        out[:, head] = sink_softmax(sc, None if sink is None else sink[head]) @ v[:, kv]
    return out


# ---- layers ------------------------------------------------------------------------------------------
ALL = frozenset({"bias", "qk_norm", "distance", "sink", "post_norm"})


def attention_mixer(h, w, name, mixer, eps, rnd=ident, has=ALL):
    hq, g, d, e = mixer["heads"], mixer["kv_heads"], mixer["dim"], mixer["vdim"]
    t = h.shape[0]
    proj = lambda n: linear(h, w[f"{name}.mix.{n}"], w[f"{name}.mix.{n}.b"] if "bias" in has else None)
    unit = (lambda a: root_mean_square_norm(a, eps)) if "qk_norm" in has else ident
    q = unit(proj("q").reshape(t, hq, d))
    k = unit(proj("k").reshape(t, g, d))
    v = proj("v").reshape(t, g, e)
    window = (mixer.get("mask") or {}).get("size", 0)
    y = attend(rnd(q), rnd(k), rnd(v), mixer["scale"], window, distance_slopes(hq) if "distance" in has else None,
               w[f"{name}.mix.sink"] if "sink" in has else None)
    return rnd(linear(rnd(y.reshape(t, hq * e)), w[f"{name}.mix.o"]))


def gated_mlp(h, w, name, rnd=ident):
    a = silu_gated(linear(h, w[f"{name}.mlp.gate"]), linear(h, w[f"{name}.mlp.up"]))
    return rnd(linear(rnd(a), w[f"{name}.mlp.down"]))


def layer(x, w, i, spec, eps, rnd=ident, has=ALL):
    n = f"l{i}"
    post = (lambda y, p: root_mean_square_norm(y, eps, w[f"{n}.{p}"])) if "post_norm" in has else (lambda y, p: y)
    y = attention_mixer(rnd(root_mean_square_norm(x, eps, w[n + ".norm1"])), w, n, spec["mixer"], eps, rnd, has)
    x = x + post(y, "norm1b")
    if spec.get("mlp"):
        y = gated_mlp(rnd(root_mean_square_norm(x, eps, w[n + ".norm2"])), w, n, rnd)
        x = x + post(y, "norm2b")
    return x


def layer_runs(cfg):
    """[(weight layer, opens a pass of the loop)] in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    one = [(i, i == a) for i in range(a, b)]
    return [(i, False) for i in range(a)] + one * loop["times"] + [(i, False) for i in range(b, n)]


def forward(tokens, w, cfg, rnd=ident, dtype=np.float64, want_layers=False, has=ALL):
    """Logits [T, vocab] of one sequence (and the residual after every layer run)."""
    eps = cfg["norm"]["eps"]
    x0 = x = w["embed"][np.asarray(tokens)].astype(dtype) * dtype(cfg["embedding"]["scale"])
    trail = []
    for i, opens in layer_runs(cfg):
        if opens:
            x = linear(np.concatenate([rnd(x), rnd(x0)], -1), w["loop.in"])
        x = layer(x, w, i, cfg["layers"][i], eps, rnd, has)
        trail.append(x)
    logits = linear(rnd(root_mean_square_norm(x, eps, w["final.norm"])), w["head"])
    return (logits, np.stack(trail)) if want_layers else logits


# ---- test models -------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    """name -> shape of every tensor a configuration asks for."""
    d, out = cfg["width"], {}
    out["embed"] = (cfg["vocab"], d)
    if cfg.get("loop"):
        out["loop.in"] = (d, 2 * d)
    for i, spec in enumerate(cfg["layers"]):
        n, m = f"l{i}", spec["mixer"]
        hq, g, kd, vd = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for p, rows in (("q", hq * kd), ("k", g * kd), ("v", g * vd)):
            out[f"{n}.mix.{p}"], out[f"{n}.mix.{p}.b"] = (rows, d), (rows,)
        out[f"{n}.mix.sink"], out[f"{n}.mix.o"] = (hq,), (d, hq * vd)
        names = ["norm1", "norm1b"]
        if spec.get("mlp"):
            f = spec["mlp"]["ff"]
            out[f"{n}.mlp.gate"], out[f"{n}.mlp.up"], out[f"{n}.mlp.down"] = (f, d), (f, d), (d, f)
            names += ["norm2", "norm2b"]
        for p in names:
            out[f"{n}.{p}"] = (d,)
    out["final.norm"], out["head"] = (d,), (cfg["vocab"], d)
    return out


def random_weights(cfg, seed, spread=1.0):
    """Weights as bf16 can hold them: projections keep unit variance (times `spread`), norms scatter around 1, biases and
    sinks are large enough to be missed."""
    from .ref_math import bf16_round

    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        if ".norm" in name or name == "final.norm":
            a = 1.0 + 0.3 * rng.normal(size=shape)
        elif name.endswith(".b"):
            a = 0.5 * rng.normal(size=shape)
        elif name.endswith(".sink"):
            a = 1.0 + rng.normal(size=shape)
        elif name == "embed":
            a = rng.normal(size=shape) / cfg["embedding"]["scale"]
        else:
            a = spread * rng.normal(size=shape) / np.sqrt(shape[1])
        out[name] = bf16_round(a.astype(np.float32)).astype(np.float64)
    return out


def write_model(folder, cfg, weights):
    """A model folder (config.json, model.safetensors) with these weights in bf16."""
    import json
    import os

    from dmlx_b200.safetensors_io import write_safetensors

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    bits = lambda a: (a.astype(np.float32).view(np.uint32) >> 16).astype(np.uint16)
    write_safetensors(os.path.join(folder, "model.safetensors"), {n: ("BF16", bits(a)) for n, a in weights.items()}, {})
