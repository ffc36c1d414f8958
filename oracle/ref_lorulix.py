"""Plain numpy restatement of the Lorulix design: one function per mechanism, every request on its own, no cache, no
batching, token after token where the design recurs; f64 unless a rounding hook is given.

Configurations are the dictionaries that a model folder's config.json holds; weights are name -> array.  `rnd` is applied
wherever a 16-bit implementation may round (matmul operands and results, convolved inputs, cached keys and values); the default
keeps full precision.  `without` names mechanisms that are left out on purpose (tests show that each of them matters).
"""
from __future__ import annotations

import math

import numpy as np

from .ref_decoder import ident, linear, root_mean_square_norm, window_mask

NOTHING = frozenset()


# ---- mechanisms --------------------------------------------------------------------------------------
def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def causal_convolution(u, taps):
    """u [T, C], taps [C, K], the last one the current token's; zeros before the first token."""
    y = np.zeros_like(u)
    for back in range(min(taps.shape[1], u.shape[0])):
        y[back:] += taps[:, -1 - back] * u[:u.shape[0] - back]
    return y


def input_convolution(h, taps):
    return h + causal_convolution(h, taps)


def distance_bucket(distance, buckets, reach):
    """Row of the distance table: one each for the near half, the far half spaced by the logarithm up to `reach`."""
    near = buckets // 2
    if distance < near:
        return distance
    return min(buckets - 1, near + math.floor(math.log(distance / near) / math.log(reach / near) * (buckets - near)))


def query_temperature(position, coef, every):
    return 1.0 + coef * math.log((position + 1) // every + 1)


def attend(q, k, v, scale, table, reach):
    """q [T, H, D], k [T, G, D], v [T, G, E], table [B, H] (or none) -> [T, H, E], causal."""
    t, h, _ = q.shape
    per = h // k.shape[1]
    seen = window_mask(t, t, 0)
    if table is not None:
        bucket = np.array([distance_bucket(n, table.shape[0], reach) for n in range(t)])
        row = bucket[np.maximum(np.arange(t)[:, None] - np.arange(t)[None, :], 0)]
    out = np.zeros((t, h, v.shape[2]), q.dtype)
    for head in range(h):
        s = q[:, head] @ k[:, head // per].T * scale
        if table is not None:
            s = s + table[row, head]
        s = np.where(seen, s, -np.inf)
        e = np.exp(s - s.max(-1, keepdims=True))
        out[:, head] = e / e.sum(-1, keepdims=True) @ v[:, head // per]
    return out


def unit_vectors(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, beta, log_decay, without=NOTHING):
    """q, k [T, H, D], v [T, H, E], beta and log_decay [T, H] -> [T, H, E], token after token."""
    t, h, d = q.shape
    s = np.zeros((h, d, v.shape[2]), q.dtype)
    out = np.zeros((t, h, v.shape[2]), q.dtype)
    for i in range(t):
        if "decay" not in without:
            s = np.exp(log_decay[i])[:, None, None] * s
        held = np.einsum("hde,hd->he", s, k[i])
        u = beta[i][:, None] * (v[i] if "delta" in without else v[i] - held)
        s = s + k[i][:, :, None] * u[:, None, :]
        out[i] = np.einsum("hde,hd->he", s, q[i])
    return out


def clamped_gate(gate, up, limit):
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def choose_experts(z, router, without=NOTHING):
    """Router logits of one token -> (experts, weights)."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    chosen = np.argsort(-s, kind="stable")[:router["top"]]
    return chosen, s[chosen] * (1.0 if "router_scale" in without else router["scale"])


# ---- sublayers ---------------------------------------------------------------------------------------
def delta_mixer(h, w, name, m, eps, shared, rnd=ident, without=NOTHING):
    heads, kv, d, e, t = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    get = lambda n: w[f"{name}.mix.{n}"]

    def part(n):
        u = rnd(linear(h, get(n)))
        if "short_conv" not in without:
            u = causal_convolution(u, get(n + ".conv"))
        return u if "conv_silu" in without else silu(u)

    q, k, v = part("q").reshape(t, kv, d), part("k").reshape(t, kv, d), part("v").reshape(t, heads, e)
    if "unit_norm" not in without:
        q, k = unit_vectors(q), unit_vectors(k)
    q, k = (np.repeat(x, heads // kv, axis=1) for x in (q * d ** -0.5, k))
    beta = np.ones((t, heads)) if "beta" in without else sigmoid(linear(h, get("b")))
    log_decay = -np.exp(get("A_log")) * softplus(linear(h, get("a")) + (0.0 if "dt_bias" in without else get("dt_bias")))
    o = root_mean_square_norm(delta_rule(q, k, v, beta, log_decay, without), eps)
    if "head_norm" not in without:
        o = o * get("norm")
    o = o.reshape(t, heads * e)
    if "out_gate" not in without:
        o = o * silu(rnd(linear(h, get("g"))))
    return rnd(linear(rnd(o), get("o")))


def attention_mixer(h, w, name, m, eps, shared, rnd=ident, without=NOTHING):
    """`shared`: layer -> its (keys, values), filled as the layers run."""
    heads, kv, d, e, t = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]
    get = lambda n: w[f"{name}.mix.{n}"]
    whole = lambda n: (lambda x: x) if "qk_norm" in without else (lambda x: root_mean_square_norm(x, eps, get(n + ".norm")))
    layer = int(name[1:])
    if m.get("kv_from") is None:
        shared[layer] = (rnd(whole("k")(rnd(linear(h, get("k"))))).reshape(t, kv, d), rnd(linear(h, get("v"))).reshape(t, kv, e))
    k, v = shared[layer if m.get("kv_from") is None else m["kv_from"]]
    q = whole("q")(rnd(linear(h, get("q"))))
    if m.get("q_temp") and "q_temp" not in without:
        q = q * np.array([query_temperature(p, m["q_temp"]["coef"], m["q_temp"]["every"]) for p in range(t)])[:, None]
    y = attend(rnd(q).reshape(t, heads, d), k, v, m["scale"], None if "distance" in without else get("rel"), m["bias_max"])
    return rnd(linear(rnd(y.reshape(t, heads * e)), get("o")))


MIXERS = {"delta": delta_mixer, "attention": attention_mixer}


def squared_relu_layers(h, w, name, rnd=ident):
    a = np.maximum(linear(h, w[f"{name}.up"]), 0.0)
    return rnd(linear(rnd(a * a), w[f"{name}.down"]))


def feed_forward(h, w, name, mlp, rnd=ident, without=NOTHING):
    n = f"{name}.mlp"
    if mlp["kind"] == "dense":
        limit = np.inf if "limit" in without else mlp["limit"]
        a = clamped_gate(linear(h, w[n + ".gate"]), linear(h, w[n + ".up"]), limit)
        return rnd(linear(rnd(a), w[n + ".down"]))
    z = linear(h, w[n + ".router"])
    y = np.zeros_like(h)
    for i in range(h.shape[0]):
        for e, weight in zip(*choose_experts(z[i], mlp["router"], without)):
            y[i] += weight * squared_relu_layers(h[i:i + 1], w, f"{n}.e{e}", rnd)[0]
    if mlp.get("shared") and "shared" not in without:
        part = squared_relu_layers(h, w, n + ".shared", rnd)
        y = y + (part if "shared_gate" in without else part * sigmoid(linear(h, w[n + ".shared.sg"])))
    return y


def sublayer(x, w, name, which, eps, f, rnd=ident, without=NOTHING):
    """x + norm(f(h + conv(h)) * sigmoid(W h + b)), h = norm(x)."""
    norm = lambda y, n: root_mean_square_norm(y, eps, (0.0 if "unit_offset" in without else 1.0) + w[f"{name}.{n}"])
    h = rnd(norm(x, f"norm{which}"))
    y = f(h if f"canon{which}" in without else rnd(input_convolution(h, w[f"{name}.canon{which}"])))
    if f"gate{which}" not in without:
        y = y * sigmoid(rnd(linear(h, w[f"{name}.rg{which}"])) + w[f"{name}.rg{which}.b"])
    return x + (y if "post_norm" in without else norm(y, f"norm{which}b"))


def forward(tokens, w, cfg, rnd=ident, want_layers=False, without=NOTHING):
    """Logits [T, vocab] of one sequence (and the residual after every layer)."""
    eps, tokens, shared, trail = cfg["norm"]["eps"], np.asarray(tokens), {}, []
    x = w["embed"][tokens]
    if "positions" not in without:
        x = x + w["pos"][:len(tokens)]
    for i, spec in enumerate(cfg["layers"]):
        n = f"l{i}"
        x = sublayer(x, w, n, 1, eps, lambda h: MIXERS[spec["type"]](h, w, n, spec["mixer"], eps, shared, rnd, without), rnd, without)
        if spec.get("mlp"):
            x = sublayer(x, w, n, 2, eps, lambda h: feed_forward(h, w, n, spec["mlp"], rnd, without), rnd, without)
        trail.append(x)
    one = 0.0 if "unit_offset" in without else 1.0
    logits = linear(rnd(root_mean_square_norm(x, eps, one + w["final.norm"])), w["head"])
    return (logits, np.stack(trail)) if want_layers else logits


# ---- test models -------------------------------------------------------------------------------------
def tensor_shapes(cfg, buckets=8):
    """name -> shape of every tensor a configuration asks for; `buckets`: rows of the distance tables, one number or a function of the layer."""
    d = cfg["width"]
    out = {"embed": (cfg["vocab"], d), "pos": (cfg["max_positions"], d), "final.norm": (d,), "head": (cfg["vocab"], d)}
    for i, spec in enumerate(cfg["layers"]):
        n, m, mlp = f"l{i}", spec["mixer"], spec.get("mlp")
        mix = f"{n}.mix."
        for s in "12" if mlp else "1":
            out[f"{n}.norm{s}"], out[f"{n}.norm{s}b"], out[f"{n}.canon{s}"] = (d,), (d,), (d, cfg["canon"]["taps"])
            out[f"{n}.rg{s}"], out[f"{n}.rg{s}.b"] = (d, d), (d,)
        if spec["type"] == "delta":
            for p, rows in (("q", m["kv_heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["heads"] * m["vdim"])):
                out[mix + p], out[f"{mix}{p}.conv"] = (rows, d), (rows, m["conv"])
            out[mix + "b"], out[mix + "a"], out[mix + "g"] = (m["heads"], d), (m["heads"], d), (m["heads"] * m["vdim"], d)
            out[mix + "A_log"], out[mix + "dt_bias"], out[mix + "norm"] = (m["heads"],), (m["heads"],), (m["vdim"],)
        else:
            h, g = m["heads"], m["kv_heads"]
            out[mix + "q"], out[mix + "q.norm"] = (h * m["dim"], d), (h * m["dim"],)
            out[mix + "rel"] = (buckets(i) if callable(buckets) else buckets, h)
            if m.get("kv_from") is None:
                out[mix + "k"], out[mix + "k.norm"], out[mix + "v"] = (g * m["dim"], d), (g * m["dim"],), (g * m["vdim"], d)
        out[mix + "o"] = (d, m["heads"] * m["vdim"])
        if not mlp:
            continue
        if mlp["kind"] == "dense":
            out[f"{n}.mlp.gate"], out[f"{n}.mlp.up"], out[f"{n}.mlp.down"] = (mlp["ff"], d), (mlp["ff"], d), (d, mlp["ff"])
            continue
        parts = [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
        out[f"{n}.mlp.router"] = (mlp["router"]["experts"], d)
        if mlp.get("shared"):
            parts.append(("shared.", mlp["shared"]["ff"]))
            out[f"{n}.mlp.shared.sg"] = (1, d)
        for p, f in parts:
            out[f"{n}.mlp.{p}up"], out[f"{n}.mlp.{p}down"] = (f, d), (d, f)
    return out


def random_weights(cfg, seed, decisive=True, buckets=8):
    """Weights as bf16 can hold them: projections keep unit variance, norm weights scatter, states remember some tens of tokens.

    `decisive`: every token id ranks the experts of a layer by levels in a few coordinates of its own, which the sublayers hardly touch,
    so that 16-bit rounding cannot swap two experts."""
    from .ref_math import bf16_round

    rng = np.random.default_rng(seed)
    most = max([s["mlp"]["router"]["experts"] for s in cfg["layers"] if s.get("mlp") and s["mlp"]["kind"] == "moe"], default=0) if decisive else 0
    out = {}
    for name, shape in tensor_shapes(cfg, buckets).items():
        part = name.split(".")[-1]
        if part in ("norm1", "norm2", "norm1b", "norm2b") or name == "final.norm":
            a = 0.3 * rng.normal(size=shape)
            a[:most] = 0.0
        elif part == "norm":
            a = 1.0 + 0.3 * rng.normal(size=shape)
        elif part in ("canon1", "canon2"):
            a = 0.5 * rng.normal(size=shape)
            a[:most] = 0.0
        elif name.endswith(("rg1.b", "rg2.b")):
            a = rng.normal(size=shape)
        elif part == "A_log":
            a = -1.5 + rng.normal(size=shape)
        elif part == "dt_bias":
            a = -1.0 + rng.normal(size=shape)
        elif part == "rel":
            a = 1.5 * rng.normal(size=shape)
        elif part == "pos":
            a = 0.7 * rng.normal(size=shape)
            a[:, :most] = 0.0
        elif part == "embed":
            a = rng.normal(size=shape)
            if most:
                a[:, :most] = np.stack([rng.permutation(np.linspace(-1.8, 1.8, most)) for _ in range(shape[0])])
        elif part == "router" and most:
            a = np.zeros(shape)
            a[np.arange(shape[0]), rng.permutation(most)[:shape[0]]] = 1.5
        elif part in ("a", "b", "sg"):
            a = 2.0 * rng.normal(size=shape) / np.sqrt(shape[1])
        else:
            a = rng.normal(size=shape) / np.sqrt(shape[-1])
            if part in ("o", "down") and most:
                a[:most] *= 0.03
        out[name] = bf16_round(np.asarray(a, np.float32)).astype(np.float64)
    return out


def write_model(folder, cfg, weights):
    from .ref_sotavik import write_model as write

    write(folder, cfg, weights)
