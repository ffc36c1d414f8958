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
    for back in range(taps.shape[1]):
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
