"""Plain numpy restatement of the Dovorax design: one function per mechanism, every request on its own, no cache, no
batching, token after token where the design recurs; f64 unless a rounding hook is given.

Configurations are the dictionaries that a model folder's config.json holds; weights are name -> array.  `rnd` is applied
wherever a 16-bit implementation may round (matmul operands and results, cached keys, values and latents); the default keeps
full precision.  `without` names mechanisms that are left out on purpose (tests show that each of them matters).
"""
from __future__ import annotations

import math

import numpy as np
from scipy.special import erf

from .ref_decoder import ident, linear, root_mean_square_norm, window_mask

NOTHING = frozenset()


# ---- mechanisms --------------------------------------------------------------------------------------
def gelu(z):
    return 0.5 * z * (1.0 + erf(z / math.sqrt(2.0)))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def softplus(z):
    return np.logaddexp(0.0, z)


def yarn_frequencies(dims, base, scaling):
    """Angles per position of the dims / 2 pairs, and the factor on both cosine and sine."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    turns = lambda t: dims * math.log(scaling["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turns(scaling["fast"])), 0)
    hi = min(math.ceil(turns(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / scaling["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(scaling["factor"]) + 1.0


def rotate_halves(x, positions, rot, without=NOTHING):
    """x [T, ..., D]: coordinates i and i + dims / 2 of the first `dims` turn together, the others stay."""
    if "rotation" in without:
        return x
    dims = rot["dims"]
    freq, size = yarn_frequencies(dims, rot["base"], None if "yarn" in without else rot.get("scaling"))
    if "yarn_size" in without:
        size = 1.0
    ang = np.asarray(positions, np.float64)[:, None] * freq[None, :]
    ang = ang.reshape(ang.shape[0], *([1] * (x.ndim - 2)), -1)
    c, s = size * np.cos(ang), size * np.sin(ang)
    u, v = x[..., :dims // 2], x[..., dims // 2:dims]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., dims:]], axis=-1)


def causal_convolution(u, taps, bias=None):
    """u [T, C], taps [C, K], the last one the current token's; zeros before the first token."""
    k = taps.shape[1]
    padded = np.concatenate([np.zeros((k - 1, u.shape[1]), u.dtype), u])
    y = sum(padded[j:j + u.shape[0]] * taps[:, j] for j in range(k))
    return y if bias is None else y + bias


def softmax(scores, one_more):
    """Softmax over the last axis; with `one_more` the denominator also holds exp(0)."""
    m = scores.max(-1, keepdims=True)
    if one_more:
        m = np.maximum(m, 0.0)
    e = np.exp(scores - m)
    total = e.sum(-1, keepdims=True)
    return e / (total + np.exp(-m) if one_more else total)


def grouped_attend(q, k, v, scale, one_more):
    """q [T, H, D], k [T, G, D], v [T, G, E] -> [T, H, E], causal."""
    t, h, _ = q.shape
    per = h // k.shape[1]
    seen = window_mask(t, t, 0)
    out = np.zeros((t, h, v.shape[2]), q.dtype)
    for head in range(h):
        s = np.where(seen, q[:, head] @ k[:, head // per].T * scale, -np.inf)
        out[:, head] = softmax(s, one_more) @ v[:, head // per]
    return out


def latent_attend(q_plain, q_rot, k_plain, k_rot, v, scale, window):
    """q_plain, k_plain [T, H, D], q_rot [T, H, R], k_rot [T, R] (one for all heads), v [T, H, E] -> [T, H, E]."""
    t, h, _ = q_plain.shape
    seen = window_mask(t, t, window)
    out = np.zeros((t, h, v.shape[2]), q_plain.dtype)
    for head in range(h):
        s = (q_plain[:, head] @ k_plain[:, head].T + q_rot[:, head] @ k_rot.T) * scale
        out[:, head] = softmax(np.where(seen, s, -np.inf), False) @ v[:, head]
    return out


def matrix_memory(q, k, v, log_in, log_forget, without=NOTHING):
    """q, k [T, H, D], v [T, H, E], log gates [T, H] -> [T, H, E], token after token."""
    t, h, d = q.shape
    s, n, m = np.zeros((h, d, v.shape[2]), q.dtype), np.zeros((h, d), q.dtype), np.zeros(h, q.dtype)
    out = np.zeros((t, h, v.shape[2]), q.dtype)
    for i in range(t):
        m_new = np.maximum(log_forget[i] + m, log_in[i])
        keep, take = np.exp(log_forget[i] + m - m_new), np.exp(log_in[i] - m_new)
        s = keep[:, None, None] * s + take[:, None, None] * k[i][:, :, None] * v[i][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[i]
        m = m_new
        qn = (n * q[i]).sum(-1)
        below = np.exp(-m) if "normaliser" in without else np.maximum(np.abs(qn), np.exp(-m))
        out[i] = (s * q[i][:, :, None]).sum(1) / (below + 1e-6)[:, None]
    return out


def gated_linear_unit_recurrence(u, log_a, gate_in):
    """u, log_a, gate_in [T, W] -> states [T, W]: S <- a S + sqrt(1 - a^2) gate_in u from zero."""
    s, out = np.zeros(u.shape[1], u.dtype), np.zeros_like(u)
    for i in range(u.shape[0]):
        a = np.exp(log_a[i])
        s = a * s + np.sqrt(-np.expm1(2.0 * log_a[i])) * gate_in[i] * u[i]
        out[i] = s
    return out


def choose_experts(z, router, without=NOTHING):
    """Router logits of one token -> (experts, weights)."""
    s = np.exp(z - z.max())
    s = s / s.sum()
    groups = router.get("groups") or {"count": 1, "keep": 1}
    by_group = s.reshape(groups["count"], -1)
    open_ = np.ones(groups["count"], bool)
    if "groups" not in without:
        open_[:] = False
        open_[np.argsort(-by_group.max(1), kind="stable")[:groups["keep"]]] = True
    choice = np.where(np.repeat(open_, by_group.shape[1]), s, -1.0)
    chosen = np.argsort(-choice, kind="stable")[:router["top"]]
    w = s[chosen]
    return chosen, w if "renormalise" in without else w / (w.sum() + 1e-20)


# ---- sublayers ---------------------------------------------------------------------------------------
def latent_pair(h, w, name, m, eps, rnd=ident, without=NOTHING):
    """What a latent attention layer caches per token: the normed latent and the rotated key part."""
    rank = m["kv_rank"]
    dkv = rnd(linear(h, w[f"{name}.mix.dkv"]))
    c = dkv[:, :rank] if "latent_norm" in without else root_mean_square_norm(dkv[:, :rank], eps, w[f"{name}.mix.dkv.norm"])
    return rnd(c), rnd(rotate_halves(dkv[:, rank:], np.arange(h.shape[0]), m["rot"], without))


def latent_mixer(h, w, name, m, eps, shared, rnd=ident, without=NOTHING):
    """`shared`: layer -> its (latent, rotated key part), filled as the layers run."""
    heads, d, r, e, t = m["heads"], m["dim"], m["rot_dim"], m["vdim"], h.shape[0]
    layer = int(name[1:])
    if m.get("kv_from") is None:
        shared[layer] = latent_pair(h, w, name, m, eps, rnd, without)
    c, k_rot = shared[layer if m.get("kv_from") is None else m["kv_from"]]
    cq = rnd(linear(h, w[f"{name}.mix.dq"]))
    if "query_norm" not in without:
        cq = rnd(root_mean_square_norm(cq, eps, w[f"{name}.mix.dq.norm"]))
    q = rnd(linear(cq, w[f"{name}.mix.uq"])).reshape(t, heads, d + r)
    k_plain = rnd(linear(c, w[f"{name}.mix.uk"])).reshape(t, heads, d)
    v = rnd(linear(c, w[f"{name}.mix.uv"])).reshape(t, heads, e)
    window = 0 if "window" in without else (m.get("mask") or {}).get("size", 0)
    y = latent_attend(q[:, :, :d], rnd(rotate_halves(q[:, :, d:], np.arange(t), m["rot"], without)), k_plain, k_rot, v, m["scale"], window)
    return rnd(linear(rnd(y.reshape(t, heads * e)), w[f"{name}.mix.o"]))


def attention_branch(h, w, name, m, eps, rnd=ident, without=NOTHING):
    heads, kv, d, e, t = m["heads"], m["kv_heads"], m["dim"], m["vdim"], h.shape[0]

    def part(n):
        u = rnd(linear(h, w[f"{name}.{n}"]))
        return u if "short_conv" in without else causal_convolution(u, w[f"{name}.{n}.conv"])

    q, k, v = part("q").reshape(t, heads, d), part("k").reshape(t, kv, d), rnd(part("v")).reshape(t, kv, e)
    if "qk_norm" not in without:
        q, k = (root_mean_square_norm(x, eps, w[f"{name}.{n}.norm"]) for x, n in ((q, "q"), (k, "k")))
    q, k = (rnd(rotate_halves(x, np.arange(t), m["rot"], without)) for x in (q, k))
    y = grouped_attend(q, k, v, m["scale"], "sink" not in without)
    return rnd(linear(rnd(y.reshape(t, heads * e)), w[f"{name}.o"]))


def memory_branch(h, w, name, m, eps, rnd=ident, without=NOTHING):
    heads, d, e, t, cap = m["heads"], m["dim"], m["vdim"], h.shape[0], m["gate_cap"]
    proj = lambda n: rnd(linear(h, w[f"{name}.{n}"]))
    bound = (lambda z: z) if "gate_cap" in without else (lambda z: cap * np.tanh(z / cap))
    gate_i, gate_f = (bound(linear(h, w[f"{name}.{g}"]) + (0.0 if "gate_bias" in without else w[f"{name}.{g}.b"])) for g in "if")
    o = matrix_memory(proj("q").reshape(t, heads, d) * d ** -0.5, proj("k").reshape(t, heads, d), proj("v").reshape(t, heads, e), gate_i,
                      -softplus(-gate_f), without)
    o = root_mean_square_norm(o, eps).reshape(t, heads * e)
    if "head_norm" not in without:
        o = o * w[f"{name}.norm"]
    if "out_gate" not in without:
        o = o * sigmoid(proj("g"))
    return rnd(linear(rnd(o), w[f"{name}.o"]))


def parallel_mixer(h, w, name, m, eps, shared, rnd=ident, without=NOTHING):
    left = attention_branch(h, w, f"{name}.mix.left", m["left"], eps, rnd, without)
    right = memory_branch(h, w, f"{name}.mix.right", m["right"], eps, rnd, without)
    return (0.0 if "left" in without else m["left_scale"]) * left + (0.0 if "right" in without else m["right_scale"]) * right


def rglru_mixer(h, w, name, m, eps, shared, rnd=ident, without=NOTHING):
    t, blocks = h.shape[0], m["blocks"]
    get = lambda n: w[f"{name}.mix.{n}"]
    y = gelu_tanh(rnd(linear(h, get("y"))) + get("y.b"))
    u = rnd(linear(h, get("x"))) + get("x.b")
    if "short_conv" not in without:
        u = rnd(causal_convolution(u, get("conv"), get("conv.b")))
    ub = u.reshape(t, blocks, -1)
    gate = lambda n: sigmoid(np.einsum("tbi,boi->tbo", ub, get(n)) + get(n + ".b")).reshape(t, -1)
    gate_in = np.ones_like(u) if "input_gate" in without else gate("ri")
    log_a = -8.0 * (1.0 if "decay_gate" in without else gate("ra")) * softplus(get("lam"))
    s = gated_linear_unit_recurrence(u, log_a, gate_in)
    return rnd(linear(rnd(s * (1.0 if "out_branch" in without else y)), get("o")))


MIXERS = {"latent_attention": latent_mixer, "parallel": parallel_mixer, "rglru": rglru_mixer}


def two_layers(h, w, name, rnd=ident):
    return rnd(linear(rnd(gelu(linear(h, w[f"{name}.up"]))), w[f"{name}.down"]))


def feed_forward(h, w, name, mlp, rnd=ident, without=NOTHING):
    if mlp["kind"] == "dense":
        return two_layers(h, w, f"{name}.mlp", rnd)
    z = linear(h, w[f"{name}.mlp.router"])
    y = np.zeros_like(h)
    for i in range(h.shape[0]):
        for e, weight in zip(*choose_experts(z[i], mlp["router"], without)):
            y[i] += weight * two_layers(h[i:i + 1], w, f"{name}.mlp.e{e}", rnd)[0]
    if mlp.get("shared") and "shared" not in without:
        y = y + two_layers(h, w, f"{name}.mlp.shared", rnd)
    return y


def forward(tokens, w, cfg, rnd=ident, want_layers=False, without=NOTHING):
    """Logits [T, vocab] of one sequence (and the residual after every layer)."""
    eps, alpha, tokens, shared, trail = cfg["norm"]["eps"], cfg["postln_alpha"], np.asarray(tokens), {}, []
    one = 0.0 if "unit_offset" in without else 1.0
    if "alpha" in without:
        alpha = 1.0
    norm = lambda x, n: root_mean_square_norm(x, eps, one + w[n])
    x = w["embed"][tokens]
    for i, spec in enumerate(cfg["layers"]):
        n = f"l{i}"
        x = norm(alpha * x + MIXERS[spec["type"]](rnd(x), w, n, spec["mixer"], eps, shared, rnd, without), n + ".norm1")
        if spec.get("mlp"):
            x = norm(alpha * x + feed_forward(rnd(x), w, n, spec["mlp"], rnd, without), n + ".norm2")
        trail.append(x)
    logits = linear(rnd(norm(x, "final.norm")), w["embed"])
    return (logits, np.stack(trail)) if want_layers else logits


# ---- test models -------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    """name -> shape of every tensor a configuration asks for."""
    d, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, spec in enumerate(cfg["layers"]):
        n, m = f"l{i}", spec["mixer"]
        mix = f"{n}.mix."
        out[f"{n}.norm1"] = (d,)
        if spec["type"] == "latent_attention":
            h = m["heads"]
            out[mix + "dq"], out[mix + "dq.norm"], out[mix + "uq"] = (m["q_rank"], d), (m["q_rank"],), (h * (m["dim"] + m["rot_dim"]), m["q_rank"])
            if m.get("kv_from") is None:
                out[mix + "dkv"], out[mix + "dkv.norm"] = (m["kv_rank"] + m["rot_dim"], d), (m["kv_rank"],)
            out[mix + "uk"], out[mix + "uv"], out[mix + "o"] = (h * m["dim"], m["kv_rank"]), (h * m["vdim"], m["kv_rank"]), (d, h * m["vdim"])
        elif spec["type"] == "parallel":
            a, r = m["left"], m["right"]
            for p, rows in (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])):
                out[f"{mix}left.{p}"] = (rows, d)
                if a.get("conv"):
                    out[f"{mix}left.{p}.conv"] = (rows, a["conv"])
            out[mix + "left.q.norm"], out[mix + "left.k.norm"], out[mix + "left.o"] = (a["dim"],), (a["dim"],), (d, a["heads"] * a["vdim"])
            for p, rows in (("q", r["dim"]), ("k", r["dim"]), ("v", r["vdim"]), ("g", r["vdim"]), ("i", 1), ("f", 1)):
                out[f"{mix}right.{p}"] = (r["heads"] * rows, d)
            out[mix + "right.i.b"], out[mix + "right.f.b"] = (r["heads"],), (r["heads"],)
            out[mix + "right.norm"], out[mix + "right.o"] = (r["heads"] * r["vdim"],), (d, r["heads"] * r["vdim"])
        else:
            w, b = m["width"], m["blocks"]
            for p in "xy":
                out[mix + p], out[f"{mix}{p}.b"] = (w, d), (w,)
            out[mix + "conv"], out[mix + "conv.b"] = (w, m["conv"]), (w,)
            for p in ("ra", "ri"):
                out[mix + p], out[f"{mix}{p}.b"] = (b, w // b, w // b), (b, w // b)
            out[mix + "lam"], out[mix + "o"] = (w,), (d, w)
        mlp = spec.get("mlp")
        if not mlp:
            continue
        out[f"{n}.norm2"] = (d,)
        if mlp["kind"] == "dense":
            parts = [("", mlp["ff"])]
        else:
            parts = [(f"e{e}.", mlp["expert"]["ff"]) for e in range(mlp["router"]["experts"])]
            out[f"{n}.mlp.router"] = (mlp["router"]["experts"], d)
            if mlp.get("shared"):
                parts.append(("shared.", mlp["shared"]["ff"]))
        for p, f in parts:
            out[f"{n}.mlp.{p}up"], out[f"{n}.mlp.{p}down"] = (f, d), (d, f)
    out["final.norm"] = (d,)
    return out


def random_weights(cfg, seed, decisive=True):
    """Weights as bf16 can hold them: projections keep unit variance, norm weights scatter, gates remember some tens of tokens.

    `decisive`: every token id ranks the experts of a layer by levels in a few coordinates of its own, which the sublayers
    hardly touch, so that 16-bit rounding cannot swap two experts."""
    from .ref_math import bf16_round

    rng = np.random.default_rng(seed)
    most = max([s["mlp"]["router"]["experts"] for s in cfg["layers"] if s.get("mlp") and s["mlp"]["kind"] == "moe"], default=0) if decisive else 0
    out = {}
    for name, shape in tensor_shapes(cfg).items():
        part = name.split(".")[-1]
        if part in ("norm1", "norm2") or name == "final.norm":
            a = 0.3 * rng.normal(size=shape)
            a[:most] = 0.0
        elif part == "norm":
            a = 1.0 + 0.3 * rng.normal(size=shape)
        elif name.endswith(".f.b"):
            a = 3.0 + rng.normal(size=shape)
        elif part == "b":
            a = rng.normal(size=shape)
        elif part == "lam":
            a = -3.0 + 1.5 * rng.normal(size=shape)
        elif part == "embed":
            a = rng.normal(size=shape)
            if most:
                a[:, :most] = np.stack([rng.permutation(np.linspace(-1.8, 1.8, most)) for _ in range(shape[0])])
        elif part == "router" and most:
            a = np.zeros(shape)
            a[np.arange(shape[0]), rng.permutation(most)[:shape[0]]] = 1.5
        elif part in ("i", "f"):
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
