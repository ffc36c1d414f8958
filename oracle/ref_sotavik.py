"""Plain numpy restatement of the Sotavik design: one function per mechanism, every request on its own, no cache, no
batching, token after token where the design recurs; f64 unless a rounding hook is given.

Configurations are the dictionaries that a model folder's config.json holds; weights are name -> array.  `rnd` is applied
wherever a 16-bit implementation may round (matmul operands and results, cached latents); the default keeps full precision.
`without` names mechanisms that are left out on purpose (tests show that each of them matters).
"""
from __future__ import annotations

import numpy as np

from .ref_decoder import ident, linear, root_mean_square_norm, silu_gated, sink_softmax

NOTHING = frozenset()


# ---- mechanisms --------------------------------------------------------------------------------------
def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def rotate_pairs(x, positions, base):
    """x [T, ..., dims]: the pair of coordinates (2i, 2i + 1) turned by positions * base^(-2i / dims)."""
    dims = x.shape[-1]
    freq = float(base) ** (-np.arange(0, dims, 2) / dims)
    ang = np.asarray(positions, np.float64)[:, None] * freq[None, :]
    ang = ang.reshape(ang.shape[0], *([1] * (x.ndim - 2)), -1)
    u, v = x[..., 0::2], x[..., 1::2]
    out = np.empty_like(x)
    out[..., 0::2] = u * np.cos(ang) - v * np.sin(ang)
    out[..., 1::2] = v * np.cos(ang) + u * np.sin(ang)
    return out


def gated_linear_recurrence(q, k, v, log_alpha):
    """q, k, log_alpha [T, H, D], v [T, H, E] -> o [T, H, E]: S <- diag(alpha) S + k v^T, o = S^T q."""
    t, h, d = q.shape
    s = np.zeros((h, d, v.shape[2]), q.dtype)
    out = np.zeros((t, h, v.shape[2]), q.dtype)
    for i in range(t):
        s = np.exp(log_alpha[i])[:, :, None] * s + k[i][:, :, None] * v[i][:, None, :]
        out[i] = (s * q[i][:, :, None]).sum(1)
    return out


def latent_attend(q_plain, q_rot, k_plain, k_rot, v, scale, sink=None):
    """q_plain, k_plain [T, H, D], q_rot [T, H, R], k_rot [T, R] (one for all heads), v [T, H, E] -> [T, H, E], causal."""
    t, h, _ = q_plain.shape
    out = np.zeros((t, h, v.shape[2]), q_plain.dtype)
    seen = np.arange(t)[None, :] <= np.arange(t)[:, None]
    for head in range(h):
        s = (q_plain[:, head] @ k_plain[:, head].T + q_rot[:, head] @ k_rot.T) * scale
        out[:, head] = sink_softmax(np.where(seen, s, -np.inf), None if sink is None else sink[head]) @ v[:, head]
    return out


def depth_average(weights, results):
    return sum(w * x for w, x in zip(weights, results))


# ---- sublayers ---------------------------------------------------------------------------------------
def gla_mixer(h, w, name, m, eps, rnd=ident, without=NOTHING):
    heads, d, e, t = m["heads"], m["dim"], m["vdim"], h.shape[0]
    proj = lambda n: rnd(linear(h, w[f"{name}.mix.{n}"]))
    q = proj("q").reshape(t, heads, d) * d ** -0.5
    k, v = proj("k").reshape(t, heads, d), proj("v").reshape(t, heads, e)
    z = linear(linear(h, w[f"{name}.mix.a1"]), w[f"{name}.mix.a2"])
    if "decay_bias" not in without:
        z = z + w[f"{name}.mix.a2.b"]
    tau = 1.0 if "tau" in without else m["tau"]
    log_alpha = 0.0 * z if "decay" in without else log_sigmoid(z) / tau
    o = gated_linear_recurrence(q, k, v, log_alpha.reshape(t, heads, d))
    if "head_norm" not in without:
        o = root_mean_square_norm(o, eps, w[f"{name}.mix.norm"])
    o = o.reshape(t, heads * e)
    if "out_gate" not in without:
        o = silu_gated(proj("g"), o)
    return rnd(linear(rnd(o), w[f"{name}.mix.o"]))


def latent_mixer(h, w, name, m, eps, rnd=ident, without=NOTHING):
    heads, d, r, e, rank, t = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], h.shape[0]
    q = rnd(linear(h, w[f"{name}.mix.q"])).reshape(t, heads, d + r)
    dkv = rnd(linear(h, w[f"{name}.mix.dkv"]))
    c = dkv[:, :rank] if "latent_norm" in without else root_mean_square_norm(dkv[:, :rank], eps, w[f"{name}.mix.dkv.norm"])
    c = rnd(c)
    turn = (lambda x: x) if "rotation" in without else (lambda x: rotate_pairs(x, np.arange(t), m["rot"]["base"]))
    k_plain = rnd(linear(c, w[f"{name}.mix.uk"])).reshape(t, heads, d)
    v = rnd(linear(c, w[f"{name}.mix.uv"])).reshape(t, heads, e)
    y = latent_attend(q[:, :, :d], rnd(turn(q[:, :, d:])), k_plain, rnd(turn(dkv[:, rank:])), v, m["scale"],
                      None if "sink" in without else w[f"{name}.mix.sink"])
    return rnd(linear(rnd(y.reshape(t, heads * e)), w[f"{name}.mix.o"]))


MIXERS = {"gla": gla_mixer, "latent_attention": latent_mixer}


def expert(h, w, name, rnd=ident):
    a = silu_gated(linear(h, w[f"{name}.gate"]), linear(h, w[f"{name}.up"]))
    return rnd(linear(rnd(a), w[f"{name}.down"]))


def table_experts(h, tokens, w, name, mlp, rnd=ident, without=NOTHING):
    """Experts by token id, each weighing 1 / top, and the shared one."""
    table = np.asarray(w[f"{name}.mlp.table"]).astype(int)
    top = table.shape[1]
    y = np.zeros((h.shape[0], w[f"{name}.mlp.e0.down"].shape[0]), h.dtype)
    for i, tok in enumerate(tokens):
        for e in table[tok]:
            y[i] += expert(h[i:i + 1], w, f"{name}.mlp.e{e}", rnd)[0] / top
    if mlp.get("shared") and "shared" not in without:
        y = y + expert(h, w, f"{name}.mlp.shared", rnd)
    return y


def forward(tokens, w, cfg, rnd=ident, want_layers=False, without=NOTHING):
    """Logits [T, vocab] of one sequence (and the residual after every layer)."""
    eps, tokens = cfg["norm"]["eps"], np.asarray(tokens)
    x = w["embed"][tokens]
    results, trail = [x], []
    for i, spec in enumerate(cfg["layers"]):
        n = f"l{i}"
        h = rnd(root_mean_square_norm(x, eps, w[n + ".norm1"]))
        y = MIXERS[spec["type"]](h, w, n, spec["mixer"], eps, rnd, without)
        if spec.get("mlp"):
            y = y + table_experts(h, tokens, w, n, spec["mlp"], rnd, without)
        x = x + y
        results.append(x)
        if "depth_average" not in without:
            x = depth_average(w[n + ".dwa"], results)
        trail.append(x)
    logits = linear(rnd(root_mean_square_norm(x, eps, w["final.norm"])), w["head"]) * cfg["logit_scale"]
    return (logits, np.stack(trail)) if want_layers else logits


# ---- test models -------------------------------------------------------------------------------------
def tensor_shapes(cfg, decay_rank=7):
    """name -> shape of every tensor a configuration asks for (the decay projection's inner width is the tensors' alone)."""
    d, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, spec in enumerate(cfg["layers"]):
        n, m = f"l{i}", spec["mixer"]
        h = m["heads"]
        out[f"{n}.norm1"] = ()
        mix = f"{n}.mix."
        if spec["type"] == "gla":
            for p, rows in (("q", m["dim"]), ("k", m["dim"]), ("v", m["vdim"]), ("g", m["vdim"])):
                out[mix + p] = (h * rows, d)
            out[mix + "o"], out[mix + "norm"] = (d, h * m["vdim"]), (m["vdim"],)
            out[mix + "a1"], out[mix + "a2"], out[mix + "a2.b"] = (decay_rank, d), (h * m["dim"], decay_rank), (h * m["dim"],)
        else:
            out[mix + "q"] = (h * (m["dim"] + m["rot_dim"]), d)
            out[mix + "dkv"], out[mix + "dkv.norm"] = (m["kv_rank"] + m["rot_dim"], d), (m["kv_rank"],)
            out[mix + "uk"], out[mix + "uv"] = (h * m["dim"], m["kv_rank"]), (h * m["vdim"], m["kv_rank"])
            out[mix + "sink"], out[mix + "o"] = (h,), (d, h * m["vdim"])
        if spec.get("mlp"):
            names = [(f"e{e}", spec["mlp"]["expert"]["ff"]) for e in range(spec["mlp"]["router"]["experts"])]
            if spec["mlp"].get("shared"):
                names.append(("shared", spec["mlp"]["shared"]["ff"]))
            for e, f in names:
                out[f"{n}.mlp.{e}.gate"], out[f"{n}.mlp.{e}.up"], out[f"{n}.mlp.{e}.down"] = (f, d), (f, d), (d, f)
            out[f"{n}.mlp.table"] = (cfg["vocab"], spec["mlp"]["router"]["top"])
        out[f"{n}.dwa"] = (i + 2,)
    out["final.norm"], out["head"] = (), (cfg["vocab"], d)
    return out


def random_weights(cfg, seed, decay_rank=7):
    """Weights as bf16 can hold them: projections keep unit variance, norm weights scatter around 1, sinks, decay biases and
    depth weights are large enough to be missed."""
    from .ref_math import bf16_round

    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in tensor_shapes(cfg, decay_rank).items():
        part = name.split(".")[-1]
        if part == "table":
            experts = cfg["layers"][int(name.split(".")[0][1:])]["mlp"]["router"]["experts"]
            out[name] = np.stack([rng.permutation(experts)[:shape[1]] for _ in range(shape[0])]).astype(np.int32)
            continue
        if part in ("norm", "norm1"):
            a = 1.0 + 0.3 * rng.normal(size=shape)
        elif part == "b":
            a = 1.0 + 2.0 * rng.normal(size=shape)
        elif part == "sink":
            a = 1.0 + rng.normal(size=shape)
        elif part == "dwa":
            a = 0.3 * rng.normal(size=shape)
            a[-1] += 0.8
        elif part == "embed":
            a = rng.normal(size=shape)
        else:
            a = rng.normal(size=shape) / np.sqrt(shape[1])
        out[name] = bf16_round(np.asarray(a, np.float32)).astype(np.float64)
    return out


def write_model(folder, cfg, weights):
    """A model folder (config.json, model.safetensors): floating-point tensors in bf16, tables in int32."""
    import json
    import os

    from dmlx_b200.safetensors_io import write_safetensors

    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    bits = lambda a: (np.asarray(a, np.float32).view(np.uint32) >> 16).astype(np.uint16)
    write_safetensors(os.path.join(folder, "model.safetensors"),
                      {n: ("I32", a) if n.endswith(".table") else ("BF16", bits(a)) for n, a in weights.items()}, {})
