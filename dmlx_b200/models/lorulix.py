"""Lorulix: gated delta rule and softmax attention layers on the configurable decoder stack.

Every sublayer reads its norm h beside a short causal convolution of it, h + conv(h); its result is gated element by element from h
and normed once more before it joins the residual.  Attention has no rotation: a learned vector per position is added to the embedding, a
table gives every head a bias by distance, and queries grow with the position; q and k are normed over all heads at once, and a layer
may read the keys and values that an earlier one caches.  Dense feed-forwards are gated and clamped; experts (square of relu, no gate)
are chosen by a router, next to an expert that serves all tokens with a weight per token.
"""
from __future__ import annotations

import os
from typing import List, Tuple

import numpy as np

from ..safetensors_io import SafetensorsFile
from . import ConfigError, Limits, LoadedModel, register

GATE_ALPHA, UP_SHIFT = 1.702, 1.0  # g sigmoid(alpha g) (u + shift) of the dense feed-forwards


def _mixer_spec(i: int, kind: str, m: dict, buckets) -> dict:
    from .. import device as dev

    shape = dict(n_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), key_dim=int(m["dim"]), value_dim=int(m["vdim"]))
    if shape["n_kv_heads"] <= 0 or shape["n_heads"] % shape["n_kv_heads"]:
        raise ConfigError(f"layer {i}: {shape['n_heads']} heads over {shape['n_kv_heads']}")
    if kind == "delta":
        return dict(mixer=dev.MIX_DELTA, conv_taps=int(m["conv"]), **shape)
    if kind == "attention":
        source, temp = m.get("kv_from"), m.get("q_temp") or {"coef": 0.0, "every": 0}
        rows, reach = int(buckets(i)), int(m["bias_max"])
        if rows < 2 or reach <= rows // 2:
            raise ConfigError(f"layer {i}: distances up to {reach} in {rows} buckets")
        return dict(mixer=dev.MIX_ATTENTION, scale=float(m["scale"]), kv_source=0 if source is None else 1 + int(source), rel_buckets=rows, rel_reach=reach,
                    q_temp_coef=float(temp["coef"]), q_temp_every=int(temp["every"]), flags=dev.DEC_QK_NORM_ROW, **shape)
    raise ConfigError(f"layer {i}: unknown mixer {kind!r}")


def layer_specs(config: dict, buckets) -> List[dict]:
    """The layers of a configuration as fields of b200_decoder_layer; `buckets(layer)` is the number of rows in a layer's distance table,
    which only the checkpoint knows."""
    from .. import device as dev

    out = []
    for i, entry in enumerate(config["layers"]):
        spec = _mixer_spec(i, entry.get("type"), entry["mixer"], buckets)
        source = spec.get("kv_source", 0) - 1
        if source >= 0:
            other = config["layers"][source] if source < i else {}
            if other.get("type") != "attention" or other["mixer"].get("kv_from") is not None:
                raise ConfigError(f"layer {i}: layer {source} caches no keys for it")
            if any(other["mixer"][k] != entry["mixer"][k] for k in ("kv_heads", "dim", "vdim")):
                raise ConfigError(f"layer {i}: its keys and values have another shape than layer {source}'s")
        spec["input_taps"] = int(config["canon"]["taps"])
        spec["flags"] = spec.get("flags", 0) | dev.DEC_POST_NORM | dev.DEC_RESULT_GATE
        mlp = entry.get("mlp")
        if mlp is not None:
            if mlp.get("kind") == "dense":
                spec.update(ffn=int(mlp["ff"]), ff_limit=float(mlp["limit"]), ff_alpha=GATE_ALPHA, ff_shift=UP_SHIFT)
            elif mlp.get("kind") == "moe":
                router, shared = mlp["router"], mlp.get("shared")
                spec["flags"] |= dev.DEC_ROUTER | dev.DEC_ROUTER_PLAIN | dev.DEC_FF_RELU2 | (dev.DEC_SHARED_GATE if shared else 0)
                spec.update(n_experts=int(router["experts"]), top_k=int(router["top"]), expert_ffn=int(mlp["expert"]["ff"]),
                            router_scale=float(router["scale"]), ffn=int(shared["ff"]) if shared else 0)
            else:
                raise ConfigError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
        out.append(spec)
    return out


_DELTA = (*((t, t) for t in "qkvo"), *((f"{t}_conv", f"{t}.conv") for t in "qkv"), ("beta", "b"), ("decay", "a"), ("a_log", "A_log"), ("dt_bias", "dt_bias"),
          ("out_gate", "g"), ("head_norm", "norm"))
_ATTENTION = (("q", "q"), ("o", "o"), ("q_norm", "q.norm"), ("distances", "rel"))
_ATTENTION_KEYS = (("k", "k"), ("v", "v"), ("k_norm", "k.norm"))


def _mixer_tensors(entry: dict):
    if entry["type"] == "delta":
        return _DELTA
    return _ATTENTION + (_ATTENTION_KEYS if entry["mixer"].get("kv_from") is None else ())


def tensor_names(config: dict) -> List[Tuple[int, str, List[str]]]:
    """[(layer, tensor of the decoder stack, names in the checkpoint)] of everything a configuration needs; the tensors of several
    names (the experts) are stacked."""
    out = [(0, "embed", ["embed"]), (0, "positions", ["pos"]), (0, "final_norm", ["final.norm"]), (0, "head", ["head"])]
    for i, entry in enumerate(config["layers"]):
        p = f"l{i}."
        mlp = entry.get("mlp")
        for s in "12" if mlp else "1":
            out += [(i, f"norm{s}", [f"{p}norm{s}"]), (i, f"postnorm{s}", [f"{p}norm{s}b"]), (i, f"in_conv{s}", [f"{p}canon{s}"]),
                    (i, f"result_gate{s}", [f"{p}rg{s}"]), (i, f"result_gate{s}_bias", [f"{p}rg{s}.b"])]
        out += [(i, which, [f"{p}mix.{name}"]) for which, name in _mixer_tensors(entry)]
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            out += [(i, t, [f"{p}mlp.{t}"]) for t in ("gate", "up", "down")]
            continue
        experts = range(int(mlp["router"]["experts"]))
        out += [(i, f"expert_{t}", [f"{p}mlp.e{e}.{t}" for e in experts]) for t in ("up", "down")]
        out.append((i, "router", [p + "mlp.router"]))
        if mlp.get("shared"):
            out += [(i, t, [f"{p}mlp.shared.{t}"]) for t in ("up", "down")]
            out.append((i, "shared_gate", [p + "mlp.shared.sg"]))
    return out


def build(config: dict, weights, dtype: str, limits: Limits):
    """Model on the device from a SafetensorsFile (or anything with its `bf16` and `shape`)."""
    from .. import device as dev

    model = dev.DecoderModel(
        hidden=int(config["width"]), vocab=int(config["vocab"]), layers=layer_specs(config, lambda i: weights.shape(f"l{i}.mix.rel")[0]),
        norm_eps=float(config["norm"]["eps"]), dtype=dev.DT_F32 if dtype == "float32" else dev.DT_BF16, max_rows=limits.max_rows,
        max_reqs=limits.max_reqs, max_seqs=limits.max_seqs, flags=dev.DEC_NORM_OFFSET, max_positions=int(config["max_positions"]))
    for layer, which, names in tensor_names(config):
        model.set_tensor(layer, which, weights.bf16(names[0]) if len(names) == 1 else np.concatenate([weights.bf16(n).ravel() for n in names]))
    model.finalize()
    return model


@register("Lorulix")
def load(config: dict, folder: str, dtype: str, limits: Limits) -> LoadedModel:
    model = build(config, SafetensorsFile(os.path.join(folder, "model.safetensors")), dtype, limits)
    return LoadedModel("Lorulix", model,
                       lambda n_pages, max_pages_per_seq: model.make_cache(n_pages, limits.max_seqs, max_pages_per_seq),
                       int(config["vocab"]), limits)
