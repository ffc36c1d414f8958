"""Dovorax: gated linear recurrences, latent attention and attention beside a matrix memory, on the configurable decoder stack.

Norms stand behind the residual sum, x = norm(alpha x + f(x)), and the sublayers read x itself.  Latent attention takes its queries
through a latent of their own, sees a sliding window, and may read the latents that an earlier layer caches.  A parallel layer runs
softmax attention (short convolutions on q, k and v, one more in the softmax's denominator) and a matrix memory on the same input.
Feed-forwards have no gate; experts are chosen by a router from the best groups, next to an expert that serves all tokens.
"""
from __future__ import annotations

import os
from typing import List, Tuple

import numpy as np

from ..safetensors_io import SafetensorsFile
from . import ConfigError, Limits, LoadedModel, register

LRU_DECAY = 8.0  # factor in the exponent of the gated linear recurrence's decay


def _rotation(where: str, rot, dims: int) -> dict:
    """Fields of a rotation of `dims` dimensions ('rotate half' pairs), with its YaRN scaling where it has one."""
    rot = rot or {}
    if not dims:
        return {}
    out = dict(rot_dim=dims, rot_base=float(rot.get("base", 10000.0)))
    scaling = rot.get("scaling")
    if scaling:
        out.update(yarn_factor=float(scaling["factor"]), yarn_original=float(scaling["original"]), yarn_fast=float(scaling["fast"]),
                   yarn_slow=float(scaling["slow"]))
    if dims % 2:
        raise ConfigError(f"{where}: {dims} rotated dimensions")
    return out


def _mixer_spec(i: int, kind: str, m: dict) -> dict:
    from .. import device as dev

    where = f"layer {i}"
    if kind == "latent_attention":
        rot_dim = int(m["rot_dim"])
        if int((m.get("rot") or {}).get("dims", rot_dim)) != rot_dim:
            raise ConfigError(f"{where}: {m['rot']['dims']} rotated dimensions in a rotated part of {rot_dim}")
        source = m.get("kv_from")
        return dict(mixer=dev.MIX_LATENT, n_heads=int(m["heads"]), n_kv_heads=1, key_dim=int(m["dim"]), value_dim=int(m["vdim"]),
                    kv_rank=int(m["kv_rank"]), q_rank=int(m["q_rank"]), scale=float(m["scale"]), window=int((m.get("mask") or {}).get("size", 0)),
                    kv_source=0 if source is None else 1 + int(source), flags=dev.DEC_ROT_HALVES, **_rotation(where, m.get("rot"), rot_dim))
    if kind == "parallel":
        left, right = m["left"], m["right"]
        rot = left.get("rot") or {}
        return dict(mixer=dev.MIX_ATTENTION, n_heads=int(left["heads"]), n_kv_heads=int(left["kv_heads"]), key_dim=int(left["dim"]),
                    value_dim=int(left["vdim"]), conv_taps=int(left.get("conv") or 0), scale=float(left["scale"]),
                    window=int((left.get("mask") or {}).get("size", 0)), mem_heads=int(right["heads"]), mem_key_dim=int(right["dim"]),
                    mem_value_dim=int(right["vdim"]), mem_gate_cap=float(right["gate_cap"]), mix_scale=float(m["left_scale"]),
                    mem_scale=float(m["right_scale"]), flags=dev.DEC_QK_NORM | dev.DEC_QK_NORM_WEIGHT | dev.DEC_SINK_ONE | dev.DEC_ROT_HALVES,
                    **_rotation(where, rot, int(rot.get("dims", 0))))
    if kind == "rglru":
        width, blocks = int(m["width"]), int(m["blocks"])
        if blocks <= 0 or width % blocks:
            raise ConfigError(f"{where}: {width} channels in {blocks} blocks")
        return dict(mixer=dev.MIX_LRU, n_heads=blocks, n_kv_heads=blocks, key_dim=width // blocks, value_dim=width // blocks,
                    conv_taps=int(m["conv"]), lru_decay=LRU_DECAY)
    raise ConfigError(f"{where}: unknown mixer {kind!r}")


def layer_specs(config: dict) -> List[dict]:
    """The layers of a configuration as fields of b200_decoder_layer."""
    from .. import device as dev

    out = []
    for i, entry in enumerate(config["layers"]):
        spec = _mixer_spec(i, entry.get("type"), entry["mixer"])
        source = spec.get("kv_source", 0) - 1
        if source >= 0:
            other = config["layers"][source] if source < i else {}
            if other.get("type") != "latent_attention" or other["mixer"].get("kv_from") is not None:
                raise ConfigError(f"layer {i}: layer {source} caches no latents for it")
            if any(other["mixer"][k] != entry["mixer"][k] for k in ("kv_rank", "rot_dim")):
                raise ConfigError(f"layer {i}: its latents have another shape than layer {source}'s")
        mlp = entry.get("mlp")
        if mlp is not None:
            spec["flags"] = spec.get("flags", 0) | dev.DEC_FF_GELU
            if mlp.get("kind") == "dense":
                spec["ffn"] = int(mlp["ff"])
            elif mlp.get("kind") == "moe":
                router = mlp["router"]
                groups = router.get("groups") or {"count": 1, "keep": 1}
                spec["flags"] |= dev.DEC_ROUTER
                spec.update(n_experts=int(router["experts"]), top_k=int(router["top"]), expert_ffn=int(mlp["expert"]["ff"]),
                            n_groups=int(groups["count"]), keep_groups=int(groups["keep"]), ffn=int(mlp["shared"]["ff"]) if mlp.get("shared") else 0)
            else:
                raise ConfigError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
        out.append(spec)
    return out


_LRU = (("lru_y", "y"), ("lru_y_bias", "y.b"), ("lru_x", "x"), ("lru_x_bias", "x.b"), ("lru_conv", "conv"), ("lru_conv_bias", "conv.b"),
        ("lru_r", "ra"), ("lru_r_bias", "ra.b"), ("lru_i", "ri"), ("lru_i_bias", "ri.b"), ("lru_lambda", "lam"), ("o", "o"))
_PARALLEL = (*((t, f"left.{t}") for t in "qkvo"), ("q_norm", "left.q.norm"), ("k_norm", "left.k.norm"), *((f"mem_{t}", f"right.{t}") for t in "qkvgoif"),
             ("mem_i_bias", "right.i.b"), ("mem_f_bias", "right.f.b"), ("mem_norm", "right.norm"))
_CONVS = tuple((f"{t}_conv", f"left.{t}.conv") for t in "qkv")
_LATENT = (("dq", "dq"), ("dq_norm", "dq.norm"), ("q", "uq"), ("uk", "uk"), ("uv", "uv"), ("o", "o"))
_LATENT_KEYS = (("dkv", "dkv"), ("dkv_norm", "dkv.norm"))


def _mixer_tensors(entry: dict):
    m = entry["mixer"]
    if entry["type"] == "latent_attention":
        return _LATENT + (_LATENT_KEYS if m.get("kv_from") is None else ())
    if entry["type"] == "parallel":
        return _PARALLEL + (_CONVS if m["left"].get("conv") else ())
    return _LRU


def tensor_names(config: dict) -> List[Tuple[int, str, List[str]]]:
    """[(layer, tensor of the decoder stack, names in the checkpoint)] of everything a configuration needs; the tensors of several
    names (the experts) are stacked."""
    out = [(0, "embed", ["embed"]), (0, "final_norm", ["final.norm"]), (0, "head", ["embed"])]
    for i, entry in enumerate(config["layers"]):
        p = f"l{i}."
        out.append((i, "norm1", [p + "norm1"]))
        out += [(i, which, [f"{p}mix.{name}"]) for which, name in _mixer_tensors(entry)]
        mlp = entry.get("mlp")
        if mlp is None:
            continue
        out.append((i, "norm2", [p + "norm2"]))
        if mlp["kind"] == "dense":
            out += [(i, t, [f"{p}mlp.{t}"]) for t in ("up", "down")]
            continue
        experts = range(int(mlp["router"]["experts"]))
        out += [(i, f"expert_{t}", [f"{p}mlp.e{e}.{t}" for e in experts]) for t in ("up", "down")]
        out.append((i, "router", [p + "mlp.router"]))
        if mlp.get("shared"):
            out += [(i, t, [f"{p}mlp.shared.{t}"]) for t in ("up", "down")]
    return out


def build(config: dict, weights, dtype: str, limits: Limits):
    """Model on the device from a SafetensorsFile (or anything with its `bf16`)."""
    from .. import device as dev

    model = dev.DecoderModel(
        hidden=int(config["width"]), vocab=int(config["vocab"]), layers=layer_specs(config), norm_eps=float(config["norm"]["eps"]),
        dtype=dev.DT_F32 if dtype == "float32" else dev.DT_BF16, max_rows=limits.max_rows, max_reqs=limits.max_reqs, max_seqs=limits.max_seqs,
        flags=dev.DEC_SUM_NORM | dev.DEC_NORM_OFFSET, residual_scale=float(config["postln_alpha"]))
    for layer, which, names in tensor_names(config):
        model.set_tensor(layer, which, weights.bf16(names[0]) if len(names) == 1 else np.concatenate([weights.bf16(n).ravel() for n in names]))
    model.finalize()
    return model


@register("Dovorax")
def load(config: dict, folder: str, dtype: str, limits: Limits) -> LoadedModel:
    model = build(config, SafetensorsFile(os.path.join(folder, "model.safetensors")), dtype, limits)
    return LoadedModel("Dovorax", model,
                       lambda n_pages, max_pages_per_seq: model.make_cache(n_pages, limits.max_seqs, max_pages_per_seq),
                       int(config["vocab"]), limits)
