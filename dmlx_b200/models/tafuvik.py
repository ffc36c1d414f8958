"""Tafuvik: a decoder whose layers may be run in a loop, on the configurable decoder stack.

Per layer: sliding-window attention with grouped queries, keys and values of different widths, biased
projections, unweighted norms on q and k, a distance bias and a learned sink per head; a SwiGLU feed-forward
(or none); norms before and after each sublayer.  A range of layers runs several times with the same weights,
and each pass starts from a projection of the residual beside the embedding output.
"""
from __future__ import annotations

import os
from typing import List, Tuple

from ..safetensors_io import SafetensorsFile
from . import ConfigError, Limits, LoadedModel, register


def layer_specs(config: dict) -> List[dict]:
    """The layers of a configuration as fields of b200_decoder_layer."""
    from .. import device as dev

    out = []
    for i, entry in enumerate(config["layers"]):
        kind = entry.get("type")
        if kind != "attention":
            raise ConfigError(f"layer {i}: unknown mixer {kind!r}")
        m, mlp = entry["mixer"], entry.get("mlp")
        if mlp is not None and mlp.get("kind") != "dense":
            raise ConfigError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
        mask = m.get("mask") or {}
        out.append(dict(
            n_heads=int(m["heads"]), n_kv_heads=int(m["kv_heads"]), key_dim=int(m["dim"]), value_dim=int(m["vdim"]),
            window=int(mask.get("size", 0)), ffn=int(mlp["ff"]) if mlp else 0, scale=float(m["scale"]),
            flags=dev.DEC_QKV_BIAS | dev.DEC_QK_NORM | dev.DEC_DISTANCE_BIAS | dev.DEC_SINK | dev.DEC_POST_NORM))
    return out


def loop_of(config: dict):
    """(start, stop, times) of the looped range, None without one."""
    loop = config.get("loop")
    return (int(loop["start"]), int(loop["stop"]), int(loop["times"])) if loop else None


def tensor_names(config: dict) -> List[Tuple[int, str, str]]:
    """[(layer, tensor of the decoder stack, name in the checkpoint)] of everything a configuration needs."""
    out = [(0, "embed", "embed"), (0, "final_norm", "final.norm"), (0, "head", "head")]
    if config.get("loop"):
        out.append((0, "loop_in", "loop.in"))
    for i, entry in enumerate(config["layers"]):
        p = f"l{i}."
        for t in ("q", "k", "v"):
            out += [(i, t, f"{p}mix.{t}"), (i, f"{t}_bias", f"{p}mix.{t}.b")]
        out += [(i, "o", p + "mix.o"), (i, "sink", p + "mix.sink"), (i, "norm1", p + "norm1"), (i, "postnorm1", p + "norm1b")]
        if entry.get("mlp"):
            out += [(i, t, f"{p}mlp.{t}") for t in ("gate", "up", "down")]
            out += [(i, "norm2", p + "norm2"), (i, "postnorm2", p + "norm2b")]
    return out


def build(config: dict, tensors, dtype: str, limits: Limits):
    """Model on the device; `tensors(name)` gives the bf16 bits of a checkpoint tensor."""
    from .. import device as dev

    model = dev.DecoderModel(
        hidden=int(config["width"]), vocab=int(config["vocab"]), layers=layer_specs(config), norm_eps=float(config["norm"]["eps"]),
        embed_scale=float(config["embedding"]["scale"]), loop=loop_of(config),
        dtype=dev.DT_F32 if dtype == "float32" else dev.DT_BF16,
        max_rows=limits.max_rows, max_reqs=limits.max_reqs, max_seqs=limits.max_seqs)
    for layer, which, name in tensor_names(config):
        model.set_tensor(layer, which, tensors(name))
    model.finalize()
    return model


@register("Tafuvik")
def load(config: dict, folder: str, dtype: str, limits: Limits) -> LoadedModel:
    weights = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    model = build(config, weights.bf16, dtype, limits)
    return LoadedModel("Tafuvik", model,
                       lambda n_pages, max_pages_per_seq: model.make_cache(n_pages, limits.max_seqs, max_pages_per_seq),
                       int(config["vocab"]), limits)
