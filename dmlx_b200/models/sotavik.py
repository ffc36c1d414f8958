"""Sotavik: gated linear attention and latent attention layers on the configurable decoder stack.

A layer normalises once, with a single learned number as the weight, and feeds mixer and feed-forward from that; their sum joins
the residual, and a learned combination of everything computed so far in depth is handed on.  The feed-forward is a mixture of
experts looked up by token id in a table, next to an expert that serves all tokens.
"""
from __future__ import annotations

import os
from typing import List, Tuple

import numpy as np

from ..safetensors_io import SafetensorsFile
from . import ConfigError, Limits, LoadedModel, register


def _mixer_spec(i: int, kind: str, m: dict, decay_rank) -> dict:
    from .. import device as dev

    if kind == "gla":
        return dict(mixer=dev.MIX_GLA, n_heads=int(m["heads"]), n_kv_heads=int(m["heads"]), key_dim=int(m["dim"]), value_dim=int(m["vdim"]),
                    decay_rank=int(decay_rank(i)), decay_tau=float(m["tau"]))
    if kind == "latent_attention":
        rot, rot_dim = m.get("rot") or {}, int(m["rot_dim"])
        if int(rot.get("dims", rot_dim)) != rot_dim:
            raise ConfigError(f"layer {i}: {rot['dims']} rotated dimensions in a rotated part of {rot_dim}")
        return dict(mixer=dev.MIX_LATENT, n_heads=int(m["heads"]), n_kv_heads=1, key_dim=int(m["dim"]), value_dim=int(m["vdim"]),
                    kv_rank=int(m["kv_rank"]), rot_dim=rot_dim, rot_base=float(rot.get("base", 10000.0)), scale=float(m["scale"]), flags=dev.DEC_SINK)
    raise ConfigError(f"layer {i}: unknown mixer {kind!r}")


def layer_specs(config: dict, decay_rank) -> List[dict]:
    """The layers of a configuration as fields of b200_decoder_layer; `decay_rank(layer)` is the inner width of a layer's decay
    projection, which only the checkpoint knows."""
    from .. import device as dev

    out = []
    for i, entry in enumerate(config["layers"]):
        spec = _mixer_spec(i, entry.get("type"), entry["mixer"], decay_rank)
        spec["flags"] = spec.get("flags", 0) | dev.DEC_PARALLEL
        mlp = entry.get("mlp")
        if mlp is not None:
            if mlp.get("kind") != "moe":
                raise ConfigError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
            spec.update(n_experts=int(mlp["router"]["experts"]), top_k=int(mlp["router"]["top"]), expert_ffn=int(mlp["expert"]["ff"]),
                        ffn=int(mlp["shared"]["ff"]) if mlp.get("shared") else 0)
        out.append(spec)
    return out


_MIXER_TENSORS = {
    "gla": (("q", "q"), ("k", "k"), ("v", "v"), ("out_gate", "g"), ("o", "o"), ("a1", "a1"), ("a2", "a2"), ("a2_bias", "a2.b"), ("head_norm", "norm")),
    "latent_attention": (("q", "q"), ("dkv", "dkv"), ("dkv_norm", "dkv.norm"), ("uk", "uk"), ("uv", "uv"), ("sink", "sink"), ("o", "o")),
}


def tensor_names(config: dict) -> List[Tuple[int, str, List[str]]]:
    """[(layer, tensor of the decoder stack, names in the checkpoint)] of everything a configuration needs; the tensors of several
    names (the experts) are stacked.  "table" is the integer table of a layer's experts."""
    out = [(0, "embed", ["embed"]), (0, "final_norm", ["final.norm"]), (0, "head", ["head"])]
    for i, entry in enumerate(config["layers"]):
        p = f"l{i}."
        out += [(i, "norm1", [p + "norm1"]), (i, "depth", [p + "dwa"])]
        out += [(i, which, [f"{p}mix.{name}"]) for which, name in _MIXER_TENSORS[entry["type"]]]
        mlp = entry.get("mlp")
        if mlp:
            experts = range(int(mlp["router"]["experts"]))
            out += [(i, f"expert_{t}", [f"{p}mlp.e{e}.{t}" for e in experts]) for t in ("gate", "up", "down")]
            out.append((i, "table", [p + "mlp.table"]))
            if mlp.get("shared"):
                out += [(i, t, [f"{p}mlp.shared.{t}"]) for t in ("gate", "up", "down")]
    return out


def build(config: dict, weights, dtype: str, limits: Limits):
    """Model on the device from a SafetensorsFile (or anything with its `bf16`, `shape` and indexing)."""
    from .. import device as dev

    model = dev.DecoderModel(
        hidden=int(config["width"]), vocab=int(config["vocab"]), layers=layer_specs(config, lambda i: weights.shape(f"l{i}.mix.a1")[0]),
        norm_eps=float(config["norm"]["eps"]), dtype=dev.DT_F32 if dtype == "float32" else dev.DT_BF16,
        max_rows=limits.max_rows, max_reqs=limits.max_reqs, max_seqs=limits.max_seqs,
        logit_scale=float(config.get("logit_scale", 1.0)), flags=dev.DEC_SCALAR_NORM | dev.DEC_DEPTH_AVERAGE)
    for layer, which, names in tensor_names(config):
        if which == "table":
            model.set_table(layer, weights[names[0]])
        else:
            model.set_tensor(layer, which, weights.bf16(names[0]) if len(names) == 1 else np.concatenate([weights.bf16(n).ravel() for n in names]))
    model.finalize()
    return model


@register("Sotavik")
def load(config: dict, folder: str, dtype: str, limits: Limits) -> LoadedModel:
    model = build(config, SafetensorsFile(os.path.join(folder, "model.safetensors")), dtype, limits)
    return LoadedModel("Sotavik", model,
                       lambda n_pages, max_pages_per_seq: model.make_cache(n_pages, limits.max_seqs, max_pages_per_seq),
                       int(config["vocab"]), limits)
