"""LLaMA-architecture checkpoints (src/models/llama.zig:40-70 LlamaConfig, src/models/llama_loader.zig:245-279 the weight
triples): bf16 projections, or affine 4-bit ones in groups of 64 (`.weight` packed, `.scales`, `.biases`).
"""
from __future__ import annotations

import os

from ..safetensors_io import SafetensorsFile
from . import ConfigError, Limits, LoadedModel, UnsupportedDtype, register

_PROJECTIONS = (("self_attn.q_proj", "W_Q"), ("self_attn.k_proj", "W_K"), ("self_attn.v_proj", "W_V"), ("self_attn.o_proj", "W_O"),
                ("mlp.gate_proj", "W_GATE"), ("mlp.up_proj", "W_UP"), ("mlp.down_proj", "W_DOWN"))


@register("LlamaForCausalLM", "llama")
def load(config: dict, folder: str, dtype: str, limits: Limits) -> LoadedModel:
    from .. import device as dev

    if dtype != "bfloat16":
        raise UnsupportedDtype("the LLaMA stack runs in bfloat16")
    heads, hidden = int(config["num_attention_heads"]), int(config["hidden_size"])
    kv_heads = int(config.get("num_key_value_heads") or heads)
    head_dim = int(config.get("head_dim") or hidden // heads)
    if config.get("rope_scaling"):
        raise ConfigError("rope_scaling is not implemented")
    n_layers, vocab = int(config["num_hidden_layers"]), int(config["vocab_size"])
    model = dev.LlamaModel(n_layers, hidden, heads, kv_heads, head_dim, int(config["intermediate_size"]), vocab, limits.max_rows,
                           limits.max_reqs, limits.max_seqs, float(config.get("rms_norm_eps", 1e-5)), float(config.get("rope_theta", 10000.0)))
    w = SafetensorsFile(os.path.join(folder, "model.safetensors"))

    def linear(layer: int, which: int, name: str):
        if name + ".scales" in w:
            model.set_linear(layer, which, dev.Q_AFFINE4_G64, w[name + ".weight"], w.bf16(name + ".scales"), w.bf16(name + ".biases"))
        else:
            model.set_linear(layer, which, dev.Q_BF16, w.bf16(name + ".weight"))

    for i in range(n_layers):
        p = f"model.layers.{i}."
        for name, which in _PROJECTIONS:
            linear(i, getattr(dev, which), p + name)
        model.set_norm(i, 0, w.bf16(p + "input_layernorm.weight"))
        model.set_norm(i, 1, w.bf16(p + "post_attention_layernorm.weight"))
    model.set_norm(-1, 0, w.bf16("model.norm.weight"))
    model.set_embedding(w.bf16("model.embed_tokens.weight"))
    linear(0, dev.W_LM_HEAD, "model.embed_tokens" if config.get("tie_word_embeddings") else "lm_head")
    model.finalize()

    def new_cache(n_pages: int, max_pages_per_seq: int):
        return dev.PagedKVCache(n_layers, kv_heads, head_dim, n_pages, limits.max_seqs, max_pages_per_seq, heads, limits.max_rows)

    return LoadedModel("LlamaForCausalLM", model, new_cache, vocab, limits)
