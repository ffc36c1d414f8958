"""The registry's other architecture: a LLaMA folder loads into the same step, engine and trace replay."""
import os

import numpy as np
import pytest

from oracle import ref_math

pytestmark = pytest.mark.gpu


def _folder(path, quantised):
    import json

    from dmlx_b200.safetensors_io import write_safetensors

    cfg = ref_math.LlamaConfig(n_layers=2, hidden=256, n_heads=4, n_kv_heads=2, head_dim=64, ffn=320, vocab=512)
    rng = np.random.default_rng(6)
    bits = lambda a: (ref_math.bf16_round(a).view(np.uint32) >> 16).astype(np.uint16)
    t = {}

    def linear(name, n, k):
        w = rng.normal(0, 0.05, (n, k)).astype(np.float32)
        if quantised:
            packed, s, b = ref_math.quantize_affine4(w)
            t[name + ".weight"], t[name + ".scales"], t[name + ".biases"] = ("U32", packed), ("BF16", bits(s)), ("BF16", bits(b))
        else:
            t[name + ".weight"] = ("BF16", bits(w))

    for i in range(cfg.n_layers):
        p = f"model.layers.{i}."
        for n, rows, k in (("self_attn.q_proj", 256, 256), ("self_attn.k_proj", 128, 256), ("self_attn.v_proj", 128, 256),
                           ("self_attn.o_proj", 256, 256), ("mlp.gate_proj", 320, 256), ("mlp.up_proj", 320, 256), ("mlp.down_proj", 256, 320)):
            linear(p + n, rows, k)
        for n in ("input_layernorm", "post_attention_layernorm"):
            t[p + n + ".weight"] = ("BF16", bits(np.ones(256, np.float32)))
    t["model.norm.weight"] = ("BF16", bits(np.ones(256, np.float32)))
    t["model.embed_tokens.weight"] = ("BF16", bits(rng.normal(0, 1, (512, 256)).astype(np.float32)))
    linear("lm_head", 512, 256)
    os.makedirs(path)
    write_safetensors(os.path.join(path, "model.safetensors"), t, {})
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump({"architectures": ["LlamaForCausalLM"], "hidden_size": 256, "num_attention_heads": 4, "num_key_value_heads": 2,
                   "num_hidden_layers": 2, "intermediate_size": 320, "vocab_size": 512, "rms_norm_eps": 1e-5, "rope_theta": 10000.0}, f)


@pytest.mark.parametrize("quantised", [False, True])
def test_llama_folder_through_the_common_step(tmp_path, quantised):
    """Portions and single tokens give the logits of the whole prompt; generation follows its argmax."""
    from dmlx_b200.models import Limits, UnsupportedDtype, load_model
    from dmlx_b200.serving import TokenFeeder, generate

    path = str(tmp_path / "m")
    _folder(path, quantised)
    with pytest.raises(UnsupportedDtype):
        load_model(path, "float32")
    loaded = load_model(path, "bfloat16", Limits(256, 4, 4))
    toks = np.random.default_rng(1).integers(0, 512, 60).tolist()
    feeder = TokenFeeder(loaded, 8)
    whole = feeder.step([("w", toks, range(60))])
    parts = [feeder.step([("p", toks[a:b], range(b - a))]) for a, b in ((0, 30), (30, 33), (33, 58), (58, 59), (59, 60))]
    scale = np.abs(whole).max()
    assert np.abs(np.concatenate(parts) - whole).max() <= 2e-2 * scale
    got = generate(loaded, [toks], 4)[0]
    top = np.sort(whole[-1])[::-1]
    assert whole[-1][got[0]] >= top[0] - 2e-2 * scale
