"""Configurations of the Lorulix tests: small, and different from one another in every size and branch."""


def dense(ff, limit=2.0):
    return {"kind": "dense", "ff": ff, "limit": limit}


def experts(count, top, ff, scale=1.5, shared=None):
    out = {"kind": "moe", "router": {"experts": count, "top": top, "scale": scale}, "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def attention(heads, kv_heads, dim, vdim, mlp=None, kv_from=None, bias_max=60, temp=(0.4, 9), scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "bias_max": bias_max, "scale": scale if scale is not None else 1.5 * dim ** -0.5,
         "q_temp": {"coef": temp[0], "every": temp[1]}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def delta(heads, kv_heads, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp}


def config(width, vocab, layers, eps=1e-5, taps=4, positions=512):
    return {"architecture": "Lorulix", "width": width, "vocab": vocab, "max_positions": positions, "norm": {"eps": eps}, "canon": {"taps": taps},
            "layers": layers}


CASES = {
    "delta_only": config(96, 150, [delta(4, 2, 24, 40, 3, dense(136)), delta(3, 3, 64, 16, 5, experts(5, 2, 40, shared=56)), delta(6, 1, 16, 24, 1)], taps=2),
    "attention_only": config(128, 200, [attention(6, 2, 24, 40, experts(6, 2, 24, 0.8, 72)), attention(6, 2, 24, 40, None, kv_from=0, bias_max=17, temp=(1.1, 4)),
                                        attention(4, 1, 64, 32, dense(88, 0.7), bias_max=200), attention(2, 2, 24, 40, dense(64)),
                                        attention(2, 1, 64, 32, None, kv_from=2, temp=(-0.3, 30))], eps=1e-3, taps=5),
    "mixed_order": config(192, 330, [delta(8, 4, 32, 48, 4, dense(64, 1.0)), attention(8, 4, 16, 24, experts(9, 4, 32, 2.5, 128), bias_max=90),
                                     delta(2, 2, 128, 64, 2, experts(4, 1, 64)), attention(8, 4, 16, 24, None, kv_from=1, temp=(0.9, 13)),
                                     attention(3, 1, 64, 24, dense(72, 3.0), bias_max=33), attention(12, 4, 16, 24, experts(6, 6, 24, 1.0, 40), kv_from=1)]),
    # nothing is a multiple of anything
    "odd_sizes": config(90, 77, [attention(6, 3, 21, 13, experts(6, 1, 51, 3.0, 30), bias_max=29, temp=(0.2, 1)), delta(5, 5, 19, 11, 6, experts(7, 7, 33, 0.5, 17)),
                                 attention(3, 3, 21, 13, dense(41, 0.4), kv_from=0), delta(6, 2, 9, 30, 2, dense(37))], eps=1e-6, taps=3),
    # one tap, convolutions of the current token alone
    "one_tap": config(64, 90, [delta(2, 1, 16, 32, 1, dense(48)), attention(4, 4, 16, 16, dense(40), bias_max=12)], taps=1),
    # wide heads, more rows per token than one tile of the attention holds, states of several column blocks
    "wide": config(256, 192, [attention(20, 1, 72, 56, experts(6, 2, 64, 1.2, 96)), delta(2, 1, 160, 200, 4, dense(128)), attention(34, 1, 72, 56, None, kv_from=0),
                              delta(1, 1, 256, 264, 4), attention(2, 1, 160, 200, dense(72))], taps=7),
    # head widths that the tensor-core kernels do not take
    "wide_heads": config(64, 130, [attention(2, 1, 288, 272, experts(3, 2, 16, shared=24)), delta(1, 1, 288, 40, 3, dense(24))]),
}
# rows of the distance tables by case and layer (8 elsewhere)
BUCKETS = {"mixed_order": {1: 32, 3: 10, 5: 6}, "odd_sizes": {0: 7, 2: 4}, "one_tap": {1: 2}, "attention_only": {2: 16}}


def buckets_of(name):
    return lambda i: BUCKETS.get(name, {}).get(i, 8)
