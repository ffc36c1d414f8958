"""Configurations of the decoder tests: small, and different from one another in every size and branch."""


def attention(heads, kv_heads, dim, vdim, window, scale=None, ff=None):
    return {"type": "attention",
            "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window},
                      "scale": scale if scale is not None else 2.0 * dim ** -0.5},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(width, vocab, layers, loop=None, eps=1e-5, embed_scale=3.0):
    return {"architecture": "Tafuvik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "layers": layers, "loop": dict(zip(("start", "stop", "times"), loop)) if loop else None}


CASES = {
    # a loop in the middle, a layer without feed-forward, windows shorter and longer than a page
    "middle_loop": config(128, 320, [attention(6, 2, 32, 48, 21, ff=192), attention(4, 4, 64, 64, 70, ff=64), attention(4, 1, 48, 16, 33)],
                          (1, 2, 2)),
    # no loop, one kv head per query head, one layer wider than the tensor-core kernel takes
    "no_loop": config(192, 200, [attention(2, 2, 128, 128, 64, ff=100), attention(3, 1, 272, 40, 9, ff=128)], None, eps=1e-3, embed_scale=0.5),
    # the loop covers the whole stack and runs once; twenty query heads on one kv head
    "whole_loop": config(64, 130, [attention(20, 1, 16, 24, 50, ff=72)], (0, 1, 1)),
    # nothing is a multiple of anything: widths, heads, vocabulary
    "odd_sizes": config(90, 77, [attention(5, 1, 21, 13, 17, ff=51), attention(3, 3, 40, 7, 1, ff=30)], (0, 2, 3), eps=1e-6, embed_scale=1.0),
    # a window over several pages and a wide head
    "wide_head": config(256, 384, [attention(4, 2, 160, 136, 100, ff=320), attention(8, 2, 72, 200, 45, ff=128)], (1, 2, 2)),
}
