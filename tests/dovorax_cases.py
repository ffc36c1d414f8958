"""Configurations of the Dovorax tests: small, and different from one another in every size and branch."""


def dense(ff):
    return {"kind": "dense", "ff": ff}


def experts(count, top, ff, groups=None, shared=None):
    out = {"kind": "moe", "router": {"experts": count, "top": top}, "expert": {"ff": ff}}
    if groups:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def rotation(dims, base=10000.0, scaling=None):
    """scaling: (factor, original, fast, slow)."""
    out = {"dims": dims, "base": base}
    if scaling:
        out["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    return out


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, window, mlp=None, kv_from=None, base=10000.0, scaling=None, scale=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "rot": rotation(rot_dim, base, scaling),
         "scale": scale if scale is not None else 1.5 * (dim + rot_dim) ** -0.5}
    if window:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def parallel(heads, kv_heads, dim, vdim, conv, rot, memory, mlp=None, scales=(0.7, 1.1), scale=None, cap=12.0):
    """memory: (heads, dim, vdim)."""
    left = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv, "rot": rot, "scale": scale if scale is not None else 2.0 * dim ** -0.5}
    right = dict(zip(("heads", "dim", "vdim"), memory), gate_cap=cap)
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def rglru(width, blocks, conv, mlp=None):
    return {"type": "rglru", "mixer": {"width": width, "blocks": blocks, "conv": conv}, "mlp": mlp}


def config(width, vocab, layers, eps=1e-5, alpha=2.0):
    return {"architecture": "Dovorax", "width": width, "vocab": vocab, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": layers}


CASES = {
    "recurrent_only": config(96, 150, [rglru(112, 2, 3, dense(136)), rglru(64, 4, 5, experts(5, 2, 40, shared=56)), rglru(48, 1, 1)], alpha=1.3),
    "latent_only": config(128, 200, [latent(5, 24, 16, 40, 72, 56, 33, experts(6, 2, 24, (3, 2), 72), base=500.0, scaling=(3.0, 64, 20.0, 1.5)),
                                     latent(3, 40, 16, 16, 72, 96, 21, None, kv_from=0, base=500.0, scaling=(3.0, 64, 20.0, 1.5)),
                                     latent(2, 64, 32, 24, 136, 64, 70, dense(88), scale=0.1)], eps=1e-3, alpha=3.5),
    "parallel_only": config(112, 170, [parallel(4, 2, 48, 32, 4, rotation(16, 300.0, (8.0, 40, 16.0, 2.0)), (3, 24, 40), experts(8, 3, 32, (4, 2))),
                                       parallel(6, 6, 16, 64, 2, rotation(16), (2, 64, 88), None, scales=(1.2, 0.4), cap=5.0)], alpha=1.0),
    "mixed_order": config(192, 330, [latent(8, 16, 8, 32, 48, 80, 45, dense(64), scaling=(2.5, 96, 32.0, 1.0)),
                                     rglru(128, 2, 4, experts(9, 4, 32, (3, 2), 128)),
                                     parallel(8, 2, 32, 48, 3, rotation(20, 1000.0, (1.7, 128, 24.0, 1.0)), (4, 32, 48), experts(4, 1, 64)),
                                     latent(4, 32, 8, 24, 48, 40, 90, None, kv_from=0, scaling=(2.5, 96, 32.0, 1.0)),
                                     parallel(3, 1, 64, 24, 4, rotation(64), (1, 128, 96), dense(72))]),
    # nothing is a multiple of anything
    "odd_sizes": config(90, 77, [parallel(6, 3, 21, 13, 6, rotation(10, 77.0), (3, 19, 27), experts(6, 1, 51, (2, 1), 30), scales=(0.3, 2.0)),
                                 latent(5, 19, 6, 11, 50, 37, 19, experts(7, 7, 33, None, 17), base=77.0, scaling=(4.0, 30, 8.0, 1.0)),
                                 rglru(75, 5, 2, dense(41)), latent(7, 9, 6, 30, 50, 13, 300, None, kv_from=1, base=77.0, scaling=(4.0, 30, 8.0, 1.0))],
                        eps=1e-6, alpha=1.9),
    # wide heads, more rows per token than one tile of the attention holds, blocks of several tiles
    "wide": config(256, 192, [latent(20, 72, 40, 56, 288, 128, 61, experts(6, 2, 64, (2, 2), 96)), parallel(2, 1, 160, 200, 4, rotation(80), (2, 160, 200), dense(128)),
                              latent(36, 16, 40, 24, 288, 192, 100, None, kv_from=0), rglru(400, 2, 4)]),
    # head widths that the tensor-core kernels do not take
    "wide_heads": config(64, 130, [parallel(2, 1, 288, 272, 3, rotation(32), (1, 272, 40), experts(3, 2, 16, None, 24)), latent(1, 8, 2, 8, 16, 8, 5, dense(8))]),
}
