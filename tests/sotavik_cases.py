"""Configurations of the Sotavik tests: small, and different from one another in every size and branch."""


def experts(count, top, ff, shared=None):
    out = {"kind": "moe", "router": {"experts": count, "top": top}, "expert": {"ff": ff}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def gla(heads, dim, vdim, tau, mlp=None):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}, "mlp": mlp}


def latent(heads, dim, rot_dim, vdim, kv_rank, mlp=None, base=10000.0, scale=None):
    return {"type": "latent_attention",
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "rot": {"base": base, "dims": rot_dim},
                      "scale": scale if scale is not None else 1.5 * (dim + rot_dim) ** -0.5},
            "mlp": mlp}


def config(width, vocab, layers, eps=1e-5, logit_scale=1.0):
    return {"architecture": "Sotavik", "width": width, "vocab": vocab, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": layers}


CASES = {
    "gla_only": config(96, 160, [gla(3, 40, 24, 4.0, experts(5, 2, 40, 56)), gla(2, 64, 88, 16.0)], logit_scale=0.25),
    "latent_only": config(128, 200, [latent(5, 24, 16, 40, 72, experts(7, 3, 24, 72), base=500.0), latent(2, 64, 32, 16, 136, None, scale=0.1)], eps=1e-3),
    "mixed_order": config(192, 330, [latent(8, 16, 8, 32, 48, experts(4, 1, 64)), gla(4, 32, 48, 8.0, experts(9, 4, 32, 128)), gla(1, 128, 96, 2.0),
                                     latent(3, 48, 64, 24, 160, experts(3, 3, 72, 40))], logit_scale=1.7),
    # nothing is a multiple of anything
    "odd_sizes": config(90, 77, [gla(3, 21, 13, 5.0, experts(5, 2, 51, 30)), latent(5, 19, 6, 11, 50, experts(6, 1, 33, 17), base=77.0),
                                 gla(2, 9, 30, 1.0, experts(2, 2, 7, 90))], eps=1e-6, logit_scale=0.5),
    # wide heads, more rows per token than one tile of the attention holds
    "wide": config(256, 192, [latent(20, 72, 40, 56, 288, experts(6, 2, 64, 96)), gla(2, 160, 200, 12.0, experts(4, 2, 128, 64)),
                              latent(3, 136, 64, 160, 520)]),
    # a state whose keys are wider than the chunk-wise kernels take
    "wide_keys": config(64, 130, [gla(1, 272, 40, 16.0, experts(3, 2, 16, 24)), latent(1, 8, 2, 8, 16, experts(2, 1, 8, 8))]),
}
