"""Tiny Bavetar configurations for the tests.  They differ from one another in every size and option: order of the two
mixers, dense, routed and absent feed-forwards, head counts, latent sizes, rotated parts and their bases, state sizes,
value sizes and groups of the recurrence (one group, several, as many as heads), taps of the convolution (one to six),
parts of the norm (one, several, parts that cut heads and parts of several heads), numbers of experts, groups and chosen
experts (with and without groups, one chosen, all groups kept), scales of the experts and of the logits, with and without
a cap, vocabulary, eps."""


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale=1.0, groups=None):
    router = {"experts": experts, "top": top, "scale": scale}
    if groups is not None:
        router["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, scale, base, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale,
                      "rot": {"dims": rot_dim, "base": base}}}


def mamba(heads, vdim, state, groups, conv, norm_groups, mlp=None):
    return {"type": "mamba2", "mlp": mlp,
            "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}}


# the recurrence first; every feed-forward kind behind both mixers; a norm part that cuts a head (3 parts of 2 heads)
BAVETAR_A = {
    "architecture": "Bavetar", "vocab": 150, "width": 64, "norm": {"eps": 1e-5}, "logit_scale": 1.5, "logit_softcap": 12.0,
    "layers": [mamba(4, 16, 16, 2, 4, 1, moe(8, 3, 40, 2.0, (4, 2))), latent(3, 16, 8, 24, 20, 40, 0.2, 1000.0, dense(72)),
               mamba(2, 24, 32, 1, 3, 3, dense(56)), latent(2, 8, 8, 8, 24, 24, 0.25, 5e4, moe(6, 2, 32, 1.3, (3, 2))),
               mamba(3, 8, 8, 3, 2, 3), latent(4, 24, 4, 16, 12, 28, 0.18, 200.0)],
}

# sizes no fast path takes: a width and feed-forwards that are no multiples of 8, odd heads, latents, states and values, an
# odd vocabulary; no groups of experts, one chosen; no cap and no scale of the logits
BAVETAR_B = {
    "architecture": "Bavetar", "vocab": 97, "width": 36, "norm": {"eps": 1e-6}, "logit_softcap": None,
    "layers": [latent(5, 6, 2, 7, 5, 11, 0.4, 10.0, moe(5, 1, 9)), mamba(3, 6, 10, 3, 6, 2, dense(27)),
               mamba(4, 5, 7, 1, 1, 5, moe(3, 3, 27, 0.5)), latent(1, 3, 4, 9, 7, 5, 0.5, 30.0, dense(13))],
}

# sizes the tensor-core attention kernels take (cached rows of 64 and 48), states of 64 and 128, values of 32 and 64
BAVETAR_C = {
    "architecture": "Bavetar", "vocab": 211, "width": 128, "norm": {"eps": 1e-6}, "logit_scale": 0.7, "logit_softcap": 25.0,
    "layers": [latent(4, 48, 16, 32, 64, 48, 0.14, 3e4, dense(192)), mamba(4, 32, 64, 2, 4, 2, moe(12, 4, 48, 1.5, (6, 3))),
               mamba(2, 64, 128, 1, 4, 1, dense(96)), latent(8, 16, 16, 16, 32, 32, 0.2, 100.0, moe(9, 2, 32, 1.0, (3, 3))),
               mamba(6, 16, 32, 3, 4, 6, moe(4, 2, 40, 0.8, (2, 1)))],
}

# one head and one group everywhere, two experts in two groups of which one is kept
BAVETAR_D = {
    "architecture": "Bavetar", "vocab": 53, "width": 40, "norm": {"eps": 1e-4}, "logit_scale": 3.0, "logit_softcap": 5.0,
    "layers": [mamba(1, 24, 16, 1, 2, 1, moe(2, 1, 16, 1.0, (2, 1))), latent(1, 8, 4, 8, 8, 12, 0.3, 50.0),
               mamba(1, 8, 24, 1, 4, 2), latent(1, 16, 2, 4, 16, 6, 0.25, 7.0, dense(24))],
}

# prompts of hundreds of tokens: cached rows of 80 on pages of 16, states of 32 x 48 and 64 x 64
BAVETAR_E = {
    "architecture": "Bavetar", "vocab": 300, "width": 96, "norm": {"eps": 1e-6}, "logit_scale": 1.2, "logit_softcap": 15.0,
    "layers": [mamba(4, 48, 32, 2, 4, 2, dense(160)), latent(5, 32, 16, 16, 48, 64, 0.14, 5e3, moe(6, 2, 32, 1.5, (3, 2))),
               mamba(2, 64, 64, 1, 4, 1, moe(6, 2, 32, 1.2))],
}

BAVETAR_CONFIGS = {"A": BAVETAR_A, "B": BAVETAR_B, "C": BAVETAR_C, "D": BAVETAR_D}
BAVETAR_PAGE = {"A": 8, "B": 4, "C": 16, "D": 2}
BAVETAR_SEEDS = {"A": 45, "B": 46, "C": 47, "D": 48}
BAVETAR_STD = {"A": 0.12, "B": 0.2, "C": 0.08, "D": 0.25}
