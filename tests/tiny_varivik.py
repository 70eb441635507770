"""Tiny Varivik configurations for the tests.  They differ from one another in every size and option: head counts and
groups, key and value sizes (equal, different, multiples of 16 and not), chunks (of one, two, shorter and longer than a
page, none), rotated shares of a head (none, part, all) with and without scaled rates, layers with and without mixed
values (from the first layer on, later, in the last alone), dense feed-forwards, experts with and without a shared one,
one and all of them chosen, layers without a feed-forward, width, vocabulary, eps."""


def bands(factor, low, high, original):
    return {"factor": factor, "low": low, "high": high, "original": original}


def rot(dims, base, scaling=None):
    r = {"dims": dims, "base": base}
    if scaling is not None:
        r["scaling"] = scaling
    return r


def attention(heads, kv_heads, dim, vdim, scale, chunk=None, turn=None, v_mix=True, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "v_mix": v_mix}
    if chunk:
        m["mask"] = {"size": chunk}
    if turn is not None:
        m["rot"] = turn
    return {"type": "attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None):
    mlp = {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}
    if shared is not None:
        mlp["shared"] = {"ff": shared}
    return mlp


# the first layer mixes nothing; chunks shorter and longer than a page and none; every kind of feed-forward
VARIVIK_A = {
    "architecture": "Varivik", "vocab": 150, "width": 64, "norm": {"eps": 1e-5},
    "layers": [attention(4, 2, 16, 32, 0.3, 9, rot(8, 1000.0, bands(4.0, 1.0, 4.0, 64)), False, dense(40)),
               attention(4, 2, 24, 16, 0.2, 20, rot(24, 5e4), True, moe(6, 2, 24, 40)),
               attention(2, 2, 8, 16, 0.35, None, rot(4, 100.0, bands(2.0, 0.5, 2.0, 16)), True, moe(5, 3, 16)),
               attention(8, 2, 16, 16, 0.25, 33, None, True, None),
               attention(6, 2, 32, 16, 0.17, 7, rot(16, 3e5, bands(16.0, 1.0, 8.0, 128)), True, dense(24))],
}

# sizes no fast path takes: a width that is no multiple of 8, odd head and feed-forward sizes, an odd vocabulary
VARIVIK_B = {
    "architecture": "Varivik", "vocab": 97, "width": 36, "norm": {"eps": 1e-6},
    "layers": [attention(3, 1, 12, 20, 0.3, 5, rot(2, 10.0), True, moe(3, 1, 9, 7)),
               attention(5, 1, 7, 20, 0.4, 3, rot(6, 50.0, bands(3.0, 0.0, 1.0, 9)), True, dense(27)),
               attention(4, 1, 10, 20, 0.3, 11, rot(10, 200.0, bands(1.0, 1.0, 2.0, 8)), True, None)],
}

# sizes the tensor-core kernels take, keys and values alike and different
VARIVIK_C = {
    "architecture": "Varivik", "vocab": 211, "width": 128, "norm": {"eps": 1e-6},
    "layers": [attention(8, 2, 64, 32, 0.125, 40, rot(32, 3e4, bands(8.0, 1.0, 4.0, 64)), True, moe(8, 2, 48, 96)),
               attention(6, 2, 32, 32, 0.2, 24, rot(32, 1e4), True, dense(72)),
               attention(4, 2, 128, 32, 0.09, None, rot(64, 1e6, bands(4.0, 1.0, 4.0, 256)), True, moe(8, 1, 48)),
               attention(4, 4, 64, 64, 0.11, 16, rot(8, 1e3), False, moe(4, 2, 32, 32))],
}

# one head, chunks of one and two, every expert chosen, no rotation in one layer, only the last layer mixes (with nothing)
VARIVIK_D = {
    "architecture": "Varivik", "vocab": 53, "width": 40, "norm": {"eps": 1e-4},
    "layers": [attention(1, 1, 8, 8, 0.5, 2, rot(0, 10.0), False, moe(3, 3, 16)),
               attention(1, 1, 8, 24, -0.4, 1, rot(8, 50.0), False, dense(16)),
               attention(2, 1, 16, 8, 0.3, None, rot(2, 30.0), True, moe(1, 1, 8, 24))],
}

# chunks that prompts of hundreds of tokens pass, at sizes of the kernels fed by TMA, on pages of 16 that are given back
VARIVIK_E = {
    "architecture": "Varivik", "vocab": 300, "width": 96, "norm": {"eps": 1e-6},
    "layers": [attention(4, 2, 64, 64, 0.125, 70, rot(32, 5e3, bands(8.0, 1.0, 4.0, 128)), True, dense(64)),
               attention(4, 2, 128, 64, 0.09, 150, rot(64, 1e4), True, moe(6, 2, 32, 64)),
               attention(8, 2, 64, 64, 0.125, None, rot(64, 1e5), True, moe(6, 2, 32))],
}

VARIVIK_CONFIGS = {"A": VARIVIK_A, "B": VARIVIK_B, "C": VARIVIK_C, "D": VARIVIK_D}
VARIVIK_PAGE = {"A": 8, "B": 4, "C": 16, "D": 2}
VARIVIK_SEEDS = {"A": 45, "B": 46, "C": 47, "D": 48}
VARIVIK_STD = {"A": 0.15, "B": 0.2, "C": 0.1, "D": 0.25}
