"""Small Depunex configurations for the tests.  They differ from one another in every size; head counts, key and value sizes, chunk sizes,
tap counts, group counts and the order of layers are unequal on purpose, and some values that models tend to make equal or 1 are not (and
some are)."""
import copy


def attention(heads, kv_heads, dim, vdim, scale, chunk=None, base=10000.0, dims=None, scaling=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if dims != 0:
        m["rot"] = {"base": base, "dims": dim if dims is None else dims}
        if scaling:
            m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    if chunk is not None:
        m["mask"] = {"size": chunk}
    return m


def scan(inner, dt_rank, state, conv):
    return {"inner": inner, "dt_rank": dt_rank, "state": state, "conv": conv}


def parallel(left, right, left_scale, right_scale):
    return {"left": left, "right": right, "left_scale": left_scale, "right_scale": right_scale}


def mamba2(heads, vdim, state, groups, conv, norm_groups):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}


def dense(ff, limit):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts, top, ff, groups=None):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def layer(kind, mixer, mlp):
    return {"type": kind, "mixer": mixer, "mlp": mlp}


# Odd sizes that only the plain kernels take; a layer without a feed-forward between others; grouped heads of both kinds; a chunk that ends
# inside a page, another smaller than one; slowed frequencies on all three sides of the two borders.
DEP_A = {
    "architecture": "Depunex", "vocab": 150, "width": 90, "norm": {"eps": 1e-5}, "logit_softcap": 6.0, "token_side": {"dim": 10},
    "embedding": {"scale": 1.7, "bigram": {"buckets": 61, "mul_prev": 13, "mul_cur": 5}},
    "layers": [
        layer("parallel", parallel(attention(3, 1, 14, 10, 0.5, 45, 50.0, 10, (3.0, 1.0, 4.0, 60)), scan(42, 5, 6, 3), 0.6, 0.9), dense(50, 0.8)),
        layer("mamba2", mamba2(6, 7, 11, 3, 3, 2), None),
        layer("parallel", parallel(attention(4, 2, 12, 18, 0.4, 20, 300.0, 6), scan(54, 3, 10, 2), 1.1, 0.7), moe(9, 3, 26, (3, 2))),
        layer("mamba2", mamba2(3, 10, 9, 1, 4, 5), moe(6, 2, 18)),
    ],
}

# Sizes the tensor-core kernels and the vector loads accept; chunks of a page and a half and of three pages.
DEP_B = {
    "architecture": "Depunex", "vocab": 352, "width": 256, "norm": {"eps": 1e-6}, "logit_softcap": 12.0, "token_side": {"dim": 32},
    "embedding": {"scale": 2.5, "bigram": {"buckets": 200, "mul_prev": 31, "mul_cur": 3}},
    "layers": [
        layer("mamba2", mamba2(4, 64, 32, 2, 4, 4), moe(8, 2, 64, (4, 2))),
        layer("parallel", parallel(attention(4, 2, 64, 32, 0.12, 96, 10000.0, 32, (8.0, 1.0, 4.0, 512)), scan(192, 32, 16, 4), 0.5, 0.8), dense(384, 2.0)),
        layer("parallel", parallel(attention(8, 8, 32, 64, 0.15, 192, 500.0, 32, (2.0, 2.0, 8.0, 100)), scan(320, 16, 8, 3), 1.0, 1.2), moe(16, 4, 96, (2, 1))),
        layer("mamba2", mamba2(2, 128, 64, 1, 2, 1), dense(320, 1.5)),
    ],
}

# One head, one tap, a state of one value, a chunk of one token, one expert of the top, everything optional left out.
DEP_C = {
    "architecture": "Depunex", "vocab": 64, "width": 48, "norm": {"eps": 1e-6},
    "layers": [
        layer("parallel", parallel(attention(1, 1, 24, 40, 0.3, 1), scan(16, 1, 1, 1), 1.0, 1.0), dense(40, 3.0)),
        layer("mamba2", mamba2(1, 8, 4, 1, 1, 1), moe(5, 1, 24)),
    ],
}

# The state alone: no layer keeps a key or a value.
DEP_D = {
    "architecture": "Depunex", "vocab": 96, "width": 64, "norm": {"eps": 1e-5}, "token_side": {"dim": 7}, "embedding": {"scale": 0.8},
    "layers": [layer("mamba2", mamba2(4, 16, 20, 2, 3, 2), None), layer("mamba2", mamba2(2, 24, 16, 1, 5, 1), dense(72, 1.1))],
}

# No mask and no rotation on one layer, a part of every head turned on the other.
DEP_E = {
    "architecture": "Depunex", "vocab": 80, "width": 72, "norm": {"eps": 1e-5}, "logit_softcap": 9.0, "embedding": {"bigram": {"buckets": 33, "mul_prev": 7, "mul_cur": 11}},
    "layers": [
        layer("parallel", parallel(attention(2, 2, 16, 8, 0.4, None, dims=0), scan(36, 4, 12, 5), 0.8, 1.0), moe(8, 3, 20, (2, 1))),
        layer("parallel", parallel(attention(6, 2, 10, 12, 0.4, 65, 100.0, 4), scan(40, 6, 20, 4), 0.9, 0.5), None),
    ],
}

ALL = {"a": DEP_A, "b": DEP_B, "c": DEP_C, "d": DEP_D, "e": DEP_E}


def config(which):
    return copy.deepcopy(ALL[which])
