"""Small Zabozen configurations for the tests.  They differ from one another in every size; head counts, key and value sizes,
windows, tap counts and the order of layers are unequal on purpose, and some values that models tend to make equal or 1 are not
(and some are)."""
import copy


def attention(heads, kv_heads, dim, vdim, scale, window=None, kv_from=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        m["mask"] = {"size": window}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return m


def latent(heads, dim, rot_dim, vdim, kv_rank, scale, base=10000.0):
    return {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale, "rot": {"base": base, "dims": rot_dim}}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": ff} if ff else None}


# Odd sizes that only the plain kernels take; two layers on another layer's keys, one with a wider window than the layer that keeps them and
# one with a narrower; a layer without a feed-forward between others; three query heads on one key head, six memory heads on two.
ZAB_A = {
    "architecture": "Zabozen", "vocab": 150, "width": 88, "norm": {"eps": 1e-5}, "residual_mult": 0.83, "logit_softcap": 9.0,
    "layers": [
        layer("delta", delta(6, 2, 12, 20, 4), 72),
        layer("attention", attention(3, 1, 20, 12, 0.4, 33), None),
        layer("latent_attention", latent(3, 10, 6, 14, 36, 0.45, base=300.0), 40),
        layer("attention", attention(3, 1, 20, 12, 0.3, 70, kv_from=1), 56),
        layer("attention", attention(3, 1, 20, 12, 0.55, 9, kv_from=1), None),
    ],
}

# Sizes the tensor-core kernels and the vector loads accept; windows of exactly one page and, on the same keys, of a little over three.
ZAB_B = {
    "architecture": "Zabozen", "vocab": 352, "width": 256, "norm": {"eps": 1e-6}, "residual_mult": 0.6, "logit_softcap": 20.0,
    "layers": [
        layer("latent_attention", latent(4, 64, 32, 64, 128, 0.11, base=200000.0), 384),
        layer("attention", attention(8, 2, 64, 32, 0.12, 64), 320),
        layer("delta", delta(8, 4, 64, 64, 2), 256),
        layer("attention", attention(8, 2, 64, 32, 0.14, 200, kv_from=1), 384),
    ],
}

# One head, one tap (a convolution that keeps nothing), a window of one token, a residual share of 1, no cap on the logits, no feed-forward
# in the last layer.
ZAB_C = {
    "architecture": "Zabozen", "vocab": 64, "width": 48, "norm": {"eps": 1e-6}, "residual_mult": 1.0,
    "layers": [
        layer("attention", attention(1, 1, 24, 40, 0.3, 1), 40),
        layer("delta", delta(1, 1, 8, 8, 1), 24),
        layer("latent_attention", latent(1, 4, 2, 6, 8, 0.5), None),
    ],
}

# The memory alone: no layer keeps a key or a value.  A key size that is no multiple of four (no kernel but the token-by-token one takes it).
ZAB_D = {
    "architecture": "Zabozen", "vocab": 96, "width": 64, "norm": {"eps": 1e-5}, "residual_mult": 0.5, "logit_softcap": 4.0,
    "layers": [layer("delta", delta(2, 2, 18, 10, 3), None), layer("delta", delta(4, 1, 16, 24, 5), 96)],
}

# Attention without a window on whose keys a windowed layer looks, and the other way round.
ZAB_E = {
    "architecture": "Zabozen", "vocab": 80, "width": 72, "norm": {"eps": 1e-5}, "residual_mult": 0.9, "logit_softcap": 30.0,
    "layers": [
        layer("attention", attention(2, 2, 16, 8, 0.4), 48),
        layer("attention", attention(4, 2, 12, 16, 0.4, 20), 48),
        layer("attention", attention(2, 2, 16, 8, 0.5, 25, kv_from=0), 40),
        layer("attention", attention(4, 2, 12, 16, 0.3, None, kv_from=1), 40),
    ],
}

ALL = {"a": ZAB_A, "b": ZAB_B, "c": ZAB_C, "d": ZAB_D, "e": ZAB_E}


def config(which):
    return copy.deepcopy(ALL[which])
