"""Plain, slow restatement of the Zabozen decoder in numpy float64: whole sequences, no cache, no state carried between
calls, one function per mechanism, nothing imported from the package under test (the model-folder reader is the
tests' own).  The GPU tests compare the library with these functions.

Notation: n tokens of one sequence at places 0 .. n-1; matrices are stored [out, in]; `w` maps tensor names (without the
layer's prefix) to arrays."""
from __future__ import annotations

import numpy as np

from plain_llama import read_model  # noqa: F401  (config dict, name -> array)

D64 = np.float64
UNIT_EPS = 1e-6          # inside the root of the delta rule's unit vectors


def unit_rms(x, eps):
    x = np.asarray(x, D64)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, scale, eps):
    return unit_rms(x, eps) * np.asarray(scale, D64)


def lin(x, w, b=None):
    y = np.asarray(x, D64) @ np.asarray(w, D64).T
    return y if b is None else y + np.asarray(b, D64)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, D64)))


def silu(z):
    return np.asarray(z, D64) * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, np.asarray(z, D64))


def heads_of(x, heads):
    return np.asarray(x, D64).reshape(x.shape[0], heads, -1)


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


# ----------------------------------------------------------------------------- pieces of the mixers
def turn_halves(x, base, dims):
    """Rotary positions on the first `dims` values of every head, x [n, heads, d]: values i and i + dims / 2 are a pair, and pair i
    at place p turns by p * base^(-2i / dims)."""
    x = np.asarray(x, D64)
    out = x.copy()
    p = np.arange(x.shape[0], dtype=D64)[:, None]
    for i in range(dims // 2):
        j = i + dims // 2
        ang = p * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(ang), np.sin(ang)
        out[:, :, i] = x[:, :, i] * c - x[:, :, j] * s
        out[:, :, j] = x[:, :, j] * c + x[:, :, i] * s
    return out


def sees(n, window=None):
    """[n, n] booleans: place i (row) sees place j (column)."""
    d = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (d >= 0) if window is None else (d >= 0) & (d < window)


def softmax_rows(s, mask):
    s = np.where(mask, s, -np.inf)
    e = np.exp(s - s.max(axis=1, keepdims=True))
    return e / e.sum(axis=1, keepdims=True)


def slopes(H):
    return [2.0 ** (-8.0 * (h + 1) / H) for h in range(H)]


def sloped_attention(q, k, v, scale, window=None):
    """q [n, H, d], k [n, G, d], v [n, G, dv]: query head h reads key head h // (H / G); its score with a key `far` places back is
    lowered by slope_h * far."""
    q, k, v = (np.asarray(a, D64) for a in (q, k, v))
    n, H, _ = q.shape
    per = H // k.shape[1]
    far = np.arange(n)[:, None] - np.arange(n)[None, :]
    out = np.zeros((n, H, v.shape[2]), D64)
    for h, slope in enumerate(slopes(H)):
        s = (q[:, h] @ k[:, h // per].T) * scale - slope * far
        out[:, h] = softmax_rows(s, sees(n, window)) @ v[:, h // per]
    return out


def short_convolution(u, taps):
    """Causal convolution over time per channel: u [n, c], taps [c, k]; the last tap weighs the token itself."""
    u = np.asarray(u, D64)
    taps = np.asarray(taps, D64)
    k = taps.shape[1]
    out = np.zeros_like(u)
    for back in range(min(k, u.shape[0])):
        out[back:] += taps[:, k - 1 - back] * u[:u.shape[0] - back]
    return out


def unit_vectors(x):
    x = np.asarray(x, D64)
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + UNIT_EPS)


def delta_rule(q, k, v, write, keep):
    """The recurrence of one head, q, k [n, d], v [n, dv], write and keep [n]: what is left of the memory forgets (times keep), the
    value it holds under the key is moved by the share `write` towards v, and the query reads the result."""
    S = np.zeros((k.shape[1], v.shape[1]), D64)
    out = np.zeros_like(np.asarray(v, D64))
    for t in range(k.shape[0]):
        S = keep[t] * S
        u = write[t] * (v[t] - S.T @ k[t])
        S = S + np.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


# ----------------------------------------------------------------------------- the three mixers
def keys_and_values(h, w, m, eps):
    """What an `attention` layer keeps of its tokens: unit-rms keys and values."""
    G = m["kv_heads"]
    return unit_rms(heads_of(lin(h, w["k"], w["k.b"]), G), eps), heads_of(lin(h, w["v"], w["v.b"]), G)


def mixer_attention(h, w, m, eps, kept=None):
    """`kept`: another layer's keys and values, for a layer that has none of its own."""
    k, v = kept if kept is not None else keys_and_values(h, w, m, eps)
    q = unit_rms(heads_of(lin(h, w["q"], w["q.b"]), m["heads"]), eps)
    o = sloped_attention(q, k, v, m["scale"], m["mask"]["size"] if m.get("mask") else None)
    return lin(o.reshape(o.shape[0], -1), w["o"], w["o.b"])


def mixer_latent(h, w, m, eps):
    H, d, r, rank = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    n = h.shape[0]
    q = heads_of(lin(h, w["q"]), H)
    low = lin(h, w["dkv"])
    c = rms_norm(low[:, :rank], w["dkv.norm"], eps)
    qr = turn_halves(q[:, :, d:], m["rot"]["base"], r)
    kr = turn_halves(low[:, None, rank:], m["rot"]["base"], r)[:, 0]
    k, v = heads_of(lin(c, w["uk"]), H), heads_of(lin(c, w["uv"]), H)
    o = np.zeros((n, H, v.shape[2]), D64)
    for i in range(H):
        s = (q[:, i, :d] @ k[:, i].T + qr[:, i] @ kr.T) * m["scale"]
        o[:, i] = softmax_rows(s, sees(n)) @ v[:, i]
    o = o * sigmoid(lin(h, w["g"]))[:, :, None]
    return lin(o.reshape(n, -1), w["o"])


def mixer_delta(h, w, m, eps):
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    n = h.shape[0]
    q = unit_vectors(heads_of(silu(short_convolution(lin(h, w["q"]), w["q.conv"])), G)) * d ** -0.5
    k = unit_vectors(heads_of(silu(short_convolution(lin(h, w["k"]), w["k.conv"])), G))
    v = heads_of(silu(short_convolution(lin(h, w["v"]), w["v.conv"])), H)
    write = sigmoid(lin(h, w["b"]))
    keep = np.exp(-np.exp(np.asarray(w["A_log"], D64)) * softplus(lin(h, w["a"]) + np.asarray(w["dt_bias"], D64)))
    o = np.stack([delta_rule(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], write[:, i], keep[:, i]) for i in range(H)], axis=1)
    o = rms_norm(o, w["norm"], eps) * silu(heads_of(lin(h, w["g"]), H))
    return lin(o.reshape(n, -1), w["o"])


MIXERS = {"attention": mixer_attention, "latent_attention": mixer_latent, "delta": mixer_delta}


def gated_unit(h, w):
    return lin(silu(lin(h, w["gate"])) * lin(h, w["up"]), w["down"])


# ----------------------------------------------------------------------------- the wiring and the whole model
def sublayer(x, w_in, w_out, eps, share, fn):
    """x + share * norm_out(fn(norm_in(x)))"""
    return x + share * rms_norm(fn(rms_norm(x, w_in, eps)), w_out, eps)


def soft_cap(z, cap):
    return cap * np.tanh(np.asarray(z, D64) / cap)


def forward(config, weights, tokens, return_layers=False):
    """Logits [n, vocab] of one sequence (and, if asked, the stream after every layer)."""
    eps, share = config["norm"]["eps"], config["residual_mult"]
    x = np.asarray(weights["embed"], D64)[np.asarray(tokens)]
    after, kept = [], {}
    for i, layer in enumerate(config["layers"]):
        w = sub(weights, "l%d." % i)
        m = layer["mixer"]

        def mixer(a):
            if layer["type"] != "attention":
                return MIXERS[layer["type"]](a, sub(w, "mix."), m, eps)
            if m.get("kv_from") is None:
                kept[i] = keys_and_values(a, sub(w, "mix."), m, eps)
            return mixer_attention(a, sub(w, "mix."), m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])

        x = sublayer(x, w["norm1"], w["norm1b"], eps, share, mixer)
        if layer.get("mlp"):
            x = sublayer(x, w["norm2"], w["norm2b"], eps, share, lambda a: gated_unit(a, sub(w, "mlp.")))
        after.append(x)
    logits = lin(rms_norm(x, weights["final.norm"], eps), weights["head"])
    if config.get("logit_softcap"):
        logits = soft_cap(logits, config["logit_softcap"])
    return (logits, np.stack(after)) if return_layers else logits
