"""Plain, slow restatement of the Depunex decoder in numpy float64: whole sequences, no cache, no state carried between
calls, one function per mechanism, nothing imported from the package under test (the model-folder reader is the
tests' own).  The GPU tests compare the library with these functions.

Notation: n tokens of one sequence at places 0 .. n-1; matrices are stored [out, in]; `w` maps tensor names (without the
layer's prefix) to arrays."""
from __future__ import annotations

import numpy as np

from plain_llama import read_model  # noqa: F401  (config dict, name -> array)

D64 = np.float64


def f64(a):
    return np.asarray(a, D64)


def rms_unit(x, eps):
    x = f64(x)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_about_one(x, w, eps):
    """RMS norm whose stored weight is the scale's distance from 1."""
    return rms_unit(x, eps) * (1.0 + f64(w))


def lin(x, w):
    return f64(x) @ f64(w).T


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-f64(z)))


def silu(z):
    return f64(z) * sigmoid(z)


def softplus(z):
    z = f64(z)
    return np.maximum(z, 0.0) + np.log1p(np.exp(-np.abs(z)))


def gelu_tanh(z):
    z = f64(z)
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


# ----------------------------------------------------------------------------- embedding
def embed(tokens, table, scale, pair_table=None, pairs=None):
    """scale * the token's row, plus (unscaled) the row of the pair table that the last two tokens choose; a sequence's first
    token takes that table's last row."""
    x = f64(table)[np.asarray(tokens)] * scale
    if pairs is None:
        return x
    n_rows = int(pairs["buckets"])
    for t in range(len(tokens)):
        if t == 0:
            row = n_rows
        else:
            row = (int(tokens[t - 1]) * int(pairs["mul_prev"]) + int(tokens[t]) * int(pairs["mul_cur"])) % n_rows
        x[t] += f64(pair_table[row])
    return x


# ----------------------------------------------------------------------------- pieces of the mixers
def conv_silu(u, taps, bias):
    """Causal convolution per channel (u [n, c], taps [c, k], the last tap is the current token's) with bias, then SiLU."""
    u, taps = f64(u), f64(taps)
    n, k = u.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((k - 1, u.shape[1])), u])
    y = np.tile(f64(bias), (n, 1))
    for j in range(k):
        y += taps[:, j] * padded[j:j + n]
    return silu(y)


def frequencies(rot):
    """base^(-2i / dims) for pair i, slowed by the wave length's place between original / high and original / low."""
    dims = int(rot["dims"])
    f = float(rot["base"]) ** (-2.0 * np.arange(dims // 2) / dims)
    sc = rot.get("scaling")
    if not sc:
        return f
    out = []
    for x in f:
        wave = 2.0 * np.pi / x
        if wave < sc["original"] / sc["high"]:
            out.append(x)
        elif wave > sc["original"] / sc["low"]:
            out.append(x / sc["factor"])
        else:
            s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
            out.append((1.0 - s) * x / sc["factor"] + s * x)
    return np.array(out, D64)


def turn(x, rot):
    """x [n, heads, d]: values i and i + dims / 2 of every head turned by place * frequency i."""
    x = f64(x)
    if not rot or not rot.get("dims"):
        return x
    half = int(rot["dims"]) // 2
    ang = np.arange(x.shape[0])[:, None] * frequencies(rot)[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    a, b = x[..., :half], x[..., half:2 * half]
    return np.concatenate([a * c - b * s, b * c + a * s, x[..., 2 * half:]], axis=-1)


def sees(n, chunk):
    """[n, n] whether place i sees place j: j <= i, both in the same chunk of `chunk` places (None: one chunk)."""
    i, j = np.arange(n)[:, None], np.arange(n)[None, :]
    return (j <= i) & ((i // chunk == j // chunk) if chunk else True)


def chunk_attention(q, k, v, scale, chunk):
    """q [n, H, d], k [n, G, d], v [n, G, dv]; query head h reads key head h // (H / G)."""
    q, k, v = f64(q), f64(k), f64(v)
    n, H, _ = q.shape
    G = k.shape[1]
    mask = sees(n, chunk)
    out = np.zeros((n, H, v.shape[2]), D64)
    for h in range(H):
        g = h // (H // G)
        s = np.where(mask, q[:, h] @ k[:, g].T * scale, -np.inf)
        e = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, h] = e @ v[:, g] / e.sum(axis=1, keepdims=True)
    return out


def attention_mixer(h, w, m):
    n, H = h.shape[0], m["heads"]
    G = m.get("kv_heads", H)
    q = turn(lin(h, w["q"]).reshape(n, H, -1), m.get("rot"))
    k = turn(lin(h, w["k"]).reshape(n, G, -1), m.get("rot"))
    v = lin(h, w["v"]).reshape(n, G, -1)
    chunk = m["mask"]["size"] if m.get("mask") else None
    return lin(chunk_attention(q, k, v, m["scale"], chunk).reshape(n, -1), w["o"])


def channel_scan(x, dt, A, B, C, D):
    """Per channel c and state value s: S <- exp(dt A) S + dt x B, y = sum_s S C + D x.  x, dt [n, c]; A [c, N]; B, C [n, N]."""
    x, dt, A, B, C, D = map(f64, (x, dt, A, B, C, D))
    S = np.zeros_like(A)
    y = np.zeros_like(x)
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y


def mamba_mixer(h, w, m):
    inner, rank, N = m["inner"], m["dt_rank"], m["state"]
    p = lin(h, w["in"])
    x, z = conv_silu(p[:, :inner], w["conv"], w["conv.b"]), p[:, inner:]
    r = lin(x, w["x"])
    dt = softplus(lin(r[:, :rank], w["dt"]) + f64(w["dt.b"]))
    y = channel_scan(x, dt, -np.exp(f64(w["A_log"])), r[:, rank:rank + N], r[:, rank + N:], w["D"])
    return lin(y * silu(z), w["o"])


def parallel_mixer(h, w, m):
    left = {k[5:]: v for k, v in w.items() if k.startswith("left.")}
    right = {k[6:]: v for k, v in w.items() if k.startswith("right.")}
    return m["left_scale"] * attention_mixer(h, left, m["left"]) + m["right_scale"] * mamba_mixer(h, right, m["right"])


def head_scan(x, dt, A_log, B, C, D):
    """x [n, H, P], dt [n, H], B, C [n, G, N]: S_h <- exp(-exp(A_log_h) dt) S_h + dt B x^T, y = S^T C + D x."""
    x, dt, B, C = map(f64, (x, dt, B, C))
    n, H, P = x.shape
    G, N = B.shape[1:]
    y = np.zeros_like(x)
    for h in range(H):
        g = h // (H // G)
        rate = -np.exp(float(A_log[h]))
        S = np.zeros((N, P), D64)
        for t in range(n):
            S = np.exp(rate * dt[t, h]) * S + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S.T @ C[t, g] + float(D[h]) * x[t, h]
    return y


def mamba2_mixer(h, w, m, eps):
    n, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m.get("groups", 1)
    inner = H * P
    p = lin(h, w["in"])
    z, u, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    u = conv_silu(u, w["conv"], w["conv.b"])
    x, B, C = u[:, :inner].reshape(n, H, P), u[:, inner:inner + G * N].reshape(n, G, N), u[:, inner + G * N:].reshape(n, G, N)
    y = head_scan(x, softplus(dt + f64(w["dt_bias"])), w["A_log"], B, C, w["D"]).reshape(n, inner)
    y = y * silu(z)
    parts = m.get("norm_groups", 1)
    y = rms_unit(y.reshape(n, parts, inner // parts), eps).reshape(n, inner) * f64(w["norm"])
    return lin(y, w["o"])


# ----------------------------------------------------------------------------- feed-forward
def clamped_unit(h, w, limit):
    g = np.minimum(lin(h, w["gate"]), limit)
    u = np.clip(lin(h, w["up"]), -limit, limit)
    return lin(g * sigmoid(1.702 * g) * (u + 1.0), w["down"])


def choose_experts(z, top, groups=None):
    """One token's router logits -> (chosen experts, weights): sigmoid scores, the `top` largest among the experts of the best
    groups (a group's score is the sum of its two largest scores), weights are the scores over their sum."""
    s = sigmoid(z)
    allowed = np.ones(len(s), bool)
    if groups:
        per = len(s) // groups["count"]
        rank = [np.sort(s[i * per:(i + 1) * per])[::-1][:2].sum() for i in range(groups["count"])]
        best = np.argsort(-np.array(rank), kind="stable")[:groups.get("keep", groups["count"])]
        allowed = np.array([e // per in best for e in range(len(s))])
    order = np.argsort(-np.where(allowed, s, -np.inf), kind="stable")[:top]
    return order, s[order] / (s[order].sum() + 1e-20)


def routed(h, w, mlp):
    z = lin(h, w["router"])
    out = np.zeros(f64(h).shape)
    for t in range(h.shape[0]):
        for e, p in zip(*choose_experts(z[t], mlp["router"]["top"], mlp["router"].get("groups"))):
            a = silu(lin(h[t], w[f"e{e}.gate"])) * lin(h[t], w[f"e{e}.up"])
            out[t] += p * lin(a, w[f"e{e}.down"])
    return out


def feed_forward(h, w, mlp):
    return clamped_unit(h, w, mlp["limit"]) if mlp["kind"] == "dense" else routed(h, w, mlp)


# ----------------------------------------------------------------------------- layer and model
def token_input(x, part, gate, proj, weight, eps):
    """x + norm(proj (gelu(gate x) * part)) with a plain weight; `part` is the layer's share of the tokens' rows."""
    y = lin(gelu_tanh(lin(x, gate)) * f64(part), proj)
    return f64(x) + rms_unit(y, eps) * f64(weight)


def under(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def layer(x, w, spec, eps, part=None):
    h = norm_about_one(x, w["norm1"], eps)
    mix = under(w, "mix.")
    y = parallel_mixer(h, mix, spec["mixer"]) if spec["type"] == "parallel" else mamba2_mixer(h, mix, spec["mixer"], eps)
    y = y * f64(w["ls1"])
    if spec.get("mlp"):
        y = y + feed_forward(h, under(w, "mlp."), spec["mlp"]) * f64(w["ls2"])
    x = x + y
    if part is not None:
        x = token_input(x, part, w["side.gate"], w["side.proj"], w["side.norm"], eps)
    return x


def forward(cfg, weights, tokens, keep_layers=None):
    """Logits [n, vocab] of one whole sequence; `keep_layers` (a list) receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    e = cfg.get("embedding") or {}
    x = embed(tokens, weights["embed"], e.get("scale", 1.0), weights.get("bigram"), e.get("bigram"))
    side = cfg.get("token_side")
    for i, spec in enumerate(cfg["layers"]):
        part = None
        if side:
            d = side["dim"]
            part = f64(weights["side.embed"])[np.asarray(tokens), i * d:(i + 1) * d]
        x = layer(x, under(weights, f"l{i}."), spec, eps, part)
        if keep_layers is not None:
            keep_layers.append(x.copy())
    z = lin(norm_about_one(x, weights["final.norm"], eps), weights["embed"])
    cap = cfg.get("logit_softcap")
    return cap * np.tanh(z / cap) if cap else z
