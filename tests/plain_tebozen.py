"""The Tebozen design once more, plain and slow: NumPy float64, whole sequences, no cache, no state carried between calls,
one function per mechanism.  It shares no code with the library; the tests compare the engine with it.  A model is a dict
``cfg`` (the parsed config.json) and a dict ``w`` of float64 arrays by tensor name.

``round16`` rounds where the bfloat16 engine rounds: the operands of the matrix products, the rotated queries, and what
the cache holds (keys, values, latents, rotated key parts); everything else stays in float64.
"""
from __future__ import annotations

import math

import numpy as np

TINY = 1e-6         # joins the matrix memory's denominator


# ----------------------------------------------------------------------------- small pieces
def round_bf16(a):
    a = np.ascontiguousarray(a, dtype=np.float32)
    u = a.view(np.uint32).astype(np.uint64)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & 0xFFFF0000
    return u.astype(np.uint32).view(np.float32).astype(np.float64).reshape(a.shape)


def product(x, W, round16=False):
    """Rows of x times W [out, in] transposed."""
    x = round_bf16(x) if round16 else np.asarray(x, dtype=np.float64)
    return x @ np.asarray(W, dtype=np.float64).T


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-np.asarray(z, dtype=np.float64)))


def unit_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_about_one(x, weight, eps):
    """RMS norm whose stored weight is the difference from 1."""
    return unit_rms(x, eps) * (1.0 + weight)


def conv_over_time(u, taps):
    """u [n, C], taps [C, J]: every channel's last J inputs, the newest times the last tap; zeros before the start."""
    n, J = u.shape[0], taps.shape[1]
    padded = np.concatenate([np.zeros((J - 1, u.shape[1])), u])
    return sum(padded[j:j + n] * taps[:, j] for j in range(J))


def turn(x, positions, base, dims, neighbours):
    """x [n, ..., size]: the first ``dims`` values of the last axis turned by pairs, pair i by the angle
    position * base^(-2 i / dims).  ``neighbours``: the pair is (2i, 2i + 1), else (i, i + dims / 2)."""
    out = np.array(x, dtype=np.float64)
    i = np.arange(dims // 2)
    angle = np.asarray(positions, dtype=np.float64)[:, None] * float(base) ** (-2.0 * i / max(dims, 1))
    angle = angle.reshape((len(angle),) + (1,) * (x.ndim - 2) + (dims // 2,))
    a, b = (2 * i, 2 * i + 1) if neighbours else (i, i + dims // 2)
    out[..., a] = x[..., a] * np.cos(angle) - x[..., b] * np.sin(angle)
    out[..., b] = x[..., b] * np.cos(angle) + x[..., a] * np.sin(angle)
    return out


def softmax(s, seen):
    s = np.where(seen, s, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def visible(n, window=None):
    """[query, key]: keys up to the query's own position, and only the last ``window`` of them."""
    back = np.arange(n)[:, None] - np.arange(n)[None, :]
    return (back >= 0) & (back < (window if window else n))


# ----------------------------------------------------------------------------- mixers
def gates(h, m, w, px, round16=False):
    """Logarithms of the input and of the forget gate, [n, heads] each."""
    cap = m["gate_cap"]
    i = cap * np.tanh((product(h, w[px + "i"], round16) + w[px + "i.b"]) / cap)
    f = cap * np.tanh((product(h, w[px + "f"], round16) + w[px + "f.b"]) / cap)
    return i, -np.logaddexp(0.0, -f)


def matrix_memory(q, k, v, i, f):
    """One head: q, k [n, K], v [n, P], log gates i, f [n] -> [n, P].  The memory and its normaliser are kept relative to
    exp(m), m a running maximum that starts at 0."""
    n, K = q.shape
    S, N, m = np.zeros((K, v.shape[1])), np.zeros(K), 0.0
    out = np.zeros((n, v.shape[1]))
    for t in range(n):
        above = max(f[t] + m, i[t])
        keep, write = math.exp(f[t] + m - above), math.exp(i[t] - above)
        S = keep * S + write * np.outer(k[t], v[t])
        N = keep * N + write * k[t]
        m = above
        out[t] = S.T @ q[t] / (max(abs(N @ q[t]), math.exp(-m)) + TINY)
    return out


def mlstm(h, m, w, px, eps, round16=False):
    n, H, K, P = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = product(h, w[px + "q"], round16).reshape(n, H, K) / math.sqrt(K)
    k = product(h, w[px + "k"], round16).reshape(n, H, K)
    v = product(h, w[px + "v"], round16).reshape(n, H, P)
    i, f = gates(h, m, w, px, round16)
    o = np.stack([matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]) for a in range(H)], axis=1)
    o = unit_rms(o, eps).reshape(n, H * P) * w[px + "norm"] * sigmoid(product(h, w[px + "g"], round16))
    return product(o, w[px + "o"], round16)


def difference_weight(w, px, diff):
    """The factor on the second map's output, one number for the layer."""
    return math.exp(np.sum(w[px + "lq1"] * w[px + "lk1"])) - math.exp(np.sum(w[px + "lq2"] * w[px + "lk2"])) + diff


def head_gate(h, o, w, px, round16=False):
    """o [n, H, P]: every head's output times one number of its own."""
    return o * sigmoid(product(h, w[px + "g"], round16))[:, :, None]


def attention(h, m, w, px, eps, round16=False):
    """Two score maps a head over the same values, their difference normed; a window; a gate a head."""
    n, H, G, K, P = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (conv_over_time(product(h, w[px + x], round16) + w[px + x + ".b"], w[px + x + ".conv"]) for x in "qkv")
    q, k, v = q.reshape(n, H, 2, K), k.reshape(n, G, 2, K), v.reshape(n, G, P)
    q, k = (turn(a, np.arange(n), m["rot"]["base"], m["rot"]["dims"], False) for a in (q, k))
    if round16:
        q, k, v = round_bf16(q), round_bf16(k), round_bf16(v)
    seen, lam = visible(n, m["mask"]["size"]), difference_weight(w, px, m["diff"])
    o = np.zeros((n, H, P))
    for a in range(H):
        g = a // (H // G)
        one, two = (softmax(q[:, a, j] @ k[:, g, j].T * m["scale"], seen) @ v[:, g] for j in range(2))
        o[:, a] = unit_rms(one - lam * two, eps) * (1.0 - m["diff"])
    return product(head_gate(h, o, w, px, round16).reshape(n, H * P), w[px + "o"], round16)


def latent_rows(h, m, w, px, eps, round16=False):
    """What the cache holds of every token: the normed latent and the rotated key part, [n, rank] and [n, rot_dim]."""
    n, L = h.shape[0], m["kv_rank"]
    d = product(h, w[px + "dkv"], round16)
    c = unit_rms(d[:, :L], eps) * w[px + "dkv.norm"]
    r = turn(d[:, L:], np.arange(n), m["rot"]["base"], m["rot"]["dims"], True)
    return (round_bf16(c), round_bf16(r)) if round16 else (c, r)


def latent_attention(h, m, w, px, eps, round16=False, rows=None):
    """Keys and values from latents: the layer's own, or another layer's ``rows``; a gate a head.  Returns (output, rows)."""
    n, H, K, R, P = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    rows = latent_rows(h, m, w, px, eps, round16) if rows is None else rows
    c, k_turned = rows
    q = product(h, w[px + "q"], round16).reshape(n, H, K + R)
    q_plain, q_turned = q[..., :K], turn(q[..., K:], np.arange(n), m["rot"]["base"], m["rot"]["dims"], True)
    if round16:
        q_plain = round_bf16(q_plain)
    k, v = product(c, w[px + "uk"]).reshape(n, H, K), product(c, w[px + "uv"]).reshape(n, H, P)
    o = np.zeros((n, H, P))
    for a in range(H):
        o[:, a] = softmax((q_plain[:, a] @ k[:, a].T + q_turned[:, a] @ k_turned.T) * m["scale"], visible(n)) @ v[:, a]
    return product(head_gate(h, o, w, px, round16).reshape(n, H * P), w[px + "o"], round16), rows


# ----------------------------------------------------------------------------- feed-forward
def expert(x, w, px, round16=False, weight=None):
    """``weight`` [n, 1] is on the expert's input (rounded, the product of a weight and rounded rows; products are linear)."""
    up = product(x, w[px + "up"], round16)
    up = up if weight is None else up * weight
    return product(np.maximum(up, 0.0) ** 2, w[px + "down"], round16)


def route(z, top):
    """Logits [n, experts] -> (chosen [n, top], weights [n, top]), best first, ties to the lower index."""
    s = sigmoid(z)
    chosen = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=-1)


def route_margin(z, top):
    """How far each token's choice is from another one, in scores."""
    s = -np.sort(-sigmoid(z), axis=-1)
    return s[:, top - 1] - s[:, top] if top < z.shape[1] else np.full(len(z), np.inf)


def experts(h, mlp, w, px, round16=False, margins=None):
    top = mlp["router"]["top"]
    z = product(h, w[px + "router"], round16)
    chosen, weights = route(z, top)
    if margins is not None:
        margins.append(route_margin(z, top))
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, k = np.nonzero(chosen == e)
        if t.size:
            out[t] += expert(h[t], w, px + f"e{e}.", round16, weight=weights[t, k][:, None])
    if mlp.get("shared"):
        out = out + expert(h, w, px + "shared.", round16)
    return out


# ----------------------------------------------------------------------------- the model
def forward(cfg, w, tokens, round16=False, taps=None, margins=None):
    """Logits [n, vocab] of one sequence; ``taps``, a list, receives the stream after every layer, ``margins`` every
    router's margin for every token."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    rows = {}
    for i, layer in enumerate(cfg["layers"]):
        px, m = f"l{i}.", layer["mixer"]
        h = norm_about_one(x, w[px + "norm1"], eps)
        if layer["type"] == "latent_attention":
            y, rows[i] = latent_attention(h, m, w, px + "mix.", eps, round16, rows=rows[m["kv_from"]] if m.get("kv_from") is not None else None)
        else:
            y = {"mlstm": mlstm, "attention": attention}[layer["type"]](h, m, w, px + "mix.", eps, round16)
        x = x + y
        if layer.get("mlp") is not None:
            x = x + experts(norm_about_one(x, w[px + "norm2"], eps), layer["mlp"], w, px + "mlp.", round16, margins)
        if taps is not None:
            taps.append(x.copy())
    return product(norm_about_one(x, w["final.norm"], eps), w["head"], round16)
