"""The Tufadra design once more, plain and slow: NumPy float64, whole sequences, no cache, one function per mechanism.
It shares no code with the library; the tests compare the engine with it.  A model is a dict ``cfg`` (the parsed
config.json) and a dict ``w`` of float64 arrays by tensor name.

``round16`` rounds where the bfloat16 engine rounds: the operands of the matrix products, the queries, and the cached
keys and values; everything else stays in float64.
"""
from __future__ import annotations

import math

import numpy as np


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
    return 1.0 / (1.0 + np.exp(-z))


_erf = np.frompyfunc(math.erf, 1, 1)


def gelu_exact(z):
    """z times the normal distribution's function at z."""
    z = np.asarray(z, dtype=np.float64)
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)).astype(np.float64))


def unit_rms(x, eps):
    """x over its root mean square along the last axis, eps inside the root."""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def norm_about_one(x, weight, eps):
    """RMS norm whose stored weight is the difference from 1."""
    return unit_rms(x, eps) * (1.0 + weight)


# ----------------------------------------------------------------------------- embedding
def embed(tokens, w):
    """Table rows plus a learned vector for each position."""
    tokens = np.asarray(tokens)
    return w["embed"][tokens] + w["pos"][np.arange(len(tokens))]


# ----------------------------------------------------------------------------- attention
def query_temperature(positions, coef, every):
    """1 + coef ln(floor((p + 1) / every) + 1): a factor on the query that grows with the position."""
    return 1.0 + coef * np.log(np.floor((np.asarray(positions, dtype=np.float64) + 1.0) / every) + 1.0)


def attention(h, m, w, px, eps, round16=False):
    """Grouped-query causal softmax attention: q and k normed over the whole projection, no rotation, a temperature on q."""
    n = h.shape[0]
    H, G, K, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms(product(h, w[px + "q"], round16), eps) * w[px + "q.norm"]
    k = unit_rms(product(h, w[px + "k"], round16), eps) * w[px + "k.norm"]
    v = product(h, w[px + "v"], round16).reshape(n, G, P)
    q = q * query_temperature(np.arange(n), m["q_temp"]["coef"], m["q_temp"]["every"])[:, None]
    q, k = q.reshape(n, H, K), k.reshape(n, G, K)
    if round16:
        q, k, v = round_bf16(q), round_bf16(k), round_bf16(v)
    seen = np.tril(np.ones((n, n), dtype=bool))
    o = np.zeros((n, H, P))
    for hd in range(H):
        g = hd // (H // G)
        s = np.where(seen, q[:, hd] @ k[:, g].T * m["scale"], -np.inf)
        e = np.exp(s - s.max(axis=-1, keepdims=True))
        o[:, hd] = e @ v[:, g] / e.sum(axis=-1, keepdims=True)
    return product(o.reshape(n, H * P), w[px + "o"], round16)


MIXERS = {"attention": attention}


# ----------------------------------------------------------------------------- feed-forward
def route(z, correction, router):
    """Router logits z [n, experts] -> (chosen [n, top], weights [n, top]), best first, ties to the lower index."""
    n, E = z.shape
    groups = router.get("groups") or {"count": 1, "keep": 1}
    count, keep, top = groups["count"], groups["keep"], router["top"]
    size = E // count
    s = sigmoid(z)
    chosen, weights = np.zeros((n, top), dtype=int), np.zeros((n, top))
    for t in range(n):
        c = s[t] + correction
        group_score = [sum(sorted(c[g * size:(g + 1) * size])[-2:]) for g in range(count)]
        kept = sorted(range(count), key=lambda g: (-group_score[g], g))[:keep]
        c = np.array([c[e] if e // size in kept else -np.inf for e in range(E)])
        chosen[t] = sorted(range(E), key=lambda e: (-c[e], e))[:top]
        weights[t] = s[t, chosen[t]]
        weights[t] *= router["scale"] / (weights[t].sum() + 1e-20)
    return chosen, weights


def route_margin(z, correction, router):
    """How far each token's choice is from another one: the least gap, in choice scores, between what is taken and the next
    best that is not (groups, and experts inside the groups that are taken)."""
    n, E = z.shape
    groups = router.get("groups") or {"count": 1, "keep": 1}
    count, keep, top = groups["count"], groups["keep"], router["top"]
    c = (sigmoid(z) + correction).reshape(n, count, E // count)
    g = np.sort(c, axis=-1)[..., -2:].sum(axis=-1)
    order = np.argsort(-g, axis=-1, kind="stable")
    ranked = np.take_along_axis(g, order, axis=-1)
    margin = ranked[:, keep - 1] - ranked[:, keep] if keep < count else np.full(n, np.inf)
    inside = -np.sort(-np.take_along_axis(c, order[:, :keep, None], axis=1).reshape(n, -1), axis=-1)
    if top < inside.shape[1]:
        margin = np.minimum(margin, inside[:, top - 1] - inside[:, top])
    return margin


def expert(h, w, px, round16=False):
    return product(gelu_exact(product(h, w[px + "up"], round16)), w[px + "down"], round16)


def shared_expert(h, w, px, round16=False):
    """Runs for every token, times a gate of one number a token."""
    return expert(h, w, px, round16) * sigmoid(product(h, w[px + "sg"], round16))


def experts(h, mlp, w, px, round16=False, margins=None):
    z = product(h, w[px + "router"], round16)
    chosen, weights = route(z, w[px + "correction"], mlp["router"])
    if margins is not None:
        margins.append(route_margin(z, w[px + "correction"], mlp["router"]))
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        t, k = np.nonzero(chosen == e)
        if t.size:
            out[t] += weights[t, k][:, None] * expert(h[t], w, px + f"e{e}.", round16)
    if mlp.get("shared"):
        out = out + shared_expert(h, w, px + "shared.", round16)
    return out


# ----------------------------------------------------------------------------- the model
def weights_layer(cfg, i):
    """The layer whose tensors layer i uses."""
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


def forward(cfg, w, tokens, round16=False, taps=None, margins=None):
    """Logits [n, vocab] of one sequence; ``taps``, a list, receives the stream after every layer, ``margins`` every
    router's margin for every token."""
    eps = cfg["norm"]["eps"]
    x = embed(tokens, w)
    for i, layer in enumerate(cfg["layers"]):
        px = f"l{weights_layer(cfg, i)}."
        h = norm_about_one(x, w[px + "norm1"], eps)
        y = MIXERS[layer["type"]](h, layer["mixer"], w, px + "mix.", eps, round16)
        if layer.get("mlp") is not None:
            y = y + experts(h, layer["mlp"], w, px + "mlp.", round16, margins)
        x = x + y
        if taps is not None:
            taps.append(x.copy())
    return product(norm_about_one(x, w["final.norm"], eps), w["embed"], round16)
