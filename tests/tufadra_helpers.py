"""Shared by the Tufadra tests: small configurations of their own, weights drawn so that every mechanism matters (O(1)
activations, corrections that move the choice and make choice scores negative, a query factor that grows fast, sharp
attention), model folders."""
from __future__ import annotations

import json
import os

import numpy as np
import torch

import plain_tufadra as pt


def attention(heads=6, kv_heads=2, dim=24, vdim=40, scale=0.3, coef=0.7, every=10):
    return {"type": "attention", "mixer": {"dim": dim, "heads": heads, "kv_heads": kv_heads, "scale": scale, "vdim": vdim,
                                           "q_temp": {"coef": coef, "every": every}}}


def moe(ff=40, experts=6, top=3, count=3, keep=2, scale=2.0, shared=56):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
            "router": {"experts": experts, "groups": {"count": count, "keep": keep}, "scale": scale, "top": top}}


def config(layers, width=64, vocab=96, eps=2e-5, max_positions=700):
    """layers: (mixer entry, mlp entry or None) pairs, or the number of an earlier layer whose tensors are used again."""
    out = []
    for i, layer in enumerate(layers):
        if isinstance(layer, int):
            out.append({**out[layer], "weights_of": layer})
        else:
            out.append({**layer[0], "mlp": layer[1]})
    return {"architecture": "Tufadra", "layers": out, "max_positions": max_positions, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# Sizes that share no value where they could be confused: key/value heads fewer than heads and as many, keys larger than
# values and the other way round, sizes of the tcgen05 prompt kernel and sizes that are no multiple of 8, groups of
# several experts, of one, and a single group, all experts chosen, layers without a feed-forward, layers that use
# another's tensors, directly and through a third.
MIXED = config([(attention(), moe()),
                (attention(heads=4, kv_heads=4, dim=16, vdim=16, coef=0.0, every=3), None),
                (attention(heads=3, kv_heads=1, dim=40, vdim=8, scale=0.2, every=33), moe(ff=24, experts=12, top=5, count=2, keep=1, shared=24)),
                0,
                (attention(heads=2, kv_heads=1, dim=64, vdim=64, scale=0.15), moe(ff=10, experts=5, top=5, count=1, keep=1, scale=0.7, shared=30)),
                1,
                (attention(heads=2, kv_heads=1, dim=12, vdim=20, coef=0.2, every=64), moe(ff=16, experts=4, top=2, count=4, keep=3, shared=8)),
                3])
# values that happen to be equal or 1
ONES = config([(attention(heads=1, kv_heads=1, dim=8, vdim=8, scale=1.0, coef=1.0, every=1), moe(ff=8, experts=1, top=1, count=1, keep=1, scale=1.0, shared=8)),
               0, (attention(heads=2, kv_heads=2, dim=8, vdim=8, every=1), moe(ff=8, experts=2, top=1, count=2, keep=1, scale=1.0, shared=1)),
               (attention(heads=1, kv_heads=1, dim=8, vdim=1), None)],
              width=16, vocab=37, eps=1e-6, max_positions=160)


def draw_weights(cfgd, seed=0, sharp=1.0):
    """float64 arrays by tensor name, every value a bfloat16 number, from the configuration alone.  ``sharp`` scales the
    query norms' weights: a sharper softmax shows a key that is seen or not seen."""
    rng = np.random.default_rng(seed)
    D, V = cfgd["width"], cfgd["vocab"]

    def matrix(*shape):
        return 1.3 * rng.standard_normal(shape) / np.sqrt(shape[-1])

    w = {"embed": rng.standard_normal((V, D)), "pos": 0.5 * rng.standard_normal((cfgd["max_positions"], D)),
         "final.norm": 0.3 * rng.standard_normal(D)}
    for i, layer in enumerate(cfgd["layers"]):
        if layer.get("weights_of") is not None:
            continue
        px, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        H, G, K, P = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        w[px + "norm1"] = 0.3 * rng.standard_normal(D)
        w[px + "mix.q"], w[px + "mix.k"], w[px + "mix.v"] = matrix(H * K, D), matrix(G * K, D), matrix(G * P, D)
        w[px + "mix.o"] = matrix(D, H * P)
        w[px + "mix.q.norm"] = sharp * (1.0 + 0.3 * rng.standard_normal(H * K))
        w[px + "mix.k.norm"] = 1.0 + 0.3 * rng.standard_normal(G * K)
        if mlp:
            p, E, F, Fs = px + "mlp.", mlp["router"]["experts"], mlp["expert"]["ff"], mlp["shared"]["ff"]
            w[p + "router"], w[p + "correction"] = 1.5 * matrix(E, D), -0.4 + 0.4 * rng.standard_normal(E)
            for e in range(E):
                w[p + f"e{e}.up"], w[p + f"e{e}.down"] = matrix(F, D), matrix(D, F)
            w[p + "shared.up"], w[p + "shared.down"], w[p + "shared.sg"] = matrix(Fs, D), matrix(D, Fs), matrix(1, D)
    return {k: pt.round_bf16(v) for k, v in w.items()}


def clear_choices(cfgd, w, n, seed, round16=False, margin=0.02):
    """A random sequence of n tokens in which no router's choice is a close call (a token with one is drawn again), and the
    plain implementation's logits: rounding then changes no choice, and every row can be held to a tolerance."""
    rng = np.random.default_rng(seed)
    tokens = rng.integers(0, cfgd["vocab"], n).tolist()
    for _ in range(20 * n):
        margins = []
        logits = pt.forward(cfgd, w, tokens, round16, margins=margins)
        close = np.nonzero(np.min(margins, axis=0) < margin)[0]
        if not close.size:
            return tokens, logits
        for i in close:
            tokens[i] = int(rng.integers(0, cfgd["vocab"]))
    raise AssertionError("no sequence without close calls was found")


def write_folder(path, cfgd, w):
    from questwend_b200.weights import write_safetensors
    os.makedirs(path, exist_ok=True)
    write_safetensors(os.path.join(path, "model.safetensors"),
                      {k: torch.from_numpy(np.asarray(v, dtype=np.float32)).to(torch.bfloat16) for k, v in w.items()})
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfgd, f)
    return str(path)
