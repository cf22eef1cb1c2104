"""Shared by the Tebozen tests: small configurations of their own, weights drawn so that every mechanism matters (O(1)
activations, gates that reach their cap, memories that last and memories that fade, a second score map that counts), model
folders."""
from __future__ import annotations

import json
import os

import numpy as np
import torch

import plain_tebozen as pz


def attention(heads=4, kv_heads=2, dim=16, vdim=24, conv=3, window=20, dims=8, base=300.0, scale=0.4, diff=0.3):
    return {"type": "attention", "mixer": {"conv": conv, "diff": diff, "dim": dim, "heads": heads, "kv_heads": kv_heads,
                                           "mask": {"size": window}, "rot": {"base": base, "dims": dims}, "scale": scale, "vdim": vdim}}


def memory(heads=3, dim=8, vdim=12, cap=4.0):
    return {"type": "mlstm", "mixer": {"dim": dim, "gate_cap": cap, "heads": heads, "vdim": vdim}}


def latent(heads=3, dim=16, rot_dim=8, vdim=24, rank=40, base=500.0, scale=0.3, kv_from=None):
    m = {"dim": dim, "heads": heads, "kv_rank": rank, "rot": {"base": base, "dims": rot_dim}, "rot_dim": rot_dim, "scale": scale, "vdim": vdim}
    return {"type": "latent_attention", "mixer": m if kv_from is None else {**m, "kv_from": kv_from}}


def moe(ff=40, experts=6, top=2, shared=56):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return {**out, "shared": {"ff": shared}} if shared else out


def config(layers, width=64, vocab=90, eps=2e-5, embedding_scale=1.7):
    """layers: (mixer entry, mlp entry or None) pairs."""
    return {"architecture": "Tebozen", "embedding": {"scale": embedding_scale}, "layers": [{**mixer, "mlp": mlp} for mixer, mlp in layers],
            "norm": {"eps": eps}, "vocab": vocab, "width": width}


# Sizes that share no value where they could be confused: key/value heads fewer than heads and as many, keys larger than
# values and the other way round, windows below, at and above a page, one to four taps, a turn of a part of a map and of all
# of it, sizes that are no multiple of 8, two latent caches and three layers that read them with heads of their own, a layer
# without a feed-forward, experts without a shared one, all experts chosen.
MIXED = config([(latent(), moe()),
                (memory(), moe(ff=24, experts=9, top=4, shared=16)),
                (attention(), moe(ff=16, experts=5, top=1, shared=72)),
                (latent(heads=5, dim=8, vdim=16, kv_from=0, scale=0.5), None),
                (attention(heads=3, kv_heads=1, dim=12, vdim=20, conv=4, window=64, dims=12, base=50.0, diff=0.7), moe(ff=10, experts=3, top=3, shared=30)),
                (memory(heads=2, dim=20, vdim=6, cap=9.0), None),
                (latent(heads=2, dim=12, rot_dim=4, vdim=10, rank=24, base=90.0), moe(shared=0)),
                (attention(heads=2, kv_heads=2, dim=32, vdim=8, conv=1, window=130, dims=32), moe(ff=8, experts=4, top=2)),
                (latent(heads=4, dim=24, rot_dim=4, vdim=8, rank=24, base=90.0, kv_from=6), moe(ff=56, experts=7, top=3, shared=8)),
                (latent(heads=1, dim=16, vdim=40, kv_from=0), None)])
# values that happen to be equal or 1
ONES = config([(memory(heads=1, dim=1, vdim=2, cap=1.0), moe(ff=8, experts=1, top=1, shared=1)),
               (attention(heads=1, kv_heads=1, dim=8, vdim=8, conv=1, window=1, dims=0, scale=1.0, diff=0.0), None),
               (latent(heads=1, dim=8, rot_dim=8, vdim=8, rank=8, scale=1.0), moe(ff=8, experts=2, top=1, shared=8)),
               (attention(heads=2, kv_heads=2, dim=8, vdim=8, conv=2, window=2, dims=8), None),
               (latent(heads=1, dim=8, rot_dim=8, vdim=8, rank=8, scale=1.0, kv_from=2), None),
               (memory(heads=8, dim=8, vdim=8, cap=8.0), None)],
              width=16, vocab=37, eps=1e-6, embedding_scale=1.0)


def draw_weights(cfgd, seed=0, lasting=False, sharp=1.0):
    """float64 arrays by tensor name, every value a bfloat16 number, from the configuration alone.  ``lasting``: forget gates
    near 1; ``sharp`` scales the query projections of both kinds of attention: a key that is seen or not seen shows."""
    rng = np.random.default_rng(seed)
    D, V = cfgd["width"], cfgd["vocab"]

    def matrix(*shape):
        return 1.3 * rng.standard_normal(shape) / np.sqrt(shape[-1])

    w = {"embed": rng.standard_normal((V, D)) / cfgd["embedding"]["scale"], "final.norm": 0.3 * rng.standard_normal(D), "head": matrix(V, D)}
    for i, layer in enumerate(cfgd["layers"]):
        px, m, mlp = f"l{i}.", layer["mixer"], layer["mlp"]
        p, H, K, P = px + "mix.", m["heads"], m["dim"], m["vdim"]
        w[px + "norm1"] = 0.3 * rng.standard_normal(D)
        w[p + "o"] = matrix(D, H * P)
        if layer["type"] == "mlstm":
            w[p + "q"], w[p + "k"], w[p + "v"], w[p + "g"] = matrix(H * K, D), matrix(H * K, D), matrix(H * P, D), matrix(H * P, D)
            w[p + "norm"] = 1.0 + 0.3 * rng.standard_normal(H * P)
            w[p + "i"], w[p + "f"] = 3.0 * matrix(H, D), (0.3 if lasting else 2.0) * matrix(H, D)
            w[p + "i.b"] = rng.standard_normal(H)
            w[p + "f.b"] = rng.uniform(8.0, 12.0, H) if lasting else rng.uniform(-1.0, 5.0, H)
        elif layer["type"] == "attention":
            G = m["kv_heads"]
            for name, n in (("q", H * 2 * K), ("k", G * 2 * K), ("v", G * P)):
                w[p + name] = (sharp if name == "q" else 1.0) * matrix(n, D)
                w[p + name + ".b"] = 0.4 * rng.standard_normal(n)
                w[p + name + ".conv"] = 0.6 * rng.standard_normal((n, m["conv"]))
            for name in ("lq1", "lk1", "lq2", "lk2"):
                w[p + name] = 0.9 * rng.standard_normal(K) / K ** 0.25
            w[p + "g"] = 1.5 * matrix(H, D)
        else:
            L, R = m["kv_rank"], m["rot_dim"]
            w[p + "q"] = sharp * matrix(H * (K + R), D)
            if m.get("kv_from") is None:
                w[p + "dkv"], w[p + "dkv.norm"] = matrix(L + R, D), 1.0 + 0.3 * rng.standard_normal(L)
            w[p + "uk"], w[p + "uv"], w[p + "g"] = matrix(H * K, L), matrix(H * P, L), 1.5 * matrix(H, D)
        if mlp:
            w[px + "norm2"] = 0.3 * rng.standard_normal(D)
            p, E, F = px + "mlp.", mlp["router"]["experts"], mlp["expert"]["ff"]
            w[p + "router"] = 1.5 * matrix(E, D)
            for e in range(E):
                w[p + f"e{e}.up"], w[p + f"e{e}.down"] = matrix(F, D), 0.6 * matrix(D, F)
            if mlp.get("shared"):
                w[p + "shared.up"], w[p + "shared.down"] = matrix(mlp["shared"]["ff"], D), 0.6 * matrix(D, mlp["shared"]["ff"])
    return {k: pz.round_bf16(v) for k, v in w.items()}


def clear_choices(cfgd, w, n, seed, round16=False, margin=0.01):
    """A random sequence of n tokens in which no router's choice is a close call (a token with one is drawn again), and the
    plain implementation's logits: rounding then changes no choice, and every row can be held to a tolerance."""
    rng = np.random.default_rng(seed)
    tokens = rng.integers(0, cfgd["vocab"], n).tolist()
    for _ in range(20 * n):
        margins = []
        logits = pz.forward(cfgd, w, tokens, round16, margins=margins)
        close = np.nonzero(np.min(margins, axis=0) < margin)[0]
        if not close.size:
            return tokens, logits
        tokens[close[0]] = int(rng.integers(0, cfgd["vocab"]))      # a token changes the choices of all after it: the first one only
    raise AssertionError("no sequence without close calls was found")


def write_folder(path, cfgd, w):
    from questwend_b200.weights import write_safetensors
    os.makedirs(path, exist_ok=True)
    write_safetensors(os.path.join(path, "model.safetensors"),
                      {k: torch.from_numpy(np.asarray(v, dtype=np.float32)).to(torch.bfloat16) for k, v in w.items()})
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfgd, f)
    return str(path)
