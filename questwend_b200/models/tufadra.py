"""Tufadra: configuration -> plan.

Every layer is ``x <- x + (mixer(h) + feed_forward(h))`` with ``h = norm1(x)``, one RMS norm whose stored weight is the
difference from 1.  The mixer is grouped-query causal softmax attention without a rotation: q and k are RMS-normed over
their whole projections (before the heads are split) and q is multiplied by a factor that grows with its position.  The
feed-forward is a set of ungated experts (exact GELU) behind a sigmoid router that chooses by corrected scores inside the
best groups of experts, plus a shared expert times a gate of one number a token.  The embedding adds a learned vector for
each position; the output head is the embedding table.  A layer with ``weights_of`` is a second run of that layer in the
schedule: the same tensors, a cache of its own.  Tensors: ``embed``, ``pos``, ``l<i>.norm1``, ``l<i>.mix.*``,
``l<i>.mlp.*``, ``final.norm``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.tufadra import ARCHITECTURE, TufadraConfig
from ..engine.plan import LayerSpec, ModelPlan, Run
from ..parts.base import PartSpec

WEIGHT_SUM_EPS = 1e-20      # on the sum that the chosen experts' scores are divided by


def _mixer(m: dict, width: int, eps: float) -> PartSpec:
    return PartSpec("score_maps_attention",
                    {"hidden_size": width, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                     "value_dim": m["vdim"], "maps": 1, "qk_norm": True, "qk_norm_over": "projection", "norm_eps": eps,
                     "scale": m["scale"], "q_temp_coef": m["q_temp"]["coef"], "q_temp_every": m["q_temp"]["every"]})


def _feed_forward(mlp, width: int):
    if mlp is None:
        return None
    router = mlp["router"]
    return PartSpec("routed_experts",
                    {"hidden_size": width, "expert_size": mlp["expert"]["ff"], "experts": router["experts"], "top": router["top"],
                     "gated": False, "activation": "gelu", "scores": "sigmoid", "correction": True,
                     "groups": router["groups"]["count"], "groups_kept": router["groups"]["keep"], "renormalize": True,
                     "sum_eps": WEIGHT_SUM_EPS, "weight_scale": router["scale"],
                     "shared_size": mlp["shared"]["ff"] if mlp["shared"] else 0, "shared_gate": True})


def tufadra_plan(cfg: TufadraConfig) -> ModelPlan:
    D, eps = cfg.width, cfg.norm_eps
    norm = {"dim": D, "eps": eps, "about_one": True}
    layers, place = [], {}
    for i, layer in enumerate(cfg.layers):
        if layer["weights_of"] is not None:
            continue
        place[i] = len(layers)
        layers.append(LayerSpec(block=PartSpec("parallel_residual", {"norm": "norm1", "mixer_prefix": "mix", "ffn_prefix": "mlp"},
                                               prefix=f"l{i}."),
                                mixer=_mixer(layer["mixer"], D, eps), feed_forward=_feed_forward(layer["mlp"], D),
                                norm=PartSpec("rms", norm)))
    return ModelPlan(
        architecture=ARCHITECTURE, hidden_size=D, vocab_size=cfg.vocab,
        embedding=PartSpec("token", {"vocab_size": cfg.vocab, "hidden_size": D, "name": "embed", "positions": "pos",
                                     "max_positions": cfg.max_positions}),
        layers=layers, schedule=[Run(place[cfg.tensors_of(i)]) for i in range(len(cfg.layers))],
        final_norm=PartSpec("rms", {**norm, "name": "final.norm"}),
        head=PartSpec("linear", {"vocab_size": cfg.vocab, "hidden_size": D, "tied": True, "name": "head", "tied_to": "embed"}),
        stop_token_ids=(), max_position=cfg.max_positions, position_limit=cfg.max_positions)


register_architecture(ARCHITECTURE, TufadraConfig, tufadra_plan, replace=True)
