"""Tebozen: configuration -> plan.

Every layer is ``x <- x + mixer(norm1(x)); x <- x + feed_forward(norm2(x))`` with RMS norms whose stored weight is the
difference from 1.  The mixer is one of three, layer by layer: the mLSTM's matrix memory; differential attention (two score
maps per head) with biases, a short convolution of q, k and v, a rotation of half-apart pairs, a sliding window and a gate
per head; attention through a latent (a rotation of neighbouring pairs, a gate per head), whose cached rows may be another
layer's (``kv_from``: the layer's run reads that run's cache).  The feed-forward is a set of ungated experts (relu squared)
behind a sigmoid router, the weights on the experts' inputs, plus a shared expert; or absent.  The embedding is scaled and
the output head is a matrix of its own.  Tensors: ``embed``, ``l<i>.norm1``, ``l<i>.norm2``, ``l<i>.mix.*``,
``l<i>.mlp.*``, ``final.norm``, ``head``.
"""
from __future__ import annotations

from ..config.registry import register_architecture
from ..config.tebozen import ARCHITECTURE, TebozenConfig
from ..engine.plan import LayerSpec, ModelPlan, Run
from ..parts.base import PartSpec

MEMORY_TINY = 1e-6      # joins the denominator of the matrix memory's output


def _mixer(kind: str, m: dict, width: int, eps: float):
    """(mixer spec, position spec or None)."""
    if kind == "mlstm":
        return PartSpec("mlstm", {"hidden_size": width, "heads": m["heads"], "key_dim": m["dim"], "vdim": m["vdim"],
                                  "gate_cap": m["gate_cap"], "norm_eps": eps, "tiny": MEMORY_TINY}), None
    rot = m["rot"]
    turn = {"theta": rot["base"], "rotary_dim": rot["dims"]}
    if kind == "attention":
        return (PartSpec("score_maps_attention",
                         {"hidden_size": width, "n_heads": m["heads"], "n_kv_heads": m["kv_heads"], "head_dim": m["dim"],
                          "value_dim": m["vdim"], "maps": 2, "biases": True, "conv": m["conv"], "norm_eps": eps, "scale": m["scale"],
                          "window": m["mask"]["size"] if m["mask"] else 0, "diff": m["diff"], "head_gate": True, "layout": "halves"}),
                PartSpec("rotary_neox", turn) if rot["dims"] else None)
    return (PartSpec("latent_attention",
                     {"hidden_size": width, "heads": m["heads"], "dim": m["dim"], "rot_dim": m["rot_dim"], "vdim": m["vdim"],
                      "kv_rank": m["kv_rank"], "scale": m["scale"], "head_gate": True, "shared_rows": m["kv_from"] is not None,
                      "norm_eps": eps}),
            PartSpec("rotary_pairs", turn) if rot["dims"] else None)


def _feed_forward(mlp, width: int):
    if mlp is None:
        return None
    return PartSpec("routed_experts",
                    {"hidden_size": width, "expert_size": mlp["expert"]["ff"], "experts": mlp["router"]["experts"],
                     "top": mlp["router"]["top"], "gated": False, "activation": "relu2", "scores": "sigmoid", "renormalize": False,
                     "weight_on": "input", "shared_size": mlp["shared"]["ff"] if mlp["shared"] else 0})


def tebozen_plan(cfg: TebozenConfig) -> ModelPlan:
    D, eps = cfg.width, cfg.norm_eps
    norm = {"dim": D, "eps": eps, "about_one": True}
    layers = []
    for i, layer in enumerate(cfg.layers):
        mixer, position = _mixer(layer["type"], layer["mixer"], D, eps)
        layers.append(LayerSpec(block=PartSpec("pre_norm", {"mixer_norm": "norm1", "ffn_norm": "norm2", "whole_names": True,
                                                            "mixer_prefix": "mix", "ffn_prefix": "mlp"}, prefix=f"l{i}."),
                                mixer=mixer, feed_forward=_feed_forward(layer["mlp"], D), norm=PartSpec("rms", norm), position=position))
    return ModelPlan(
        architecture=ARCHITECTURE, hidden_size=D, vocab_size=cfg.vocab,
        embedding=PartSpec("token", {"vocab_size": cfg.vocab, "hidden_size": D, "name": "embed", "scale": cfg.embedding_scale}),
        layers=layers, schedule=[Run(i, cache_of=layer["mixer"].get("kv_from")) for i, layer in enumerate(cfg.layers)],
        final_norm=PartSpec("rms", {**norm, "name": "final.norm"}),
        head=PartSpec("linear", {"vocab_size": cfg.vocab, "hidden_size": D, "tied": False, "name": "head", "tied_to": "embed"}),
        stop_token_ids=(), max_position=None)


register_architecture(ARCHITECTURE, TebozenConfig, tebozen_plan, replace=True)
