"""Configuration of the Tebozen design: a decoder whose layers are listed one by one, each with one of three mixers (the
mLSTM's matrix memory; differential attention behind a short convolution, within a sliding window; attention through a
latent, whose cached rows may be another layer's) and routed experts with a shared one, or no feed-forward.

config.json:  ``architecture`` (the design's name), ``vocab``, ``width``, ``norm.eps``, ``embedding.scale``, ``layers``: a
list of ``{"type": <mixer>, "mixer": {sizes and constants}, "mlp": {"kind": "moe", "expert": {"ff"}, "router": {"experts",
"top"}, "shared": {"ff"}} | null}``.  Every size and constant that can differ between two models of the design is read from
there.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from ..kernels.limits import conv_taps_refusal, latent_refusal, maps_attention_refusal, moe_refusal, state_matrix_refusal
from .base import ConfigError, ConfigReader, ModelConfig

ARCHITECTURE = "Tebozen"
MIXER_TYPES = ("mlstm", "attention", "latent_attention")


def _sub(r: ConfigReader, key: str, optional: bool = False):
    m = r.mapping(key, None) if optional else r.mapping(key)
    return None if m is None else ConfigReader(m, f"{r.where}: '{key}'")


def _refuse(where: str, refusal):
    if refusal:
        raise ConfigError(f"{where}: {refusal}")


def _read_rotation(r: ConfigReader, limit_key: str, limit: int) -> dict:
    rot = _sub(r, "rot")
    out = {"base": rot.number("base", positive=True), "dims": rot.integer("dims", minimum=0)}
    if out["dims"] % 2 or out["dims"] > limit:
        raise ConfigError(f"{rot.where}: key 'dims' ({out['dims']}) must be even and at most '{limit_key}' ({limit})")
    if not out["base"] > 1:
        raise ConfigError(f"{rot.where}: key 'base' must be > 1, got {out['base']}")
    return out


def _read_mixer(kind: str, r: ConfigReader) -> dict:
    w = r.where
    if kind == "mlstm":
        m = {k: r.integer(k, minimum=1) for k in ("dim", "heads", "vdim")}
        m["gate_cap"] = r.number("gate_cap", positive=True)
        _refuse(f"{w}: keys 'dim' and 'vdim'", state_matrix_refusal(m["dim"], m["vdim"]))
        return m
    if kind == "attention":
        m = {k: r.integer(k, minimum=1) for k in ("conv", "dim", "heads", "kv_heads", "vdim")}
        if m["heads"] % m["kv_heads"]:
            raise ConfigError(f"{w}: key 'heads' ({m['heads']}) must be a multiple of 'kv_heads' ({m['kv_heads']})")
        m["scale"] = r.number("scale", positive=True)
        m["diff"] = r.number("diff")
        mask = _sub(r, "mask", optional=True)
        m["mask"] = None if mask is None else {"size": mask.integer("size", minimum=1)}
        m["rot"] = _read_rotation(r, "dim", m["dim"])
        _refuse(f"{w}: key 'conv'", conv_taps_refusal(m["conv"]))
        _refuse(f"{w}: keys 'dim' and 'vdim'", maps_attention_refusal(2, m["dim"], m["vdim"]))
        return m
    m = {k: r.integer(k, minimum=1) for k in ("dim", "heads", "kv_rank", "vdim")}
    m["rot_dim"] = r.integer("rot_dim", minimum=0)
    m["scale"] = r.number("scale", positive=True)
    m["kv_from"] = r.integer("kv_from", None, minimum=0)
    m["rot"] = _read_rotation(r, "rot_dim", m["rot_dim"])
    _refuse(f"{w}: keys 'kv_rank' and 'rot_dim'", latent_refusal(m["kv_rank"], m["rot_dim"]))
    return m


def _read_mlp(r: ConfigReader | None):
    if r is None:
        return None
    kind = r.string("kind")
    if kind != "moe":
        raise ConfigError(f"{r.where}: key 'kind' must be 'moe', got {kind!r}")
    router = _sub(r, "router")
    experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
    _refuse(f"{router.where}: keys 'experts' and 'top'", moe_refusal(experts, top))
    shared = _sub(r, "shared", optional=True)
    return {"kind": "moe", "expert": {"ff": _sub(r, "expert").integer("ff", minimum=1)}, "router": {"experts": experts, "top": top},
            "shared": None if shared is None else {"ff": shared.integer("ff", minimum=1)}}


@dataclass(frozen=True)
class TebozenConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float = 1.0
    layers: tuple = field(default_factory=tuple)     # dicts: {"type", "mixer": {...}, "mlp": {...} | None}

    architecture = ARCHITECTURE

    @classmethod
    def from_reader(cls, r: ConfigReader) -> "TebozenConfig":
        vocab = r.integer("vocab", minimum=1)
        width = r.integer("width", minimum=1)
        eps = _sub(r, "norm").number("eps", positive=True)
        emb = _sub(r, "embedding", optional=True)
        scale = emb.number("scale", 1.0) if emb is not None else 1.0
        r.read_keys.add("layers")
        raw = r.data.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError(f"{r.where}: key 'layers' must be a list with at least one layer")
        layers = []
        for i, entry in enumerate(raw):
            lr = ConfigReader(entry, f"{r.where}: layers[{i}]")
            kind = lr.string("type")
            if kind not in MIXER_TYPES:
                raise ConfigError(f"{lr.where}: key 'type' must be one of {', '.join(MIXER_TYPES)}, got {kind!r}")
            layers.append({"type": kind, "mixer": _read_mixer(kind, _sub(lr, "mixer")), "mlp": _read_mlp(_sub(lr, "mlp", optional=True))})
        for i, layer in enumerate(layers):
            j = layer["mixer"].get("kv_from")
            if j is None:
                continue
            where = f"{r.where}: layers[{i}]: key 'kv_from' ({j})"
            if j >= i or layers[j]["type"] != "latent_attention" or layers[j]["mixer"]["kv_from"] is not None:
                raise ConfigError(f"{where} must name an earlier latent_attention layer with rows of its own")
            for k in ("kv_rank", "rot_dim", "rot"):
                if layer["mixer"][k] != layers[j]["mixer"][k]:
                    raise ConfigError(f"{where}: key '{k}' differs from that of layer {j}")
        return cls(vocab=vocab, width=width, norm_eps=eps, embedding_scale=scale, layers=tuple(layers))

    def to_dict(self) -> dict:
        import copy
        out = {"architecture": ARCHITECTURE, "embedding": {"scale": self.embedding_scale}, "layers": copy.deepcopy(list(self.layers)),
               "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        for layer in out["layers"]:                      # keys that stand for "none" are left out again
            for k in ("mask", "kv_from"):
                if k in layer["mixer"] and layer["mixer"][k] is None:
                    del layer["mixer"][k]
            if layer["mlp"] is not None and layer["mlp"]["shared"] is None:
                del layer["mlp"]["shared"]
        return out
