"""Configuration of the Tufadra design: a decoder whose layers are listed one by one, every layer softmax attention and
routed experts side by side behind one norm: ``x <- x + (attention(h) + experts(h))``, ``h = norm1(x)``.  Positions enter
through a learned vector per position on the embedding and a factor on the queries that grows with the position; q and k
are normed over their whole projections.  A layer may use another layer's tensors with a cache of its own
(``weights_of``).  The output head is the embedding table.

config.json:  ``architecture`` (the design's name), ``vocab``, ``width``, ``norm.eps``, ``max_positions`` (rows of the
position table), ``layers``: a list of ``{"type": "attention", "mixer": {sizes and constants}, "mlp": {"kind": "moe",
"expert": {"ff"}, "router": {"experts", "top", "scale", "groups": {"count", "keep"}}, "shared": {"ff"}} | null,
"weights_of": j}``.  Every size and constant that can differ between two models of the design is read from there.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from ..kernels.limits import maps_attention_refusal, moe_refusal
from .base import ConfigError, ConfigReader, ModelConfig

ARCHITECTURE = "Tufadra"
MIXER_TYPES = ("attention",)


def _sub(r: ConfigReader, key: str, optional: bool = False):
    m = r.mapping(key, None) if optional else r.mapping(key)
    return None if m is None else ConfigReader(m, f"{r.where}: '{key}'")


def _refuse(where: str, refusal):
    if refusal:
        raise ConfigError(f"{where}: {refusal}")


def _read_mixer(r: ConfigReader) -> dict:
    m = {k: r.integer(k, minimum=1) for k in ("dim", "heads", "kv_heads", "vdim")}
    if m["heads"] % m["kv_heads"]:
        raise ConfigError(f"{r.where}: key 'heads' ({m['heads']}) must be a multiple of 'kv_heads' ({m['kv_heads']})")
    m["scale"] = r.number("scale", positive=True)
    temp = _sub(r, "q_temp", optional=True)
    m["q_temp"] = {"coef": 0.0, "every": 1.0} if temp is None else {"coef": temp.number("coef"), "every": temp.number("every", positive=True)}
    _refuse(f"{r.where}: keys 'dim' and 'vdim'", maps_attention_refusal(1, m["dim"], m["vdim"]))
    return m


def _read_mlp(r: ConfigReader | None):
    if r is None:
        return None
    kind = r.string("kind")
    if kind != "moe":
        raise ConfigError(f"{r.where}: key 'kind' must be 'moe', got {kind!r}")
    router = _sub(r, "router")
    experts, top = router.integer("experts", minimum=1), router.integer("top", minimum=1)
    groups = _sub(router, "groups", optional=True)
    count, keep = (1, 1) if groups is None else (groups.integer("count", minimum=1), groups.integer("keep", minimum=1))
    where = router.where if groups is None else groups.where
    _refuse(f"{router.where}: keys 'experts' and 'top'", moe_refusal(experts, top))
    _refuse(f"{where}: keys 'count' and 'keep'", moe_refusal(experts, top, count, keep))
    out = {"kind": "moe", "expert": {"ff": _sub(r, "expert").integer("ff", minimum=1)},
           "router": {"experts": experts, "groups": {"count": count, "keep": keep}, "scale": router.number("scale", 1.0), "top": top}}
    shared = _sub(r, "shared", optional=True)
    out["shared"] = None if shared is None else {"ff": shared.integer("ff", minimum=1)}
    return out


@dataclass(frozen=True)
class TufadraConfig(ModelConfig):
    vocab: int
    width: int
    norm_eps: float
    max_positions: int
    layers: tuple = field(default_factory=tuple)     # dicts: {"type", "mixer": {...}, "mlp": {...} | None, "weights_of": j | None}

    architecture = ARCHITECTURE

    @property
    def max_position_embeddings(self) -> int:        # the longest sequence, under the name that other configurations give it
        return self.max_positions

    def tensors_of(self, i: int) -> int:
        """The layer whose tensors layer i uses (itself, for most)."""
        while self.layers[i]["weights_of"] is not None:
            i = self.layers[i]["weights_of"]
        return i

    @classmethod
    def from_reader(cls, r: ConfigReader) -> "TufadraConfig":
        vocab = r.integer("vocab", minimum=1)
        width = r.integer("width", minimum=1)
        eps = _sub(r, "norm").number("eps", positive=True)
        max_positions = r.integer("max_positions", minimum=1)
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
            of = lr.integer("weights_of", None, minimum=0)
            if of is not None and of >= len(raw):
                raise ConfigError(f"{lr.where}: key 'weights_of' ({of}) names no layer; there are {len(raw)}")
            layers.append({"type": kind, "mixer": _read_mixer(_sub(lr, "mixer")), "mlp": _read_mlp(_sub(lr, "mlp", optional=True)),
                           "weights_of": of})
        for i, layer in enumerate(layers):
            seen, j = {i}, layer["weights_of"]
            while j is not None:
                if j in seen:
                    raise ConfigError(f"{r.where}: layers[{i}]: key 'weights_of' leads back to layer {j}: no layer holds the tensors")
                seen.add(j)
                if any(layer[k] != layers[j][k] for k in ("type", "mixer", "mlp")):
                    raise ConfigError(f"{r.where}: layers[{i}]: key 'weights_of': the entry differs from that of layer {j}")
                j = layers[j]["weights_of"]
        return cls(vocab=vocab, width=width, norm_eps=eps, max_positions=max_positions, layers=tuple(layers))

    def to_dict(self) -> dict:
        import copy
        out = {"architecture": ARCHITECTURE, "layers": copy.deepcopy(list(self.layers)), "max_positions": self.max_positions,
               "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        for layer in out["layers"]:                      # keys that stand for "none" are left out again
            if layer["weights_of"] is None:
                del layer["weights_of"]
            if layer["mlp"] is not None and layer["mlp"]["shared"] is None:
                del layer["mlp"]["shared"]
        return out
