"""FopezenConfig: the sizes, constants and order of layers of a Fopezen decoder, from config.json.

The file is nested like the other in-house families': `layers` lists the layers, each with its `type` (the mixer:
`attention` or `attention_2`, two forms of grouped-query attention), the mixer's sizes and constants under `mixer`, and
its feed-forward under `mlp` (null: none; `kind` dense with width `ff`). Model-wide: `vocab`, `width` and `norm.eps`.
Every layer states its own sizes, so two layers of a model may differ in all of them.

A mixer: `heads`, `kv_heads`, `dim` (query/key width of a head), `vdim` (value width), `scale` (multiplies q . k), `mask`
(`size` positions of a sliding window, the query's own included, and `keep_first`, absent 0: how many of the sequence's
first positions stay visible behind it; no `mask`: every earlier position is seen) and `v_mix` (absent false: whether the
layer's values are mixed with those of the first layer that says so; such layers have equally many value columns).
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .base import ConfigError, KeyReader

LAYER_TYPES = ("attention", "attention_2")


@dataclass(frozen=True)
class FopezenMixerConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None             # positions of the sliding window; None: no window
    keep_first: int
    v_mix: bool


@dataclass(frozen=True)
class FopezenDenseConfig:
    ff: int


@dataclass(frozen=True)
class FopezenLayerConfig:
    type: str
    mixer: FopezenMixerConfig
    mlp: FopezenDenseConfig | None


@dataclass(frozen=True)
class FopezenConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    layers: tuple[FopezenLayerConfig, ...]
    raw: dict = field(default_factory=dict, compare=False, repr=False)

    @property
    def first_mixed(self) -> int | None:
        """The first layer whose configuration says `v_mix`: the one whose values the later ones take in."""
        return next((i for i, l in enumerate(self.layers) if l.mixer.v_mix), None)

    def to_json_dict(self) -> dict:
        """The config.json that reads back as this record."""
        def mixer(m: FopezenMixerConfig):
            out = {"dim": m.dim, "heads": m.heads, "kv_heads": m.kv_heads, "scale": m.scale, "v_mix": m.v_mix, "vdim": m.vdim}
            if m.window is not None:
                out["mask"] = {"keep_first": m.keep_first, "size": m.window}
            return out
        return {"architecture": self.architecture,
                "layers": [{"mixer": mixer(l.mixer), "mlp": None if l.mlp is None else {"ff": l.mlp.ff, "kind": "dense"}, "type": l.type}
                           for l in self.layers],
                "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "FopezenConfig":
        r = KeyReader(raw, where)
        name = r.string("architecture", default=None)
        if name is None:
            archs = r.any("architectures")
            if not (isinstance(archs, list) and archs and isinstance(archs[0], str)):
                raise ConfigError(f"{where}: 'architecture' must name the model")
            name = archs[0]
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        eps = KeyReader(_obj(r, "norm", where), where + ":norm").number("eps", positive=True)
        entries = r.any("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError(f"{where}: 'layers' must be a list with an entry per layer")
        layers = tuple(_layer(e, f"{where}:layers[{i}]") for i, e in enumerate(entries))
        mixed = {l.mixer.kv_heads * l.mixer.vdim for l in layers if l.mixer.v_mix}
        if len(mixed) > 1:
            raise ConfigError(f"{where}: the layers with 'v_mix' have different numbers of value columns ({sorted(mixed)})")
        return cls(name, vocab, width, eps, layers, raw)


def _obj(r: KeyReader, key: str, where: str) -> dict:
    v = r.any(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: {key!r} must be an object")
    return v


def _layer(e, where: str) -> FopezenLayerConfig:
    r = KeyReader(e, where)
    kind = r.string("type", choices=LAYER_TYPES)
    mw = where + ":mixer"
    m = KeyReader(_obj(r, "mixer", where), mw)
    heads, kv_heads = m.integer("heads", minimum=1), m.integer("kv_heads", minimum=1)
    if heads % kv_heads:
        raise ConfigError(f"{mw}: {heads} heads cannot share {kv_heads} key/value heads")
    dim, vdim = m.integer("dim", minimum=1), m.integer("vdim", minimum=1)
    if dim > 512 or vdim > 512:
        raise ConfigError(f"{mw}: heads of {dim} and {vdim}; the attention kernels take widths up to 512")
    window, keep = None, 0
    if m.any("mask") is not None:
        mask = KeyReader(_obj(m, "mask", mw), mw + ":mask")
        window, keep = mask.integer("size", minimum=1), mask.integer("keep_first", default=0, minimum=0)
    mixer = FopezenMixerConfig(heads, kv_heads, dim, vdim, m.number("scale"), window, keep, m.boolean("v_mix", default=False))
    mlp = r.any("mlp")
    ff = None
    if mlp is not None:
        f = KeyReader(mlp, where + ":mlp")
        f.string("kind", choices=("dense",))
        ff = FopezenDenseConfig(f.integer("ff", minimum=1))
    return FopezenLayerConfig(kind, mixer, ff)
