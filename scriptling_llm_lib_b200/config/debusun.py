"""DebusunConfig: the sizes, constants and order of layers of a Debusun decoder, from config.json.

The file is nested like the other in-house families': `layers` lists the layers, each with its `type` (the mixer:
`attention`, `latent_attention` or `mamba2`), the mixer's sizes and constants under `mixer` and its feed-forward under
`mlp` (null: none; `kind` dense with width `ff`). Model-wide: `vocab`, `width`, `norm.eps`, `embedding` (`scale`, absent
1, multiplies the token's row; `bigram` with `buckets`, `mul_prev`, `mul_cur`, absent: no pair table) and `loop` (`start`,
`stop`, `times`: the run of layers from `start` up to, not including, `stop` is gone through that many times on one set
of weights; absent: every layer once). Every layer states its own sizes, so two layers of a model may differ in all of them.

An `attention` mixer: `heads`, `kv_heads`, `dim` (query/key width of a head), `vdim` (value width), `scale` (multiplies
q . k), `mask.size` (positions of a sliding window, the query's own included; no `mask`: every earlier key), `rot` (`dims`
leading dims of a head that turn in neighbouring pairs, `base`; no `rot` or `dims` 0: no rotation). A `latent_attention`
mixer: `heads`, `dim` and `rot_dim` (unrotated and rotated query/key dims of a head), `vdim`, `kv_rank`, `scale`, `mask`, `rot`
(`base`, `dims` = `rot_dim`, optionally `scaling` with `factor`, `original`, `fast`, `slow`). A `mamba2` mixer: `heads`, `vdim`
(channels of a head), `state` (state size), `groups` (runs of heads that share input and read-out vectors), `conv` (taps of
the short convolution) and `norm_groups` (equal runs of columns the read-out's norm takes apart).
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .base import ConfigError, KeyReader

LAYER_TYPES = ("attention", "latent_attention", "mamba2")


@dataclass(frozen=True)
class DebusunRotation:
    dims: int
    base: float
    scaling: dict | None       # {"factor", "original", "fast", "slow"} or None


@dataclass(frozen=True)
class DebusunAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int | None
    rot: DebusunRotation | None


@dataclass(frozen=True)
class DebusunLatentConfig:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int | None
    rot: DebusunRotation | None


@dataclass(frozen=True)
class DebusunMamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int


@dataclass(frozen=True)
class DebusunLayerConfig:
    type: str
    mixer: DebusunAttentionConfig | DebusunLatentConfig | DebusunMamba2Config
    ff: int | None             # width of the dense feed-forward; None: the layer has none


@dataclass(frozen=True)
class DebusunBigram:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class DebusunLoop:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class DebusunConfig:
    architecture: str
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    bigram: DebusunBigram | None
    loop: DebusunLoop | None
    layers: tuple[DebusunLayerConfig, ...]
    raw: dict = field(default_factory=dict, compare=False, repr=False)

    def to_json_dict(self) -> dict:
        """The config.json that reads back as this record."""
        def mixer(m):
            if isinstance(m, DebusunMamba2Config):
                return {"conv": m.conv, "groups": m.groups, "heads": m.heads, "norm_groups": m.norm_groups, "state": m.state,
                        "vdim": m.vdim}
            out = {"dim": m.dim, "heads": m.heads, "scale": m.scale, "vdim": m.vdim}
            if isinstance(m, DebusunAttentionConfig):
                out["kv_heads"] = m.kv_heads
            else:
                out.update(kv_rank=m.kv_rank, rot_dim=m.rot_dim)
            if m.window is not None:
                out["mask"] = {"size": m.window}
            if m.rot is not None:
                out["rot"] = {"base": m.rot.base, "dims": m.rot.dims}
                if m.rot.scaling is not None:
                    out["rot"]["scaling"] = dict(m.rot.scaling)
            return out
        embedding = {"scale": self.embedding_scale}
        if self.bigram is not None:
            embedding["bigram"] = {"buckets": self.bigram.buckets, "mul_cur": self.bigram.mul_cur, "mul_prev": self.bigram.mul_prev}
        out = {"architecture": self.architecture, "embedding": embedding,
               "layers": [{"mixer": mixer(l.mixer), "mlp": None if l.ff is None else {"ff": l.ff, "kind": "dense"}, "type": l.type}
                          for l in self.layers],
               "norm": {"eps": self.norm_eps}, "vocab": self.vocab, "width": self.width}
        if self.loop is not None:
            out["loop"] = {"start": self.loop.start, "stop": self.loop.stop, "times": self.loop.times}
        return out

    @classmethod
    def from_dict(cls, raw: dict, where: str = "config.json") -> "DebusunConfig":
        r = KeyReader(raw, where)
        name = r.string("architecture", default=None)
        if name is None:
            archs = r.any("architectures")
            if not (isinstance(archs, list) and archs and isinstance(archs[0], str)):
                raise ConfigError(f"{where}: 'architecture' must name the model")
            name = archs[0]
        vocab, width = r.integer("vocab", minimum=1), r.integer("width", minimum=1)
        eps = KeyReader(_obj(r, "norm", where), where + ":norm").number("eps", positive=True)
        scale, bigram = 1.0, None
        if r.any("embedding") is not None:
            e = KeyReader(_obj(r, "embedding", where), where + ":embedding")
            scale = e.number("scale", default=1.0)
            if e.any("bigram") is not None:
                b = KeyReader(_obj(e, "bigram", where + ":embedding"), where + ":embedding:bigram")
                bigram = DebusunBigram(b.integer("buckets", minimum=1), b.integer("mul_prev", minimum=0), b.integer("mul_cur", minimum=0))
        entries = r.any("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError(f"{where}: 'layers' must be a list with an entry per layer")
        layers = tuple(_layer(e, f"{where}:layers[{i}]") for i, e in enumerate(entries))
        loop = None
        if r.any("loop") is not None:
            lw = where + ":loop"
            lo = KeyReader(_obj(r, "loop", where), lw)
            loop = DebusunLoop(lo.integer("start", minimum=0), lo.integer("stop", minimum=0), lo.integer("times", minimum=1))
            if not loop.start < loop.stop <= len(layers):
                raise ConfigError(f"{lw}: layers {loop.start} .. {loop.stop - 1} are not a run of the model's {len(layers)} layers")
        return cls(name, vocab, width, eps, scale, bigram, loop, layers, raw)


def _obj(r: KeyReader, key: str, where: str) -> dict:
    v = r.any(key)
    if not isinstance(v, dict):
        raise ConfigError(f"{where}: {key!r} must be an object")
    return v


def _rotation(m: KeyReader, mw: str, width: int) -> DebusunRotation | None:
    if m.any("rot") is None:
        return None
    rw = mw + ":rot"
    rot = KeyReader(_obj(m, "rot", mw), rw)
    dims = rot.integer("dims", minimum=0)
    if dims % 2 or dims > width:
        raise ConfigError(f"{rw}: 'dims' ({dims}) must be even and at most the width that turns ({width})")
    if dims < 2:
        return None
    base = rot.number("base", positive=True)
    scaling = rot.any("scaling")
    if scaling is not None:
        s = KeyReader(scaling, rw + ":scaling")
        scaling = {k: s.number(k, positive=True) for k in ("factor", "original", "fast", "slow")}
        if base == 1.0:
            raise ConfigError(f"{rw}: a rescaled rotation needs a base other than 1")
    return DebusunRotation(dims, base, scaling)


def _layer(e, where: str) -> DebusunLayerConfig:
    r = KeyReader(e, where)
    kind = r.string("type", choices=LAYER_TYPES)
    mw = where + ":mixer"
    m = KeyReader(_obj(r, "mixer", where), mw)
    heads, vdim = m.integer("heads", minimum=1), m.integer("vdim", minimum=1)
    if kind == "mamba2":
        state, groups = m.integer("state", minimum=1), m.integer("groups", minimum=1)
        conv, norm_groups = m.integer("conv", minimum=1), m.integer("norm_groups", minimum=1)
        if heads % groups:
            raise ConfigError(f"{mw}: {heads} heads do not fall into {groups} equal 'groups'")
        if heads * vdim % norm_groups:
            raise ConfigError(f"{mw}: {heads * vdim} columns do not fall into {norm_groups} equal 'norm_groups'")
        mixer = DebusunMamba2Config(heads, vdim, state, groups, conv, norm_groups)
    else:
        window = None
        if m.any("mask") is not None:
            window = KeyReader(_obj(m, "mask", mw), mw + ":mask").integer("size", minimum=1)
        dim, scale = m.integer("dim", minimum=1 if kind == "attention" else 0), m.number("scale")
        if kind == "attention":
            kv_heads = m.integer("kv_heads", minimum=1)
            if heads % kv_heads:
                raise ConfigError(f"{mw}: {heads} heads cannot share {kv_heads} key/value heads")
            if dim > 512 or vdim > 512:
                raise ConfigError(f"{mw}: heads of {dim} and {vdim}; the attention kernels take widths up to 512")
            mixer = DebusunAttentionConfig(heads, kv_heads, dim, vdim, scale, window, _rotation(m, mw, dim))
        else:
            rot_dim = m.integer("rot_dim", minimum=0)
            mixer = DebusunLatentConfig(heads, dim, rot_dim, vdim, m.integer("kv_rank", minimum=1), scale, window,
                                        _rotation(m, mw, rot_dim))
    ff = None
    if r.any("mlp") is not None:
        f = KeyReader(_obj(r, "mlp", where), where + ":mlp")
        f.string("kind", choices=("dense",))
        ff = f.integer("ff", minimum=1)
    return DebusunLayerConfig(kind, mixer, ff)
