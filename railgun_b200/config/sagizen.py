"""Typed reading of a Sagizen model's config.json.

``layers`` lists the layers one by one: ``type`` names the mixer ("mamba2" or
"parallel"), ``mixer`` holds its sizes and constants and ``mlp`` the
feed-forward (``kind`` "dense" with ``ff``; null for a layer without one).  A
"mamba2" mixer has ``heads``, ``vdim``, ``state``, ``groups``, ``conv`` taps
and ``norm_groups``.  A "parallel" mixer has two halves and a constant for
each (``left_scale``, ``right_scale``): ``left`` (``heads``, ``kv_heads``,
``dim``, ``vdim``, ``scale``, ``rot`` with ``dims``, ``base`` and
``scaling.factor``, ``mask`` with ``size`` and ``pool``) and ``right``
(``heads``, ``dim``).  Model-wide: ``width``, ``vocab`` and ``norm.eps``.
``architecture`` (a string) names the design; ``max_position`` is optional
(default 2^20: positions are computed, not tabulated).
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .base import ConfigError, KeyReader

DEFAULT_MAX_POSITION = 1 << 20


def _required(r: KeyReader, key: str) -> KeyReader:
    o = r.obj(key)
    if o is None:
        raise ConfigError(f"{r.where}: required key '{key}' is missing")
    return o


@dataclass(frozen=True)
class Mamba2Config:
    heads: int
    vdim: int
    state: int
    groups: int             # of B and C
    conv: int               # taps
    norm_groups: int        # parts of the gated output, each normed by itself

    @staticmethod
    def from_reader(r: KeyReader) -> "Mamba2Config":
        c = Mamba2Config(**{k: r.integer(k, minimum=1) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")})
        if c.heads % c.groups:
            raise ConfigError(f"{r.where}: {c.heads} heads cannot share {c.groups} groups")
        if (c.heads * c.vdim) % c.norm_groups:
            raise ConfigError(f"{r.where}: {c.heads * c.vdim} numbers do not split into {c.norm_groups} equal parts")
        return c

    def to_dict(self) -> dict:
        return dict(conv=self.conv, groups=self.groups, heads=self.heads, norm_groups=self.norm_groups,
                    state=self.state, vdim=self.vdim)


@dataclass(frozen=True)
class PooledAttentionConfig:
    """The left half of a "parallel" mixer: a sliding window beside pooled blocks of what has left it."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    size: int               # of the window
    pool: int               # tokens per block
    rot_dims: int
    rot_base: float
    rot_factor: float       # what the rotation's frequencies are divided by

    @staticmethod
    def from_reader(r: KeyReader) -> "PooledAttentionConfig":
        heads, kv = r.integer("heads", minimum=1), r.integer("kv_heads", minimum=1)
        if heads % kv:
            raise ConfigError(f"{r.where}: {heads} heads cannot share {kv} key/value heads")
        dim, rot, mask = r.integer("dim", minimum=1), r.obj("rot"), _required(r, "mask")
        dims, base, factor = 0, 10000.0, 1.0
        if rot is not None:
            dims, base = rot.integer("dims", minimum=0), rot.number("base", positive=True)
            scaling = rot.obj("scaling")
            if scaling is not None:
                factor = scaling.number("factor", positive=True)
        if dims % 2 or dims > dim:
            raise ConfigError(f"{r.where}: rot.dims {dims} must be even and at most dim {dim}")
        return PooledAttentionConfig(
            heads=heads, kv_heads=kv, dim=dim, vdim=r.integer("vdim", minimum=1), scale=r.number("scale"),
            size=mask.integer("size", minimum=1), pool=mask.integer("pool", minimum=1), rot_dims=dims, rot_base=base,
            rot_factor=factor)

    def to_dict(self) -> dict:
        d = dict(dim=self.dim, heads=self.heads, kv_heads=self.kv_heads, mask=dict(pool=self.pool, size=self.size),
                 scale=self.scale, vdim=self.vdim)
        if self.rot_dims:
            d["rot"] = dict(base=self.rot_base, dims=self.rot_dims)
            if self.rot_factor != 1.0:
                d["rot"]["scaling"] = dict(factor=self.rot_factor)
        return d


@dataclass(frozen=True)
class RwkvConfig:
    """The right half of a "parallel" mixer."""
    heads: int
    dim: int

    @staticmethod
    def from_reader(r: KeyReader) -> "RwkvConfig":
        return RwkvConfig(heads=r.integer("heads", minimum=1), dim=r.integer("dim", minimum=1))

    def to_dict(self) -> dict:
        return dict(dim=self.dim, heads=self.heads)


@dataclass(frozen=True)
class PairConfig:
    left: PooledAttentionConfig
    right: RwkvConfig
    left_scale: float
    right_scale: float

    @staticmethod
    def from_reader(r: KeyReader) -> "PairConfig":
        return PairConfig(PooledAttentionConfig.from_reader(_required(r, "left")),
                          RwkvConfig.from_reader(_required(r, "right")), r.number("left_scale"), r.number("right_scale"))

    def to_dict(self) -> dict:
        return dict(left=self.left.to_dict(), left_scale=self.left_scale, right=self.right.to_dict(),
                    right_scale=self.right_scale)


_MIXERS = {"mamba2": Mamba2Config, "parallel": PairConfig}


@dataclass(frozen=True)
class SagizenLayerConfig:
    type: str
    mixer: object
    ff: int                 # inner size of the feed-forward; 0: none

    @staticmethod
    def from_reader(r: KeyReader) -> "SagizenLayerConfig":
        kind = r.string("type")
        if kind not in _MIXERS:
            raise ConfigError(f"{r.where}: layer type {kind!r} is not known; known: {sorted(_MIXERS)}")
        mixer, mlp, ff = _required(r, "mixer"), r.obj("mlp"), 0
        if mlp is not None:
            if mlp.string("kind") != "dense":
                raise ConfigError(f"{mlp.where}: feed-forward kind {mlp.string('kind')!r} is not known; known: ['dense']")
            ff = mlp.integer("ff", minimum=1)
        return SagizenLayerConfig(kind, _MIXERS[kind].from_reader(mixer), ff)

    def to_dict(self) -> dict:
        return dict(mixer=self.mixer.to_dict(), mlp=dict(ff=self.ff, kind="dense") if self.ff else None, type=self.type)


@dataclass
class SagizenConfig:
    architecture: str
    width: int
    vocab: int
    layers: tuple
    norm_eps: float
    max_position: int = DEFAULT_MAX_POSITION
    eos_token_id: tuple = field(default_factory=tuple)

    ARCHITECTURE = "Sagizen"

    @staticmethod
    def from_dict(data: dict, where: str = "config.json") -> "SagizenConfig":
        r = KeyReader(data, where)
        raw_layers = data.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers = tuple(SagizenLayerConfig.from_reader(KeyReader(x, f"{where}:layers[{i}]"))
                       for i, x in enumerate(raw_layers))
        return SagizenConfig(
            architecture=r.string("architecture", SagizenConfig.ARCHITECTURE),
            width=r.integer("width", minimum=1), vocab=r.integer("vocab", minimum=1), layers=layers,
            norm_eps=_required(r, "norm").number("eps", positive=True),
            max_position=r.integer("max_position", DEFAULT_MAX_POSITION, minimum=1),
            eos_token_id=r.int_list("eos_token_id", ()))

    def to_dict(self) -> dict:
        d = dict(architecture=self.architecture, layers=[x.to_dict() for x in self.layers],
                 norm=dict(eps=self.norm_eps), vocab=self.vocab, width=self.width)
        if self.max_position != DEFAULT_MAX_POSITION:
            d["max_position"] = self.max_position
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d
