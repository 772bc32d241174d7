"""Typed reading of a Bunudra model's config.json.

``layers`` lists the layers one by one: ``type`` names the mixer
("attention", "latent_attention" or "mlstm"), ``mixer`` holds its sizes and
constants and ``mlp`` the feed-forward (null for a layer without one).  An
"attention" mixer has ``heads``, ``kv_heads``, ``dim``, ``vdim``, ``scale``,
``rot`` (``dims``, ``base``) and ``mask.size``, the length of its chunks; a
"latent_attention" mixer ``heads``, ``dim``, ``rot_dim``, ``vdim``,
``kv_rank``, ``scale``, ``rot`` (``dims``, ``base`` and ``scaling`` with
``factor``, ``original``, ``fast``, ``slow``) and ``mask.size``, its window;
an "mlstm" mixer ``heads``, ``dim``, ``vdim`` and ``gate_cap``.  A
feed-forward of kind "moe" has ``router`` (``experts``, ``top``, ``scale``,
``groups`` with ``count`` and ``keep``), ``expert.ff`` and ``shared.ff``.
Model-wide: ``width``, ``vocab``, ``norm.eps`` and ``embedding.scale``.
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
class YarnConfig:
    factor: float
    original: float
    fast: float
    slow: float

    @staticmethod
    def from_reader(r: KeyReader) -> "YarnConfig":
        return YarnConfig(**{k: r.number(k, positive=True) for k in ("factor", "original", "fast", "slow")})

    def to_dict(self) -> dict:
        return dict(factor=self.factor, fast=self.fast, original=self.original, slow=self.slow)


@dataclass(frozen=True)
class RotaryConfig:
    dims: int = 0               # 0: nothing is rotated
    base: float = 10000.0
    scaling: YarnConfig | None = None

    @staticmethod
    def from_reader(r: KeyReader | None, most: int, scaling: bool) -> "RotaryConfig":
        if r is None:
            return RotaryConfig()
        dims = r.integer("dims", minimum=0)
        if dims % 2 or dims > most:
            raise ConfigError(f"{r.where}: rot.dims {dims} must be even and at most {most}")
        s = r.obj("scaling")
        if s is not None and not scaling:
            raise ConfigError(f"{r.where}: this mixer's rotation has no scaling")
        return RotaryConfig(dims, r.number("base", positive=True), YarnConfig.from_reader(s) if s is not None else None)

    def to_dict(self) -> dict:
        d = dict(base=self.base, dims=self.dims)
        if self.scaling:
            d["scaling"] = self.scaling.to_dict()
        return d


@dataclass(frozen=True)
class ChunkedAttentionConfig:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    size: int                   # of a chunk
    rot: RotaryConfig

    @staticmethod
    def from_reader(r: KeyReader) -> "ChunkedAttentionConfig":
        heads, kv, dim = (r.integer(k, minimum=1) for k in ("heads", "kv_heads", "dim"))
        if heads % kv:
            raise ConfigError(f"{r.where}: {heads} heads cannot share {kv} key/value heads")
        return ChunkedAttentionConfig(heads, kv, dim, r.integer("vdim", minimum=1), r.number("scale"),
                                      _required(r, "mask").integer("size", minimum=1),
                                      RotaryConfig.from_reader(r.obj("rot"), dim, scaling=False))

    def to_dict(self) -> dict:
        return dict(dim=self.dim, heads=self.heads, kv_heads=self.kv_heads, mask=dict(size=self.size), rot=self.rot.to_dict(),
                    scale=self.scale, vdim=self.vdim)


@dataclass(frozen=True)
class WindowedLatentConfig:
    heads: int
    dim: int                    # unrotated query/key numbers per head
    rot_dim: int                # rotated ones
    vdim: int
    kv_rank: int
    scale: float
    size: int                   # of the window
    rot: RotaryConfig

    @staticmethod
    def from_reader(r: KeyReader) -> "WindowedLatentConfig":
        rot_dim = r.integer("rot_dim", minimum=0)
        return WindowedLatentConfig(
            heads=r.integer("heads", minimum=1), dim=r.integer("dim", minimum=1), rot_dim=rot_dim,
            vdim=r.integer("vdim", minimum=1), kv_rank=r.integer("kv_rank", minimum=1), scale=r.number("scale"),
            size=_required(r, "mask").integer("size", minimum=1),
            rot=RotaryConfig.from_reader(r.obj("rot"), rot_dim, scaling=True))

    def to_dict(self) -> dict:
        return dict(dim=self.dim, heads=self.heads, kv_rank=self.kv_rank, mask=dict(size=self.size), rot=self.rot.to_dict(),
                    rot_dim=self.rot_dim, scale=self.scale, vdim=self.vdim)


@dataclass(frozen=True)
class MLSTMConfig:
    heads: int
    dim: int
    vdim: int
    gate_cap: float

    @staticmethod
    def from_reader(r: KeyReader) -> "MLSTMConfig":
        return MLSTMConfig(*(r.integer(k, minimum=1) for k in ("heads", "dim", "vdim")), r.number("gate_cap", positive=True))

    def to_dict(self) -> dict:
        return dict(dim=self.dim, gate_cap=self.gate_cap, heads=self.heads, vdim=self.vdim)


_MIXERS = {"attention": ChunkedAttentionConfig, "latent_attention": WindowedLatentConfig, "mlstm": MLSTMConfig}


@dataclass(frozen=True)
class GroupedMixtureConfig:
    experts: int
    top: int
    scale: float
    groups: tuple | None        # (count, keep)
    expert_ff: int
    shared_ff: int              # 0: no shared expert

    @staticmethod
    def from_reader(r: KeyReader) -> "GroupedMixtureConfig":
        if r.string("kind") != "moe":
            raise ConfigError(f"{r.where}: feed-forward kind {r.string('kind')!r} is not known; known: ['moe']")
        router, shared = _required(r, "router"), r.obj("shared")
        experts, top, g = router.integer("experts", minimum=1), router.integer("top", minimum=1), router.obj("groups")
        groups, choice = None, experts
        if g is not None:
            groups = (g.integer("count", minimum=1), g.integer("keep", minimum=1))
            if experts % groups[0] or groups[1] > groups[0]:
                raise ConfigError(f"{r.where}: {experts} experts in {groups[0]} equal groups of which {groups[1]} are kept")
            choice = experts // groups[0] * groups[1]
        if top > choice:
            raise ConfigError(f"{r.where}: top {top} is more than the {choice} experts there are to choose from")
        return GroupedMixtureConfig(experts, top, router.number("scale", 1.0), groups,
                                    _required(r, "expert").integer("ff", minimum=1),
                                    shared.integer("ff", minimum=1) if shared is not None else 0)

    def to_dict(self) -> dict:
        router = dict(experts=self.experts, scale=self.scale, top=self.top)
        if self.groups:
            router["groups"] = dict(count=self.groups[0], keep=self.groups[1])
        return dict(expert=dict(ff=self.expert_ff), kind="moe", router=router,
                    shared=dict(ff=self.shared_ff) if self.shared_ff else None)


@dataclass(frozen=True)
class BunudraLayerConfig:
    type: str
    mixer: object
    mlp: GroupedMixtureConfig | None

    @staticmethod
    def from_reader(r: KeyReader) -> "BunudraLayerConfig":
        kind = r.string("type")
        if kind not in _MIXERS:
            raise ConfigError(f"{r.where}: layer type {kind!r} is not known; known: {sorted(_MIXERS)}")
        mlp = r.obj("mlp")
        return BunudraLayerConfig(kind, _MIXERS[kind].from_reader(_required(r, "mixer")),
                                  GroupedMixtureConfig.from_reader(mlp) if mlp is not None else None)

    def to_dict(self) -> dict:
        return dict(mixer=self.mixer.to_dict(), mlp=self.mlp.to_dict() if self.mlp else None, type=self.type)


@dataclass
class BunudraConfig:
    architecture: str
    width: int
    vocab: int
    layers: tuple
    norm_eps: float
    embedding_scale: float = 1.0
    max_position: int = DEFAULT_MAX_POSITION
    eos_token_id: tuple = field(default_factory=tuple)

    ARCHITECTURE = "Bunudra"

    @staticmethod
    def from_dict(data: dict, where: str = "config.json") -> "BunudraConfig":
        r = KeyReader(data, where)
        raw_layers = data.get("layers")
        if not isinstance(raw_layers, list) or not raw_layers:
            raise ConfigError(f"{where}: 'layers' must be a non-empty list")
        layers = tuple(BunudraLayerConfig.from_reader(KeyReader(x, f"{where}:layers[{i}]"))
                       for i, x in enumerate(raw_layers))
        embedding = r.obj("embedding")
        return BunudraConfig(
            architecture=r.string("architecture", BunudraConfig.ARCHITECTURE),
            width=r.integer("width", minimum=1), vocab=r.integer("vocab", minimum=1), layers=layers,
            norm_eps=_required(r, "norm").number("eps", positive=True),
            embedding_scale=embedding.number("scale", 1.0) if embedding is not None else 1.0,
            max_position=r.integer("max_position", DEFAULT_MAX_POSITION, minimum=1),
            eos_token_id=r.int_list("eos_token_id", ()))

    def to_dict(self) -> dict:
        d = dict(architecture=self.architecture, embedding=dict(scale=self.embedding_scale),
                 layers=[x.to_dict() for x in self.layers], norm=dict(eps=self.norm_eps), vocab=self.vocab, width=self.width)
        if self.max_position != DEFAULT_MAX_POSITION:
            d["max_position"] = self.max_position
        if self.eos_token_id:
            d["eos_token_id"] = list(self.eos_token_id)
        return d
