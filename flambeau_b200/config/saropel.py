"""SaropelConfig: the keys of a Saropel config.json, typed.

The file is nested: `vocab`, `width`, `norm.eps`, `embedding.bigram` (buckets, mul_prev, mul_cur: a second embedding
table indexed by a hash of two neighbouring tokens; absent or null: none), `token_side.dim` (columns that a token's id
gives to every layer; absent or null: none), `loop` (start, stop, times: the stretch of layers that runs several times
in a row; absent or null: none), and a list `layers` whose entries give the layer's `type` (its mixer: 'attention' or
'attention_2'), the mixer's sizes and constants (`mixer`) and its feed-forward (`mlp`: kind 'dense' or 'moe', or null
for none).  Every layer has its own sizes.  Field names are the file's keys; `to_dict` writes the same nesting back.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .base import BadValue, ConfigReader, WrongArchitecture, read_config_json

ARCHITECTURE = "Saropel"
# what sets the two mixers apart, by type name: whether the projected keys are the values too
VALUES_FROM_KEYS = {"attention": False, "attention_2": True}


@dataclass(frozen=True)
class RotationConfig:
    """`rot`: the first `dims` dimensions of a head turn; `scaling` stretches the slow waves."""
    base: float
    dims: int
    scaling: Optional[dict] = None       # factor, original, fast, slow

    @classmethod
    def from_reader(cls, r: ConfigReader, where: str, size: int) -> Optional["RotationConfig"]:
        rot = r.section("rot", default=None, where=where)
        if rot is None:
            return None
        dims = rot.integer("dims", default=size, minimum=0)
        if dims % 2 or dims > size:
            raise BadValue(f"{where}.rot.dims", dims, f"must be even and at most the head size {size}")
        if dims == 0:
            return None
        s = rot.section("scaling", default=None, where=where + ".rot")
        scaling = None
        if s is not None:
            scaling = {k: s.number(k, positive=True) for k in ("factor", "original", "fast", "slow")}
        return cls(base=rot.number("base", positive=True), dims=dims, scaling=scaling)

    def to_dict(self) -> dict:
        d = dict(base=self.base, dims=self.dims)
        if self.scaling is not None:
            d["scaling"] = dict(self.scaling)
        return d

    def __hash__(self):
        return hash((self.base, self.dims, tuple(sorted((self.scaling or {}).items()))))


@dataclass(frozen=True)
class AttentionConfig:
    heads: int
    kv_heads: int
    dim: int                 # query/key size of a head
    vdim: int                # value size of a head
    window: int              # mask.size: the last keys a query sees, itself included (0: no mask, all earlier keys)
    scale: float
    softcap: float           # 0: scores are not capped
    rot: Optional[RotationConfig]

    @classmethod
    def from_reader(cls, kind: str, r: ConfigReader, where: str) -> "AttentionConfig":
        heads, dim = r.integer("heads", minimum=1), r.integer("dim", minimum=1)
        kv_heads = r.integer("kv_heads", default=heads, minimum=1)
        if heads % kv_heads:
            raise BadValue(f"{where}.kv_heads", kv_heads, f"must divide the {heads} query heads")
        vdim = r.integer("vdim", default=dim, minimum=1)
        if VALUES_FROM_KEYS[kind] and vdim != dim:
            raise BadValue(f"{where}.vdim", vdim, f"the values are the keys: it must be dim = {dim}")
        mask = r.section("mask", default=None, where=where)
        softcap = r.number("softcap", default=None, positive=True)
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim,
                   window=mask.integer("size", minimum=1) if mask is not None else 0,
                   scale=r.number("scale", positive=True), softcap=softcap or 0.0,
                   rot=RotationConfig.from_reader(r, where, dim))

    def to_dict(self) -> dict:
        d = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale)
        if self.window:
            d["mask"] = dict(size=self.window)
        if self.softcap:
            d["softcap"] = self.softcap
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class DenseMlpConfig:
    ff: int
    kind: str = "dense"

    def to_dict(self) -> dict:
        return dict(kind=self.kind, ff=self.ff)


@dataclass(frozen=True)
class ExpertConfig:
    """`expert` and `shared`: the inner size of a small feed-forward and where its operands are cut off."""
    ff: int
    limit: float

    @classmethod
    def from_reader(cls, r: ConfigReader) -> "ExpertConfig":
        return cls(ff=r.integer("ff", minimum=1), limit=r.number("limit", positive=True))

    def to_dict(self) -> dict:
        return dict(ff=self.ff, limit=self.limit)


@dataclass(frozen=True)
class RoutedMlpConfig:
    """`mlp` of kind 'moe': `router.experts` experts of which a token uses `router.top`, chosen among those of the best
    `router.groups.keep` of `router.groups.count` equal groups (no `groups`: among all); `shared` is the expert that
    every token uses (None: there is none)."""
    experts: int
    top: int
    expert: ExpertConfig
    groups: int = 1
    keep_groups: int = 0                 # 0: the choice is among all experts
    shared: Optional[ExpertConfig] = None
    kind: str = "moe"

    @classmethod
    def from_reader(cls, r: ConfigReader, where: str) -> "RoutedMlpConfig":
        router = r.section("router", where=where)
        experts = router.integer("experts", minimum=1)
        top = router.integer("top", minimum=1)
        count, keep, eligible = 1, 0, experts
        g = router.section("groups", default=None, where=where + ".router")
        if g is not None:
            count, keep = g.integer("count", minimum=1), g.integer("keep", minimum=1)
            if experts % count:
                raise BadValue(f"{where}.router.groups.count", count, f"must divide the {experts} experts")
            if keep > count:
                raise BadValue(f"{where}.router.groups.keep", keep, f"is more than the {count} groups")
            eligible = keep * (experts // count)
        if top > eligible:
            raise BadValue(f"{where}.router.top", top, f"is more than the {eligible} experts it may choose from")
        shared = r.section("shared", default=None, where=where)
        return cls(experts=experts, top=top, expert=ExpertConfig.from_reader(r.section("expert", where=where)),
                   groups=count, keep_groups=keep,
                   shared=ExpertConfig.from_reader(shared) if shared is not None else None)

    def to_dict(self) -> dict:
        router = dict(experts=self.experts, top=self.top)
        if self.keep_groups:
            router["groups"] = dict(count=self.groups, keep=self.keep_groups)
        d = dict(kind=self.kind, router=router, expert=self.expert.to_dict())
        if self.shared is not None:
            d["shared"] = self.shared.to_dict()
        return d


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int

    def to_dict(self) -> dict:
        return dict(buckets=self.buckets, mul_prev=self.mul_prev, mul_cur=self.mul_cur)


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int

    def to_dict(self) -> dict:
        return dict(start=self.start, stop=self.stop, times=self.times)


@dataclass(frozen=True)
class SaropelLayer:
    type: str
    mixer: AttentionConfig
    mlp: object              # DenseMlpConfig, RoutedMlpConfig or None

    def to_dict(self) -> dict:
        return dict(type=self.type, mixer=self.mixer.to_dict(), mlp=self.mlp.to_dict() if self.mlp else None)


@dataclass(frozen=True)
class SaropelConfig:
    vocab: int
    width: int
    norm_eps: float
    bigram: Optional[BigramConfig]
    side_dim: int                       # 0: a token's id gives the layers nothing of its own
    loop: Optional[LoopConfig]
    layers: tuple                       # of SaropelLayer

    architecture = ARCHITECTURE

    @classmethod
    def from_dict(cls, raw: dict) -> "SaropelConfig":
        r = ConfigReader(raw)
        if r.architecture() != ARCHITECTURE:
            raise WrongArchitecture(raw.get("architecture", raw.get("architectures")), ARCHITECTURE)
        layers_raw = raw.get("layers")
        if not isinstance(layers_raw, list) or not layers_raw:
            raise BadValue("layers", layers_raw, "must be a non-empty list of layer objects")
        layers = []
        for i, lr in enumerate(layers_raw):
            L = ConfigReader(lr)
            where = f"layers[{i}]"
            kind = L.string("type")
            if kind not in VALUES_FROM_KEYS:
                raise BadValue(f"{where}.type", kind, "known mixers: " + ", ".join(VALUES_FROM_KEYS))
            mixer = AttentionConfig.from_reader(kind, L.section("mixer", where=where), where + ".mixer")
            mlp = None
            mr = L.section("mlp", default=None, where=where)
            if mr is not None:
                mk = mr.string("kind")
                if mk == "dense":
                    mlp = DenseMlpConfig(ff=mr.integer("ff", minimum=1))
                elif mk == "moe":
                    mlp = RoutedMlpConfig.from_reader(mr, where + ".mlp")
                else:
                    raise BadValue(f"{where}.mlp.kind", mk, "known feed-forwards: dense, moe")
            layers.append(SaropelLayer(type=kind, mixer=mixer, mlp=mlp))
        bigram = None
        emb = r.section("embedding", default=None)
        b = emb.section("bigram", default=None, where="embedding") if emb is not None else None
        if b is not None:
            bigram = BigramConfig(buckets=b.integer("buckets", minimum=1), mul_prev=b.integer("mul_prev"),
                                  mul_cur=b.integer("mul_cur"))
        side = r.section("token_side", default=None)
        loop = None
        lp = r.section("loop", default=None)
        if lp is not None:
            loop = LoopConfig(start=lp.integer("start", minimum=0), stop=lp.integer("stop", minimum=0),
                              times=lp.integer("times", minimum=1))
            if not loop.start <= loop.stop <= len(layers):
                raise BadValue("loop", lp.raw, f"needs start <= stop <= {len(layers)} layers")
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   norm_eps=r.section("norm").number("eps", positive=True), bigram=bigram,
                   side_dim=side.integer("dim", minimum=1) if side is not None else 0, loop=loop, layers=tuple(layers))

    @classmethod
    def from_json(cls, folder_or_file) -> "SaropelConfig":
        return cls.from_dict(read_config_json(folder_or_file))

    def to_dict(self) -> dict:
        d = dict(architecture=ARCHITECTURE, layers=[l.to_dict() for l in self.layers], norm=dict(eps=self.norm_eps),
                 vocab=self.vocab, width=self.width)
        if self.bigram is not None:
            d["embedding"] = dict(bigram=self.bigram.to_dict())
        if self.side_dim:
            d["token_side"] = dict(dim=self.side_dim)
        if self.loop is not None:
            d["loop"] = self.loop.to_dict()
        return d
