"""SisadraConfig: the keys of a Sisadra config.json, typed.

The file is nested: `vocab`, `width`, `norm.eps`, `logit_softcap` (absent or null: logits are not capped), `embedding`
(`scale`, and `bigram`: buckets, mul_prev, mul_cur of a second table indexed by a hash of two neighbouring tokens; absent or
null: none), and a list `layers` whose entries give the layer's `type` (its mixer: 'attention', 'latent_attention' or
'channel_delta'), the mixer's sizes and constants (`mixer`) and its feed-forward (`mlp`: kind 'dense', or null for none).
Every layer has its own sizes.  Field names are the file's keys; `to_dict` writes the same nesting back.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

from .base import BadValue, ConfigReader, WrongArchitecture, read_config_json
from .saropel import BigramConfig

ARCHITECTURE = "Sisadra"


def _heads(r: ConfigReader, where: str) -> tuple:
    heads = r.integer("heads", minimum=1)
    kv_heads = r.integer("kv_heads", default=heads, minimum=1)
    if heads % kv_heads:
        raise BadValue(f"{where}.kv_heads", kv_heads, f"must divide the {heads} heads")
    return heads, kv_heads


@dataclass(frozen=True)
class BandedRotationConfig:
    """`rot`: the first `dims` dimensions of every map of a head turn; `scaling` (factor, low, high, original) slows the
    waves that are long against `original` positions."""
    base: float
    dims: int
    scaling: Optional[dict] = None

    KEYS = ("factor", "low", "high", "original")

    @classmethod
    def from_reader(cls, r: ConfigReader, where: str, size: int) -> Optional["BandedRotationConfig"]:
        rot = r.section("rot", default=None, where=where)
        if rot is None:
            return None
        dims = rot.integer("dims", default=size, minimum=0)
        if dims % 2 or dims > size:
            raise BadValue(f"{where}.rot.dims", dims, f"must be even and at most the head size {size}")
        if dims == 0:
            return None
        s = rot.section("scaling", default=None, where=where + ".rot")
        scaling = {k: s.number(k, positive=True) for k in cls.KEYS} if s is not None else None
        if scaling and scaling["low"] > scaling["high"]:
            raise BadValue(f"{where}.rot.scaling.low", scaling["low"], f"is more than high = {scaling['high']}")
        return cls(base=rot.number("base", positive=True), dims=dims, scaling=scaling)

    def to_dict(self) -> dict:
        d = dict(base=self.base, dims=self.dims)
        if self.scaling is not None:
            d["scaling"] = dict(self.scaling)
        return d

    def __hash__(self):
        return hash((self.base, self.dims, tuple(sorted((self.scaling or {}).items()))))


@dataclass(frozen=True)
class DifferentialAttentionConfig:
    """`mixer` of type 'attention': two score maps a head, a query seeing its own chunk of positions."""
    heads: int
    kv_heads: int
    dim: int                 # query/key size of one map of a head
    vdim: int                # value size of a head
    chunk: int               # mask.size: positions of a chunk (0: no mask, all earlier keys)
    scale: float
    diff: float
    rot: Optional[BandedRotationConfig]

    @classmethod
    def from_reader(cls, r: ConfigReader, where: str) -> "DifferentialAttentionConfig":
        heads, kv_heads = _heads(r, where)
        dim = r.integer("dim", minimum=1)
        mask = r.section("mask", default=None, where=where)
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=r.integer("vdim", default=dim, minimum=1),
                   chunk=mask.integer("size", minimum=1) if mask is not None else 0,
                   scale=r.number("scale", positive=True), diff=r.number("diff"),
                   rot=BandedRotationConfig.from_reader(r, where, dim))

    def to_dict(self) -> dict:
        d = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, scale=self.scale, diff=self.diff)
        if self.chunk:
            d["mask"] = dict(size=self.chunk)
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        return d


@dataclass(frozen=True)
class LatentAttentionConfig:
    """`mixer` of type 'latent_attention'."""
    heads: int
    dim: int                 # query/key size of a head
    vdim: int                # value size of a head
    kv_rank: int             # size of the latent that is cached
    scale: float

    @classmethod
    def from_reader(cls, r: ConfigReader, where: str) -> "LatentAttentionConfig":
        dim = r.integer("dim", minimum=1)
        return cls(heads=r.integer("heads", minimum=1), dim=dim, vdim=r.integer("vdim", default=dim, minimum=1),
                   kv_rank=r.integer("kv_rank", minimum=1), scale=r.number("scale", positive=True))

    def to_dict(self) -> dict:
        return dict(heads=self.heads, dim=self.dim, vdim=self.vdim, kv_rank=self.kv_rank, scale=self.scale)


@dataclass(frozen=True)
class ChannelDeltaConfig:
    """`mixer` of type 'channel_delta': the gated delta rule with a decay per key channel."""
    heads: int               # value heads (one state matrix each)
    kv_heads: int            # query/key heads
    dim: int
    vdim: int
    conv: int                # taps of the short convolution

    @classmethod
    def from_reader(cls, r: ConfigReader, where: str) -> "ChannelDeltaConfig":
        heads, kv_heads = _heads(r, where)
        dim = r.integer("dim", minimum=1)
        return cls(heads=heads, kv_heads=kv_heads, dim=dim, vdim=r.integer("vdim", default=dim, minimum=1),
                   conv=r.integer("conv", minimum=1))

    def to_dict(self) -> dict:
        return dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.vdim, conv=self.conv)


MIXERS = {"attention": DifferentialAttentionConfig, "latent_attention": LatentAttentionConfig,
          "channel_delta": ChannelDeltaConfig}


@dataclass(frozen=True)
class SisadraLayer:
    type: str
    mixer: object            # one of MIXERS
    ff: int                  # inner size of the dense feed-forward (0: the layer has none)

    def to_dict(self) -> dict:
        return dict(type=self.type, mixer=self.mixer.to_dict(), mlp=dict(kind="dense", ff=self.ff) if self.ff else None)


@dataclass(frozen=True)
class SisadraConfig:
    vocab: int
    width: int
    norm_eps: float
    embedding_scale: float
    bigram: Optional[BigramConfig]
    logit_softcap: float                # 0: logits are not capped
    layers: tuple                       # of SisadraLayer

    architecture = ARCHITECTURE

    @classmethod
    def from_dict(cls, raw: dict) -> "SisadraConfig":
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
            if kind not in MIXERS:
                raise BadValue(f"{where}.type", kind, "known mixers: " + ", ".join(MIXERS))
            ff = 0
            mr = L.section("mlp", default=None, where=where)
            if mr is not None:
                mk = mr.string("kind")
                if mk != "dense":
                    raise BadValue(f"{where}.mlp.kind", mk, "known feed-forwards: dense")
                ff = mr.integer("ff", minimum=1)
            layers.append(SisadraLayer(type=kind, ff=ff, mixer=MIXERS[kind].from_reader(
                L.section("mixer", where=where), where + ".mixer")))
        emb = r.section("embedding", default=None)
        b = emb.section("bigram", default=None, where="embedding") if emb is not None else None
        bigram = BigramConfig(buckets=b.integer("buckets", minimum=1), mul_prev=b.integer("mul_prev"),
                              mul_cur=b.integer("mul_cur")) if b is not None else None
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   norm_eps=r.section("norm").number("eps", positive=True),
                   embedding_scale=emb.number("scale", default=1.0) if emb is not None else 1.0, bigram=bigram,
                   logit_softcap=r.number("logit_softcap", default=None, positive=True) or 0.0, layers=tuple(layers))

    @classmethod
    def from_json(cls, folder_or_file) -> "SisadraConfig":
        return cls.from_dict(read_config_json(folder_or_file))

    def to_dict(self) -> dict:
        embedding = dict(scale=self.embedding_scale)
        if self.bigram is not None:
            embedding["bigram"] = self.bigram.to_dict()
        d = dict(architecture=ARCHITECTURE, embedding=embedding, layers=[l.to_dict() for l in self.layers],
                 norm=dict(eps=self.norm_eps), vocab=self.vocab, width=self.width)
        if self.logit_softcap:
            d["logit_softcap"] = self.logit_softcap
        return d
