"""Configuration of the Sosepel design (config.json "architecture": "Sosepel").

A decoder whose layers are listed one by one: each entry of `layers` gives its mixer (`type`, `mixer`) and its feed-forward
(`mlp`, or null).  The mixer is differential attention: two softmax maps a head over the same values, a temperature of the
queries that grows with the position and a cap on the scores.  The feed-forward is dense with the square of relu, or a
mixture of gated experts chosen by sigmoid scores within groups, with a gated shared expert.  A stretch of layers may run
several times (`loop`), each pass begun by joining the residual with the embedding's output; the embedding is scaled and may
add a row of a table of token pairs (`embedding.bigram`).  Every size and every constant that can differ between two models
of the design is read here; nothing of them stands in code.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .base import ConfigError, ConfigReader

ARCHITECTURE = "Sosepel"
MIXERS = ("attention",)
MLP_KINDS = ("dense", "moe")


@dataclass(frozen=True)
class QueryTemperature:
    coef: float
    every: int


@dataclass(frozen=True)
class DifferentialConfig:
    heads: int
    kv_heads: int
    dim: int                 # per head and map: query/key entries
    vdim: int                # per head: value entries, shared by the two maps
    scale: float
    diff: float              # the constant in the second map's weight, and in the output's factor 1 - diff
    softcap: float | None    # scores become cap * tanh(score / cap)
    q_temp: QueryTemperature | None


@dataclass(frozen=True)
class MlpConfig:
    kind: str                # "dense" or "moe"
    ff: int                  # inner width (of an expert, for "moe")
    experts: int = 0
    top: int = 0
    groups: int = 1          # equal groups of neighbouring experts
    keep: int = 1            # groups whose experts can be chosen
    shared_ff: int | None = None


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: DifferentialConfig
    mlp: MlpConfig | None


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class BigramConfig:
    buckets: int
    mul_prev: int
    mul_cur: int


@dataclass(frozen=True)
class SosepelConfig:
    vocab: int
    width: int
    layers: tuple
    norm_eps: float
    embedding_scale: float
    bigram: BigramConfig | None
    loop: LoopConfig | None
    logit_softcap: float | None
    raw: dict = field(compare=False, repr=False, default_factory=dict)

    architecture = ARCHITECTURE

    @classmethod
    def from_dict(cls, data: dict, source: str = "config.json") -> "SosepelConfig":
        r = ConfigReader(data, source)
        entries = data.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError(f"{source}: key 'layers' must be a list with at least one layer")
        layers = tuple(cls._layer(entry, f"{source}: layers[{i}]") for i, entry in enumerate(entries))
        loop = None
        if data.get("loop") is not None:
            loop = LoopConfig(start=r.integer("loop.start", minimum=0), stop=r.integer("loop.stop", minimum=0),
                              times=r.integer("loop.times", minimum=1))
            if not (loop.start <= loop.stop <= len(layers)):
                raise ConfigError(f"{source}: loop.start {loop.start} and loop.stop {loop.stop} must lie in order within the {len(layers)} layers")
        bigram = None
        if isinstance(data.get("embedding"), dict) and data["embedding"].get("bigram") is not None:
            bigram = BigramConfig(buckets=r.integer("embedding.bigram.buckets", minimum=1),
                                  mul_prev=r.integer("embedding.bigram.mul_prev", minimum=0),
                                  mul_cur=r.integer("embedding.bigram.mul_cur", minimum=0))
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1), layers=layers,
                   norm_eps=r.number("norm.eps", exclusive_minimum=0.0), embedding_scale=r.number("embedding.scale", default=1.0),
                   bigram=bigram, loop=loop, logit_softcap=r.number("logit_softcap", default=None, exclusive_minimum=0.0), raw=data)

    @staticmethod
    def _layer(entry, where: str) -> LayerConfig:
        if not isinstance(entry, dict):
            raise ConfigError(f"{where} must be an object")
        e = ConfigReader(entry, where)
        kind = e.string("type")
        if kind not in MIXERS:
            raise ConfigError(f"{where}: type '{kind}' is not known (known: {', '.join(MIXERS)})")
        temp = None
        if isinstance(entry.get("mixer"), dict) and entry["mixer"].get("q_temp") is not None:
            temp = QueryTemperature(coef=e.number("mixer.q_temp.coef"), every=e.integer("mixer.q_temp.every", minimum=1))
        mixer = DifferentialConfig(
            heads=e.integer("mixer.heads", minimum=1), kv_heads=e.integer("mixer.kv_heads", minimum=1), dim=e.integer("mixer.dim", minimum=1),
            vdim=e.integer("mixer.vdim", minimum=1), scale=e.number("mixer.scale", exclusive_minimum=0.0), diff=e.number("mixer.diff"),
            softcap=e.number("mixer.softcap", default=None, exclusive_minimum=0.0), q_temp=temp)
        if mixer.heads % mixer.kv_heads:
            raise ConfigError(f"{where}: mixer.heads {mixer.heads} is not a multiple of mixer.kv_heads {mixer.kv_heads}")
        if entry.get("mlp") is None:
            return LayerConfig(kind, mixer, None)
        mlp_kind = e.string("mlp.kind")
        if mlp_kind not in MLP_KINDS:
            raise ConfigError(f"{where}: mlp.kind '{mlp_kind}' is not known (known: {', '.join(MLP_KINDS)})")
        if mlp_kind == "dense":
            return LayerConfig(kind, mixer, MlpConfig("dense", ff=e.integer("mlp.ff", minimum=1)))
        groups, keep = 1, 1
        if (entry["mlp"].get("router") or {}).get("groups") is not None:
            groups, keep = e.integer("mlp.router.groups.count", minimum=1), e.integer("mlp.router.groups.keep", minimum=1)
        mlp = MlpConfig("moe", ff=e.integer("mlp.expert.ff", minimum=1), experts=e.integer("mlp.router.experts", minimum=1),
                        top=e.integer("mlp.router.top", minimum=1), groups=groups, keep=keep,
                        shared_ff=e.integer("mlp.shared.ff", default=None, minimum=1))
        if mlp.experts % groups:
            raise ConfigError(f"{where}: mlp.router.experts {mlp.experts} is not a multiple of mlp.router.groups.count {groups}")
        if keep > groups:
            raise ConfigError(f"{where}: mlp.router.groups.keep {keep} is more than mlp.router.groups.count {groups}")
        if mlp.top > keep * (mlp.experts // groups):
            raise ConfigError(f"{where}: mlp.router.top {mlp.top} is more than the {keep * (mlp.experts // groups)} experts of the groups kept")
        return LayerConfig(kind, mixer, mlp)

    def runs(self) -> list:
        """[(layer, whether a pass of the loop begins with it)] in the order the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        a, b = self.loop.start, self.loop.stop
        return [(i, False) for i in range(a)] + [(i, i == a) for i in range(a, b)] * self.loop.times + [(i, False) for i in range(b, n)]

    # (what the command line prints about a loaded model)
    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def hidden_size(self) -> int:
        return self.width

    @property
    def vocab_size(self) -> int:
        return self.vocab

    def to_dict(self) -> dict:
        """config.json form of this configuration."""
        layers = []
        for l in self.layers:
            m, f = l.mixer, l.mlp
            mixer = dict(heads=m.heads, kv_heads=m.kv_heads, dim=m.dim, vdim=m.vdim, scale=m.scale, diff=m.diff)
            if m.softcap is not None:
                mixer["softcap"] = m.softcap
            if m.q_temp is not None:
                mixer["q_temp"] = dict(coef=m.q_temp.coef, every=m.q_temp.every)
            mlp = None
            if f is not None and f.kind == "dense":
                mlp = dict(kind="dense", ff=f.ff)
            elif f is not None:
                router = dict(experts=f.experts, top=f.top)
                if f.groups > 1:
                    router["groups"] = dict(count=f.groups, keep=f.keep)
                mlp = dict(kind="moe", expert=dict(ff=f.ff), router=router)
                if f.shared_ff is not None:
                    mlp["shared"] = dict(ff=f.shared_ff)
            layers.append(dict(type=l.type, mixer=mixer, mlp=mlp))
        d = dict(architecture=ARCHITECTURE, vocab=self.vocab, width=self.width, layers=layers, norm=dict(eps=self.norm_eps),
                 embedding=dict(scale=self.embedding_scale))
        if self.bigram is not None:
            d["embedding"]["bigram"] = dict(buckets=self.bigram.buckets, mul_prev=self.bigram.mul_prev, mul_cur=self.bigram.mul_cur)
        if self.loop is not None:
            d["loop"] = dict(start=self.loop.start, stop=self.loop.stop, times=self.loop.times)
        if self.logit_softcap is not None:
            d["logit_softcap"] = self.logit_softcap
        return d

    def describe(self) -> dict:
        return self.to_dict()
