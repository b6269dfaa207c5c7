"""Configuration of the Gomerax design (config.json "architecture": "Gomerax").

A decoder whose layers are listed one by one: each entry of `layers` gives its mixer (`type`, `mixer`) and its feed-forward
(`mlp`, or null).  The mixer is latent attention whose queries come out of a latent vector of their own, in a sliding window
(`mask.size`), with a sink a head.  The feed-forward is dense, SiLU-gated and biased, or a mixture of clamped gated experts chosen
by softmax scores with a correction, within groups, beside a shared expert with sizes and a limit of its own.  A stretch of
layers may run several times (`loop`).  Positions are rotated into a part of every query and key and also have a stored vector
each (`max_positions`).  Every size and every constant that can differ between two models of the design is read here.
"""
from __future__ import annotations

from dataclasses import dataclass, field

from .base import ConfigError, ConfigReader

ARCHITECTURE = "Gomerax"
MIXERS = ("latent_attention",)
MLP_KINDS = ("dense", "moe")


@dataclass(frozen=True)
class LatentAttentionConfig:
    heads: int
    dim: int                 # per head: query/key entries that are not rotated
    rot_dim: int             # per head: rotated query entries; the width of the one rotated key part
    vdim: int
    q_rank: int              # width of the queries' latent vector
    kv_rank: int
    scale: float
    rot_dims: int            # entries of the rotated part that turn (all of them)
    rot_base: float
    window: int | None


@dataclass(frozen=True)
class MlpConfig:
    kind: str                # "dense" or "moe"
    ff: int                  # inner width (of an expert, for "moe")
    limit: float = 0.0       # of an expert's clamps
    experts: int = 0
    top: int = 0
    groups: int = 1          # equal groups of neighbouring experts
    keep: int = 1            # groups whose experts can be chosen
    scale: float = 1.0       # of the weights
    shared_ff: int | None = None
    shared_limit: float = 0.0


@dataclass(frozen=True)
class LayerConfig:
    type: str
    mixer: LatentAttentionConfig
    mlp: MlpConfig | None


@dataclass(frozen=True)
class LoopConfig:
    start: int
    stop: int
    times: int


@dataclass(frozen=True)
class GomeraxConfig:
    vocab: int
    width: int
    max_positions: int
    layers: tuple
    norm_eps: float
    embedding_scale: float
    loop: LoopConfig | None
    raw: dict = field(compare=False, repr=False, default_factory=dict)

    architecture = ARCHITECTURE

    @classmethod
    def from_dict(cls, data: dict, source: str = "config.json") -> "GomeraxConfig":
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
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1), max_positions=r.integer("max_positions", minimum=1),
                   layers=layers, norm_eps=r.number("norm.eps", exclusive_minimum=0.0), embedding_scale=r.number("embedding.scale", default=1.0),
                   loop=loop, raw=data)

    @classmethod
    def _layer(cls, entry, where: str) -> LayerConfig:
        if not isinstance(entry, dict):
            raise ConfigError(f"{where} must be an object")
        e = ConfigReader(entry, where)
        kind = e.string("type")
        if kind not in MIXERS:
            raise ConfigError(f"{where}: type '{kind}' is not known (known: {', '.join(MIXERS)})")
        rot_dim = e.integer("mixer.rot_dim", minimum=0)
        mixer = LatentAttentionConfig(
            heads=e.integer("mixer.heads", minimum=1), dim=e.integer("mixer.dim", minimum=1), rot_dim=rot_dim,
            vdim=e.integer("mixer.vdim", minimum=1), q_rank=e.integer("mixer.q_rank", minimum=1), kv_rank=e.integer("mixer.kv_rank", minimum=1),
            scale=e.number("mixer.scale", exclusive_minimum=0.0), rot_dims=e.integer("mixer.rot.dims", default=rot_dim, minimum=0),
            rot_base=e.number("mixer.rot.base", default=10000.0, exclusive_minimum=0.0), window=e.integer("mixer.mask.size", default=None, minimum=1))
        if mixer.rot_dims % 2 or mixer.rot_dims > rot_dim:
            raise ConfigError(f"{where}: mixer.rot.dims {mixer.rot_dims} must be even and at most mixer.rot_dim {rot_dim}")
        return LayerConfig(kind, mixer, cls._mlp(entry, e, where) if entry.get("mlp") is not None else None)

    @staticmethod
    def _mlp(entry, e: ConfigReader, where: str) -> MlpConfig:
        kind = e.string("mlp.kind")
        if kind not in MLP_KINDS:
            raise ConfigError(f"{where}: mlp.kind '{kind}' is not known (known: {', '.join(MLP_KINDS)})")
        if kind == "dense":
            return MlpConfig("dense", ff=e.integer("mlp.ff", minimum=1))
        groups, keep = 1, 1
        if (entry["mlp"].get("router") or {}).get("groups") is not None:
            groups, keep = e.integer("mlp.router.groups.count", minimum=1), e.integer("mlp.router.groups.keep", minimum=1)
        shared_ff = e.integer("mlp.shared.ff", default=None, minimum=1)
        mlp = MlpConfig("moe", ff=e.integer("mlp.expert.ff", minimum=1), limit=e.number("mlp.expert.limit", exclusive_minimum=0.0),
                        experts=e.integer("mlp.router.experts", minimum=1), top=e.integer("mlp.router.top", minimum=1), groups=groups, keep=keep,
                        scale=e.number("mlp.router.scale", default=1.0), shared_ff=shared_ff,
                        shared_limit=0.0 if shared_ff is None else e.number("mlp.shared.limit", exclusive_minimum=0.0))
        if mlp.experts % groups:
            raise ConfigError(f"{where}: mlp.router.experts {mlp.experts} is not a multiple of mlp.router.groups.count {groups}")
        if keep > groups:
            raise ConfigError(f"{where}: mlp.router.groups.keep {keep} is more than mlp.router.groups.count {groups}")
        if mlp.top > keep * (mlp.experts // groups):
            raise ConfigError(f"{where}: mlp.router.top {mlp.top} is more than the {keep * (mlp.experts // groups)} experts of the groups kept")
        return mlp

    def runs(self) -> list:
        """[(layer, whether the embedding's output is added in front of it)] in the order the layers run: at the beginning of every
        pass of the loop but the first."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, False) for i in range(n)]
        a, b = self.loop.start, self.loop.stop
        passes = [(i, k > 0 and i == a) for k in range(self.loop.times) for i in range(a, b)]
        return [(i, False) for i in range(a)] + passes + [(i, False) for i in range(b, n)]

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
            mixer = dict(heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, q_rank=m.q_rank, kv_rank=m.kv_rank, scale=m.scale,
                         rot=dict(dims=m.rot_dims, base=m.rot_base))
            if m.window is not None:
                mixer["mask"] = dict(size=m.window)
            mlp = None
            if f is not None and f.kind == "dense":
                mlp = dict(kind="dense", ff=f.ff)
            elif f is not None:
                router = dict(experts=f.experts, top=f.top, scale=f.scale)
                if f.groups > 1:
                    router["groups"] = dict(count=f.groups, keep=f.keep)
                mlp = dict(kind="moe", expert=dict(ff=f.ff, limit=f.limit), router=router)
                if f.shared_ff is not None:
                    mlp["shared"] = dict(ff=f.shared_ff, limit=f.shared_limit)
            layers.append(dict(type=l.type, mixer=mixer, mlp=mlp))
        d = dict(architecture=ARCHITECTURE, vocab=self.vocab, width=self.width, max_positions=self.max_positions, layers=layers,
                 norm=dict(eps=self.norm_eps), embedding=dict(scale=self.embedding_scale))
        if self.loop is not None:
            d["loop"] = dict(start=self.loop.start, stop=self.loop.stop, times=self.loop.times)
        return d

    def describe(self) -> dict:
        return self.to_dict()
