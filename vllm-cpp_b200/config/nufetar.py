"""Nufetar configuration, from the keys of its config.json.

The file lists the layers one by one::

    {"architecture": "Nufetar", "vocab": V, "width": W, "norm": {"eps": e},
     "layers": [{"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": s, "mask": {"size": c} | null,
                           "rot": {"base": b, "dims": r}},
                 "mlp": {"kind": "dense", "ff": F} | null},
                {"type": "latent_attention",
                 "mixer": {"heads": H, "dim": d, "rot_dim": r, "vdim": dv, "kv_rank": k, "scale": s,
                           "mask": {"size": w} | null, "rot": {"base": b, "dims": r}},
                 "mlp": ...},
                {"type": "wkv", "mixer": {"heads": H, "dim": d}, "mlp": ...}, ...]}

Every size and constant is read from there; a layer may differ from the next in all of them.  ``mask`` is the size of
the chunks of an "attention" mixer and of the sliding window of a "latent_attention" one; left out or null, every
earlier token is seen.  ``mlp`` left out or null is a layer without a feed-forward.  The rank of the low-rank pair
behind a "wkv" mixer's decay is not in the file: it is the shape of the tensors (``rank``, optional, names it for a model
that is written from a configuration).  ``max_positions`` (optional) bounds a sequence's length.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from .base import ConfigError, KeyReader, ModelConfig

MLP_KINDS = ("dense",)
DEFAULT_MAX_POSITIONS = 1 << 20      # the design itself has no limit: positions are turned into angles on the fly


@dataclass(frozen=True)
class Rotation:
    base: float
    dims: int

    @classmethod
    def from_dict(cls, data, where, default_dims=None):
        if not isinstance(data, dict):
            raise ConfigError(f"{where}: required key 'rot' is missing")
        r = KeyReader(data, where + ".rot")
        dims = r.integer("dims", minimum=0) if default_dims is None else r.integer("dims", default_dims, minimum=0)
        if dims % 2:
            raise ConfigError(f"{where}.rot: 'dims' must be even (lanes turn in pairs)")
        return cls(base=r.number("base", positive=True), dims=dims)

    def to_dict(self):
        return {"base": self.base, "dims": self.dims}


def _mask_size(data, where) -> int:
    mask = data.get("mask")
    if mask is None:
        return 0
    return KeyReader(mask, where + ".mask").integer("size", minimum=1)


@dataclass(frozen=True)
class ChunkAttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: int             # 0: every earlier token is seen
    rot: Rotation

    @classmethod
    def from_dict(cls, data, where):
        r = KeyReader(data, where)
        heads = r.integer("heads", minimum=1)
        out = cls(heads=heads, kv_heads=r.integer("kv_heads", heads, minimum=1), dim=r.integer("dim", minimum=1),
                  vdim=r.integer("vdim", minimum=1), scale=r.number("scale"), chunk=_mask_size(data, where),
                  rot=Rotation.from_dict(data.get("rot"), where))
        if out.heads % out.kv_heads:
            raise ConfigError(f"{where}: 'kv_heads' must divide 'heads'")
        if out.rot.dims > out.dim:
            raise ConfigError(f"{where}.rot: {out.rot.dims} turning lanes in heads of {out.dim}")
        return out

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
             "rot": self.rot.to_dict()}
        if self.chunk:
            d["mask"] = {"size": self.chunk}
        return d


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int               # lanes of a head's query and key that do not turn
    rot_dim: int           # lanes that turn; the key's are shared by all heads
    vdim: int
    kv_rank: int
    scale: float
    window: int            # 0: every earlier token is seen
    rot: Rotation

    @classmethod
    def from_dict(cls, data, where):
        r = KeyReader(data, where)
        rot_dim = r.integer("rot_dim", minimum=0)
        out = cls(heads=r.integer("heads", minimum=1), dim=r.integer("dim", minimum=1), rot_dim=rot_dim,
                  vdim=r.integer("vdim", minimum=1), kv_rank=r.integer("kv_rank", minimum=1), scale=r.number("scale"),
                  window=_mask_size(data, where), rot=Rotation.from_dict(data.get("rot"), where, rot_dim))
        if out.rot.dims != out.rot_dim:
            raise ConfigError(f"{where}.rot: 'dims' is {out.rot.dims}, the turning part has {out.rot_dim} lanes ('rot_dim')")
        return out

    def to_dict(self):
        d = {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim, "kv_rank": self.kv_rank,
             "scale": self.scale, "rot": self.rot.to_dict()}
        if self.window:
            d["mask"] = {"size": self.window}
        return d


@dataclass(frozen=True)
class WkvSpec:
    heads: int
    dim: int               # lanes of a head's r, k and v alike
    rank: int = 0          # of the decay's low-rank projection; 0: whatever the tensors' shape says

    @classmethod
    def from_dict(cls, data, where):
        r = KeyReader(data, where)
        return cls(heads=r.integer("heads", minimum=1), dim=r.integer("dim", minimum=1), rank=r.integer("rank", 0, minimum=0) or 0)

    def to_dict(self):
        d = {"heads": self.heads, "dim": self.dim}
        if self.rank:
            d["rank"] = self.rank
        return d


MIXER_SPECS = {"attention": ChunkAttentionSpec, "latent_attention": LatentSpec, "wkv": WkvSpec}
MIXER_TYPES = tuple(MIXER_SPECS)


@dataclass(frozen=True)
class NufetarMlp:
    kind: str
    ff: int

    @classmethod
    def from_dict(cls, data, where):
        r = KeyReader(data, where)
        kind = r.string("kind")
        if kind not in MLP_KINDS:
            raise ConfigError(f"{where}: kind '{kind}' is not one of {MLP_KINDS}")
        return cls(kind, ff=r.integer("ff", minimum=1))

    def to_dict(self):
        return {"kind": self.kind, "ff": self.ff}


@dataclass(frozen=True)
class NufetarLayer:
    type: str
    mixer: Any
    mlp: NufetarMlp | None = None

    @classmethod
    def from_dict(cls, data, where):
        r = KeyReader(data, where)
        kind = r.string("type")
        if kind not in MIXER_SPECS:
            raise ConfigError(f"{where}: layer type '{kind}' is not one of {MIXER_TYPES}")
        if not isinstance(data.get("mixer"), dict):
            raise ConfigError(f"{where}: required key 'mixer' is missing")
        mlp = data.get("mlp")
        return cls(kind, MIXER_SPECS[kind].from_dict(data["mixer"], where + ".mixer"),
                   None if mlp is None else NufetarMlp.from_dict(mlp, where + ".mlp"))

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class NufetarConfig(ModelConfig):
    vocab: int
    width: int
    layers: tuple
    norm_eps: float = 1e-6
    max_positions: int = DEFAULT_MAX_POSITIONS
    architecture: str = "Nufetar"
    extra: dict = field(default_factory=dict, compare=False)

    def __post_init__(self):
        object.__setattr__(self, "layers", tuple(self.layers))
        if not self.layers:
            raise ConfigError("a model needs at least one layer")

    @classmethod
    def from_dict(cls, data: dict[str, Any]) -> "NufetarConfig":
        r = KeyReader(data)
        layers = data.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        norm = KeyReader(data.get("norm") or {}, "config.json.norm")
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   layers=tuple(NufetarLayer.from_dict(l, f"config.json.layers[{i}]") for i, l in enumerate(layers)),
                   norm_eps=norm.number("eps", positive=True),
                   max_positions=r.integer("max_positions", DEFAULT_MAX_POSITIONS, minimum=1),
                   architecture=r.string("architecture", "Nufetar"))

    def to_dict(self) -> dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "layers": [l.to_dict() for l in self.layers]}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d
