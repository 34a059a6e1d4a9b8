"""Disorax configuration, from the keys of its config.json.

The file lists the layers one by one::

    {"architecture": "Disorax", "vocab": V, "width": W, "norm": {"eps": e}, "residual_mult": m,
     "layers": [{"type": "attention",
                 "mixer": {"heads": H, "kv_heads": G, "dim": d, "vdim": dv, "scale": s, "v_mix": true | false,
                           "mask": {"size": w, "keep_first": f} | null, "rot": {"base": b, "dims": r}},
                 "mlp": {"kind": "moe", "expert": {"ff": F}, "router": {"experts": E, "top": k},
                         "shared": {"ff": Fs} | null} | null},
                {"type": "latent_attention",
                 "mixer": {"heads": H, "dim": d, "vdim": dv, "kv_rank": k, "scale": s}, "mlp": ...},
                {"type": "latent_attention_2",
                 "mixer": {"heads": H, "dim": d, "vdim": dv, "kv_rank": k, "scale": s, "mask": {"size": w} | null},
                 "mlp": ...}, ...]}

Every size and constant is read from there; a layer may differ from the next in all of them.  ``mask`` left out or null
means every earlier token is seen, ``keep_first`` left out that a window keeps no first tokens, ``v_mix`` left out that
values are not mixed, ``mlp`` left out or null a layer without a feed-forward, ``shared`` experts without a shared one,
``residual_mult`` left out 1.  ``max_positions`` (optional) bounds a sequence's length.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any

from .base import ConfigError, KeyReader, ModelConfig

MLP_KINDS = ("moe",)
DEFAULT_MAX_POSITIONS = 1 << 20      # the design itself has no limit: positions are turned into angles on the fly


def _mask(data, where) -> tuple:
    """(window size, kept first tokens); (0, 0) without a mask."""
    if data.get("mask") is None:
        return 0, 0
    r = KeyReader(data["mask"], where + ".mask")
    return r.integer("size", minimum=1), r.integer("keep_first", 0, minimum=0)


@dataclass(frozen=True)
class AttentionSpec:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rope_base: float
    rope_dims: int
    window: int = 0        # 0: every earlier token is seen
    keep_first: int = 0
    v_mix: bool = False

    @classmethod
    def from_dict(cls, data, where):
        r = KeyReader(data, where)
        if not isinstance(data.get("rot"), dict):
            raise ConfigError(f"{where}: required key 'rot' is missing")
        rot = KeyReader(data["rot"], where + ".rot")
        heads = r.integer("heads", minimum=1)
        window, keep_first = _mask(data, where)
        out = cls(heads=heads, kv_heads=r.integer("kv_heads", heads, minimum=1), dim=r.integer("dim", minimum=1),
                  vdim=r.integer("vdim", minimum=1), scale=r.number("scale"), rope_base=rot.number("base", positive=True),
                  rope_dims=rot.integer("dims", minimum=0), window=window, keep_first=keep_first, v_mix=r.boolean("v_mix", False))
        if out.heads % out.kv_heads:
            raise ConfigError(f"{where}: 'kv_heads' must divide 'heads'")
        if out.rope_dims % 2 or out.rope_dims > out.dim:
            raise ConfigError(f"{where}.rot: {out.rope_dims} turning lanes in heads of {out.dim} (an even number up to the head size)")
        return out

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale,
             "v_mix": self.v_mix, "rot": {"base": self.rope_base, "dims": self.rope_dims}}
        if self.window:
            d["mask"] = {"size": self.window, "keep_first": self.keep_first}
        return d


@dataclass(frozen=True)
class LatentSpec:
    heads: int
    dim: int
    vdim: int
    kv_rank: int
    scale: float
    window: int = 0        # 0: every earlier token is seen

    @classmethod
    def from_dict(cls, data, where):
        r = KeyReader(data, where)
        window, keep_first = _mask(data, where)
        if keep_first:
            raise ConfigError(f"{where}.mask: a window over latent rows keeps no first tokens")
        return cls(heads=r.integer("heads", minimum=1), dim=r.integer("dim", minimum=1), vdim=r.integer("vdim", minimum=1),
                   kv_rank=r.integer("kv_rank", minimum=1), scale=r.number("scale"), window=window)

    def to_dict(self):
        d = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim, "kv_rank": self.kv_rank, "scale": self.scale}
        if self.window:
            d["mask"] = {"size": self.window}
        return d


MIXER_SPECS = {"attention": AttentionSpec, "latent_attention": LatentSpec, "latent_attention_2": LatentSpec}
MIXER_TYPES = tuple(MIXER_SPECS)


@dataclass(frozen=True)
class DisoraxMlp:
    kind: str
    ff: int                # an expert's hidden size
    experts: int
    top: int
    shared_ff: int = 0     # 0: no shared expert

    @classmethod
    def from_dict(cls, data, where):
        r = KeyReader(data, where)
        kind = r.string("kind")
        if kind not in MLP_KINDS:
            raise ConfigError(f"{where}: kind '{kind}' is not one of {MLP_KINDS}")
        for key in ("router", "expert"):
            if not isinstance(data.get(key), dict):
                raise ConfigError(f"{where}: required key '{key}' is missing")
        router = KeyReader(data["router"], where + ".router")
        shared = data.get("shared")
        out = cls(kind, ff=KeyReader(data["expert"], where + ".expert").integer("ff", minimum=1),
                  experts=router.integer("experts", minimum=1), top=router.integer("top", minimum=1),
                  shared_ff=0 if shared is None else KeyReader(shared, where + ".shared").integer("ff", minimum=1))
        if out.top > out.experts:
            raise ConfigError(f"{where}.router: 'top' exceeds 'experts'")
        return out

    def to_dict(self):
        d = {"kind": self.kind, "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}
        if self.shared_ff:
            d["shared"] = {"ff": self.shared_ff}
        return d


@dataclass(frozen=True)
class DisoraxLayer:
    type: str
    mixer: Any
    mlp: DisoraxMlp | None = None

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
                   None if mlp is None else DisoraxMlp.from_dict(mlp, where + ".mlp"))

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class DisoraxConfig(ModelConfig):
    vocab: int
    width: int
    layers: tuple
    norm_eps: float = 1e-6
    residual_mult: float = 1.0
    max_positions: int = DEFAULT_MAX_POSITIONS
    architecture: str = "Disorax"
    extra: dict = field(default_factory=dict, compare=False)

    def __post_init__(self):
        object.__setattr__(self, "layers", tuple(self.layers))
        if not self.layers:
            raise ConfigError("a model needs at least one layer")
        mixing = {(l.mixer.kv_heads, l.mixer.vdim) for l in self.layers if l.type == "attention" and l.mixer.v_mix}
        if len(mixing) > 1:
            raise ConfigError(f"layers that mix their values need values of one size, found {sorted(mixing)} (heads, lanes)")

    @classmethod
    def from_dict(cls, data: dict[str, Any]) -> "DisoraxConfig":
        r = KeyReader(data)
        layers = data.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        norm = KeyReader(data.get("norm") or {}, "config.json.norm")
        return cls(vocab=r.integer("vocab", minimum=1), width=r.integer("width", minimum=1),
                   layers=tuple(DisoraxLayer.from_dict(l, f"config.json.layers[{i}]") for i, l in enumerate(layers)),
                   norm_eps=norm.number("eps", positive=True), residual_mult=r.number("residual_mult", 1.0),
                   max_positions=r.integer("max_positions", DEFAULT_MAX_POSITIONS, minimum=1),
                   architecture=r.string("architecture", "Disorax"))

    def to_dict(self) -> dict[str, Any]:
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "norm": {"eps": self.norm_eps},
             "residual_mult": self.residual_mult, "layers": [l.to_dict() for l in self.layers]}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        return d
