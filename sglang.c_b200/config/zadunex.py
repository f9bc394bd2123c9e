"""Typed configuration of the Zadunex architecture: a decoder over several residual streams whose
config.json lists its layers one by one.  A layer is pre-norm: a mixer, then a feed-forward, each of which
reads one combination of the streams and writes into all of them.  The mixer is a selective state
space ("mamba2") or softmax attention with biases, norms over the whole query and key projections, a partial
rotation and a constant in the softmax's denominator ("attention"); the feed-forward is dense with
bounded gates, a mixture of experts, or absent.  A run of consecutive layers may be repeated several
times with the same weights (`loop`).  Every size and every constant that may differ between models
comes from the file:

    {"architecture": "Zadunex", "vocab": V, "width": E, "streams": s, "norm": {"eps": e}, "logit_scale": c,
     "loop": {"start": a, "stop": b, "times": n},            (optional)
     "layers": [{"type": "mamba2", "mixer": {"heads", "vdim", "state", "groups", "conv", "norm_groups"},
                 "mlp": {"kind": "dense", "ff": F, "limit": L}},
                {"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "rot": {"base", "dims"}},
                 "mlp": {"kind": "moe", "expert": {"ff": F}, "router": {"experts", "top"}}},
                {"type": ..., "mixer": {...}, "mlp": null}]}

`rot` may be left out: nothing is turned then.  An optional `max_positions` bounds a request's length
(positions are computed, not looked up).
"""
from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigError, LayerLoop, get_float, get_int, get_str

DEFAULT_MAX_POSITIONS = 1 << 16


def _obj(d, key, where):
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return v


@dataclass(frozen=True)
class StateSpaceMixer:
    heads: int
    vdim: int
    state: int
    groups: int
    conv: int
    norm_groups: int

    @classmethod
    def read(cls, m, where):
        self = cls(*(get_int(m, k, minimum=1) for k in ("heads", "vdim", "state", "groups", "conv", "norm_groups")))
        if self.heads % self.groups:
            raise ConfigError(f"config.json: key 'heads' ({self.heads}) must be a multiple of 'groups' ({self.groups})")
        if (self.heads * self.vdim) % self.norm_groups:
            raise ConfigError(f"config.json: heads x vdim ({self.heads * self.vdim}) must be a multiple of "
                              f"'norm_groups' ({self.norm_groups})")
        return self

    def to_dict(self):
        return {"heads": self.heads, "vdim": self.vdim, "state": self.state, "groups": self.groups, "conv": self.conv,
                "norm_groups": self.norm_groups}


@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot_dims: int = 0
    rot_base: float = 10000.0

    @classmethod
    def read(cls, m, where):
        heads, kv = get_int(m, "heads", minimum=1), get_int(m, "kv_heads", minimum=1)
        if heads % kv:
            raise ConfigError(f"config.json: key 'heads' ({heads}) must be a multiple of 'kv_heads' ({kv})")
        dim = get_int(m, "dim", minimum=1)
        more = {}
        if m.get("rot") is not None:
            rot = _obj(m, "rot", where)
            dims = get_int(rot, "dims", minimum=0)
            if dims > dim or dims % 2:
                raise ConfigError(f"config.json: key 'dims' ({dims}) must be even and at most 'dim' ({dim})")
            more = {"rot_dims": dims, "rot_base": get_float(rot, "base", positive=True)}
        return cls(heads, kv, dim, get_int(m, "vdim", minimum=1), get_float(m, "scale"), **more)

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.rot_dims:
            d["rot"] = {"base": self.rot_base, "dims": self.rot_dims}
        return d


_MIXERS = {"mamba2": StateSpaceMixer, "attention": AttentionMixer}


@dataclass(frozen=True)
class ZadunexMlp:
    kind: str                         # "dense" | "moe"
    ff: int                           # dense: inner width; moe: an expert's inner width
    limit: float = 0.0                # dense: the bound of gate and up values
    experts: int = 0
    top: int = 0

    @classmethod
    def read(cls, mlp, where):
        if mlp is None:
            return None
        if not isinstance(mlp, dict):
            raise ConfigError(f"config.json: {where}.mlp must be null or an object")
        kind = get_str(mlp, "kind", choices={"dense", "moe"})
        if kind == "dense":
            return cls("dense", get_int(mlp, "ff", minimum=1), limit=get_float(mlp, "limit", positive=True))
        router = _obj(mlp, "router", where + ".mlp")
        experts, top = get_int(router, "experts", minimum=1), get_int(router, "top", minimum=1)
        if top > experts:
            raise ConfigError(f"config.json: key 'top' ({top}) must be at most 'experts' ({experts})")
        return cls("moe", get_int(_obj(mlp, "expert", where + ".mlp"), "ff", minimum=1), experts=experts, top=top)

    def to_dict(self):
        if self.kind == "dense":
            return {"kind": "dense", "ff": self.ff, "limit": self.limit}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": {"experts": self.experts, "top": self.top}}


@dataclass(frozen=True)
class ZadunexLayer:
    type: str
    mixer: object                     # StateSpaceMixer | AttentionMixer
    mlp: Optional[ZadunexMlp]

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


@dataclass(frozen=True)
class ZadunexConfig:
    vocab: int
    width: int
    streams: int
    norm_eps: float
    logit_scale: float
    layers: Tuple[ZadunexLayer, ...]
    loop: Optional[LayerLoop] = None
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_id: Optional[int] = None
    architecture: str = "Zadunex"

    @classmethod
    def from_dict(cls, d):
        norm = d.get("norm")
        if not isinstance(norm, dict):
            raise ConfigError("config.json: key 'norm' must be an object with 'eps'")
        raw = d.get("layers")
        if not isinstance(raw, list) or not raw:
            raise ConfigError("config.json: key 'layers' must be a non-empty list")
        layers = []
        for i, entry in enumerate(raw):
            where = f"layers[{i}]"
            if not isinstance(entry, dict) or not isinstance(entry.get("mixer"), dict):
                raise ConfigError(f"config.json: {where} must be an object with 'type' and 'mixer'")
            kind = get_str(entry, "type", choices=set(_MIXERS))
            try:
                layers.append(ZadunexLayer(kind, _MIXERS[kind].read(entry["mixer"], where + ".mixer"),
                                           ZadunexMlp.read(entry.get("mlp"), where)))
            except ConfigError as e:
                raise ConfigError(f"{e} (in {where})") from None
        return cls(vocab=get_int(d, "vocab", minimum=1), width=get_int(d, "width", minimum=1),
                   streams=get_int(d, "streams", minimum=1), norm_eps=get_float(norm, "eps", positive=True),
                   logit_scale=get_float(d, "logit_scale", default=1.0), layers=tuple(layers),
                   loop=LayerLoop.read(d.get("loop"), len(layers)),
                   max_positions=get_int(d, "max_positions", default=DEFAULT_MAX_POSITIONS, minimum=1),
                   eos_token_id=get_int(d, "eos_token_id", default=None))

    def to_dict(self):
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width, "streams": self.streams,
             "norm": {"eps": self.norm_eps}, "logit_scale": self.logit_scale,
             "layers": [layer.to_dict() for layer in self.layers]}
        if self.loop is not None:
            d["loop"] = self.loop.to_dict()
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d
