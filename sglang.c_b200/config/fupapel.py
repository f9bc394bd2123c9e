"""Typed configuration of the Fupapel architecture: a decoder whose config.json lists its layers one
by one.  A layer adds a mixer's result and a feed-forward's (if it has one), each behind a norm of its
own, both of the same stream, times one number (`residual_mult`); the mixer reads its normed rows
moved towards the token before.  The mixer is chunked attention with gated results ("attention"),
chunked attention behind short convolutions, with a factor and a sink per head ("attention_2", which
may read the keys and values of an earlier layer: `kv_from`), or latent attention with a sink and a
gate per head ("latent_attention").  The feed-forward is a mixture of experts, some of which hand their
input on as it is.  Every size and every constant that may differ between models comes from the file:

    {"architecture": "Fupapel", "vocab": V, "width": E, "norm": {"eps": e}, "residual_mult": m,
     "layers": [{"type": "attention",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size"}, "rot": {"base", "dims"}},
                 "mlp": {"kind": "moe", "expert": {"ff": F},
                         "router": {"experts", "top", "identity", "groups": {"count", "keep"}}}},
                {"type": "attention_2",
                 "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "conv", "mask": {"size"}, "kv_from": j,
                           "rot": {"base", "dims", "scaling": {"factor", "low", "high", "original"}}},
                 "mlp": null},
                {"type": "latent_attention",
                 "mixer": {"heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank", "scale", "rot": {...}},
                 "mlp": ...}]}

`mask`, `rot`, `scaling`, `kv_from`, `identity` and `groups` may be absent: the model then has no such
thing.  An optional `max_positions` bounds a request's length (positions are computed, not looked up).
"""
from dataclasses import dataclass
from typing import Optional, Tuple

from .base import ConfigError, get_float, get_int, get_str

LAYER_TYPES = ("attention", "attention_2", "latent_attention")
DEFAULT_MAX_POSITIONS = 1 << 16


@dataclass(frozen=True)
class WavelengthScaling:
    """Pairs of long wavelength are slowed by `factor`, short ones kept, the rest blended."""
    factor: float
    low: float
    high: float
    original: float

    def to_dict(self):
        return {"factor": self.factor, "low": self.low, "high": self.high, "original": self.original}


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    scaling: Optional[WavelengthScaling] = None

    def to_dict(self):
        d = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = self.scaling.to_dict()
        return d


@dataclass(frozen=True)
class AttentionMixer:
    """The "attention" and "attention_2" mixers (`conv` and `kv_from` belong to the second)."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    chunk: Optional[int] = None
    rot: Optional[Rotation] = None
    conv: Optional[int] = None
    kv_from: Optional[int] = None

    def to_dict(self):
        d = {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim, "scale": self.scale}
        if self.chunk is not None:
            d["mask"] = {"size": self.chunk}
        if self.rot is not None:
            d["rot"] = self.rot.to_dict()
        if self.conv is not None:
            d["conv"] = self.conv
        if self.kv_from is not None:
            d["kv_from"] = self.kv_from
        return d


@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int
    rot_dim: int
    vdim: int
    kv_rank: int
    q_rank: int
    scale: float
    rot: Rotation

    def to_dict(self):
        return {"heads": self.heads, "dim": self.dim, "rot_dim": self.rot_dim, "vdim": self.vdim,
                "kv_rank": self.kv_rank, "q_rank": self.q_rank, "scale": self.scale, "rot": self.rot.to_dict()}


@dataclass(frozen=True)
class RoutedMlp:
    ff: int                           # an expert's inner width
    experts: int
    top: int
    identity: int = 0                 # experts behind the others that hand their input on
    groups: int = 1
    keep: int = 1

    def to_dict(self):
        r = {"experts": self.experts, "top": self.top}
        if self.identity:
            r["identity"] = self.identity
        if self.groups != 1:
            r["groups"] = {"count": self.groups, "keep": self.keep}
        return {"kind": "moe", "expert": {"ff": self.ff}, "router": r}


@dataclass(frozen=True)
class FupapelLayer:
    type: str
    mixer: object                     # AttentionMixer | LatentMixer
    mlp: Optional[RoutedMlp]

    def to_dict(self):
        return {"type": self.type, "mixer": self.mixer.to_dict(), "mlp": None if self.mlp is None else self.mlp.to_dict()}


def _obj(d, key, where):
    v = d.get(key)
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return v


def _read_rotation(m, where, dim):
    r = _obj(m, "rot", where)
    dims = get_int(r, "dims", minimum=0)
    if dims > dim or dims % 2:
        raise ConfigError(f"config.json: key 'dims' ({dims}) must be even and at most {dim}")
    scaling = None
    if r.get("scaling") is not None:
        s = _obj(r, "scaling", where + ".rot")
        scaling = WavelengthScaling(*(get_float(s, k, positive=True) for k in ("factor", "low", "high", "original")))
        if scaling.high < scaling.low:
            raise ConfigError(f"config.json: key 'high' ({scaling.high}) must not be below 'low' ({scaling.low})")
    return Rotation(dims, get_float(r, "base", positive=True), scaling)


def _read_mixer(kind, m, where):
    if kind == "latent_attention":
        rot_dim = get_int(m, "rot_dim", minimum=0)
        rot = _read_rotation(m, where, rot_dim)
        return LatentMixer(get_int(m, "heads", minimum=1), get_int(m, "dim", minimum=1), rot_dim,
                           get_int(m, "vdim", minimum=1), get_int(m, "kv_rank", minimum=1),
                           get_int(m, "q_rank", minimum=1), get_float(m, "scale", positive=True), rot)
    heads, kv = get_int(m, "heads", minimum=1), get_int(m, "kv_heads", minimum=1)
    if heads % kv:
        raise ConfigError(f"config.json: key 'heads' ({heads}) must be a multiple of 'kv_heads' ({kv})")
    dim = get_int(m, "dim", minimum=1)
    chunk = get_int(_obj(m, "mask", where), "size", minimum=1) if m.get("mask") is not None else None
    rot = _read_rotation(m, where, dim) if m.get("rot") is not None else None
    conv = kv_from = None
    if kind == "attention_2":
        conv = get_int(m, "conv", minimum=1)
        kv_from = get_int(m, "kv_from", default=None, minimum=0)
    return AttentionMixer(heads, kv, dim, get_int(m, "vdim", minimum=1), get_float(m, "scale", positive=True), chunk, rot,
                          conv, kv_from)


def _read_mlp(mlp, where):
    if mlp is None:
        return None
    if not isinstance(mlp, dict):
        raise ConfigError(f"config.json: {where}.mlp must be null or an object")
    get_str(mlp, "kind", choices={"moe"})
    router = _obj(mlp, "router", where + ".mlp")
    experts, top = get_int(router, "experts", minimum=1), get_int(router, "top", minimum=1)
    identity = get_int(router, "identity", default=0, minimum=0)
    count = keep = 1
    if router.get("groups") is not None:
        g = _obj(router, "groups", where + ".mlp.router")
        count, keep = get_int(g, "count", minimum=1), get_int(g, "keep", minimum=1)
    n = experts + identity
    if n % count:
        raise ConfigError(f"config.json: {where}.mlp.router: {n} router outputs do not form {count} equal groups")
    if keep > count:
        raise ConfigError(f"config.json: {where}.mlp.router.groups: keep ({keep}) is more than count ({count})")
    if top > keep * (n // count):
        raise ConfigError(f"config.json: {where}.mlp.router: top ({top}) is more than the kept groups hold")
    return RoutedMlp(get_int(_obj(mlp, "expert", where + ".mlp"), "ff", minimum=1), experts, top, identity, count, keep)


@dataclass(frozen=True)
class FupapelConfig:
    vocab: int
    width: int
    norm_eps: float
    residual_mult: float
    layers: Tuple[FupapelLayer, ...]
    max_positions: int = DEFAULT_MAX_POSITIONS
    eos_token_id: Optional[int] = None
    architecture: str = "Fupapel"

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
            kind = get_str(entry, "type", choices=set(LAYER_TYPES))
            try:
                mixer = _read_mixer(kind, entry["mixer"], where + ".mixer")
                mlp = _read_mlp(entry.get("mlp"), where)
            except ConfigError as e:
                raise ConfigError(f"{e} (in {where})") from None
            if kind == "attention_2" and mixer.kv_from is not None:
                j = mixer.kv_from
                src = layers[j].mixer if j < i and layers[j].type == "attention_2" else None
                if src is None or src.kv_from is not None:
                    raise ConfigError(f"config.json: {where}.mixer.kv_from = {j} must name an earlier attention_2 "
                                      "layer with keys and values of its own")
                if (src.kv_heads, src.dim, src.vdim, src.rot) != (mixer.kv_heads, mixer.dim, mixer.vdim, mixer.rot):
                    raise ConfigError(f"config.json: {where} reads the keys and values of layer {j}, whose key/value "
                                      "heads, sizes or rotation differ")
            layers.append(FupapelLayer(kind, mixer, mlp))
        return cls(vocab=get_int(d, "vocab", minimum=1), width=get_int(d, "width", minimum=1),
                   norm_eps=get_float(norm, "eps", positive=True),
                   residual_mult=get_float(d, "residual_mult", positive=True), layers=tuple(layers),
                   max_positions=get_int(d, "max_positions", default=DEFAULT_MAX_POSITIONS, minimum=1),
                   eos_token_id=get_int(d, "eos_token_id", default=None))

    def to_dict(self):
        d = {"architecture": self.architecture, "vocab": self.vocab, "width": self.width,
             "norm": {"eps": self.norm_eps}, "residual_mult": self.residual_mult,
             "layers": [layer.to_dict() for layer in self.layers]}
        if self.max_positions != DEFAULT_MAX_POSITIONS:
            d["max_positions"] = self.max_positions
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d
