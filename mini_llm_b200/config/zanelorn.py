"""ZanelornConfig: the keys of a Zanelorn config.json, typed and checked.

A Zanelorn model is a list of layers.  Every entry names its mixer ("retention" or "parallel") with that mixer's sizes and
constants, and its feed-forward (dense, a mixture of experts, or none).  Nothing is assumed equal between layers: every size
is read per entry.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Union

from .base import ConfigError, ModelConfig
from .finuvik import _int, _num

LAYER_TYPES = ("retention", "parallel")
FF_KINDS = ("dense", "moe")


@dataclass
class Rotation:
    base: float
    dims: int
    factor: Optional[float] = None       # every frequency is divided by it (None: as it is)


@dataclass
class RetentionSizes:
    heads: int
    dim: int                  # rows of a head's state: a query's and a key's entries
    vdim: int                 # columns of it: a value's entries
    decay: List[float]        # one per head
    rot: Rotation = None


@dataclass
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    rot: Rotation
    window: Optional[int] = None      # keys a query sees, itself included; None: all
    keep_first: int = 0               # first tokens that stay visible beyond the window


@dataclass
class MambaSizes:
    inner: int
    state: int
    dt_rank: int
    conv: int                 # taps of the convolution


@dataclass
class ParallelSizes:
    left: AttentionSizes
    right: MambaSizes
    left_scale: float
    right_scale: float


@dataclass
class DenseSizes:
    ff: int


@dataclass
class ExpertsSizes:
    experts: int
    identity: int             # router outputs behind the experts' whose experts give their input back
    top: int
    ff: int
    limit: float
    shared_ff: Optional[int] = None
    shared_limit: Optional[float] = None


@dataclass
class ZanelornLayer:
    type: str
    mixer: Union[RetentionSizes, ParallelSizes]
    mlp: Optional[Union[DenseSizes, ExpertsSizes]] = None


def _obj(d: dict, key: str, where: str, optional: bool = False):
    v = d.get(key)
    if v is None and optional:
        return None
    if not isinstance(v, dict):
        raise ConfigError(f"config.json: {where}.{key} must be an object")
    return v


def _positive(d: dict, key: str, where: str) -> float:
    v = _num(d, key, where)
    if not v > 0:
        raise ConfigError(f"config.json: {where}.{key} must be positive, got {v!r}")
    return v


@dataclass
class ZanelornConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-5
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    side_dim: int = 0
    layers: List[ZanelornLayer] = field(default_factory=list)
    eos_token_id: Optional[int] = None
    max_positions: Optional[int] = None
    raw: Dict[str, Any] = field(default_factory=dict, repr=False)

    @staticmethod
    def _rotation(m: dict, dim: int, where: str) -> Rotation:
        rot = _obj(m, "rot", where)
        where += ".rot"
        dims = _int(rot, "dims", where, minimum=0)
        if dims % 2 or dims > dim:
            raise ConfigError(f"config.json: {where}.dims={dims} must be even and at most dim={dim}")
        scaling = _obj(rot, "scaling", where, optional=True)
        return Rotation(base=_positive(rot, "base", where), dims=dims,
                        factor=None if scaling is None else _positive(scaling, "factor", where + ".scaling"))

    @classmethod
    def _retention(cls, m: dict, where: str) -> RetentionSizes:
        heads, dim = _int(m, "heads", where), _int(m, "dim", where)
        decay = m.get("decay")
        if not isinstance(decay, list) or len(decay) != heads or any(isinstance(a, bool) or not isinstance(a, (int, float)) for a in decay):
            raise ConfigError(f"config.json: {where}.decay must be a list of {heads} numbers, one per head")
        return RetentionSizes(heads=heads, dim=dim, vdim=_int(m, "vdim", where), decay=[float(a) for a in decay],
                              rot=cls._rotation(m, dim, where))

    @classmethod
    def _attention(cls, m: dict, where: str) -> AttentionSizes:
        heads, kv, dim = _int(m, "heads", where), _int(m, "kv_heads", where), _int(m, "dim", where)
        if heads % kv:
            raise ConfigError(f"config.json: {where}: heads={heads} is not a multiple of kv_heads={kv}")
        mask = _obj(m, "mask", where, optional=True)
        out = AttentionSizes(heads=heads, kv_heads=kv, dim=dim, vdim=_int(m, "vdim", where), scale=_num(m, "scale", where),
                             rot=cls._rotation(m, dim, where))
        if mask is not None:
            out.window = _int(mask, "size", where + ".mask")
            if mask.get("keep_first") is not None:
                out.keep_first = _int(mask, "keep_first", where + ".mask", minimum=0)
        return out

    @classmethod
    def _parallel(cls, m: dict, where: str) -> ParallelSizes:
        left, right = _obj(m, "left", where), _obj(m, "right", where)
        wr = where + ".right"
        return ParallelSizes(left=cls._attention(left, where + ".left"),
                             right=MambaSizes(inner=_int(right, "inner", wr), state=_int(right, "state", wr),
                                              dt_rank=_int(right, "dt_rank", wr), conv=_int(right, "conv", wr)),
                             left_scale=_num(m, "left_scale", where), right_scale=_num(m, "right_scale", where))

    @staticmethod
    def _mlp(m: dict, where: str):
        if m.get("kind") not in FF_KINDS:
            raise ConfigError(f"config.json: {where}.kind must be one of {FF_KINDS}, got {m.get('kind')!r}")
        if m["kind"] == "dense":
            return DenseSizes(ff=_int(m, "ff", where))
        expert, router, shared = _obj(m, "expert", where), _obj(m, "router", where), _obj(m, "shared", where, optional=True)
        wr = where + ".router"
        out = ExpertsSizes(experts=_int(router, "experts", wr),
                           identity=_int(router, "identity", wr, minimum=0) if router.get("identity") is not None else 0,
                           top=_int(router, "top", wr), ff=_int(expert, "ff", where + ".expert"),
                           limit=_positive(expert, "limit", where + ".expert"))
        if out.top > out.experts + out.identity:
            raise ConfigError(f"config.json: {wr}.top={out.top} of {out.experts} + {out.identity} experts")
        if shared is not None:
            out.shared_ff = _int(shared, "ff", where + ".shared")
            out.shared_limit = _positive(shared, "limit", where + ".shared")
        return out

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ZanelornConfig":
        for key in ("vocab", "width", "norm", "embedding", "residual_mult", "token_side", "layers"):
            if d.get(key) is None:
                raise ConfigError(f"config.json: missing required key {key!r}")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        layers: List[ZanelornLayer] = []
        for i, e in enumerate(d["layers"]):
            where = f"layers[{i}]"
            if not isinstance(e, dict):
                raise ConfigError(f"config.json: {where} must be an object")
            if e.get("type") not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}.type must be one of {LAYER_TYPES}, got {e.get('type')!r}")
            m = _obj(e, "mixer", where)
            mixer = (cls._retention if e["type"] == "retention" else cls._parallel)(m, where + ".mixer")
            mlp = _obj(e, "mlp", where, optional=True)
            layers.append(ZanelornLayer(type=e["type"], mixer=mixer, mlp=None if mlp is None else cls._mlp(mlp, where + ".mlp")))
        vocab = _int(d, "vocab", "config")
        eos = d.get("eos_token_id")
        if eos is not None and (isinstance(eos, bool) or not isinstance(eos, int) or not (0 <= eos < vocab)):
            raise ConfigError(f"config.json: eos_token_id {eos!r} is not a token of the vocabulary")
        mp = d.get("max_positions")
        cfg = cls(vocab=vocab, width=_int(d, "width", "config"), norm_eps=_positive(_obj(d, "norm", "config"), "eps", "norm"),
                  embedding_scale=_num(_obj(d, "embedding", "config"), "scale", "embedding"),
                  residual_mult=_num(d, "residual_mult", "config"), side_dim=_int(_obj(d, "token_side", "config"), "dim", "token_side"),
                  layers=layers, eos_token_id=eos, max_positions=None if mp is None else _int(d, "max_positions", "config"),
                  raw=copy.deepcopy(d))
        cfg.architecture = "Zanelorn"
        return cfg

    def to_dict(self) -> Dict[str, Any]:
        d = copy.deepcopy(self.raw)
        d["architecture"] = "Zanelorn"
        return d
