"""ZadenexConfig: the keys of a Zadenex config.json, typed and checked.

A Zadenex model is a list of layers.  Every entry names its mixer ("attention", "latent_attention" or "mlstm") with that
mixer's sizes and constants, and its feed-forward (dense) or none.  Nothing is assumed equal between layers: every size is
read per entry.  ``loop`` names a stretch of layers that runs several times in a row with the same weights.
"""
from __future__ import annotations

import copy
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Tuple

from .base import ConfigError, ModelConfig
from .finuvik import _int, _num

LAYER_TYPES = ("attention", "latent_attention", "mlstm")
FF_KINDS = ("dense",)


@dataclass
class AttentionSizes:
    heads: int
    kv_heads: int
    dim: int                  # a query's and a key's entries per head
    vdim: int
    scale: float              # factor on the scores, before they are mixed over the heads
    window: Optional[int] = None      # keys a query sees, itself included; None: all


@dataclass
class LatentSizes:
    heads: int
    dim: int                  # unrotated query/key entries per head
    rot_dim: int              # rotated ones (the key's are shared by all heads)
    vdim: int
    q_rank: int               # size of the queries' latent
    kv_rank: int              # size of the cached latent
    scale: float
    rot_dims: int
    rot_base: float


@dataclass
class MatrixMemorySizes:
    heads: int
    dim: int                  # rows of a head's state
    vdim: int                 # columns of it
    gate_cap: float           # cap on both gates' logarithms


@dataclass
class DenseSizes:
    ff: int


@dataclass
class Loop:
    start: int
    stop: int                 # one past the last layer of the stretch
    times: int


@dataclass
class ZadenexLayer:
    type: str
    mixer: Any
    mlp: Optional[DenseSizes] = None


@dataclass
class ZadenexConfig(ModelConfig):
    vocab: int = 0
    width: int = 0
    norm_eps: float = 1e-5
    embedding_scale: float = 1.0
    residual_mult: float = 1.0
    layers: List[ZadenexLayer] = field(default_factory=list)
    loop: Optional[Loop] = None
    eos_token_id: Optional[int] = None
    max_positions: Optional[int] = None
    raw: Dict[str, Any] = field(default_factory=dict, repr=False)

    @staticmethod
    def _attention(m: dict, where: str) -> AttentionSizes:
        heads, kv = _int(m, "heads", where), _int(m, "kv_heads", where)
        if heads % kv:
            raise ConfigError(f"config.json: {where}: heads={heads} is not a multiple of kv_heads={kv}")
        mask = m.get("mask")
        if mask is not None and not isinstance(mask, dict):
            raise ConfigError(f"config.json: {where}.mask must be an object with 'size', or null")
        return AttentionSizes(heads=heads, kv_heads=kv, dim=_int(m, "dim", where), vdim=_int(m, "vdim", where),
                              scale=_num(m, "scale", where),
                              window=_int(mask, "size", where + ".mask") if mask is not None else None)

    @staticmethod
    def _latent(m: dict, where: str) -> LatentSizes:
        rot = m.get("rot")
        if not isinstance(rot, dict):
            raise ConfigError(f"config.json: {where}.rot must be an object with 'base' and 'dims'")
        rot_dim = _int(m, "rot_dim", where, minimum=0)
        dims = _int(rot, "dims", where + ".rot", minimum=0)
        if dims % 2 or dims > rot_dim:
            raise ConfigError(f"config.json: {where}.rot.dims={dims} must be even and at most rot_dim={rot_dim}")
        base = _num(rot, "base", where + ".rot")
        if not base > 0:
            raise ConfigError(f"config.json: {where}.rot.base must be positive")
        return LatentSizes(heads=_int(m, "heads", where), dim=_int(m, "dim", where), rot_dim=rot_dim, vdim=_int(m, "vdim", where),
                           q_rank=_int(m, "q_rank", where), kv_rank=_int(m, "kv_rank", where), scale=_num(m, "scale", where),
                           rot_dims=dims, rot_base=base)

    @staticmethod
    def _memory(m: dict, where: str) -> MatrixMemorySizes:
        cap = _num(m, "gate_cap", where)
        if not cap > 0:
            raise ConfigError(f"config.json: {where}.gate_cap must be positive, got {cap!r}")
        return MatrixMemorySizes(heads=_int(m, "heads", where), dim=_int(m, "dim", where), vdim=_int(m, "vdim", where), gate_cap=cap)

    @classmethod
    def from_dict(cls, d: Dict[str, Any]) -> "ZadenexConfig":
        for key in ("vocab", "width", "norm", "embedding", "residual_mult", "layers"):
            if d.get(key) is None:
                raise ConfigError(f"config.json: missing required key {key!r}")
        if not isinstance(d["norm"], dict):
            raise ConfigError("config.json: 'norm' must be an object with 'eps'")
        eps = _num(d["norm"], "eps", "norm")
        if not eps > 0:
            raise ConfigError(f"config.json: norm.eps must be positive, got {eps!r}")
        if not isinstance(d["embedding"], dict):
            raise ConfigError("config.json: 'embedding' must be an object with 'scale'")
        if not isinstance(d["layers"], list) or not d["layers"]:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        read = {"attention": cls._attention, "latent_attention": cls._latent, "mlstm": cls._memory}
        layers: List[ZadenexLayer] = []
        for i, e in enumerate(d["layers"]):
            where = f"layers[{i}]"
            if not isinstance(e, dict):
                raise ConfigError(f"config.json: {where} must be an object")
            if e.get("type") not in LAYER_TYPES:
                raise ConfigError(f"config.json: {where}.type must be one of {LAYER_TYPES}, got {e.get('type')!r}")
            m = e.get("mixer")
            if not isinstance(m, dict):
                raise ConfigError(f"config.json: {where}.mixer must be an object")
            mixer = read[e["type"]](m, where + ".mixer")
            mlp = e.get("mlp")
            if mlp is not None:
                if not isinstance(mlp, dict):
                    raise ConfigError(f"config.json: {where}.mlp must be an object or null")
                if mlp.get("kind") not in FF_KINDS:
                    raise ConfigError(f"config.json: {where}.mlp.kind must be one of {FF_KINDS}, got {mlp.get('kind')!r}")
                mlp = DenseSizes(ff=_int(mlp, "ff", where + ".mlp"))
            layers.append(ZadenexLayer(type=e["type"], mixer=mixer, mlp=mlp))
        loop = d.get("loop")
        if loop is not None:
            if not isinstance(loop, dict):
                raise ConfigError("config.json: 'loop' must be an object with 'start', 'stop' and 'times', or null")
            loop = Loop(start=_int(loop, "start", "loop", minimum=0), stop=_int(loop, "stop", "loop", minimum=0),
                        times=_int(loop, "times", "loop"))
            if not (loop.start < loop.stop <= len(layers)):
                raise ConfigError(f"config.json: loop {loop.start}..{loop.stop} is no stretch of the {len(layers)} layers")
        vocab = _int(d, "vocab", "config")
        eos = d.get("eos_token_id")
        if eos is not None and (isinstance(eos, bool) or not isinstance(eos, int) or not (0 <= eos < vocab)):
            raise ConfigError(f"config.json: eos_token_id {eos!r} is not a token of the vocabulary")
        mp = d.get("max_positions")
        if mp is not None:
            mp = _int(d, "max_positions", "config")
        cfg = cls(vocab=vocab, width=_int(d, "width", "config"), norm_eps=eps,
                  embedding_scale=_num(d["embedding"], "scale", "embedding"), residual_mult=_num(d, "residual_mult", "config"),
                  layers=layers, loop=loop, eos_token_id=eos, max_positions=mp, raw=copy.deepcopy(d))
        cfg.architecture = "Zadenex"
        return cfg

    def layer_runs(self) -> List[Tuple[int, Optional[int]]]:
        """(layer, number of the pass that begins with this run, or None) in the order the layers run."""
        n = len(self.layers)
        if self.loop is None:
            return [(i, None) for i in range(n)]
        lp = self.loop
        runs: List[Tuple[int, Optional[int]]] = [(i, None) for i in range(lp.start)]
        for t in range(lp.times):
            runs += [(i, t if i == lp.start else None) for i in range(lp.start, lp.stop)]
        return runs + [(i, None) for i in range(lp.stop, n)]

    def to_dict(self) -> Dict[str, Any]:
        d = copy.deepcopy(self.raw)
        d["architecture"] = "Zadenex"
        return d
