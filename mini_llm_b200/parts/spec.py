"""The description of a model as data.

An architecture's ``build_spec(config)`` returns a ``ModelSpec``: which part
(by registry key) stands where, with which constants and which checkpoint
tensors, layer by layer, and in which order the layers run.  Nothing in here
executes; ``parts.model.Model`` builds the parts from it.

The reference has no such level: GPT2Model hard-wires twelve identical blocks
(src/model/gpt2_model.cu:271-365, 402-406).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional, Sequence, Tuple


@dataclass
class WeightRef:
    """Where one parameter of a part comes from in the checkpoint.

    ``names``: accepted tensor names, the first is canonical (the one written by
    the random-weights mode).  ``transpose``: the checkpoint stores the matrix
    [in, out] (GPT-2's Conv1D, scripts/export_weights.py:48-52) while parts keep
    matrices [out, in].  ``init``: ("normal", std) | ("ones",) | ("zeros",) for
    the random-weights mode.  ``shared_with``: canonical name of a tensor that
    this parameter aliases (a tied head), so it is neither stored nor missed.
    """

    names: Sequence[str]
    transpose: bool = False
    init: Tuple = ("normal", 0.02)
    shared_with: Optional[str] = None

    @property
    def canonical(self) -> str:
        return self.names[0]


@dataclass
class PartSpec:
    """One part: registry key, constructor constants, checkpoint tensors."""

    kind: str
    params: Dict[str, Any] = field(default_factory=dict)
    weights: Dict[str, WeightRef] = field(default_factory=dict)


@dataclass
class LayerSpec:
    """One block: a mixer and a feed-forward, each behind its norm.

    ``arrangement`` names how they are wired (registry ``ARRANGEMENTS``), e.g.
    "pre_norm": x += mixer(norm(x)); x += ff(norm(x)); "parallel": both read the
    same x.  ``ff`` and ``ff_norm`` are None for a layer without a feed-forward.  ``mixer_join`` / ``ff_join`` (registry
    category "join") say how a branch's result reaches the residual when that is more than a sum: a norm and a learned
    scale per column on the result, say ("sandwich" arrangement); None: the branch adds itself.
    """

    mixer: PartSpec
    ff: Optional[PartSpec]
    mixer_norm: Optional[PartSpec]      # None (with ``ff_norm`` None): the arrangement norms after the sum, in its joins
    ff_norm: Optional[PartSpec]
    arrangement: str = "pre_norm"
    mixer_join: Optional[PartSpec] = None
    ff_join: Optional[PartSpec] = None
    side: Optional[PartSpec] = None          # category "token_side": a third branch that reads the token itself
    side_join: Optional[PartSpec] = None


@dataclass
class ScheduleEntry:
    """One run of a layer.  ``cache_of``: the layer whose cache (pages or state)
    this run uses; when it differs from ``layer`` the run only reads that cache
    and writes nothing to it.  ``private_cache``: the run has a cache and a state
    of its own (of the kind its layer's mixer needs) that no other run touches:
    a layer that runs several times with the same weights, each run with its own
    history.  ``enters_pass`` t: before this run the model's ``pass_input`` part makes the residual anew for pass t of a
    looped stretch.  ``cache_unit`` (set by ModelSpec) is the id under which the cache
    manager keeps the run's cache: the layer's index, or a number beyond the
    layers for a private one."""

    layer: int
    cache_of: Optional[int] = None
    private_cache: bool = False
    enters_pass: Optional[int] = None
    cache_unit: Optional[int] = None

    def __post_init__(self):
        if self.cache_of is None:
            self.cache_of = self.layer
        if self.private_cache and self.cache_of != self.layer:
            raise ValueError("a run with a private cache cannot also borrow another layer's")


@dataclass
class ModelSpec:
    hidden_size: int
    vocab_size: int
    embedding: PartSpec
    positions: PartSpec
    layers: List[LayerSpec]
    final_norm: PartSpec
    head: PartSpec
    schedule: Optional[List[ScheduleEntry]] = None
    token_table: Optional[PartSpec] = None   # category "token_table": what the layers' ``side`` branches read of a token
    pass_input: Optional[PartSpec] = None    # category "pass_input": runs before every entry that enters a pass
    max_positions: Optional[int] = None      # None: the position encoding sets no limit
    eos_token_id: Optional[int] = None
    ignored_tensors: List[str] = field(default_factory=list)   # regexes of checkpoint tensors to skip

    def __post_init__(self):
        if self.schedule is None:
            self.schedule = [ScheduleEntry(i) for i in range(len(self.layers))]
        n = len(self.layers)
        if self.pass_input is None and any(e.enters_pass is not None for e in self.schedule):
            raise ValueError("the schedule enters a pass but the model names no pass_input part")
        if self.token_table is None and any(l.side is not None for l in self.layers):
            raise ValueError("a layer has a side branch but the model names no token_table part")
        private = 0
        for e in self.schedule:
            if not (0 <= e.layer < n) or not (0 <= e.cache_of < n):
                raise ValueError(f"schedule entry {e} names a layer outside 0..{n - 1}")
            if e.private_cache:
                e.cache_unit = n + private
                private += 1
            else:
                e.cache_unit = e.cache_of

    def all_part_specs(self):
        """(label, PartSpec) of every part, in a fixed order."""
        yield "embedding", self.embedding
        yield "positions", self.positions
        if self.token_table is not None:
            yield "token_table", self.token_table
        if self.pass_input is not None:
            yield "pass_input", self.pass_input
        for i, l in enumerate(self.layers):
            if l.mixer_norm is not None:
                yield f"layers.{i}.mixer_norm", l.mixer_norm
            yield f"layers.{i}.mixer", l.mixer
            if l.mixer_join is not None:
                yield f"layers.{i}.mixer_join", l.mixer_join
            if l.ff is not None:
                if l.ff_norm is not None:
                    yield f"layers.{i}.ff_norm", l.ff_norm
                yield f"layers.{i}.ff", l.ff
                if l.ff_join is not None:
                    yield f"layers.{i}.ff_join", l.ff_join
            if l.side is not None:
                yield f"layers.{i}.side", l.side
                if l.side_join is not None:
                    yield f"layers.{i}.side_join", l.side_join
        yield "final_norm", self.final_norm
        yield "head", self.head
