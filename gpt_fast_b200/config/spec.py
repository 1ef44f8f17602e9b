"""Data that describes a model to build: which parts, with which sizes and
constants, in which order.

Nothing here knows an architecture.  An architecture (see `registry.py`)
turns its typed configuration into a `ModelSpec`; `engine.model.Transformer`
builds itself from the spec alone.  Every size a part needs is in its
`PartSpec.params`; the order in which layers run is the `schedule` list.
"""
from dataclasses import dataclass, field
from typing import Any, Dict, List, Optional


@dataclass(frozen=True)
class PartSpec:
    """One part: `kind` is a key of the matching registry in `parts`, `params`
    are the constructor's keyword arguments (sizes and constants only)."""
    kind: str
    params: Dict[str, Any] = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """One set of layer parameters.  `block` names the arrangement of the
    parts (for instance pre-norm residual); `parts` gives one `PartSpec` per
    role the arrangement declares (`parts.BLOCKS[block].roles`: for 'prenorm'
    mixer, feed_forward, mixer_norm, ffn_norm), so an arrangement with other
    roles (one shared norm, post-norms, no feed-forward) needs no change here.
    Each layer picks its own parts, so layers of one model may differ."""
    block: str
    parts: Dict[str, PartSpec]
    position: Optional[PartSpec] = None   # position encoding the layer's mixers apply
    block_params: Dict[str, Any] = field(default_factory=dict)   # constants of the arrangement itself (a factor on its branches, ...)


@dataclass(frozen=True)
class ScheduleEntry:
    """One run of a layer.  `layer` indexes `ModelSpec.layers` (a layer may be
    named by several entries: its weights are then shared).  `cache` is the id
    of the cache entry the run's mixer uses; with `owns_cache=False` the run
    appends nothing and reads what the entry's owner wrote earlier in the
    same step.  `kv_from` (or None) is the id of another entry whose keys and values the run's mixer reads in place
    of keys and values of its own, while per-sequence state (if the mixer keeps any) stays in its own entry `cache`."""
    layer: int
    cache: int
    owns_cache: bool = True
    kv_from: Optional[int] = None
    junction: Optional[int] = None        # index into `ModelSpec.junctions`: what happens to the stream right before this run
    turn: int = 0                         # which time that junction is passed (a loop's pass), counted from 0


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    dim: int
    vocab_size: int
    layers: List[LayerSpec]
    schedule: List[ScheduleEntry]
    final_norm: PartSpec
    tie_embeddings: bool = False
    max_position: int = 0                 # longest sequence the model allows
    stop_tokens: tuple = ()               # default stop tokens of generation
    bos_token: Optional[int] = None
    embed_scale: Optional[float] = None   # factor on the embedding rows (None: 1)
    logit_cap: Optional[float] = None     # soft cap on the logits, cap * tanh(logits / cap) (None: none)
    embedding: Optional[PartSpec] = None  # what is added to the token embedding (a part of `parts.EMBEDDINGS`; None: nothing)
    junctions: List[PartSpec] = field(default_factory=list)   # parts of `parts.JUNCTIONS` that schedule entries name
    token_table: int = 0                  # columns of the per-token side table that layers' token inputs read (0: none)
    streams: int = 0                      # residual streams per token (0: the one ordinary stream); every block then takes streams
    launch_overlap: bool = True           # kernels of a step may start while their predecessor drains; False: strictly in turn

    def validate(self) -> None:
        if self.logit_cap is not None and not self.logit_cap > 0:
            raise ValueError(f"ModelSpec.logit_cap = {self.logit_cap}: a soft cap must be positive")
        if self.embed_scale is not None and self.embed_scale != self.embed_scale:
            raise ValueError("ModelSpec.embed_scale is not a number")
        if self.streams < 0 or (self.streams and self.junctions):
            raise ValueError(f"ModelSpec.streams = {self.streams}: not negative, and without junctions")
        owners = {}
        for i, e in enumerate(self.schedule):
            if not 0 <= e.layer < len(self.layers):
                raise ValueError(f"schedule[{i}] names layer {e.layer}, the model has {len(self.layers)}")
            if e.junction is not None and not 0 <= e.junction < len(self.junctions):
                raise ValueError(f"schedule[{i}] names junction {e.junction}, the model has {len(self.junctions)}")
            if e.owns_cache:
                if e.cache in owners:
                    raise ValueError(f"cache entry {e.cache} has two owners: schedule[{owners[e.cache]}] and [{i}]")
                owners[e.cache] = i
            elif e.cache not in owners:
                raise ValueError(f"schedule[{i}] reads cache entry {e.cache} before any run wrote it")
            if e.kv_from is not None and (e.kv_from not in owners or owners[e.kv_from] >= i):
                raise ValueError(f"schedule[{i}] reads the keys and values of entry {e.kv_from} before any run wrote them")
