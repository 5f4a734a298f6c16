"""Architecture-neutral description of a decoder: what the parts are built from.

A model configuration (config.json of some architecture) is translated once
into a :class:`ModelSpec`.  Everything below the configuration layer — parts,
cache manager, step function, weight loader — reads only these specs, so no
part knows which architecture it serves.

* :class:`PartSpec`: ``kind`` (a name in one of the part registries) plus the
  sizes and constants of that part.  Parameters are free-form so that a part
  registered from outside the package can carry its own.
* :class:`BlockSpec`: which parts one layer has, under which role names, how
  they are arranged (``kind``) and the tensor-name prefix of each.
* :class:`ScheduleEntry`: one run of a block.  The schedule is data: a block
  may appear twice, and an entry may read the cache of an earlier entry
  instead of owning one.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional, Sequence, Tuple


@dataclass(frozen=True)
class PartSpec:
    """``kind`` selects the implementation; ``params`` are its sizes and constants."""

    kind: str
    params: Mapping[str, Any] = field(default_factory=dict)

    def __getitem__(self, key: str) -> Any:
        return self.params[key]

    def get(self, key: str, default: Any = None) -> Any:
        return self.params.get(key, default)

    def replace(self, **changes: Any) -> "PartSpec":
        merged = dict(self.params)
        merged.update(changes)
        return PartSpec(self.kind, merged)


# The four parts of a pre-norm decoder layer and LitInfer's tensor-name stems for them
# (python/llaisys/models/qwen2.py:156-190).  Other arrangements name their own roles.
DEFAULT_PREFIXES = {
    "mixer": "self_attn.",
    "feed_forward": "mlp.",
    "mixer_norm": "input_layernorm.",
    "feed_forward_norm": "post_attention_layernorm.",
}


@dataclass(frozen=True)
class BlockSpec:
    """One layer: an arrangement (``kind``) of parts, each under a role name.

    ``parts`` maps a role (``mixer``, ``feed_forward``, ``mixer_norm``, ``feed_forward_norm``, or whatever else
    the arrangement knows: a norm after the mixer, a second mixer) to the part's spec; ``prefixes`` maps a role
    to the part's tensor-name prefix below the layer's own ``prefix`` (for instance ``model.layers.3.``), with
    ``<role>.`` as the default for roles outside :data:`DEFAULT_PREFIXES`.  An arrangement takes the roles it
    wants and may do without any of them (a layer without a feed-forward has no such entry).
    """

    kind: str
    prefix: str
    parts: Mapping[str, PartSpec] = field(default_factory=dict)
    prefixes: Mapping[str, str] = field(default_factory=dict)

    @classmethod
    def of(cls, kind: str, prefix: str, prefixes: Optional[Mapping[str, str]] = None, **parts: Optional[PartSpec]) -> "BlockSpec":
        """``BlockSpec.of("prenorm", "model.layers.0.", mixer=..., feed_forward=..., mixer_norm=..., feed_forward_norm=...)``."""
        return cls(kind, prefix, {r: p for r, p in parts.items() if p is not None}, dict(prefixes or {}))

    def part(self, role: str) -> Optional[PartSpec]:
        return self.parts.get(role)

    def prefix_of(self, role: str) -> str:
        """Full tensor-name prefix of the part under ``role``."""
        return self.prefix + self.prefixes.get(role, DEFAULT_PREFIXES.get(role, role + "."))

    def with_part(self, role: str, spec: Optional[PartSpec], prefix: Optional[str] = None) -> "BlockSpec":
        """A copy with the part under ``role`` replaced (``None`` removes it) and, if given, its prefix."""
        parts = dict(self.parts)
        if spec is None:
            parts.pop(role, None)
        else:
            parts[role] = spec
        prefixes = dict(self.prefixes)
        if prefix is not None:
            prefixes[role] = prefix
        return BlockSpec(self.kind, self.prefix, parts, prefixes)

    def with_kind(self, kind: str) -> "BlockSpec":
        return BlockSpec(kind, self.prefix, dict(self.parts), dict(self.prefixes))


@dataclass(frozen=True)
class ScheduleEntry:
    """Run block ``block``.  ``cache_from`` None: this entry owns a cache (or
    state); otherwise it reads what schedule entry ``cache_from`` wrote in
    this step and writes nothing.  ``add``: (name of a table in ``ModelSpec.stream_tables``, row): that row is added to the
    residual stream right before the block runs (a vector per pass of a span of layers that runs several times).  ``join``: the name
    of a map in ``ModelSpec.stream_maps``; before anything of ``add``, the stream x becomes ``M [x; x0]`` with x0 the embedding
    output (a span that reads the embedding anew at the start of every pass)."""

    block: int
    cache_from: Optional[int] = None
    add: Optional[Tuple[str, int]] = None
    join: Optional[str] = None


@dataclass(frozen=True)
class ModelSpec:
    architecture: str
    vocab_size: int
    hidden_size: int
    blocks: Tuple[BlockSpec, ...]
    schedule: Tuple[ScheduleEntry, ...]
    final_norm: PartSpec
    tie_word_embeddings: bool
    max_position_embeddings: int
    eos_token_ids: Tuple[int, ...] = ()
    embedding_name: str = "model.embed_tokens.weight"
    final_norm_prefix: str = "model.norm."
    lm_head_name: str = "lm_head.weight"
    # a position encoding of the whole model, applied to the residual stream right after the embedding (learned
    # absolute positions, say); None: positions are the mixers' business
    position: Optional[PartSpec] = None
    position_prefix: str = "model."
    # factor on the embedding rows and cap of the logits (cap * tanh(logits / cap)); None: neither
    embedding_scale: Optional[float] = None
    logit_cap: Optional[float] = None
    # the residual stream is kept as this many streams (hyper-connections): copies of the embedding at the start, their
    # sum at the end; every block then is of an arrangement that takes them (also for 1, where those arrangements still
    # weigh what they read and write).  None: the plain single stream
    streams: Optional[int] = None
    # tables of vectors that schedule entries add to the residual stream (``ScheduleEntry.add``): tensor name -> rows
    stream_tables: Mapping[str, int] = field(default_factory=dict)
    # maps [hidden, 2 hidden] that schedule entries put the residual stream beside the embedding output through
    # (``ScheduleEntry.join``; the embedding output is the stream as it enters the first block): tensor names
    stream_maps: Tuple[str, ...] = ()
    # parts that add something to the residual stream right after the embedding and may keep a state per request for it
    # (an embedding of token pairs): (spec, tensor-name prefix) each, kinds of the registry of stream inputs
    stream_inputs: Tuple[Tuple[PartSpec, str], ...] = ()
    # tables with a row per token of the vocabulary that layers read by token id (``parts.base.TokenInput``): tensor name -> columns
    token_tables: Mapping[str, int] = field(default_factory=dict)
    # other names under which a declared tensor may be stored: declared name -> names tried after it
    aliases: Mapping[str, Tuple[str, ...]] = field(default_factory=dict)

    def with_schedule(self, schedule: Sequence[ScheduleEntry]) -> "ModelSpec":
        from dataclasses import replace

        return replace(self, schedule=tuple(schedule))


def default_schedule(num_blocks: int) -> Tuple[ScheduleEntry, ...]:
    return tuple(ScheduleEntry(i) for i in range(num_blocks))


def validate_schedule(spec: ModelSpec) -> None:
    for i, e in enumerate(spec.schedule):
        if not 0 <= e.block < len(spec.blocks):
            raise ValueError(f"schedule entry {i} names block {e.block}, the model has {len(spec.blocks)}")
        if e.add is not None:
            name, row = e.add
            if name not in spec.stream_tables or not 0 <= int(row) < int(spec.stream_tables[name]):
                raise ValueError(f"schedule entry {i} adds row {row} of '{name}', which the model's stream tables do not have")
        if e.join is not None and (e.join not in spec.stream_maps or spec.streams is not None):
            raise ValueError(f"schedule entry {i} puts the stream through '{e.join}', which is not among the model's stream maps (of a single stream)")
        if e.cache_from is not None:
            if not 0 <= e.cache_from < i:
                raise ValueError(f"schedule entry {i} reads the cache of entry {e.cache_from}, which does not run before it")
            if spec.schedule[e.cache_from].cache_from is not None:
                raise ValueError(f"schedule entry {i} reads entry {e.cache_from}, which owns no cache itself")
