"""The description of a model as data: which parts make each layer, in which
order the layers run and whose cache each run reads.

An architecture turns its typed configuration into a :class:`ModelPlan`; the
engine builds the parts from it without knowing the architecture.  The
reference writes one file per architecture and repeats norm, rotary, attention
and experts in each (src/minimax.rs:31-126 beside src/rope.rs:26-108); here they
are parts chosen layer by layer.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Mapping, Optional


@dataclass(frozen=True)
class PartSpec:
    """One part of a layer: a registered kind, its constants, and the checkpoint
    names of its tensors (local name -> name in the safetensors file; a name
    may hold ``{e}`` where the part enumerates experts)."""

    kind: str
    args: Mapping[str, Any] = field(default_factory=dict)
    tensors: Mapping[str, str] = field(default_factory=dict)


@dataclass(frozen=True)
class LayerSpec:
    """A layer: a block arrangement over a mixer and a feed-forward, each with its norm (where the norm
    sits, before the sublayer or on its output, is the block's business).  A layer without a feed-forward
    has ``feed_forward`` and ``feed_forward_norm`` None.  ``addition`` names a part that adds to the stream once more
    after the block (category ``addition``: a further input per layer that reads the stream and the step's tokens)."""

    block: str
    mixer: PartSpec
    feed_forward: Optional[PartSpec]
    mixer_norm: PartSpec
    feed_forward_norm: Optional[PartSpec]
    addition: Optional[PartSpec] = None
    # norms behind the sublayers, for a block that has a norm on both sides of each (``sandwich_norm``)
    mixer_out_norm: Optional[PartSpec] = None
    feed_forward_out_norm: Optional[PartSpec] = None
    # a part between the mixer's norm and the mixer (category ``mixer_input``), which may keep a state of its own
    mixer_input: Optional[PartSpec] = None
    # how the sublayers read and write a stream that is kept as several copies (category ``stream_connection``)
    connections: Optional[PartSpec] = None


@dataclass(frozen=True)
class RunSpec:
    """One entry of the run order.  ``layer`` indexes :attr:`ModelPlan.layers`
    (the same layer may run twice).  ``cache_line`` names the line of the cache
    this run reads; ``writes_cache`` is false for a run that reads a line which
    an earlier run wrote.  ``connector`` names a part that rewrites the whole stream before the run (a model
    that runs a stretch of layers several times mixes the embedding back in at the start of every pass)."""

    layer: int
    cache_line: int
    writes_cache: bool = True
    # (index into ModelPlan.connectors, number of the pass): the stream goes through that connector before this run
    connector: Optional[tuple[int, int]] = None


@dataclass(frozen=True)
class ModelPlan:
    architecture: str
    hidden_size: int
    vocab_size: int
    embedding: PartSpec
    layers: tuple[LayerSpec, ...]
    run_order: tuple[RunSpec, ...]
    final_norm: PartSpec
    head: PartSpec
    eos_token_id: tuple[int, ...] = ()
    connectors: tuple[PartSpec, ...] = ()
    # copies of the residual stream that the layers' connections work on, all equal to the embedding's rows at the start
    # and added up in front of the final norm; 0: one plain stream
    streams: int = 0

    def check(self) -> None:
        if self.streams < 0 or any((layer.connections is not None) != (self.streams > 0) for layer in self.layers):
            raise ValueError(f"a plan with {self.streams} copies of the stream: every layer has connections to them, or, with 0, none")
        if self.streams and (self.connectors or any(layer.addition is not None for layer in self.layers)):
            raise ValueError("connectors and additions work on a single stream, not on copies of it")
        written: set[int] = set()
        for step, run in enumerate(self.run_order):
            if run.connector is not None and not 0 <= run.connector[0] < len(self.connectors):
                raise ValueError(f"run order entry {step} names connector {run.connector[0]}, the plan has "
                                 f"{len(self.connectors)}")
            if not 0 <= run.layer < len(self.layers):
                raise ValueError(f"run order entry {step} names layer {run.layer}, the plan has {len(self.layers)}")
            if run.writes_cache:
                if run.cache_line in written:
                    raise ValueError(f"run order entry {step} writes cache line {run.cache_line} a second time")
                written.add(run.cache_line)
            elif run.cache_line not in written:
                raise ValueError(
                    f"run order entry {step} reads cache line {run.cache_line} before any entry wrote it")


def default_run_order(num_layers: int) -> tuple[RunSpec, ...]:
    """Each layer once, in order, each with a cache line of its own."""
    return tuple(RunSpec(layer=i, cache_line=i) for i in range(num_layers))
