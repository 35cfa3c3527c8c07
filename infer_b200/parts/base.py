"""Interfaces of the parts a layer is made of, and the registries that map a spec's ``kind`` to a class.

A part is built from its own ``PartSpec`` alone: it knows its sizes and constants, the local
names and shapes of its parameters, and what it needs from the cache manager.  It does not know
which architecture, which layer index or which model it is in.

To add a part: subclass the matching interface below, decorate it with
``@register_mixer("name")`` (or the feed-forward / norm / position / block / embedding / head
variant), and let an architecture's ``to_spec`` name that kind.  No framework file changes.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, Mapping, Optional, Tuple

import torch

from ..config.specs import PartSpec


# ----------------------------------------------------------------------------- cache needs

@dataclass(frozen=True)
class PagedKVNeed:
    """Keys and values of every position (or of the last ``window`` positions) in pages."""
    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None     # None: all positions stay; n: only the last n are ever read
    v_head_dim: Optional[int] = None  # size of a value where it differs from a key's (None: head_dim)
    values_in_keys: bool = False      # True: a position's value is the first v_head_dim channels of its key row (one
                                      # row per position serves both, as in attention through a shared latent); there
                                      # are no value pages and the view's ``v`` is None
    keep_first: int = 0               # with a window: the positions below this stay readable for every later query
    chunk: Optional[int] = None       # n: a query reads keys of its own chunk of n positions only (counted from position 0)

    @property
    def value_dim(self) -> int:
        return int(self.v_head_dim or self.head_dim)

    @property
    def stored_value_dim(self) -> int:
        """Channels per position and kv head that the value pages hold."""
        return 0 if self.values_in_keys else self.value_dim


@dataclass(frozen=True)
class StateNeed:
    """A fixed-size state per request, zeroed when the request is admitted.

    shapes maps a state tensor's name to (shape without the slot dimension, torch dtype); a dtype of None stands
    for the model's compute dtype (copies of activations, as opposed to sums that must stay float32)."""
    shapes: Mapping[str, Tuple[Tuple[int, ...], Optional[torch.dtype]]]


@dataclass(frozen=True)
class CompositeNeed:
    """Several needs of one cache entry, by name: a mixer that keeps pages AND a fixed-size state (attention whose
    projections pass a filter over time), or mixers that run side by side on one input. The cache manager gives such
    an entry a dict ``name -> view`` of the same shape (nested where a need is itself composite)."""
    parts: Mapping[str, Any]         # name -> PagedKVNeed | StateNeed | CompositeNeed | None


# ----------------------------------------------------------------------------- interfaces

class Part:
    """Common surface of every part."""

    def __init__(self, spec: PartSpec, runtime: "Runtime"):
        self.spec = spec
        self.rt = runtime

    @classmethod
    def param_shapes(cls, spec: PartSpec) -> Dict[str, Tuple[int, ...]]:
        """Local parameter name -> shape, as the checkpoint stores them under ``spec.prefix``."""
        return {}

    @classmethod
    def init_params(cls, spec: PartSpec, name: str, shape: Tuple[int, ...], gen: torch.Generator) -> torch.Tensor:
        """Random value for one parameter (float32, on the generator's device): matrices and
        biases N(0, 0.02).  Parts whose parameters want another distribution override this."""
        return torch.randn(shape, generator=gen, dtype=torch.float32, device=gen.device) * 0.02

    # False: the part's forward() cannot be captured into a CUDA graph (it reads device memory on the host, allocates
    # outside the stream's pool, or launches by data). The engine then runs every step of the model eagerly.
    graph_safe = True

    def load(self, params: Mapping[str, torch.Tensor]) -> None:
        """Receives the part's parameters (CPU tensors in their stored dtype) and moves what it
        needs to the device, in the layout its kernels want."""


class DeferredNorm:
    """The float32 rows ``h`` with a norm that has not been applied yet. A part that declares
    ``accepts_deferred_norm`` may receive this instead of the normalised tensor and hand it to a kernel that
    normalises on the fly; ``materialize()`` applies the norm the ordinary way."""

    def __init__(self, norm: "Norm", h: torch.Tensor):
        self.norm, self.h = norm, h
        self._value = None

    @property
    def shape(self):
        return self.h.shape

    def materialize(self) -> torch.Tensor:
        if self._value is None:
            self._value = self.norm.forward(self.h)
        return self._value


class ProjectedInput:
    """What a block hands its parts in place of the normalised rows when it has joined their first matrix products
    (every one of them reads the same rows) into fewer, larger ones: the results' rows, and for each part that took
    part, where its own columns start. ``of(part)`` gives that part's (rows, first column) or None; ``rows_in`` are
    the normalised rows themselves (possibly a DeferredNorm) for parts that did not take part.

    A part takes part by offering ``input_product() -> (Linear, "compute" | "float32")``, its first product and the
    dtype of the result it wants, and by starting ``forward`` from ``x.of(self)`` when x is a ProjectedInput. The block
    calls ``drop_input_product()`` on it after joining, so that the matrix lives once."""

    def __init__(self, rows_in):
        self.rows_in = rows_in
        self._where = {}

    def place(self, part, rows, col0: int) -> None:
        self._where[id(part)] = (rows, col0)

    def of(self, part):
        return self._where.get(id(part))


def own_or_projected(part, x, linear, out_dtype=None):
    """(rows, first column) of a part's first product: its slice of a joined product, or its own ``linear`` on x."""
    if isinstance(x, ProjectedInput):
        got = x.of(part)
        if got is not None:
            return got
        x = x.rows_in
    return linear(x, out_dtype=out_dtype), 0


class Norm(Part):
    def forward(self, x: torch.Tensor, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
        """x [rows, size] float32 (the residual stream) -> normalised rows in the compute dtype."""
        raise NotImplementedError


class PositionEncoding(Part):
    def apply(self, q: torch.Tensor, k: torch.Tensor, positions: torch.Tensor) -> None:
        """Encodes positions into q [T, heads, head_dim] and k [T, kv_heads, head_dim] in place.
        positions: int32 [T], absolute."""
        raise NotImplementedError

    def rotary_tables(self):
        """(cos, sin) float32 [max_positions, head_dim/2] if this encoding is a half-split rotation
        that a mixer's fused kernel may apply itself; None otherwise."""
        return None


class Mixer(Part):
    accepts_deferred_norm = False    # True: forward() may get a DeferredNorm as x
    # True: a block whose sublayers read the residual stream itself hands forward() the float32 rows of the stream as x,
    # whatever the compute dtype (a mixer that combines rows in float32 before its first matrix product)
    reads_stream = False

    def cache_need(self):
        """PagedKVNeed, StateNeed, CompositeNeed or None."""
        return None

    def forward(self, x: torch.Tensor, step: "StepContext", cache: Any, residual: torch.Tensor,
                write_cache: bool = True) -> torch.Tensor:
        """x: normalised rows [T, hidden] in the compute dtype; residual: float32 [T, hidden].
        Returns residual + mixer(x) as float32 [T, hidden] (it may overwrite ``residual``); with ``residual`` None,
        mixer(x) alone as float32 (for blocks that weigh or gate a sublayer's result before they add it).
        ``cache`` is what the cache manager made for this part's need: a ``PagedKVView``,
        a dict of state tensors [slots, ...], or None."""
        raise NotImplementedError


class FeedForward(Part):
    accepts_deferred_norm = False

    def forward(self, x: torch.Tensor, residual: torch.Tensor) -> torch.Tensor:
        """Returns residual + feed_forward(x), float32 [T, hidden] (may overwrite ``residual``); with ``residual``
        None, feed_forward(x) alone as float32."""
        raise NotImplementedError


class Gate(Part):
    """Multipliers for sublayer results, computed from the rows the sublayers read."""

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        """x: normalised rows [T, hidden] in the compute dtype -> float32 gate logits [T, n * hidden], n the number
        of sublayers this part gates; the block's sum applies the squashing function."""
        raise NotImplementedError


class Connection(Part):
    """How one sublayer reads from and writes to a residual stream that is more than one row per token."""


class Stream(Part):
    """The residual stream of a model whose blocks pass on something else than float32 rows [T, hidden]: how it starts
    from the embedding's rows and how it ends in front of the head. A model without one passes the rows themselves."""

    def open(self, rows: torch.Tensor):
        """float32 [T, hidden] from the embedding -> what the first block's forward() gets as h."""
        raise NotImplementedError

    def close(self, h, norm: "Norm", rows: torch.Tensor) -> torch.Tensor:
        """What the last block returned -> the final norm of the wanted rows (int32 ``rows``), in the compute dtype."""
        raise NotImplementedError


class Embedding(Part):
    """Token ids -> float32 rows of the residual stream."""

    def forward(self, step: "StepContext") -> torch.Tensor:
        """float32 [T, hidden] for ``step.token_ids`` (an id of -1 stands for the request's last sampled token, kept
        on the device in ``step.feedback[step.seg_slot[step.token_seg[t]]]``)."""
        raise NotImplementedError

    def table(self) -> Optional[torch.Tensor]:
        """The [vocab, hidden] matrix on the device, for a head that is tied to it; None if there is none."""
        return None


class Head(Part):
    """Normalised rows -> float32 logits [rows, vocab]."""

    def tie(self, embedding: Embedding) -> None:
        """Called once after loading, with the model's embedding part; a tied head takes its matrix from there."""

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


class Block:
    """An arrangement of parts into a layer. ``parts`` maps the slot names of the layer's spec to the built and
    loaded parts, in the spec's order; each is also an attribute of the block under its slot name. A block class
    defines which slots it wants and how ``forward`` runs them."""

    def __init__(self, **parts: Part):
        self.parts: Dict[str, Part] = dict(parts)
        for slot, part in parts.items():
            setattr(self, slot, part)

    def cache_need(self):
        """What the layer needs from the cache manager per run-order entry: the need of its one part that has one."""
        needs = [n for n in (p.cache_need() for p in self.parts.values() if hasattr(p, "cache_need")) if n is not None]
        if len(needs) > 1:
            raise ValueError("a block with more than one stateful part must define cache_need() itself")
        return needs[0] if needs else None

    def forward(self, h: torch.Tensor, step: "StepContext", cache: Any, write_cache: bool) -> torch.Tensor:
        raise NotImplementedError


# ----------------------------------------------------------------------------- registries

_REGISTRIES: Dict[str, Dict[str, type]] = {"mixer": {}, "feed_forward": {}, "norm": {}, "position": {}, "block": {},
                                           "embedding": {}, "head": {}, "gate": {}, "connection": {}, "stream": {}}


def _register(family: str, name: str) -> Callable[[type], type]:
    def deco(cls: type) -> type:
        if name in _REGISTRIES[family] and _REGISTRIES[family][name] is not cls:
            raise ValueError(f"{family} kind {name!r} is already registered")
        _REGISTRIES[family][name] = cls
        return cls
    return deco


def register_mixer(name: str): return _register("mixer", name)
def register_feed_forward(name: str): return _register("feed_forward", name)
def register_norm(name: str): return _register("norm", name)
def register_position(name: str): return _register("position", name)
def register_block(name: str): return _register("block", name)
def register_embedding(name: str): return _register("embedding", name)
def register_head(name: str): return _register("head", name)
def register_gate(name: str): return _register("gate", name)
def register_connection(name: str): return _register("connection", name)
def register_stream(name: str): return _register("stream", name)


def unregister(family: str, name: str) -> None:
    _REGISTRIES[family].pop(name, None)


def part_class(family: str, kind: str) -> type:
    try:
        return _REGISTRIES[family][kind]
    except KeyError:
        known = ", ".join(sorted(_REGISTRIES[family])) or "(none)"
        raise KeyError(f"no {family} part of kind {kind!r} is registered; known: {known}") from None


def build_part(family: str, spec: PartSpec, runtime: "Runtime") -> Part:
    return part_class(family, spec.kind)(spec, runtime)
