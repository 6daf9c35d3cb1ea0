"""Interfaces of the parts a decoder is put together from, and their registry.

A part is built from the parameters of its :class:`PartSpec` alone; it learns its
sizes and constants there and never which model it is in.  It declares the tensors
it needs by names relative to itself; the model prefixes them and the loader fills
them by name.

Kinds of part and what each must provide:

``Norm``            ``forward(h, delta, rows=None, bias=None)``: adds ``delta`` (may be None;
                    a tensor, split-K partial sums, or either with a multiplier as
                    ``ops.Scaled``, or normed first as ``ops.PostNormed``) and the vector ``bias`` into the 32-bit residual ``h``
                    in place and returns the normed rows in the activation dtype; with
                    ``rows`` it returns the norm of the picked rows of ``h + delta`` and
                    leaves ``h`` alone.
``PositionEncoding````tables()``: what the mixer's kernels need to place a token.
``Mixer``           ``cache_need()``: a :class:`KVCacheNeed`, a :class:`StateNeed`
                    or None, or several by name; ``forward(x, step, cache)`` mixes tokens of the same
                    request, reading and writing only its own cache; what it hands to later layers
                    of the same step (per token) goes into ``step.carried``.
``FeedForward``     ``forward(x)``: works on each token alone.
``Block``           ``mixer`` attribute and ``forward(h, pending, step, cache, bias=None)``:
                    arranges norms, mixer, feed-forward and residual sums; returns
                    the update not yet added into ``h``.  ``bias`` is a vector the model
                    adds to the residual stream right before this run of the layer.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable, Optional

import torch

from ..config.spec import PartSpec


# ------------------------------------------------------------------ declarations
@dataclass(frozen=True)
class TensorSpec:
    """A tensor a part needs.  ``init`` says how the random-weights mode fills it:
    ``matrix`` normal(0, 0.02), ``norm`` 1 + U(-0.1, 0.1), ``around_zero`` U(-0.1, 0.1), ``unit`` U(0, 1), ``zeros``; ``integer``
    tensors are kept as int32, others in the run's dtype (bfloat16 or float32)
    unless the file stores them in 32-bit, in which case they stay so.

    A dimension of -1 is free: the file gives it (the rank of a low-rank pair of matrices that no
    configuration key names); the part reads it from the tensor it is bound to.  ``free`` is the size the
    random-weights mode gives such a dimension."""

    shape: tuple[int, ...]
    init: str = "matrix"
    optional: bool = False
    integer: bool = False
    free: int = 16

    def fits(self, shape) -> bool:
        shape = tuple(shape)
        return len(shape) == len(self.shape) and all(a == -1 and b > 0 or a == b for a, b in zip(self.shape, shape))

    def concrete(self) -> tuple[int, ...]:
        return tuple(self.free if a == -1 else a for a in self.shape)


@dataclass(frozen=True)
class KVCacheNeed:
    """Keys and values per token in pages.  ``window`` None: every earlier key stays
    visible; an integer w: a query at position i reads keys i-w+1 .. i, and pages
    wholly behind that may be given back.  ``values`` False: the pages hold keys only (a mixer
    whose values are part of its key rows, such as a latent shared by keys and values).
    ``value_dim``: the size of a value when it differs from a key's (None: ``head_dim``).  ``keep_first``:
    with a window, the request's first tokens that stay visible to every later query, so that the pages
    which hold them are never given back.  ``tokens_per_entry`` P: the pages hold ONE key and value per P tokens (means over
    blocks of tokens): entry e belongs to positions e P .. e P + P - 1, has its place from the step that brings the last
    of them, and is never given back before the request ends (no window).  Runs that share a cache may want different windows; the cache
    then keeps what the most demanding of them reads (:meth:`merged`)."""

    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    values: bool = True
    value_dim: Optional[int] = None
    keep_first: int = 0
    tokens_per_entry: int = 1

    def same_pages(self, other: "KVCacheNeed") -> bool:
        """Whether both describe pages of the same layout (whatever they keep of them)."""
        return (self.num_kv_heads, self.head_dim, self.values, self.value_dim or self.head_dim, self.tokens_per_entry) == \
            (other.num_kv_heads, other.head_dim, other.values, other.value_dim or other.head_dim, other.tokens_per_entry)

    def merged(self, other: "KVCacheNeed") -> "KVCacheNeed":
        """The need of a cache that serves both: the wider window (none if either has none), the longer kept start."""
        window = None if self.window is None or other.window is None else max(self.window, other.window)
        keep = 0 if window is None else max(self.keep_first, other.keep_first)
        return KVCacheNeed(self.num_kv_heads, self.head_dim, window, self.values, self.value_dim, keep, self.tokens_per_entry)


@dataclass(frozen=True)
class StateNeed:
    """A fixed-size state per request (zero when the request starts)."""

    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass
class BuildContext:
    """What a part may use while it is built."""

    device: torch.device
    dtype: torch.dtype                      # activations and matrices: float32 or bfloat16
    max_positions: int                      # the engine's limit on a request's length
    shared: dict = field(default_factory=dict)   # tables shared by equal parts (rotary tables)


class Part:
    def __init__(self, params: dict[str, Any], ctx: BuildContext):
        self.params = params
        self.ctx = ctx

    def tensor_specs(self) -> dict[str, TensorSpec]:
        return {}

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        """Receives the device tensors named in :meth:`tensor_specs`."""


class Norm(Part):
    def forward(self, h: torch.Tensor, delta, rows: Optional[torch.Tensor] = None,
                bias: Optional[torch.Tensor] = None) -> torch.Tensor:
        raise NotImplementedError


class PositionEncoding(Part):
    pass


class Mixer(Part):
    # True if forward() only launches kernels that read the step's device arrays (no
    # host-side loop over requests, no synchronisation): decode steps of a model whose
    # mixers all say so are replayed from CUDA graphs.
    graph_safe = False

    def cache_need(self):
        return None

    def forward(self, x: torch.Tensor, step, cache) -> torch.Tensor:
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


class Block(Part):
    mixer: Mixer

    def forward(self, h: torch.Tensor, pending, step, cache, bias: Optional[torch.Tensor] = None):
        raise NotImplementedError


# ---------------------------------------------------------------------- registry
_PARTS: dict[str, Callable[[dict, BuildContext], Part]] = {}


def register_part(kind: str, factory: Callable[[dict, BuildContext], Part], *, replace: bool = False) -> None:
    if kind in _PARTS and not replace:
        raise ValueError(f"part kind {kind!r} is already registered")
    _PARTS[kind] = factory


def unregister_part(kind: str) -> None:
    _PARTS.pop(kind, None)


def make_part(spec: PartSpec, ctx: BuildContext) -> Part:
    if spec.kind not in _PARTS:
        raise KeyError(f"no part of kind {spec.kind!r}; registered: {', '.join(sorted(_PARTS))}")
    return _PARTS[spec.kind](dict(spec.params), ctx)


def prefixed(prefix: str, specs: dict[str, TensorSpec]) -> dict[str, TensorSpec]:
    return {prefix + k: v for k, v in specs.items()}


def take(tensors: dict[str, torch.Tensor], prefix: str) -> dict[str, torch.Tensor]:
    """The tensors under ``prefix``, with the prefix removed."""
    n = len(prefix)
    return {k[n:]: v for k, v in tensors.items() if k.startswith(prefix)}
