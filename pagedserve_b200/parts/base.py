"""Interfaces of the parts and the part registry.

A part is built from a :class:`PartSpec` (its constants), declares the tensors
it needs (:meth:`Part.param_specs`), receives them (:meth:`Part.bind`) and then
runs.  No part knows which model it is in: sizes, names of tensors and every
constant are parameters.

Categories and what each must provide
-------------------------------------
``embedding``          ``forward(ctx) -> hidden``: float32 ``[T, H]`` residual stream.
``positions``          ``embedding_table()`` (a table to add to the token embedding, or None),
                       ``add_to_hidden(hidden, ctx)`` and ``rotate(q, k, ctx)`` hooks.
``norm``               ``forward(x, out=None, rows=None) -> normed`` (compute dtype).
``mixer``              ``cache_need()``, ``state_need()``,
                       ``forward(x, residual, ctx, layer)``: adds its output into ``residual``.
``feed_forward``       ``forward(x, residual, ctx)``: adds its output into ``residual``.
``block``              ``forward(hidden, ctx, layer)``: runs norms, mixer, feed-forward in its arrangement.
``head``               ``forward(x_rows) -> float32 logits [R, V]``.

``ctx`` is the :class:`pagedserve_b200.engine.batch.StepContext` of the step;
``layer`` is a :class:`LayerContext` that carries what this run of the layer
may touch of the cache (pages of its cache layer, its slot state).
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Callable, Dict, List, Optional, Tuple

import torch

from pagedserve_b200.cache.manager import KVNeed, StateNeed
from pagedserve_b200.weights.loader import ParamSpec

Init = Tuple[str, float]            # ("normal" | "ones_plus_normal", std)


@dataclass
class PartEnv:
    """What every part gets at construction."""

    ops: object                      # pagedserve_b200.kernels.Ops (None on a host without kernels)
    dtype: torch.dtype               # compute dtype
    device: object


@dataclass
class LayerContext:
    layer: int                       # index of the layer whose parameters run
    cache_layer: int                 # index of the cache layer it uses
    positions: "PositionEncoding"
    k_pool: Optional[torch.Tensor] = None      # [pages, kv heads, page size, head dim] view
    v_pool: Optional[torch.Tensor] = None
    page_stride: int = 0             # elements between consecutive pages
    page_size: int = 0
    pool: Optional[torch.Tensor] = None        # the group's whole pool [pages, layers, 2, kv heads, page, head dim]
    pool_layer: int = 0                        # index of this cache layer inside the pool
    block_table: Optional[torch.Tensor] = None  # int32 [slots + 1, max pages] of the layer's group, by request slot
    state: Optional[torch.Tensor] = None        # [max slots, *state shape] of this cache layer


class Part:
    category = ""
    # True when ``forward`` only launches work whose shapes and addresses depend on the batch size alone
    # and reads the batch from ``ctx``'s device arrays: such a step can be captured once as a CUDA graph
    # and replayed. A part that branches on host data (``ctx.host``) leaves this False, and a model
    # with such a part runs every step eagerly.
    graph_safe = False

    # A factor per coordinate (float32 [H]) that an arrangement puts on what a mixer or a feed-forward adds to the residual
    # rows (:meth:`set_result_factor`); parts that can apply it where their last product is stored say so.
    result_factor = None
    takes_result_factor = False

    def set_result_factor(self, factor: torch.Tensor) -> None:
        if not self.takes_result_factor:
            raise ValueError(f"{type(self).__name__} cannot multiply its result by a factor per coordinate")
        self.result_factor = factor

    def __init__(self, params: dict, prefix: str, env: PartEnv):
        self.params = dict(params)
        self.prefix = prefix
        self.env = env

    # name helper: tensors are named prefix + local name
    def _n(self, local: str) -> str:
        return self.prefix + local

    def param_specs(self) -> List[Tuple[ParamSpec, Init]]:
        """Tensors this part needs, each with the rule by which random weights are drawn."""
        return []

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Receive the loaded tensors (by canonical name)."""


class Embedding(Part):
    category = "embedding"

    def state_need(self) -> Optional[StateNeed]:
        """Per-request state of the embedding itself (a table indexed by more than the current token); the model
        gives it a cache layer of its own behind those of the schedule and passes the tensor to ``forward`` as
        ``state``."""
        return None

    def forward(self, ctx, positions: "PositionEncoding") -> torch.Tensor:
        raise NotImplementedError


class PositionEncoding(Part):
    category = "positions"

    def embedding_table(self) -> Optional[torch.Tensor]:
        """A ``[positions, H]`` table to be added to the token embedding, if this encoding has one."""
        return None

    def sinusoids(self) -> Optional[torch.Tensor]:
        """Frequencies ``[ceil(H / 2), 2]`` ((high, low) floats) of sines and cosines of the position that are added to the
        token embedding, if this encoding is made of them."""
        return None

    def add_to_hidden(self, hidden: torch.Tensor, ctx) -> None:
        """Add a position term to the embedded tokens (absolute encodings)."""

    def rotate(self, q: torch.Tensor, k: torch.Tensor, ctx) -> None:
        """Transform queries and keys in place by position (rotary encodings)."""

    def max_positions(self) -> Optional[int]:
        return None


@dataclass
class NormPrologue:
    """What a matrix product needs to compute a norm of the form ``(x - mean?) * rsqrt(var + eps) * weight
    (+ bias)`` over the last axis inside its own kernel, in float32."""

    weight: torch.Tensor                 # float32 [width]
    bias: Optional[torch.Tensor]         # float32 [width] or None
    eps: float
    has_mean: bool                       # False: the RMS form


class Norm(Part):
    category = "norm"

    def forward(self, x: torch.Tensor, out: Optional[torch.Tensor] = None,
                rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        raise NotImplementedError

    def fused_prologue(self) -> Optional[NormPrologue]:
        """A norm that a consuming product may fold into its prologue says how here (any norm of the form
        :class:`NormPrologue` describes, whatever its class); None: it has to run as its own kernel."""
        return None


class Mixer(Part):
    category = "mixer"

    def cache_need(self) -> Optional[KVNeed]:
        return None

    def state_need(self) -> Optional[StateNeed]:
        return None

    # What ``forward`` adds is the mixer's result divided by this common factor (1 for nearly all of them): a block that
    # norms the result multiplies by it first (``Block.takes_output_scale``), other blocks refuse such a mixer.
    output_scale = 1.0

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx, layer: LayerContext) -> None:
        raise NotImplementedError

    # A mixer that can stand beside others, behind one product that makes all their inputs and in front of one that
    # takes all their results (``parts/parallel.py``), cuts its ``forward`` into these.
    def joint_in(self):
        """(matrix [rows, hidden], bias [rows] or None) of its projections, stacked; after ``bind``."""
        raise NotImplementedError

    def joint_out(self):
        """(matrix [hidden, columns], bias [hidden] or None) of its output projection."""
        raise NotImplementedError

    scales_joint = False        # whether ``joint_mix`` can multiply its result by a factor in float32

    def joint_mix(self, projected: torch.Tensor, context: torch.Tensor, ctx, layer: LayerContext, factor: float = 1.0) -> None:
        """From its columns of the projections' rows (compute dtype) to its columns of the rows that the output
        projection reads."""
        raise NotImplementedError


class FeedForward(Part):
    category = "feed_forward"

    def forward(self, x: torch.Tensor, residual: torch.Tensor, ctx) -> None:
        raise NotImplementedError


class Block(Part):
    category = "block"

    def __init__(self, params, prefix, env, mixer: Mixer, feed_forward: FeedForward, norms: Dict[str, Norm]):
        super().__init__(params, prefix, env)
        self.mixer = mixer
        self.feed_forward = feed_forward
        self.norms = norms
        if mixer.output_scale != 1.0 and not self.takes_output_scale:
            raise ValueError("this arrangement cannot multiply a mixer's result by a factor")

    required_norms: Tuple[str, ...] = ()
    takes_output_scale = False

    # What a run of the layer needs of the cache: the mixer's needs, unless the arrangement keeps state of its own
    # (``state_need``: it then hands the mixer its share of ``layer.state``).
    def cache_need(self) -> Optional[KVNeed]:
        return self.mixer.cache_need()

    def state_need(self) -> Optional[StateNeed]:
        return self.mixer.state_need()

    def forward(self, hidden: torch.Tensor, ctx, layer: LayerContext) -> None:
        raise NotImplementedError

    # What runs through the layers need not be the one float32 row per token that the embedding makes: an
    # arrangement with a carrier of its own (several residual streams, say) builds it from the embedded rows
    # before the first layer (``begin``), gets it as ``hidden`` in every ``forward``, and turns it back into one
    # row per token behind the last layer (``end``).  ``following`` is the block of the next run of the
    # schedule (None behind the last): what a block leaves undone for the next one to fold into its first pass.
    # All blocks of a model share one kind of carrier.
    def begin(self, hidden: torch.Tensor, ctx):
        return hidden

    def end(self, carrier, ctx) -> torch.Tensor:
        return carrier


class Head(Part):
    category = "head"

    def forward(self, x_rows: torch.Tensor, embedding: Embedding) -> torch.Tensor:
        raise NotImplementedError


# ---------------------------------------------------------------------------- registry
_PARTS: Dict[Tuple[str, str], Callable] = {}
CATEGORIES = ("embedding", "positions", "norm", "mixer", "feed_forward", "block", "head")


def register_part(category: str, kind: str, replace: bool = False):
    """Class decorator: make ``kind`` available to ModelSpecs under ``category``."""
    if category not in CATEGORIES:
        raise ValueError(f"unknown part category {category!r}; one of {CATEGORIES}")

    def decorate(cls):
        key = (category, kind)
        if key in _PARTS and not replace:
            raise ValueError(f"part {kind!r} is already registered as a {category}")
        _PARTS[key] = cls
        return cls

    return decorate


def part_kinds(category: str) -> List[str]:
    return sorted(kind for (cat, kind) in _PARTS if cat == category)


def create_part(category: str, spec, env: PartEnv, **extra) -> Part:
    key = (category, spec.kind)
    if key not in _PARTS:
        raise ValueError(f"no {category} part named {spec.kind!r}; registered: {part_kinds(category)}")
    return _PARTS[key](spec.params, spec.prefix, env, **extra)
