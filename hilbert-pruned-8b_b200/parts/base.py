"""Interfaces and registries of the parts a decoder layer is put together from.

Kinds of part: mixer (attention, or anything else that mixes tokens of a sequence),
feed-forward, norm, position encoding, block (the arrangement of the four in a layer),
embedding and head.  Each kind has one registry from a name to a class; a configuration
chooses parts by name, layer by layer.  No part knows which model it is in: sizes and
constants arrive as parameters of its ``PartSpec``.

What a part must provide:

* ``params()``: its weight tensors as ``ParamSpec`` rows (name local to the part, shape,
  kind).  The loader, the random-weights mode and the byte accounting all read this one
  table, as the reference does with its shape table
  (cleanroom-transformer/src/shapes.c:12-39, model.c:246-257).
* ``bind(tensors)``: receives the loaded tensors by local name and may fuse them.
* mixers: ``cache_need()`` (keys and values per token, or None), ``state_need()``
  (fixed-size state per sequence, or None) and
  ``forward(h, residual, step, cache, state, append)`` which ADDS the mixer's output to the
  32-bit ``residual`` in place.
* feed-forwards: ``forward(h, residual, step)``, adding likewise.
* norms: ``forward(x, out, rows=None)``.
* token filters: ``state_need()`` and ``forward(x, out, step, state, norm=None)``.
* position encodings: ``rotation_table(step)`` when the encoding is a rotation of pairs of
  head dimensions by position-dependent angles (the kernels then turn queries and keys
  themselves), else ``apply(q, k, step)`` which turns them in place; see ``PositionEncoding``.
* residual gates: ``logits(h, step)`` (32-bit, without the bias) and ``bias``.
* residual scales: ``factors`` (32-bit ``[width]``), one factor per channel of a sublayer's result.
* stream vectors: ``vector(i)`` (32-bit ``[width]``), what a plan entry adds to every token's stream in front of itself.
* token sides: ``forward(h, x, step, copy=None)``, adding to the 32-bit stream ``x``.
* blocks (``parts/block.py``): ``ROLES``, ``named_parts()``, ``cache_need()``, ``state_need()``,
  ``forward(x, step, cache, state, append)``.
* optional, ``folds_norms = True`` on mixers, feed-forwards and blocks: the norms between two
  matrix products may be folded into them for steps of few tokens; see ``Mixer`` and
  ``Norm.fold_request`` below and ``Block`` in ``parts/block.py``.
* ``graph_safe`` (class attribute, default True): whether ``forward`` only enqueues work on
  the current stream, so that a decode step can be captured in a CUDA graph.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, List, Optional, Tuple

import torch

from ..config.spec import PartSpec


@dataclass(frozen=True)
class ParamSpec:
    name: str
    shape: Tuple[int, ...]
    kind: str = "matrix"        # "matrix" | "vector" | "int_table"
    init: str = "normal"        # random-weights mode: "normal" | "ones" | "zeros"
    absolute: bool = False      # name is not below the decoder's prefix (lm_head.weight)
    optional: bool = False      # may be absent (and is then not an error)


@dataclass(frozen=True)
class CacheNeed:
    """Keys and values a mixer keeps per token: ``window`` None keeps all of them; with a window
    the sequence's first ``keep_first`` tokens stay visible (and stored) for good.  ``v_head_dim``:
    the size of a value head where it differs from a key head's.  ``stride`` above 1: one key and
    value per WHOLE run of ``stride`` tokens (entry ``e`` stands for the positions ``e * stride`` to
    ``e * stride + stride - 1`` and exists once the sequence holds them all), which is what a mixer
    that keeps pooled summaries of its past needs.  ``store_f32``: 32-bit storage whatever the
    cache's dtype.  A mixer may ask for several needs at once (a tuple): it then gets a view per need."""

    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    v_head_dim: Optional[int] = None
    keep_first: int = 0
    stride: int = 1
    store_f32: bool = False

    @property
    def value_dim(self) -> int:
        return self.head_dim if self.v_head_dim is None else self.v_head_dim


@dataclass(frozen=True)
class StateNeed:
    """Fixed-size state a mixer keeps per sequence (zeroed when a sequence starts)."""

    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass
class BuildContext:
    """What parts need to build themselves: device, activation dtype, kernels, scratch."""

    device: torch.device
    dtype: torch.dtype                      # torch.bfloat16 or torch.float32
    ops: Any                                # the kernel library (kernels.ops)
    workspace: Any                          # engine.workspace.Workspace
    max_step_tokens: int
    _shared: Dict[str, Any] = None          # parts shared between layers, by spec

    def shared_part(self, registry: "Registry", spec: PartSpec) -> Any:
        if self._shared is None:
            self._shared = {}
        key = registry.kind + ":" + repr(spec)
        if key not in self._shared:
            self._shared[key] = registry.build(spec, self)
        return self._shared[key]


class Part:
    # False for a part whose forward reads device values on the host or allocates: the engine
    # then runs its decode steps eagerly instead of replaying a captured CUDA graph
    graph_safe = True

    def __init__(self, spec: PartSpec, ctx: BuildContext):
        self.spec = spec
        self.ctx = ctx

    def params(self) -> List[ParamSpec]:
        return []

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        pass

    def weight_bytes(self) -> int:
        """Bytes of weights a step reads from this part (for roofline accounting)."""
        return 0


class Mixer(Part):
    """Reads the normed input ``h``, adds its result to the 32-bit ``residual``.

    A part with ``folds_norms = True`` also takes two keyword arguments, by which a block folds
    the norms around it into its matrix products for steps of few tokens (no norm kernel):
    ``prepared`` (a ``kernels.ops.PreparedNorm``: ``h`` holds the norm's input times the norm's
    weight WITHOUT the per-token factor, which the part's first product applies to its rows),
    and ``prepare`` (what ``Norm.fold_request`` returned for the norm that reads ``residual``
    next: the part's last product fills that norm's buffer).  ``forward`` then returns the
    ``PreparedNorm`` for the next reader, or None when it prepared nothing (the block runs the
    norm).  Parts without the attribute are called without the two arguments.

    A part with ``can_overwrite = True`` also takes ``accumulate=False``: it then WRITES its result
    to ``residual`` (which is then some other 32-bit buffer of the same shape) instead of adding
    it.  Blocks that put something between a sublayer and the residual stream (a norm on the
    sublayer's output, a weighted sum of several mixers) use it; for other parts they zero the
    buffer first."""

    folds_norms = False
    can_overwrite = False

    # ``takes_guest = True``: the mixer's first product can carry further rows for a part that reads the same input (a
    # residual gate).  The block sets ``guest`` before weights are bound; ``bind`` takes the guest's rows
    # (``guest.host_rows(dtype)``, None: the guest keeps them) and ``forward`` hands it the columns they gave
    # (``guest.receive(view)``).
    takes_guest = False
    guest = None

    def cache_need(self) -> Optional[CacheNeed]:
        return None

    def state_need(self) -> Optional[StateNeed]:
        return None

    def forward(self, h, residual, step, cache, state, append: bool):
        raise NotImplementedError


class FeedForward(Part):
    """As ``Mixer``: reads ``h``, adds to ``residual``; ``folds_norms`` and ``can_overwrite`` as there.

    ``sums_entries = True`` (may depend on the part's options): ``forward_entries(h, step)`` returns ``(rows, n)``, 32-bit rows
    ``[tokens * n, width]`` of which n per token add up to the result, for a caller whose own kernel forms that sum."""

    sums_entries = False

    # ``weighs_entries = True`` (may depend on the part's options): ``forward_weighted(h, step)`` returns ``(rows, n, weights, base)``: the
    # result of token t is ``base[t] + sum_k weights[t, k] * rows[t * n + k]``, all 32-bit, ``base`` None: nothing, for a caller whose own
    # kernel forms that sum.
    weighs_entries = False

    folds_norms = False
    can_overwrite = False

    def forward(self, h, residual, step):
        raise NotImplementedError


class TokenFilter(Part):
    """Changes what a mixer reads by looking at a few earlier tokens of the same sequence (a short
    convolution over time).  ``state_need()``: what it keeps per sequence between steps;
    ``forward(x, out, step, state, norm=None)`` writes ``out`` from ``x``; a filter with
    ``fuses_norm(norm)`` true can be handed the residual stream and the norm in front of it
    (``norm=``) and applies both in one pass."""

    def state_need(self) -> Optional[StateNeed]:
        return None

    def fuses_norm(self, norm) -> bool:
        return False

    def forward(self, x, out, step, state, norm=None) -> None:
        raise NotImplementedError


class Norm(Part):
    out_dtype: torch.dtype

    def forward(self, x, out, rows=None) -> None:
        raise NotImplementedError

    def add_normed(self, y, x, then=None, then_out=None) -> bool:
        """``x += norm(y)`` for a norm that sits on a sublayer's OUTPUT (``x`` the 32-bit residual stream, ``y`` the
        sublayer's 32-bit result).  ``then``/``then_out``: the norm that reads ``x`` next and its output buffer; a norm
        that can make both in one pass does and returns True, else it returns False and the caller runs ``then``."""
        raise NotImplementedError(f"{type(self).__name__} cannot sit on a sublayer's output")

    def fold_request(self, out):
        """What the product that writes this norm's input needs in order to prepare it
        (``Ops.linear(..., prepare=...)``): ``(weight, offset, eps, out)`` for a norm of the form
        ``x * rsqrt(mean(x^2) + eps) * (offset + weight)``; None: the norm cannot be folded."""
        return None


class PositionEncoding(Part):
    """How a mixer's queries and keys learn their positions.  A mixer uses one of two forms:

    * ``rotation_table(step)`` returns ``(table, rotary_dim)``: ``table[t, i] = (cos a, sin a)``
      in 32-bit, ``[tokens, rotary_dim / 2, 2]``, for the step's token ``t`` and the pair
      ``(i, i + rotary_dim / 2)`` of every head; the attention kernels turn queries and keys by
      it (dimensions from ``rotary_dim`` on stay).  ``fusable`` says whether a kernel that does
      more than turning (decode attention that also appends and attends) may take the table;
      a part sets it False to keep the rotation a step of its own.
    * ``rotation_table`` returns None: the encoding is something else, and ``apply(q, k, step)``
      changes ``q [tokens, heads, head_dim]`` and ``k [tokens, kv_heads, head_dim]`` (views of
      the step's projections) in place before the keys are cached; no kernel rotates.

    ``prepare(step)`` may compute what all layers of a step share into ``step.shared``."""

    fusable = True

    def prepare(self, step) -> None:
        pass

    def rotation_table(self, step):
        return None

    def apply(self, q, k, step) -> None:
        raise NotImplementedError(f"{type(self).__name__} gives neither a rotation table nor apply()")


def stack_rows(rows: List[torch.Tensor], width: int, guest=None) -> Tuple[torch.Tensor, Optional[int]]:
    """The matrices ``[n, width]`` one below the other as one product's weight, with zero rows up to a multiple of 8 rows,
    then the rows of a ``guest`` that lends them (``Mixer.takes_guest``), padded likewise: ``(matrix, first guest row)``,
    the second None without a guest."""
    def pad(n):
        return [torch.zeros(n, width, dtype=rows[0].dtype, device=rows[0].device)] if n else []
    total = sum(r.shape[0] for r in rows)
    out, at = list(rows) + pad(-total % 8), None
    lent = guest.host_rows(rows[0].dtype) if guest is not None else None
    if lent is not None:
        at = total + -total % 8
        out += [lent] + pad(-lent.shape[0] % 8)
    return torch.cat(out, dim=0).contiguous(), at


class Registry:
    def __init__(self, kind: str):
        self.kind = kind
        self._classes: Dict[str, Callable[..., Any]] = {}

    def register(self, name: str) -> Callable[[Any], Any]:
        def deco(cls):
            self._classes[name] = cls
            return cls
        return deco

    def unregister(self, name: str) -> None:
        self._classes.pop(name, None)

    def names(self) -> List[str]:
        return sorted(self._classes)

    def get(self, name: str) -> Callable[..., Any]:
        if name not in self._classes:
            raise KeyError(f"no {self.kind} named {name!r} is registered ({', '.join(self.names())})")
        return self._classes[name]

    def build(self, spec: PartSpec, ctx: BuildContext) -> Any:
        return self.get(spec.kind)(spec, ctx)


MIXERS = Registry("mixer")
TOKEN_FILTERS = Registry("token filter")
FEED_FORWARDS = Registry("feed-forward")
NORMS = Registry("norm")
POSITION_ENCODINGS = Registry("position encoding")
BLOCKS = Registry("block")
EMBEDDINGS = Registry("embedding")
HEADS = Registry("head")
RESIDUAL_GATES = Registry("residual gate")
RESIDUAL_SCALES = Registry("residual scale")
STREAM_VECTORS = Registry("stream vectors")
TOKEN_SIDES = Registry("token side input")
