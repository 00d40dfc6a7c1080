"""What a part is: the interfaces of mixer, feed-forward, norm, position
encoding, block, embedding and head, and the registries that name them.

A part is built from keyword arguments alone (its sizes, constants and tensor
names); it never learns which model it is in.  A model is a list of blocks
whose parts are chosen layer by layer through `PartSpec(kind, args)`.

Life of a part:
  1. `Part(**args)`                      sizes and names are fixed;
  2. `params()`                          the tensors it wants from the model folder;
  3. `bind(tensors, rt)`                 it takes them (and may fuse or drop them);
  4. `forward(...)`                      once per step, enqueueing kernels on the
                                         current stream; no host synchronisation.

A part that says `graph_safe = True` promises that its `forward` may be captured in a
CUDA graph once and replayed for other steps of the same shape: it reads sequence
numbers, slots, positions and page tables from the step's DEVICE tensors only (the host
copies change between replays), sizes its launches by what holds for every replay
(`step.n_rows` token rows, `step.n_seq_cap` sequences, some of them padding), skips rows
of sequence -1, keeps nothing on the host from one call to the next, and calls nothing
that synchronises or allocates outside torch's stream-ordered allocator.  The default is
False: a model with one such part runs every step eagerly, which is always right.
"""
from __future__ import annotations

import dataclasses
from typing import Any, Callable

import torch

from ..cache import KVRequest


@dataclasses.dataclass(frozen=True)
class ParamSpec:
    """One tensor of the model folder.

    init: how random-weights mode fills it: "matrix" N(0, 0.02), "norm" 1 + N(0, 0.1), "near_zero" N(0, 0.1),
    "logit" N(0, 1),
    "unit" 0.5 + N(0, 0.15) (mixing weights and lower bounds between 0 and 1), "decay"
    -2 + N(0, 1) (what a double exponential turns into a decay), "zeros", or "int_table"
    (int32 zeros).  alias_of: the name of another tensor that stands in when this one is
    absent (a tied head).  A dimension of -1 in `shape` takes whatever the model folder
    holds (a size that no configuration key gives); `shape_if_random` is then the shape
    that random-weights mode writes.  optional: a tensor that a folder may hold or lack; no part
    reads it and random-weights mode does not write it.
    """
    name: str
    shape: tuple[int, ...]
    init: str = "matrix"
    alias_of: str | None = None
    shape_if_random: tuple[int, ...] | None = None
    optional: bool = False

    def matches(self, shape) -> bool:
        shape = tuple(shape)
        return len(shape) == len(self.shape) and all(w in (-1, h) for w, h in zip(self.shape, shape))

    @property
    def concrete_shape(self) -> tuple[int, ...]:
        shape = self.shape_if_random if (self.shape_if_random is not None and -1 in self.shape) else self.shape
        if -1 in shape:
            raise ValueError(f"tensor '{self.name}': a dimension of its shape {self.shape} is known from a model folder only")
        return tuple(shape)

    @property
    def is_integer(self) -> bool:
        return self.init == "int_table"


@dataclasses.dataclass(frozen=True)
class PartSpec:
    kind: str
    args: dict = dataclasses.field(default_factory=dict)


class Part:
    """Base of all parts."""

    def params(self) -> list[ParamSpec]:
        return []

    def bind(self, tensors: dict[str, torch.Tensor], rt) -> None:
        pass

    # May this part's forward be captured in a CUDA graph and replayed (see the module's text)?
    graph_safe = False

    def kernel_groups(self) -> set[str]:
        """Kernel libraries this part launches (compiled before the first step)."""
        return set()

    def notes(self, rt) -> list[str]:
        """What a user should know at load about how this part will run with its sizes (a size that
        a fast kernel does not take and what runs instead); printed once, never an error."""
        return []


class ResidualAdded:
    """The answer of `Runtime.linear(..., add_to=x)` when the product has added its result to
    the residual stream x itself (in its epilogue): nothing is left to add.  A block turns it
    into "no pending update" before the next norm sees it."""


class Biased:
    """An update of the residual stream that still lacks a bias: `update` (a tensor, or
    `ResidualAdded()` when the product has added itself already) plus `bias` [width] on every row.
    Whoever adds the update (the next norm, a block's extra) adds the bias with it."""

    def __init__(self, update, bias: torch.Tensor):
        self.update, self.bias = update, bias


class Several(list):
    """Several updates of the residual stream that are pending at once (a block whose mixer and feed-forward
    read the same input answers both): tensors [n, width] or [parts, n, width], added in their order.  Only a
    norm that says `takes_several` may follow; it gets them as a list in place of `delta`."""


class Scaled:
    """Updates of the residual stream that are to be added times a factor: x += factor * (sum of the updates).
    `update`: what a mixer or feed-forward answers (a tensor, `Several`, `Biased`, None).  Only a norm that says
    `takes_scale` may follow; it gets the factor as the keyword `scale=`."""

    def __init__(self, update, factor: float):
        self.update, self.factor = update, float(factor)


class Combined(list):
    """An update that is a sum of terms, each a tensor ([n, width] or partial sums) times a factor, optionally times a
    number per row, optionally divided by its own root mean square and multiplied by a weight first (`ops.Term`): what a
    mixer of two branches answers.  Only a norm that says `takes_terms` may follow."""


class Normed:
    """An update that passes a norm of its own before it is added: x += weight * u / rms(u), u the sum of `update`
    (a tensor, `Several` or `Combined`); with `center` a layer norm, x += weight * (u - mean(u)) / std(u) + bias.  Only a
    norm that says `takes_terms` may follow; it does the sum, this norm, the add and its own norm in one kernel."""

    def __init__(self, update, weight: torch.Tensor, eps: float, bias: torch.Tensor | None = None, center: bool = False):
        self.update, self.weight, self.eps, self.bias, self.center = update, weight, float(eps), bias, bool(center)


class Streamed:
    """An update of a residual that consists of several streams X[0] .. X[s-1] (`x` is [s, n, width]): with u the sum of
    `update` (a tensor, `Biased`, `Several`, `Combined`), every stream becomes X[j] <- sum_i mix[i, j] X[i] + out[j] u, all of
    them at once from the old ones.  mix: float32 [s, s] (from, to), out: float32 [s].  Only a norm that says `takes_streams`
    may follow."""

    def __init__(self, update, mix: torch.Tensor, out: torch.Tensor):
        self.update, self.mix, self.out = update, mix, out


def update_factor(pending) -> float:
    """The factor on a pending update (1 unless it is `Scaled`)."""
    return pending.factor if isinstance(pending, Scaled) else 1.0


def split_update(pending):
    """(delta, bias) of what a mixer or feed-forward answered: each a tensor or None (delta a list of
    tensors for `Several`).  The factor of a `Scaled` update is asked for with `update_factor`."""
    bias = None
    if isinstance(pending, (Normed, Combined, Streamed)):
        return pending, None
    if isinstance(pending, Scaled):
        pending = pending.update
    if isinstance(pending, Biased):
        pending, bias = pending.update, pending.bias
    if isinstance(pending, ResidualAdded):
        pending = None
    if isinstance(pending, Several):
        kept = [u for u in pending if u is not None and not isinstance(u, ResidualAdded)]
        pending = None if not kept else kept[0] if len(kept) == 1 else kept
    return pending, bias


class Norm(Part):
    def forward(self, rt, x: torch.Tensor, delta, rows: torch.Tensor | None = None):
        """x: the 32-bit residual stream [n, width], updated in place by `delta`
        (None, [n, width] or [splits, n, width]); returns the normalised rows in
        the runtime's element type.  rows: gather these rows only (x untouched).
        A norm that sets `takes_bias` also takes a keyword `bias=` ([width], added to every
        row with the update); only such a norm may follow a part that answers `Biased`."""
        raise NotImplementedError

    takes_bias = False
    takes_several = False   # `delta` may be a list of up to three updates
    takes_scale = False     # takes a keyword `scale=`: x += scale * (the updates)
    takes_terms = False     # `delta` may be `Combined` or `Normed`
    takes_streams = False   # x is [streams, n, width] and `delta` None or `Streamed`

    can_norm_updates = False  # may stand on a sublayer's output (has `as_update_norm`)

    def as_update_norm(self, update) -> Normed:
        """`update` with this norm on it, for whoever adds it (a norm on a sublayer's output)."""
        raise NotImplementedError


class PositionEncoding(Part):
    def prepare(self, rt, n_positions: int) -> None:
        """Build whatever tables positions [0, n_positions) need."""

    def rotation(self):
        """(cos, sin, rotary_dim) tables [n_positions, rotary_dim/2] of 32-bit floats for
        mixers that rotate q and k, or None."""
        return None

    def on_embedding(self, rt, step, x: torch.Tensor) -> None:
        """Hook for encodings that act on the embedded tokens (in place)."""


class Mixer(Part):
    def cache_request(self) -> KVRequest | None:
        """Keys and values this mixer keeps per token, or None."""
        return None

    def state_bytes(self) -> int:
        """Bytes of fixed-size state this mixer keeps per sequence."""
        return 0

    # A mixer or feed-forward that sets this also takes a keyword `residual=` (the 32-bit
    # residual stream its update is meant for) and may pass it to its last product as
    # `Runtime.linear(..., add_to=residual)`, returning whatever that returns.
    takes_residual = False

    def forward(self, rt, step, h: torch.Tensor, entry: int) -> torch.Tensor:
        """h: [T, width] normalised input.  entry: index of the schedule entry being run
        (names the cache line and the state through `step`).  Returns the update of the
        residual stream, [T, width] or [splits, T, width]."""
        raise NotImplementedError


class FeedForward(Part):
    takes_residual = False  # as for Mixer

    def forward(self, rt, step, h: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


class Connection(Part):
    """How a sublayer's output joins a residual that is more than one stream."""

    def join(self, update) -> Streamed:
        raise NotImplementedError


class Block(Part):
    def forward(self, rt, step, x: torch.Tensor, pending, entry: int):
        """x: residual stream (in place); pending: an update not yet added to it (None, [n, width]
        or [splits, n, width]).  Returns (x, pending)."""
        raise NotImplementedError

    @property
    def mixer(self) -> Mixer:
        raise NotImplementedError


class BlockExtra(Part):
    """What a block does to the residual stream after its mixer and feed-forward (an input of its
    own from the tokens, for instance)."""

    def forward(self, rt, step, x: torch.Tensor, pending):
        """x: the residual stream; pending: the update not yet added (as a mixer answers it).
        Returns (x, pending)."""
        raise NotImplementedError


class Embedding(Part):
    def forward(self, rt, step) -> torch.Tensor:
        raise NotImplementedError


class Head(Part):
    def forward(self, rt, step, h: torch.Tensor) -> torch.Tensor:
        """h: [rows, width] normalised; returns 32-bit logits [rows, vocab]."""
        raise NotImplementedError


# ---------------------------------------------------------------- registries
_REGISTRIES: dict[str, dict[str, Callable[..., Any]]] = {
    "mixer": {}, "feed_forward": {}, "norm": {}, "position_encoding": {}, "block": {}, "block_extra": {},
    "connection": {}, "embedding": {}, "head": {},
}


def register_part(role: str, kind: str):
    """Class decorator: make `kind` buildable wherever a part of `role` is wanted."""
    if role not in _REGISTRIES:
        raise KeyError(f"unknown part role '{role}' (known: {', '.join(_REGISTRIES)})")

    def deco(cls):
        _REGISTRIES[role][kind] = cls
        return cls
    return deco


def build_part(role: str, spec: PartSpec):
    table = _REGISTRIES[role]
    if spec.kind not in table:
        raise KeyError(f"no {role} named '{spec.kind}' is registered (known: {', '.join(sorted(table)) or 'none'})")
    return table[spec.kind](**spec.args)
