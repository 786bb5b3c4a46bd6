"""Interfaces of the parts a layer is put together from, and the registries that map a
``PartSpec.kind`` to its class.

A part is built from its spec and a :class:`BuildEnv` (width of the residual stream,
dtype, device); it declares its tensors (:class:`~.spec.ParamDecl`), receives them with
``bind`` and then computes on device tensors.  No part knows which model it is in.

Adding a part: subclass the interface, then ``MIXERS.register("name", Class)`` (or
``FEED_FORWARDS``, ``NORMS``, ``POSITIONS``, ``FILTERS``, ``CONNECTIONS``, ``BLOCKS``, ``EMBEDDINGS``, ``HEADS``).  A model
description refers to it as ``part("name", ...)``.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any

import torch

from .spec import ParamDecl, PartSpec


class Registry:
    def __init__(self, what: str):
        self.what = what
        self._classes: dict[str, type] = {}

    def register(self, kind: str, cls: type, replace: bool = False) -> None:
        if kind in self._classes and not replace:
            raise ValueError(f"{self.what} {kind!r} is already registered")
        self._classes[kind] = cls

    def unregister(self, kind: str) -> None:
        self._classes.pop(kind, None)

    def get(self, kind: str) -> type:
        if kind not in self._classes:
            raise KeyError(f"unknown {self.what} {kind!r}; registered: {sorted(self._classes)}")
        return self._classes[kind]

    def kinds(self) -> list[str]:
        return sorted(self._classes)


EMBEDDINGS = Registry("embedding")
HEADS = Registry("output head")
MIXERS = Registry("mixer")
FEED_FORWARDS = Registry("feed-forward")
NORMS = Registry("norm")
POSITIONS = Registry("position encoding")
FILTERS = Registry("input filter")
CONNECTIONS = Registry("stream connection")
BLOCKS = Registry("block arrangement")


@dataclass(frozen=True)
class PagedKVNeed:
    """Keys and values of every token (or of the last ``window`` tokens, or of the current chunk of ``chunk``
    positions) in pages.  ``keep_first``: with a window, the keys of the first ``keep_first`` positions stay as well.  ``v_head_dim``: the size of a value head where it differs from a key head's; a page row then
    has room for the larger of the two and each kind uses its leading elements.  ``planes``: 2 for a key and a value
    plane per page; 1 for pages that hold one row per token and head (a latent vector that is key and value at once)."""
    num_kv_heads: int
    head_dim: int
    window: int | None = None
    v_head_dim: int | None = None
    chunk: int | None = None
    planes: int = 2
    keep_first: int = 0

    @property
    def row_dim(self) -> int:
        return max(self.head_dim, self.v_head_dim or self.head_dim)


@dataclass(frozen=True)
class FixedStateNeed:
    """A tensor of fixed shape per live request (``dtype``: "float32" or "model")."""
    shape: tuple[int, ...]
    dtype: str = "float32"


@dataclass(frozen=True)
class SharedPagesNeed:
    """The place of a paged need in a run that reads another run's pages (``LayerRun.cache_from``) instead of keeping
    its own: nothing is allocated for it, and the run's view shows the other run's pages, not to be written."""


@dataclass(frozen=True)
class CompositeNeed:
    """Several things kept by one mixer (a mixer made of mixers, or one with pages and a state): the run's
    :class:`CacheView` then has one child view per entry, in this order."""
    parts: tuple


def need_leaves(need) -> list:
    """The paged / fixed-state / shared needs that a need is made of (a composite's entries, flattened in order)."""
    if need is None:
        return []
    if isinstance(need, CompositeNeed):
        return [leaf for sub in need.parts for leaf in need_leaves(sub)]
    return [need]


def with_shared_pages(need):
    """The same need with every paged entry replaced by :class:`SharedPagesNeed`; what else a run keeps (fixed-size
    state of its mixer or of its block) stays its own."""
    if isinstance(need, CompositeNeed):
        return CompositeNeed(tuple(with_shared_pages(sub) for sub in need.parts))
    if isinstance(need, PagedKVNeed):
        return SharedPagesNeed()
    return need


class BuildEnv:
    """What a part may know about its surroundings."""

    def __init__(self, hidden_size: int, dtype: torch.dtype, device: torch.device | str, max_position: int):
        self.hidden_size = hidden_size
        self.dtype = dtype
        self.device = torch.device(device)
        self.max_position = max_position
        self._positions: dict[PartSpec, "PositionEncoding"] = {}

    def position(self, spec: PartSpec | None):
        """The position encoding for ``spec``; equal specs share one object (one table on the device)."""
        if spec is None:
            return None
        if spec not in self._positions:
            self._positions[spec] = POSITIONS.get(spec.kind)(spec, self)
        return self._positions[spec]


class Part:
    def __init__(self, spec: PartSpec, env: BuildEnv):
        self.spec = spec
        self.env = env

    def params(self) -> list[ParamDecl]:
        return []

    def bind(self, tensors: dict[str, torch.Tensor]) -> None:
        """Receive the tensors declared by ``params`` (keyed by their local names)."""
        for name, t in tensors.items():
            setattr(self, "w_" + name.replace(".", "_"), t)

    def streamed_weights(self) -> list[tuple[torch.Tensor, int]]:
        """The matrices that a decode step reads once from end to end, with the mode in which
        ``kernels.ops`` streams them (0: plain product, 1: fp32 logits, 2: [gate; up] rows with SiLU).  The
        engine may keep a second copy of each, laid out for the weight-streaming kernel.  Default: none."""
        return []

    def new(self, *shape, dtype=None) -> torch.Tensor:
        return torch.empty(*shape, dtype=dtype or self.env.dtype, device=self.env.device)


@dataclass
class CacheView:
    """What one run of a mixer sees of the cache.

    Paged: ``pages`` [num_pages, 2, kv_heads, page_size, head_dim] of this run (or of the run it
    reads from), ``tables`` the step's block tables and slot mapping for the run's group,
    ``writes`` False if the run must not store keys and values.
    Fixed state: ``state`` [num_slots, *shape]; the step's slots are ``batch.state_slots``.
    Composite need: ``children``, one view per entry of the need.
    """
    pages: torch.Tensor | None = None
    tables: Any = None
    writes: bool = True
    state: torch.Tensor | None = None
    children: tuple = ()


@dataclass
class Pending:
    """Sub-block outputs that are not yet added to a float32 residual stream: the stream becomes
    stream + sum(coef * tensor) over ``terms`` ((tensor in the model's dtype, coef), ...), summed in 32-bit inside the
    next norm.  Blocks that keep their stream in float32 hand this on in place of a hidden tensor.
    ``post``: a norm that the (single) term still has to pass before it is added (blocks that norm a sub-block's
    output as well as its input); the next norm applies it inside its own kernel where it can, else through
    :meth:`settled`.
    ``rounded``: the stream itself rounded to the model's type, where the block before has it at hand (nothing pending);
    a block whose sub-blocks read the stream unnormed takes it from here instead of rounding the stream again.
    ``connection``: the residual stream is several copies per token, [T, S, width], and the (single) term reaches them
    through this :class:`StreamConnection`'s matrices; the next norm applies them."""
    terms: tuple = ()
    post: "Norm | None" = None
    rounded: "torch.Tensor | None" = None
    connection: "StreamConnection | None" = None

    def settled(self) -> "Pending":
        """The same sum with ``post`` applied by that norm's own ``forward`` (rounded to the model's type)."""
        if self.post is None:
            return self
        return Pending(tuple((self.post.forward(t), c) for t, c in self.terms))


class Mixer(Part):
    def forward_terms(self, x: torch.Tensor, batch, cache: "CacheView") -> tuple:
        """The mixer's output as a weighted sum ((tensor, coef), ...) that the caller may add term by term in 32-bit
        instead of receiving one rounded tensor.  Default: the one tensor of ``forward``."""
        return ((self.forward(x, batch, cache), 1.0),)

    def forward_normed_terms(self, x: torch.Tensor, batch, cache: "CacheView") -> tuple:
        """The mixer's output as ((tensor, coef, weight or None), ...): a weighted sum whose terms may each still have to
        pass an RMS norm over the model width with that weight (eps: ``self.side_eps``).  A block that norms the mixer's
        output anyway does these norms in the same kernel.  Default: the terms of ``forward_terms``, no norms."""
        return tuple((t, c, None) for t, c in self.forward_terms(x, batch, cache))

    def cache_need(self) -> "PagedKVNeed | FixedStateNeed | CompositeNeed | None":
        return None

    def forward(self, x: torch.Tensor, batch, cache: CacheView) -> torch.Tensor:
        """x [T, hidden] (normed) -> [T, hidden]; tokens of all requests of the step, packed."""
        raise NotImplementedError


class FeedForward(Part):
    def forward(self, x: torch.Tensor, batch) -> torch.Tensor:
        raise NotImplementedError


class Norm(Part):
    def forward(self, x: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError

    def forward_add(self, x, residual: torch.Tensor) -> torch.Tensor:
        """residual += x (in place, fp32 sum rounded once); returns norm of the unrounded sum.  ``x`` may be a
        :class:`Pending` over a float32 ``residual``: the weighted terms are added in 32-bit."""
        raise NotImplementedError

    def forward_add_rows(self, x: torch.Tensor, residual: torch.Tensor, rows: torch.Tensor) -> torch.Tensor:
        """Norm of (x + residual) at the given rows only; nothing is written back."""
        raise NotImplementedError

    def forward_streams(self, x: Pending, streams: torch.Tensor, connection: "StreamConnection"):
        """For a residual stream of several copies, ``streams`` [T, S, width] float32 (or [T, 1, width] while they are
        all equal): the pending output joins the copies through its own connection, and the sum that ``connection``
        reads of the new copies is normed.  Returns (the normed sum, the new copies)."""
        raise NotImplementedError

    def add_normed(self, terms: tuple, residual: torch.Tensor, side_eps=None, want_rounded: bool = True):
        """residual (float32, in place) += norm(sum of ``terms``), terms as ``Mixer.forward_normed_terms`` gives them: for
        blocks that norm a sub-block's output.  Returns the new stream rounded to the model's type (or None)."""
        raise NotImplementedError


class InputFilter(Part):
    """Something a sub-block's input passes on its way from the norm (a short filter over time, for instance).
    ``state_need()``: what it keeps per request between steps (a :class:`FixedStateNeed`) or None.  Filters of one
    block that read the same input may share one state; the block that arranges them decides."""

    def state_need(self):
        return None

    def forward(self, x: torch.Tensor, batch, state) -> torch.Tensor:
        raise NotImplementedError


class StreamConnection(Part):
    """How one sub-block is connected to a residual stream kept as ``streams`` copies: ``read`` [S] (the weights of the
    sum that it reads), ``write`` [S] (how its output joins each copy) and ``mix`` [S, S] (indexed [from, to]: how the
    copies are rebuilt from one another), float32 tensors."""
    streams: int
    read: torch.Tensor
    write: torch.Tensor
    mix: torch.Tensor


class PositionEncoding(Part):
    """How positions enter the model.  ``rotary()`` gives (table [max_position, rotary_dim] fp32 with
    cos then sin halves, rotary_dim) for mixers that rotate queries and keys, or None;
    ``add_to_embeddings`` lets an absolute encoding change the embedded tokens."""

    def rotary(self):
        return None

    def add_to_embeddings(self, h: torch.Tensor, batch) -> torch.Tensor:
        return h


class Embedding(Part):
    """Token ids to the first hidden states.  ``forward(token_ids [T] int32, batch) -> [T, hidden]``."""

    def forward(self, token_ids: torch.Tensor, batch) -> torch.Tensor:
        raise NotImplementedError


class Head(Part):
    """Hidden states of the wanted rows (after the final norm) to fp32 logits [rows, vocab].  ``tied`` True: the
    head owns no table and is handed the embedding part with ``tie`` once the tensors are bound."""
    tied = False

    def tie(self, embedding: Embedding) -> None:
        raise NotImplementedError

    def forward(self, rows_hidden: torch.Tensor) -> torch.Tensor:
        raise NotImplementedError


class Block:
    """The arrangement of a layer's parts.  ``SLOTS`` names the parts this kind of block arranges and the
    registry each is built from; ``OPTIONAL`` those a layer may leave out.  The model builds them and hands
    them over as ``parts`` (name -> part; each is also set as an attribute of that name).  ``forward`` takes and
    returns (hidden, residual): the sub-block output not yet added, and the residual stream; residual None means
    "first layer".  ``cache_owner`` is the part whose ``cache_need`` decides what a run of this layer keeps
    between steps (one per layer)."""
    SLOTS: dict[str, Registry] = {"mixer": MIXERS, "mixer_norm": NORMS, "ffn": FEED_FORWARDS, "ffn_norm": NORMS}
    OPTIONAL: tuple[str, ...] = ()

    def __init__(self, spec: PartSpec, parts: dict[str, Part]):
        self.spec = spec
        self.parts = dict(parts)
        for name, obj in parts.items():
            setattr(self, name, obj)

    @property
    def cache_owner(self) -> Mixer | None:
        return self.parts.get("mixer")

    def cache_need(self):
        """What a run of this layer keeps between steps: by default what its ``cache_owner`` needs.  A block that
        keeps something itself returns a :class:`CompositeNeed` and hands each part its child view."""
        owner = self.cache_owner
        return owner.cache_need() if owner is not None else None

    def forward(self, hidden, residual, batch, cache: CacheView):
        raise NotImplementedError
