"""Interfaces of the parts a layer is put together from, and their registries.

A model is data: a list of layers, each naming a block arrangement, two norms, a
mixer and a feed-forward by their registry names with their parameters, and a
list that says in which order layers run and which cache each run uses.  The
parts know their own sizes and constants and nothing about the model they sit
in.  A new part is a class registered under a new name; nothing else changes.

The reference builds one fixed module tree (DELTA/Engine/DELTA/model.py:130-137,
330-336) whose sizes come through ``ModelArgs``; the parts below are the same
units (RMSNorm 521-532, Attention 362-492, FeedForward 495-518,
TransformerBlock 330-341) made exchangeable.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Any, Callable, Dict, Optional

import torch


# ---------------------------------------------------------------- tensors

@dataclass(frozen=True)
class TensorSpec:
    """One tensor a part needs from the model folder.

    ``kind``: "matrix" (operand of a matrix product, kept in the compute type),
    "vector" (norm weights and the like; a tensor stored in 32 bit stays so),
    "table" (embedding rows, kept in the compute type), "int" (integer tables,
    kept as int32).  ``init`` names how random weights are drawn: "normal"
    N(0, 0.02), "norm" 1 + U(-0.1, 0.1), "zeros".
    """
    name: str
    shape: tuple
    kind: str = "matrix"
    init: str = "normal"


PAGE = "page"     # the axis of a page layout that counts the tokens of the page


@dataclass(frozen=True)
class CacheSpec:
    """What a mixer keeps per token, and how far back it reads.

    ``layout`` is the shape of one page of one layer with the token axis written
    as ``PAGE``: keys and values per head are ``(2, kv_heads, PAGE, head_dim)``, one
    latent vector per token is ``(PAGE, width)``, keys and values of different
    widths can be packed as ``(kv_heads, PAGE, k_width + v_width)``.  The cache
    manager allocates ``[layers of the group, pages, *layout]`` with the page size
    in place of ``PAGE`` and knows nothing else about the contents.  Mixers with
    equal specs share a cache group (one pool of pages, one block table per
    request); ``window`` None means every token is kept.  ``chunk`` C: position i reads the positions of its own
    chunk only, i // C == j // C (None: not).  ``run_tokens``: the mixer reads
    a request's pages fastest when the pages of this many consecutive tokens follow one another
    in the pool; the pool then hands pages out in aligned runs of that length where it can
    (0: any order is as good)."""
    layout: tuple
    window: Optional[int] = None
    run_tokens: int = 0
    chunk: Optional[int] = None

    def __post_init__(self):
        if self.window and self.chunk:
            raise ValueError("a cache keeps a window or a chunk of tokens, not both")
        if tuple(self.layout).count(PAGE) != 1:
            raise ValueError(f"a page layout names the token axis once, as PAGE: {self.layout}")
        object.__setattr__(self, "layout", tuple(self.layout))

    def page_shape(self, page_size: int) -> tuple:
        return tuple(page_size if a == PAGE else int(a) for a in self.layout)

    @property
    def reach(self) -> Optional[int]:
        """The most tokens a query reads, its own included (None: all of them)."""
        return self.window or self.chunk or None

    def first_needed(self, new_len: int) -> int:
        """The first position that queries at positions >= ``new_len`` may read."""
        if self.window:      # the next query reads keys > new_len - window
            return max(0, new_len - self.window + 1)
        return new_len // self.chunk * self.chunk if self.chunk else 0

    def describe(self) -> str:
        return ("x".join("P" if a == PAGE else str(a) for a in self.layout) + (f"w{self.window}" if self.window else "")
                + (f"c{self.chunk}" if self.chunk else ""))


@dataclass(frozen=True)
class StateSpec:
    """Per-request state of fixed size, one slot per request slot.  Parts that name
    the same key share the tensor.  ``fill`` is the value a slot is reset to when a
    request is admitted."""
    shape: tuple
    dtype: torch.dtype = torch.float32
    fill: float = 0.0


# ------------------------------------------------------------------ parts

class Part:
    """Anything with weights.  ``prefix`` is the tensor-name prefix in the model folder."""

    def tensor_specs(self) -> list[TensorSpec]:
        return []

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Takes the tensors named by ``tensor_specs`` (on the device, already in
        the type their kind asks for)."""

    def state_specs(self) -> Dict[str, StateSpec]:
        return {}

    def begin_step(self, ctx) -> None:
        """Called once per step before any layer runs."""

    def decode_rows_differ(self) -> bool:
        """True when the part treats a row flagged ``ROW_DECODE`` otherwise than the same
        token inside a prompt portion.  The scheduler then never folds generated tokens
        into a prompt portion: a request that is recomputed feeds them one per step."""
        return False


class Norm(Part):
    """``forward(ctx, x, out=None, add=None, rows=None)``: normalises rows of x [T, d].
    With ``add`` the sum x + add is written back to x first (the residual sum,
    fused); with ``rows`` only those rows are read and the output has len(rows) rows."""

    def forward(self, ctx, x, add=None, rows=None):
        raise NotImplementedError


class PositionEncoding(Part):
    """Position information a mixer applies to its queries and keys.  ``table(device)``
    returns what the mixer's kernel needs (for rotary positions: cos and sin)."""

    def table(self, device):
        raise NotImplementedError


class Mixer(Part):
    """The part of a layer that mixes tokens.  ``cache_spec()`` says what it keeps per
    token (None: nothing); ``forward(ctx, x, cache)`` maps normalised rows x [T, d]
    to [T, d], appending to ``cache`` when ``cache.writes`` and reading from it."""

    def cache_spec(self) -> Optional[CacheSpec]:
        return None

    def forward(self, ctx, x, cache):
        raise NotImplementedError


class RunState:
    """What a mixer with a recurrent state gets for one run of its layer: ``state[name]`` is the tensor
    [slots, *shape] of the state it declared under that name in ``run_state_specs`` (every run of a layer has
    tensors of its own, so a layer that runs several times in a pass keeps one state per run)."""

    def __init__(self, state: Dict[str, torch.Tensor], writes: bool = True):
        self.state = state
        self.writes = writes


class FeedForward(Part):
    """``forward(ctx, x)``: rows [T, d] to rows [T, d], token by token."""

    def forward(self, ctx, x):
        raise NotImplementedError


class TokenInput(Part):
    """What a layer takes from the step's tokens themselves, beside the embedding.  ``forward(ctx, x)`` reads the settled stream x [T, d] in
    the compute type and returns (y, weight, eps): y [T, d] joins the stream through an RMS norm with this float32 weight."""

    def forward(self, ctx, x):
        raise NotImplementedError


class Block(Part):
    """Arrangement of parts around the residual stream.  A block is built from a dict
    of parts, ``{role: part}``; which roles it needs is the block's own business (the
    pre-norm block: norm1, mixer, norm2, feed_forward; another block may take more
    norms, no feed-forward, two mixers).  ``forward(ctx, x, pending, cache)`` takes the
    stream x [T, d] and a not yet added update ``pending`` (or None) and returns the
    same pair."""

    roles: tuple = ()
    optional_roles: tuple = ()      # roles a layer may leave out (their attributes are None then)

    def __init__(self, parts: Dict[str, Part]):
        missing = [r for r in self.roles if r not in parts]
        extra = [r for r in parts if r not in self.roles and r not in self.optional_roles]
        if missing or extra:
            raise ValueError(f"{type(self).__name__} takes the parts {list(self.roles)} and may take {list(self.optional_roles)}; "
                             f"missing {missing}, not taken {extra}")
        self._parts = dict(parts)
        for role in self.optional_roles:
            setattr(self, role, None)
        for role, part in parts.items():
            setattr(self, role, part)

    def parts(self) -> list:
        return list(self._parts.values())

    def cache_spec(self) -> Optional[CacheSpec]:
        """What a run of this block appends to its cache: that of its first part that keeps one."""
        for p in self._parts.values():
            cs = p.cache_spec() if hasattr(p, "cache_spec") else None
            if cs is not None:
                return cs
        return None

    def run_state_specs(self) -> Dict[str, StateSpec]:
        """The per-run state of its parts (see ``Mixer.run_state_specs``)."""
        out: Dict[str, StateSpec] = {}
        for p in self._parts.values():
            if hasattr(p, "run_state_specs"):
                out.update(p.run_state_specs())
        return out

    def forward(self, ctx, x, pending, cache):
        raise NotImplementedError


class Stream(Part):
    """The residual stream of a model: how it starts from the embedding table, what a block hands on as ``pending``
    means, and how it ends in the rows the output matrix reads.

    ``start(ctx, table)`` returns the stream tensor of the step's tokens; ``finish(ctx, x, pending, norm, rows)`` returns
    the normalised rows [len(rows), d] in the compute type; ``total(ctx, x, pending)`` returns the settled stream
    [T, d] in float32 (for inspection: what the layers so far have summed up)."""

    def start(self, ctx, table):
        raise NotImplementedError

    def initial_pending(self):
        """What the first block gets as ``pending`` (None: nothing is pending after ``start``)."""
        return None

    def enter_pass(self, ctx, x, pending, number: int):
        """Called before the first layer of pass ``number`` of a span of layers that runs several times; returns
        (x, pending).  Streams of models without such a span never see it."""
        raise NotImplementedError(f"{type(self).__name__} has nothing to do at the start of a pass")

    def finish(self, ctx, x, pending, norm, rows):
        raise NotImplementedError

    def total(self, ctx, x, pending):
        raise NotImplementedError


# Flags of a row of a step (``RowInput.flags``, ``ctx.row_flags``), for parts to interpret.
ROW_DECODE = 1      # a single token at or after the end of the request's prompt


# -------------------------------------------------------------- registries

class Registry:
    def __init__(self, what: str):
        self.what = what
        self._items: Dict[str, Callable[..., Any]] = {}

    def register(self, name: str):
        def deco(cls):
            if name in self._items and self._items[name] is not cls:
                raise ValueError(f"{self.what} '{name}' is registered already")
            self._items[name] = cls
            return cls
        return deco

    def unregister(self, name: str) -> None:
        self._items.pop(name, None)

    def create(self, kind: str, /, **params):
        if kind not in self._items:
            raise KeyError(f"unknown {self.what} '{kind}'; known: {', '.join(sorted(self._items)) or 'none'}")
        return self._items[kind](**params)

    def names(self) -> list[str]:
        return sorted(self._items)

    def __contains__(self, name: str) -> bool:
        return name in self._items


NORMS = Registry("norm")
POSITION_ENCODINGS = Registry("position encoding")
MIXERS = Registry("mixer")
FEED_FORWARDS = Registry("feed-forward")
BLOCKS = Registry("block")
STREAMS = Registry("residual stream")
STREAM_MIXINGS = Registry("stream mixing")
TOKEN_INPUTS = Registry("token input")


REGISTRIES = {"norm": NORMS, "position": POSITION_ENCODINGS, "mixer": MIXERS, "feed_forward": FEED_FORWARDS,
              "block": BLOCKS, "stream": STREAMS, "stream_mixing": STREAM_MIXINGS, "token_input": TOKEN_INPUTS}


@dataclass(frozen=True)
class PartSpec:
    """Registry name of a part, its parameters, and the registry it is looked up in
    ("norm", "position", "mixer", "feed_forward", "block", "stream", "stream_mixing", "token_input")."""
    kind: str
    params: dict = field(default_factory=dict)
    category: str = ""

    def build(self, registry: Optional[Registry] = None, **extra):
        if registry is None:
            if self.category not in REGISTRIES:
                raise KeyError(f"part '{self.kind}' names no registry (category '{self.category}'); known: {', '.join(REGISTRIES)}")
            registry = REGISTRIES[self.category]
        return registry.create(self.kind, **{**self.params, **extra})
