"""Interfaces of the parts a model is put together from.

A part is built from the parameters of its :class:`PartSpec` plus the build
context (device, storage dtype, checkpoint prefix).  It declares its tensors
as :class:`ParamSpec` (checkpoint names, shapes, packing), what cache it needs,
and runs on the tensors of one step.  No part knows the model it is in.

Kinds of parts and what each must offer
---------------------------------------
norm            ``forward(x) -> y`` and ``add(x, residual) -> (y, new_residual)``,
                optionally ``add_rows(x, residual, rows) -> y`` on chosen rows.  A norm
                that is y = x * rsqrt(mean(x^2) + eps) * weight with attributes
                ``weight`` [width] and ``eps`` may set ``folds_into_product = True``:
                a projection right behind it may then apply it inside its own kernel
position        built by the mixer that names it in its spec; ``finalize()`` makes its
                tables.  One whose tables the fused q/k kernels are to apply has
                float32 ``cos`` and ``sin`` [positions, head_dim / 2] and declares
                ``pairing = "half_split"``; any other pairing is refused by those
                kernels with a clear error (it needs a kernel, or a mixer, of its own)
mixer           ``cache_need() -> KVNeed | StateNeed | tuple of them | None`` and
                ``forward(x, ctx, run) -> y`` where ``ctx`` is the step's
                :class:`StepContext` and ``run`` the index in the run list;
                optionally ``forward_normed(hidden, residual, norm, ctx, run)
                -> (y, new_residual)`` (takes its pre-norm into its first
                projection; ``hidden`` is None when the part before added its
                output to the residual itself, and ``y`` may be None for the
                same reason), ``streamed_weights()`` (the large weights in the
                order a step reads them), ``takes_tensor_memory_tiles(page_size)``
                and ``scratch_floats(rows, chunks) -> int`` (float32 scratch its
                kernels may ask of ``ctx.workspace`` for a step of ``rows`` single
                tokens whose keys are cut into ``chunks`` chunks; it is set aside
                before decode steps are captured as graphs)
feed_forward    ``forward(x, ctx) -> y``, optionally ``forward_normed`` and
                ``streamed_weights`` as above
block           ``forward(hidden, residual, ctx, run) -> (hidden, residual)``;
                ``residual`` is None for the first block, ``hidden`` is None
                (on the way in or out) when it is in the residual already.
                The engine asks the block, never its insides: ``cache_need()``
                (one per run of the block), ``takes_tensor_memory_tiles(page_size)``
                and ``scratch_floats(rows, chunks)``; :class:`Block` answers them
                from an attribute ``mixer``, a block arranged otherwise answers
                them itself
embedding       ``forward(token_ids) -> hidden``, or ``forward_step(ctx) -> hidden`` where
                more of the step is needed than its tokens; optionally ``state_need()
                -> StateNeed`` for what it carries from token to token of a request
                (``ctx.storage.state_of(parts.base.EMBEDDING)``)
head            ``forward(hidden_rows) -> logits`` (float32)
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable

import torch


@dataclass(frozen=True)
class ParamSource:
    """One checkpoint tensor and the rows of the destination it fills; with ``cols`` it fills
    only the columns ``col_start .. col_start + cols`` of those rows (weights packed side by
    side along their input axis)."""

    name: str
    row_start: int
    rows: int
    col_start: int = 0
    cols: int | None = None


@dataclass(frozen=True)
class ParamSpec:
    """One device tensor of a part.

    ``sources`` lists the checkpoint tensors that are packed along the first
    dimension.  ``role``: "matrix" and "table" tensors take the storage dtype;
    a "vector" that the file stores in 32-bit stays in 32-bit; "integer"
    tensors become int32; a "scalar" is stored without a shape and bound as one element.
    ``init`` is the law of the random-weights mode: "normal" draws N(0, 0.02), "around_one"
    draws 1 + U(-0.1, 0.1), "unit_interval" draws U(0, 1), "even" draws 1 / n + N(0, 0.02) with n the first dimension.
    """

    attr: str
    shape: tuple[int, ...]
    sources: tuple[ParamSource, ...]
    role: str = "matrix"
    init: str = "normal"
    optional: bool = False        # a checkpoint may lack it: the part is then bound None (random weights draw none)
    free_rows: bool = False       # the checkpoint decides the first dimension (one source); ``shape[0]`` is only
                                  # what random weights are drawn with, and the part reads the size off the tensor
    free_cols: bool = False       # the same for the last dimension of a matrix

    @staticmethod
    def single(attr: str, name: str, shape: tuple[int, ...], *, role: str = "matrix",
               init: str = "normal", optional: bool = False, free_rows: bool = False,
               free_cols: bool = False) -> "ParamSpec":
        return ParamSpec(attr, shape, (ParamSource(name, 0, shape[0]),), role, init, optional, free_rows, free_cols)

    @staticmethod
    def scalar(attr: str, name: str, *, init: str = "unit_interval") -> "ParamSpec":
        return ParamSpec(attr, (1,), (ParamSource(name, 0, 1),), "scalar", init)

    @staticmethod
    def side_by_side(attr: str, rows: int, names_cols: list[tuple[str, int]]) -> "ParamSpec":
        """[rows, sum of cols]: every source fills its own columns of all rows."""
        sources, start = [], 0
        for name, cols in names_cols:
            sources.append(ParamSource(name, 0, rows, start, cols))
            start += cols
        return ParamSpec(attr, (rows, start), tuple(sources))

    @staticmethod
    def packed(attr: str, names_rows: list[tuple[str, int]], cols: int) -> "ParamSpec":
        sources, start = [], 0
        for name, rows in names_rows:
            sources.append(ParamSource(name, start, rows))
            start += rows
        return ParamSpec(attr, (start, cols), tuple(sources))


@dataclass(frozen=True)
class KVNeed:
    """A growing cache of keys and values, ``window`` keys long if given.  ``value_dim``: the size
    of a value where it differs from that of a key (``head_dim``).  ``keep_first``: a windowed
    cache never lets go of its first so many tokens (queries keep seeing them).  ``value_offset``:
    the value is not stored apart but is the ``value_dim`` elements from there on of the key's row
    (attention over a latent that serves as key and value at once): the cache holds no value pages."""

    num_kv_heads: int
    head_dim: int
    window: int | None = None
    value_dim: int | None = None
    keep_first: int = 0
    value_offset: int | None = None

    @property
    def value_size(self) -> int:
        return self.head_dim if self.value_dim is None else self.value_dim

    def geometry(self) -> tuple:
        """What two runs must agree on to share pages and block tables."""
        return (self.num_kv_heads, self.head_dim, self.value_size, self.window,
                self.keep_first if self.window is not None else 0, self.value_offset)


@dataclass(frozen=True)
class StateNeed:
    """Per-request state of fixed size, zero when a request starts.  A mixer with several states (or with a
    state beside pages of keys and values) declares a tuple of needs and tells its states apart by ``name``:
    ``storage.state_of(run, name)``."""

    shape: tuple[int, ...]
    dtype: torch.dtype = torch.float32
    name: str = ""


EMBEDDING = "embedding"           # the storage key of an embedding's state, in place of a run's index


def kv_need(need) -> KVNeed | None:
    """The growing cache among what a run declares (a need, a tuple of needs or None)."""
    found = [n for n in (need if isinstance(need, tuple) else (need,)) if isinstance(n, KVNeed)]
    if len(found) > 1:
        raise ValueError("a run keeps one cache of keys and values")
    return found[0] if found else None


def state_needs(need) -> tuple[StateNeed, ...]:
    """The fixed-size states among what a run declares."""
    found = tuple(n for n in (need if isinstance(need, tuple) else (need,)) if isinstance(n, StateNeed))
    if len({n.name for n in found}) != len(found):
        raise ValueError("the states of a run need names of their own")
    return found


@dataclass
class BuildContext:
    """What every part constructor receives besides its own parameters."""

    device: torch.device
    dtype: torch.dtype          # storage dtype: torch.bfloat16 or torch.float32
    prefix: str = ""            # checkpoint prefix of the layer, "" for top-level parts
    build: Callable[..., Any] | None = None   # build(kind_group, PartSpec, ctx) for nested parts

    def child(self, name: str) -> "BuildContext":
        prefix = f"{self.prefix}.{name}" if self.prefix else name
        return BuildContext(self.device, self.dtype, prefix, self.build)


class Part:
    """Base of all parts: tensors by declaration, nested parts by listing."""

    def param_specs(self) -> list[ParamSpec]:
        return []

    def children(self) -> list["Part"]:
        return []

    def bind(self, attr: str, tensor: torch.Tensor) -> None:
        setattr(self, attr, tensor)

    def all_parts(self) -> list["Part"]:
        found = [self]
        for child in self.children():
            found.extend(child.all_parts())
        return found


class Block(Part):
    """Base of block arrangements.  The engine talks to a block only through these methods and
    ``forward``; the defaults pass the questions on to ``self.mixer``."""

    mixer = None

    def cache_need(self):
        """What one run of this block needs of the cache: KVNeed, StateNeed, a tuple of them or None."""
        return self.mixer.cache_need() if self.mixer is not None else None

    def takes_tensor_memory_tiles(self, page_size: int) -> bool:
        """Whether prompt portions of this block may be cut into the tile lists of the
        tensor-memory attention kernel (a block without attention does not care: True)."""
        if self.mixer is None:
            return True
        asked = getattr(self.mixer, "takes_tensor_memory_tiles", None)
        return bool(asked(page_size)) if asked is not None else False

    def scratch_floats(self, rows: int, chunks: int) -> int:
        asked = getattr(self.mixer, "scratch_floats", None) if self.mixer is not None else None
        return int(asked(rows, chunks)) if asked is not None else 0
