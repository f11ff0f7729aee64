"""Interfaces of the parts a decoder is put together from, and their registries.

A part is built from its spec (``config.specs``) and the model's hidden size, says
which tensors it wants (:meth:`Part.param_specs`), receives them
(:meth:`Part.bind`) and then runs on the step's batch.  No part knows which model
it is in: sizes and constants come from the spec alone.

Interfaces
----------
Norm            ``forward(x_f32[T,H], rows=None) -> [n,H]`` in the compute dtype.
PositionEncoding ``rotate_append(qkv, batch, cache, nh, nkv, hd) -> q``: encodes the
                position into queries and keys and appends keys and values to
                the cache pages of the tokens' positions.
Mixer           ``cache_request()`` says what cache it needs (paged keys/values,
                a fixed-size state per request, or nothing);
                ``forward(x, residual, batch, cache, owns_cache)`` adds its output
                to ``residual`` (float32 [T,H]) in place; ``owns_cache`` is false
                when this run reads the cache of another run and must not write it.
                Mixers and feed-forwards that take ``accumulate=False`` WRITE their output to
                ``residual`` instead (a block that norms the output before adding it needs that);
                ``accumulate=None`` writes too, and may leave the last product's sum open
                (``Linear.write_to``) for a reader that takes open sums (the hyper block's kernel).
FeedForward     ``forward(x, residual, batch)`` adds its output to ``residual``.
Block           ``forward(residual, batch, cache)`` arranges norms, mixer and
                feed-forward.

Registering: ``register_mixer("kind", Class)`` (and ``register_ffn``,
``register_norm``, ``register_position``, ``register_block``); ``Class(spec,
hidden_size, ctx)`` builds it.  The spec is any object with a ``kind`` attribute.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Callable, Dict, List, Optional, Tuple

import torch


@dataclass(frozen=True)
class ParamSpec:
    """One tensor a part wants, named relative to the part's prefix.

    role: ``"matrix"`` (operand of a matrix product or an embedding table: held in
    the compute dtype), ``"gain"`` / ``"bias"`` (vectors: a 32-bit stored tensor
    stays 32-bit), ``"int_table"`` (held as int32).  ``init``: how the
    random-weights mode fills it (``"normal"``, ``"ones"``, ``"bias_normal"``,
    ``"zeros"``).  A size of -1 in ``shape`` is taken from the stored tensor (a size that the
    configuration does not state); the random-weights mode cannot fill such a tensor.
    """
    name: str
    shape: Tuple[int, ...]
    role: str = "matrix"
    init: str = "normal"
    optional: bool = False


@dataclass(frozen=True)
class BuildContext:
    device: torch.device
    dtype: torch.dtype  # torch.float32 (true 32-bit path) or torch.bfloat16


@dataclass(frozen=True)
class PagedKVRequest:
    """A mixer's need for paged keys and values: per token ``2 * num_kv_heads *
    head_dim`` elements; ``window``: only that many latest tokens stay needed, and with ``keep_first`` the
    first so many tokens of a request as well.  ``single_plane``: keys and values are the same rows (a mixer
    whose values are a part of its key rows): one plane is kept and both views show it."""
    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    keep_first: int = 0
    single_plane: bool = False


@dataclass(frozen=True)
class FixedStateRequest:
    """A mixer's need for a state of fixed size per request (zeroed at admission)."""
    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class BorrowedCache:
    """The cache view of a run that reads another run's cache and keeps something itself."""
    shared: Any    # the other run's view
    own: Any       # what the run asked for with ``borrower_request``


def flatten_cache_requests(request) -> tuple:
    """A run's cache request as a tuple of single needs: a run may ask for several things at once (pages for its
    mixer and a state for the block around it) by returning a tuple; None: nothing."""
    if request is None:
        return ()
    if isinstance(request, (tuple, list)):
        return tuple(r for r in request if r is not None)
    return (request,)


class Part:
    def param_specs(self) -> List[ParamSpec]:
        return []

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Receives the tensors named by :meth:`param_specs` (device, final dtype)."""


class Norm(Part):
    # True: forward() reads x only through ops.rmsnorm, which adds a sum that a matrix product left
    # outstanding for x (ops.gemm_tc_deferred) while it normalises.  False: whoever calls forward()
    # calls ops.resolve_pending() first.
    adds_pending = False

    def forward(self, x: torch.Tensor, rows: Optional[torch.Tensor] = None) -> torch.Tensor:
        raise NotImplementedError


class PositionEncoding(Part):
    def rotate_append(self, qkv, batch, cache, nh: int, nkv: int, hd: int, append: bool = True) -> torch.Tensor:
        """qkv [T, (nh + 2 nkv) * hd] float32 -> encoded queries [T, nh * hd]; encoded keys and raw
        values are written to the cache when ``append``."""
        raise NotImplementedError

    def norm_rotate_append(self, qkv, batch, cache, nh: int, nkv: int, dq: int, dv: int, q_gain, k_gain, eps: float,
                           append: bool = True, per_head: bool = False, q_temp=None, has_kv: bool = True,
                           v_eps: float = 0.0, v_mix=None, q_head_mult=None, kv_shared: bool = False,
                           v_scale: float = 1.0) -> torch.Tensor:
        """The general form of :meth:`rotate_append`: qkv [T, nh*dq + nkv*dq + nkv*dv] float32; with gains,
        all query channels of a token (and all its key channels) are RMS-normed together first; the cache's
        head size may exceed dq and dv (the rest is written as zeros).  ``per_head``: every head is normed by
        itself (gains of dq entries, shared by the heads) and qkv may have further columns, which are left
        alone; ``q_temp`` (coef, every): the queries are multiplied by 1 + coef log(1 + n), n the whole periods of ``every`` positions in p + 1;
        ``has_kv=False``: qkv holds queries only and nothing is appended; ``v_eps`` > 0: every value head is divided
        by sqrt(mean(v^2) + v_eps) before it is written; ``v_mix`` = (v_first float32 [T, nkv * dv], lam: one float32 number
        on the device): the values are written as (1 - lam) v + lam v_first (``per_head`` only).  Also ``per_head`` only: ``q_head_mult`` (float32
        [nh]) multiplies every query head by its own number; ``kv_shared``: qkv holds no values, the key projection before
        norm and rotation is written as the values; ``v_scale`` multiplies the values as they are written."""
        raise NotImplementedError

    def fuse_projection(self, weight: torch.Tensor, bias: Optional[torch.Tensor], nh: int, nkv: int, hd: int):
        """Optional: an encoding that can run inside the q/k/v projection returns a callable
        ``project(x, batch, cache, append) -> queries`` that replaces projection plus
        :meth:`rotate_append` (it may keep its own copy of ``weight`` and ``bias`` in another
        row order).  None: the mixer projects and calls :meth:`rotate_append`."""
        return None


class Mixer(Part):
    graph_safe = True  # False: forward() does host work between kernels; decode steps then run uncaptured

    def cache_request(self):
        return None

    def forward(self, x, residual, batch, cache, owns_cache: bool = True) -> None:
        raise NotImplementedError

    # A mixer that can stand beside another one on the same input (``parts/side_by_side.py``) also offers
    #   input_projection()   the Linear that makes everything it reads of its input in one product (None: it has none),
    #   take_projection()    hands that Linear's weight over: a wider product makes its rows from now on,
    #   from_projection(proj, batch, cache, owns_cache)   from those rows (float32) to what its output projection ``o`` reads.

    def borrower_request(self):
        """What a run that reads another run's cache (``ScheduleEntry.cache_of``) still keeps of its own; None: nothing.  With
        something of its own, the run's cache view is a :class:`BorrowedCache`."""
        return None


class FeedForward(Part):
    def forward(self, x, residual, batch) -> None:
        raise NotImplementedError


class Block(Part):
    mixer: Mixer
    # True: forward() may be entered, and may return, with a sum outstanding for the residual stream
    # (ops.gemm_tc_deferred) and sees to it that no part reads the stream before the sum is made.
    takes_pending = False

    def cache_request(self):
        """What a run of this block owns in the cache manager: the mixer's need, or a tuple of needs when the block
        keeps something of its own per request (the run's cache view is then a tuple in the same order)."""
        return self.mixer.cache_request()

    def borrower_request(self):
        """What a run of this block still owns when it reads another run's cache (see :class:`BorrowedCache`)."""
        fn = getattr(self.mixer, "borrower_request", None)
        return fn() if fn is not None else None

    def forward(self, residual, batch, cache, owns_cache: bool = True) -> None:
        raise NotImplementedError


_REG: Dict[str, Dict[str, Callable[..., Any]]] = {
    "mixer": {}, "ffn": {}, "norm": {}, "position": {}, "block": {}}


def _register(family: str, kind: str, cls) -> None:
    _REG[family][kind] = cls


def register_mixer(kind: str, cls): _register("mixer", kind, cls)
def register_ffn(kind: str, cls): _register("ffn", kind, cls)
def register_norm(kind: str, cls): _register("norm", kind, cls)
def register_position(kind: str, cls): _register("position", kind, cls)
def register_block(kind: str, cls): _register("block", kind, cls)


def _build(family: str, spec, *args):
    kind = getattr(spec, "kind", None)
    table = _REG[family]
    if kind not in table:
        raise KeyError(f"no {family} registered for kind {kind!r}; registered: {sorted(table)}")
    return table[kind](spec, *args)


def build_mixer(spec, hidden_size: int, ctx: BuildContext) -> Mixer:
    return _build("mixer", spec, hidden_size, ctx)


def build_ffn(spec, hidden_size: int, ctx: BuildContext) -> FeedForward:
    return _build("ffn", spec, hidden_size, ctx)


def build_norm(spec, hidden_size: int, ctx: BuildContext) -> Norm:
    return _build("norm", spec, hidden_size, ctx)


def build_position(spec, head_dim: int, ctx: BuildContext) -> PositionEncoding:
    return _build("position", spec, head_dim, ctx)


def build_block(layer_spec, hidden_size: int, ctx: BuildContext) -> Block:
    table = _REG["block"]
    if layer_spec.block not in table:
        raise KeyError(f"no block registered for arrangement {layer_spec.block!r}; registered: {sorted(table)}")
    return table[layer_spec.block](layer_spec, hidden_size, ctx)
