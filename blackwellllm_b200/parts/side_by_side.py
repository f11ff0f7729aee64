"""Two mixers side by side: both read the same input, their outputs become one.

``combine`` "sum": ``left(h) + right(h)`` (a factor on either is the child's own constant).  "norm_mean":
``(rms(left(h)) * gl + rms(right(h)) * gr) / 2``, the norms over the model's width, each with a gain.

The children are mixers of any registered kind, built from their own specs; each keeps its own needs in the cache manager
(pages, states) and its own kernels.  What they read of the input is ONE product: the rows of both projections are joined
at load (padded with zero rows to a multiple of eight, so that the result's rows stay 16-byte aligned), and each child gets
its range of columns.  A sum is two output products into the same tensor; of a mean of two norms the two outputs stay apart
(``ops.NormedPair``) for a block that norms a sublayer's output anyway (:meth:`forward_open`), so that its kernel reads
each of them once.  For a few tokens either product leaves its K splits to that reader.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..kernels import ops
from .base import BuildContext, Mixer, ParamSpec, build_mixer, flatten_cache_requests, register_mixer
from .linear import Linear


class SideBySide(Mixer):
    def __init__(self, spec, hidden_size: int, ctx: BuildContext):
        if spec.combine not in ("sum", "norm_mean"):
            raise ValueError(f"combine must be 'sum' or 'norm_mean', got {spec.combine!r}")
        self.children = [build_mixer(s, hidden_size, ctx) for s in (spec.left, spec.right)]
        self.prefixes = tuple(spec.prefixes)
        self.norm_mean = spec.combine == "norm_mean"
        self.norm_names, self.eps = tuple(spec.out_norms), float(spec.norm_eps)
        self.graph_safe = all(getattr(c, "graph_safe", True) for c in self.children)
        self.hidden_size = hidden_size
        self.ctx = ctx
        self.proj: Linear = None      # both children's projections, where both have one
        self.columns = None           # each child's range of its result's columns
        self.gains = None
        # which of the run's cache views belong to which child
        needs = [flatten_cache_requests(c.cache_request()) for c in self.children]
        self._needs, self._tuples = needs, [isinstance(c.cache_request(), (tuple, list)) for c in self.children]

    def cache_request(self):
        return tuple(self._needs[0]) + tuple(self._needs[1])

    def _views(self, cache):
        n = len(self._needs[0])
        out = []
        for part, as_tuple in zip((cache[:n], cache[n:]), self._tuples):
            out.append(part if as_tuple else (part[0] if part else None))
        return out

    def param_specs(self) -> List[ParamSpec]:
        out = [ParamSpec(prefix + p.name, p.shape, p.role, p.init, p.optional)
               for prefix, child in zip(self.prefixes, self.children) for p in child.param_specs()]
        if self.norm_mean:
            out += [ParamSpec(n, (self.hidden_size,), role="gain", init="ones") for n in self.norm_names]
        return out

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        for prefix, child in zip(self.prefixes, self.children):
            child.bind({k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)})
        if self.norm_mean:
            self.gains = [tensors[n].float().contiguous() for n in self.norm_names]
        if all(getattr(c, "input_projection", lambda: None)() is not None for c in self.children):
            left, right = (c.take_projection() for c in self.children)
            a, b = left.shape[0], right.shape[0]
            pad = torch.zeros((-(a + b) % 8, left.shape[1]), dtype=left.dtype, device=left.device)
            self.proj = Linear(torch.cat([left, right, pad], dim=0))
            self.columns = ((0, a), (a, a + b))

    def _read(self, x, batch, cache, owns_cache):
        """What the two output projections read (only where the children's projections are joined)."""
        rows = self.proj(x, out_dtype=torch.float32)
        return [c.from_projection(rows[:, lo:hi], batch, view, owns_cache)
                for c, (lo, hi), view in zip(self.children, self.columns, self._views(cache))]

    def forward_open(self, x, batch, cache, owns_cache: bool = True):
        """The mixer's output for a reader of its own (``ops.row_step``): a float32 tensor [T, hidden], whose last product may
        still be open, or the pair of outputs whose norms' mean it is."""
        out = torch.empty((x.shape[0], self.hidden_size), dtype=torch.float32, device=x.device)
        if not self.norm_mean:
            self.forward(x, out, batch, cache, owns_cache, accumulate=None)
            return out
        other = torch.empty_like(out)
        if self.proj is None:
            for child, view, o in zip(self.children, self._views(cache), (out, other)):
                child.forward(x, o, batch, view, owns_cache, accumulate=False)
            return ops.NormedPair(out, self.gains[0], other, self.gains[1], self.eps)
        left, right = self._read(x, batch, cache, owns_cache)
        y = self.children[0].o.planes(left)
        if y is None:
            y = out
            self.children[0].o(left, out=out)
        z = self.children[1].o.planes(right, behind=y if y.dim() == 3 else None)
        if z is None:
            if y.dim() == 3:       # no room behind the first one's planes: nothing may be written over them
                self.children[0].o(left, out=out)
                y = out
            z = other
            self.children[1].o(right, out=other)
        return ops.NormedPair(y, self.gains[0], z, self.gains[1], self.eps)

    def forward(self, x, residual, batch, cache, owns_cache: bool = True, accumulate: bool = True) -> None:
        if self.norm_mean:
            pair = self.forward_open(x, batch, cache, owns_cache)
            if not accumulate:
                residual.zero_()
            ops.row_step(residual, pair)
            return
        if self.proj is None:
            for k, (child, view) in enumerate(zip(self.children, self._views(cache))):
                child.forward(x, residual, batch, view, owns_cache, accumulate=True if k else accumulate)
            return
        left, right = self._read(x, batch, cache, owns_cache)
        if accumulate:
            self.children[0].o.add_to(left, residual)
        elif accumulate is None:
            self.children[0].o.write_to(left, residual)
        else:
            self.children[0].o(left, out=residual)
        if accumulate is False:
            self.children[1].o(right, out=residual, accumulate=True)
        else:
            self.children[1].o.add_to(right, residual)


register_mixer("side_by_side", SideBySide)
