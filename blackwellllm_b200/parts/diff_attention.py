"""Differential attention: two softmax maps over the same values, their difference normed head by head.

    q, k, v = conv(W_q x), conv(W_k x), conv(W_v x)        conv: causal over time, per channel, few taps, no activation
    a1, a2 = softmax(scale q1 k1^T) v, softmax(scale q2 k2^T) v        per head; q = [q1, q2], k = [k1, k2]
    o = a1 - lambda a2        lambda = exp(lq1 . lk1) - exp(lq2 . lk2) + diff, one number for the layer
    y = W_o concat_heads(o / rms(o) * (1 - diff) * sigmoid(W_g x)_head)

No position is encoded; a query may be kept from looking out of its own block of positions (``chunk``).

A key row of the cache is [k1, k2] of one key head, so keys and values are kept once.  The attention kernels see two query heads
per head: the first is [q1, 0], the second [0, q2], and both meet the key row in a plain product; any of the framework's attention
kernels serves.  ``ops.conv_heads`` makes these rows, keys and values in one kernel from the float32 projections (the gate's
columns ride in the same product); the maps become heads in the attention kernels' epilogues (bfloat16) or in
``ops.diff_combine``.

The convolution's earlier inputs live in the request's slot of the cache manager's fixed-size state (position p at entry
p mod taps).  A run that reads another run's keys and values (``shares_kv``) has a query projection and convolution of its own and
keeps the earlier inputs of that one alone.
"""
from __future__ import annotations

import math
from typing import Dict, List

import torch

from ..kernels import ops
from .base import BuildContext, FixedStateRequest, Mixer, PagedKVRequest, ParamSpec, register_mixer
from .linear import Linear

_DEFAULT_NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "o": "o_proj.weight", "g": "g_proj.weight",
                  "q_conv": "q_conv.weight", "k_conv": "k_conv.weight", "v_conv": "v_conv.weight", "lq1": "lambda_q1",
                  "lk1": "lambda_k1", "lq2": "lambda_q2", "lk2": "lambda_k2"}
MAPS = 2


class DifferentialAttention(Mixer):
    def __init__(self, spec, hidden_size: int, ctx: BuildContext):
        self.nh, self.nkv, self.hd, self.dv = int(spec.num_heads), int(spec.num_kv_heads), int(spec.head_dim), int(spec.v_head_dim)
        if self.nh % self.nkv:
            raise ValueError(f"num_heads {self.nh} is not a multiple of num_kv_heads {self.nkv}")
        self.taps, self.chunk = int(spec.conv_taps), spec.chunk
        if self.taps < 1:
            raise ValueError("conv_taps must be at least 1")
        self.diff, self.eps, self.scale = float(spec.diff), float(spec.norm_eps), float(spec.softmax_scale)
        self.gated, self.shares_kv = bool(spec.gate_per_head), bool(spec.shares_kv)
        self.names = dict(_DEFAULT_NAMES)
        self.names.update(dict(spec.names or ()))
        self.hidden_size, self.ctx = hidden_size, ctx
        step = 16 if ctx.dtype == torch.bfloat16 else 2
        self.dpad = -(-max(MAPS * self.hd, self.dv) // step) * step      # a row of the cache
        ops.check_attention_supported(ctx.dtype, self.dpad)
        self.Q, self.K, self.V = self.nh * MAPS * self.hd, self.nkv * MAPS * self.hd, self.nkv * self.dv
        self.C = self.Q if self.shares_kv else self.Q + self.K + self.V  # channels of the convolution
        self.proj: Linear = None
        self.o: Linear = None
        self.conv = self.lam = None

    def cache_request(self):
        return (PagedKVRequest(self.nkv, self.dpad), FixedStateRequest((self.taps, self.C), torch.float32))

    def borrower_request(self):
        return FixedStateRequest((self.taps, self.C), torch.float32) if self.shares_kv else None

    def _branches(self):
        return ("q",) if self.shares_kv else ("q", "k", "v")

    def param_specs(self) -> List[ParamSpec]:
        H, n = self.hidden_size, self.names
        rows = {"q": self.Q, "k": self.K, "v": self.V}
        specs = [ParamSpec(n[r], (rows[r], H)) for r in self._branches()]
        specs += [ParamSpec(n[r + "_conv"], (rows[r], self.taps), role="bias", init="bias_normal") for r in self._branches()]
        specs += [ParamSpec(n[r], (self.hd,), role="bias", init="bias_normal") for r in ("lq1", "lk1", "lq2", "lk2")]
        if self.gated:
            specs.append(ParamSpec(n["g"], (self.nh, H)))
        return specs + [ParamSpec(n["o"], (H, self.nh * self.dv))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = self.names
        w = torch.cat([tensors[n[r]] for r in self._branches()] + ([tensors[n["g"]]] if self.gated else []), dim=0)
        if w.shape[0] % 8:       # zero rows: the result's rows stay 16-byte aligned
            w = torch.cat([w, torch.zeros((-w.shape[0] % 8, w.shape[1]), dtype=w.dtype, device=w.device)])
        self.proj = Linear(w)
        self.conv = torch.cat([tensors[n[r + "_conv"]].float() for r in self._branches()], dim=0).t().contiguous()
        lq1, lk1, lq2, lk2 = (tensors[n[r]].double() for r in ("lq1", "lk1", "lq2", "lk2"))
        lam = math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + self.diff
        self.lam = torch.tensor([lam], dtype=torch.float32, device=w.device)
        wo = tensors[n["o"]]
        if self.dpad != self.dv:      # a head's output has dpad channels; those beyond dv are zeros
            wo = torch.nn.functional.pad(wo.view(wo.shape[0], self.nh, self.dv), (0, self.dpad - self.dv)) \
                .reshape(wo.shape[0], self.nh * self.dpad)
        self.o = Linear(wo)

    def input_projection(self):
        return self.proj

    def take_projection(self) -> torch.Tensor:
        w, self.proj = self.proj.weight, None
        return w

    def from_projection(self, rows, batch, cache, owns_cache: bool = True):
        if owns_cache == self.shares_kv:
            raise ops.KernelError("differential attention: a run with keys of its own owns its cache, one without reads another run's")
        if owns_cache:
            pages, inputs = cache
        else:
            shared, inputs = cache.shared, cache.own
            pages = shared[0] if isinstance(shared, (tuple, list)) else shared
        table = batch.block_tables[pages.group]
        q = ops.conv_heads(rows, self.conv, inputs.state, batch, table, pages.k_pages, pages.v_pages, MAPS * self.nh, self.hd, MAPS,
                           self.nkv, self.dv, has_kv=owns_cache)
        gate = (rows[:, self.C:self.C + self.nh], self.dv, "head") if self.gated else None
        return ops.paged_attention(q, pages.k_pages, pages.v_pages, batch, table, MAPS * self.nh, None, self.scale, self.chunk,
                                   gate=gate, diff=(self.lam, self.eps, 1.0 - self.diff, self.dv))

    def forward(self, x, residual, batch, cache, owns_cache: bool = True, accumulate: bool = True) -> None:
        y = self.from_projection(self.proj(x, out_dtype=torch.float32), batch, cache, owns_cache)
        if accumulate:
            self.o.add_to(y, residual)
        elif accumulate is None:
            self.o.write_to(y, residual)
        else:
            self.o(y, out=residual)


register_mixer("differential_attention", DifferentialAttention)
