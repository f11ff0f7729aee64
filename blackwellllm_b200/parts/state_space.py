"""A state-space mixer with one decay per head (Mamba-2): a recurrent mixer with a [state_dim, value_dim] state per head.

    [z | x | B | C | dt] = W_in h                      inner, inner, groups * state_dim, the same, heads; inner = heads * value_dim
    x, B, C <- silu(conv([x | B | C]) + bias)          causal over time, per channel, few taps
    dt <- softplus(dt + dt_bias)     a = exp(-exp(A_log) dt)                           one number each per head
    S <- a S + dt B x^T        y = S^T C + D x                     per head, token by token; B, C of the head's group
    out = W_o (rms_parts(y * silu(z)) * gain)          the root mean square over each of norm_groups equal parts

The state S and the convolution's last inputs are float32, live in the request's slots of the cache manager's fixed-size
state and are carried from step to step.  The projection's results are float32.  Three kernels follow: ``ops.short_conv``
(convolution, bias, silu, and dt with its decay), the recurrence with one decay per head, the keys B times dt, queries C,
heads of a group sharing both (``ops.gla_scan`` token by token in the 32-bit path and in steps of single tokens,
``ops.chunk_scan`` for portions of prompts) and ``ops.ssd_out`` (D x, the gate, the norm of the parts).
Everything but the projections is float32.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..kernels import ops
from .base import BuildContext, FixedStateRequest, Mixer, ParamSpec, register_mixer
from .linear import Linear

_DEFAULT_NAMES = {"in": "in_proj.weight", "conv": "conv1d.weight", "conv_bias": "conv1d.bias", "dt_bias": "dt_bias",
                  "A_log": "A_log", "D": "D", "norm": "norm.weight", "o": "out_proj.weight"}


class StateSpaceMixer(Mixer):
    def __init__(self, spec, hidden_size: int, ctx: BuildContext):
        self.heads, self.dv, self.N = int(spec.num_heads), int(spec.value_dim), int(spec.state_dim)
        self.groups, self.taps, self.parts = int(spec.groups), int(spec.conv_taps), int(spec.norm_groups)
        self.eps = float(spec.norm_eps)
        self.inner = self.heads * self.dv
        if self.heads % self.groups:
            raise ValueError(f"num_heads {self.heads} is not a multiple of groups {self.groups}")
        if self.inner % self.parts:
            raise ValueError(f"the {self.inner} channels of all heads do not divide into {self.parts} parts")
        if self.N > ops.GLA_MAX_KEY_DIM:
            raise ops.KernelError(f"state space: state size {self.N} exceeds the scan's {ops.GLA_MAX_KEY_DIM}")
        self.hidden_size = hidden_size
        self.ctx = ctx
        self.names = dict(_DEFAULT_NAMES)
        self.names.update(dict(getattr(spec, "names", ()) or ()))
        self.GN = self.groups * self.N
        self.C = self.inner + 2 * self.GN                  # channels of the convolution
        self.segments = ((self.heads, self.dv, None), (2 * self.groups, self.N, None))
        self.proj: Linear = None
        self.o: Linear = None
        self.conv = self.conv_bias = self.A = self.dt_bias = self.D = self.gain = None

    def cache_request(self):
        # the state of every head (rows padded to a multiple of four floats), and
        # the convolution's earlier inputs (position p at entry p mod taps)
        return (FixedStateRequest((self.heads, self.N, -(-self.dv // 4) * 4), torch.float32),
                FixedStateRequest((self.taps, self.C), torch.float32))

    def param_specs(self) -> List[ParamSpec]:
        H, n = self.hidden_size, self.names
        return [ParamSpec(n["in"], (self.inner + self.C + self.heads, H)),
                ParamSpec(n["conv"], (self.C, self.taps), role="bias", init="bias_normal"),
                ParamSpec(n["conv_bias"], (self.C,), role="bias", init="bias_normal"),
                ParamSpec(n["dt_bias"], (self.heads,), role="bias", init="bias_normal"),
                ParamSpec(n["A_log"], (self.heads,), role="bias", init="bias_normal"),
                ParamSpec(n["D"], (self.heads,), role="bias", init="ones"),
                ParamSpec(n["norm"], (self.inner,), role="gain", init="ones"),
                ParamSpec(n["o"], (H, self.inner))]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = self.names
        self.proj = Linear(tensors[n["in"]])
        self.o = Linear(tensors[n["o"]])
        self.conv = tensors[n["conv"]].float().t().contiguous()
        self.conv_bias = tensors[n["conv_bias"]].float().contiguous()
        self.A = -torch.exp(tensors[n["A_log"]].float()).contiguous()
        self.dt_bias = tensors[n["dt_bias"]].float().contiguous()
        self.D = tensors[n["D"]].float().contiguous()
        self.gain = tensors[n["norm"]].float().contiguous()

    def input_projection(self):
        return self.proj

    def take_projection(self) -> torch.Tensor:
        w, self.proj = self.proj.weight, None
        return w

    def from_projection(self, proj, batch, cache, owns_cache: bool = True):
        if not owns_cache:
            raise ops.KernelError("state space: a run cannot read another run's state")
        state, inputs = cache
        xbc, a, dt = ops.short_conv(proj[:, self.inner:], self.conv, self.conv_bias, inputs.state, batch, self.segments,
                                    gates=(proj, self.inner + self.C, None, self.A, self.dt_bias))
        rep = self.heads // self.groups
        if self.ctx.dtype == torch.bfloat16 and batch.T > batch.R:      # portions: a chunk of tokens at a time
            y = ops.chunk_scan(False, xbc, self.inner + self.GN, self.inner, 0, a, dt, batch, state.state, self.heads, rep,
                               self.N, self.dv)
        else:
            y = ops.gla_scan(xbc, self.inner + self.GN, self.inner, 0, a, batch, state.state, self.heads, self.N, self.dv, 1.0,
                             k_scale=dt, scalar_decay=True, qk_rep=rep)
        return ops.ssd_out(y, xbc, proj, self.D, self.gain, self.dv, self.parts, self.eps, self.ctx.dtype)

    def forward(self, x, residual, batch, cache, owns_cache: bool = True, accumulate: bool = True) -> None:
        y = self.from_projection(self.proj(x, out_dtype=torch.float32), batch, cache, owns_cache)
        if accumulate:
            self.o.add_to(y, residual)
        elif accumulate is None:
            self.o.write_to(y, residual)
        else:
            self.o(y, out=residual)


register_mixer("state_space", StateSpaceMixer)
