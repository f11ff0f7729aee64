"""The gated delta rule: a recurrent mixer whose memory is a [key_dim, value_dim] matrix per head.

    q, k, v = silu(conv(W_q x)), silu(conv(W_k x)), silu(conv(W_v x))      conv: causal over time, per channel, few taps
    q <- q / |q| / sqrt(key_dim)     k <- k / |k|                          per head, |x| = sqrt(sum(x^2) + 1e-6)
    beta = sigmoid(W_b x)     g = exp(-exp(A_log) softplus(W_a x + dt_bias))        one number each per head
    S <- g S        u = beta (v - S^T k)        S <- S + k u^T        o = S^T q       per head, token by token
    y = W_o (concat_heads(o / rms(o) * gain * silu(W_g x)))

Options: ``channel_decay``, one decay per head and KEY CHANNEL, g = exp(-exp(A_log) softplus(W_a2 (W_a1 x) + dt_bias)), each acting on
its row of S; ``lowrank_gate``, the output gate sigmoid(W_g2 (W_g1 x)).  The first halves ride in the joined projection, the second
halves with what is made of them are one kernel (``ops.lowrank_gates``).

Queries and keys may have fewer heads than values (head h uses number floor(h / (heads / kv_heads))).  The state S and the
convolution's last inputs are float32, live in the request's slots of the cache manager's fixed-size state and are carried
from step to step.  q, k, v, b, a (or the first halves) and the output gate's projection are one matrix made at load; its results
are float32.
Three kernels follow: ``ops.short_conv`` (convolution, silu, unit norms, and the two gates), the recurrence
(``ops.delta_scan`` token by token in the 32-bit path and in steps of single tokens, ``ops.chunk_scan`` for portions of
prompts) and ``ops.gla_gate`` (head norm, gain, gate).  A constant on the output rides in the gain.  Everything but the
projections is float32.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..kernels import ops
from .base import BuildContext, FixedStateRequest, Mixer, ParamSpec, register_mixer
from .linear import Linear

_DEFAULT_NAMES = {"q": "q_proj.weight", "k": "k_proj.weight", "v": "v_proj.weight", "g": "g_proj.weight", "b": "b_proj.weight",
                  "a": "a_proj.weight", "a1": "a_proj.0.weight", "a2": "a_proj.1.weight", "g1": "g_proj.0.weight",
                  "g2": "g_proj.1.weight", "o": "o_proj.weight", "norm": "o_norm.weight", "q_conv": "q_conv.weight",
                  "k_conv": "k_conv.weight", "v_conv": "v_conv.weight", "A_log": "A_log", "dt_bias": "dt_bias"}

UNIT_EPS = 1e-6   # under the root of a query's or key's sum of squares


class GatedDeltaRule(Mixer):
    def __init__(self, spec, hidden_size: int, ctx: BuildContext):
        self.heads, self.kv_heads = int(spec.num_heads), int(spec.num_kv_heads)
        self.dk, self.dv, self.taps = int(spec.key_dim), int(spec.value_dim), int(spec.conv_taps)
        self.eps, self.scale = float(spec.norm_eps), float(getattr(spec, "output_scale", 1.0))
        if self.heads % self.kv_heads:
            raise ValueError(f"num_heads {self.heads} is not a multiple of num_kv_heads {self.kv_heads}")
        if self.dk > ops.DELTA_MAX_KEY_DIM:
            raise ops.KernelError(f"gated delta rule: key size {self.dk} exceeds the scan's {ops.DELTA_MAX_KEY_DIM}")
        self.channel_decay = bool(getattr(spec, "channel_decay", False))
        self.lowrank_gate = bool(getattr(spec, "lowrank_gate", False))
        self.ranks = (getattr(spec, "decay_rank", None), getattr(spec, "gate_rank", None))
        self.hidden_size = hidden_size
        self.ctx = ctx
        self.names = dict(_DEFAULT_NAMES)
        self.names.update(dict(getattr(spec, "names", ()) or ()))
        self.K, self.V = self.kv_heads * self.dk, self.heads * self.dv
        self.C = 2 * self.K + self.V                       # channels of the convolution
        self.segments = ((self.kv_heads, self.dk, self.dk ** -0.5), (self.kv_heads, self.dk, 1.0), (self.heads, self.dv, None))
        self.proj: Linear = None
        self.o: Linear = None
        self.conv = self.A = self.dt_bias = self.gain = None
        self.a2 = self.g2 = None
        self.columns: Dict[str, int] = {}      # where each part's columns begin in the projection's rows

    def cache_request(self):
        # the memory of every head, and the convolution's earlier inputs (position p at entry p mod taps)
        return (FixedStateRequest((self.heads, self.dk, self.dv), torch.float32),
                FixedStateRequest((self.taps, self.C), torch.float32))

    def param_specs(self) -> List[ParamSpec]:
        H, n = self.hidden_size, self.names
        ra, rg = (-1 if r is None else int(r) for r in self.ranks)
        decay = [ParamSpec(n["a1"], (ra, H)), ParamSpec(n["a2"], (self.heads * self.dk, ra))] if self.channel_decay \
            else [ParamSpec(n["a"], (self.heads, H))]
        gate = [ParamSpec(n["g1"], (rg, H)), ParamSpec(n["g2"], (self.V, rg))] if self.lowrank_gate else [ParamSpec(n["g"], (self.V, H))]
        return decay + gate + [
                ParamSpec(n["q"], (self.K, H)), ParamSpec(n["k"], (self.K, H)), ParamSpec(n["v"], (self.V, H)),
                ParamSpec(n["q_conv"], (self.K, self.taps), role="bias", init="bias_normal"),
                ParamSpec(n["k_conv"], (self.K, self.taps), role="bias", init="bias_normal"),
                ParamSpec(n["v_conv"], (self.V, self.taps), role="bias", init="bias_normal"),
                ParamSpec(n["b"], (self.heads, H)),
                ParamSpec(n["A_log"], (self.heads,), role="bias", init="bias_normal"),
                ParamSpec(n["dt_bias"], (self.heads * (self.dk if self.channel_decay else 1),), role="bias", init="bias_normal"),
                ParamSpec(n["o"], (H, self.V)),
                ParamSpec(n["norm"], (self.dv,), role="gain", init="ones")]

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        n = self.names
        parts = ["q", "k", "v"] + (["a1"] if self.channel_decay else []) + (["g1"] if self.lowrank_gate else ["g"]) + ["b"] \
            + ([] if self.channel_decay else ["a"])
        at = 0
        for r in parts:
            self.columns[r] = at
            at += tensors[n[r]].shape[0]
        self.proj = Linear(torch.cat([tensors[n[r]] for r in parts], dim=0))
        if self.channel_decay:
            self.a2 = tensors[n["a2"]].contiguous()
        if self.lowrank_gate:
            self.g2 = tensors[n["g2"]].contiguous()
        for first, second in (("a1", self.a2), ("g1", self.g2)):
            if second is not None and second.shape[1] != tensors[n[first]].shape[0]:
                raise ValueError(f"gated delta rule: {n[first]} has {tensors[n[first]].shape[0]} rows, its second half {second.shape[1]} columns")
        self.o = Linear(tensors[n["o"]])
        self.conv = torch.cat([tensors[n[r]].float() for r in ("q_conv", "k_conv", "v_conv")], dim=0).t().contiguous()
        self.A = -torch.exp(tensors[n["A_log"]].float()).contiguous()
        self.dt_bias = tensors[n["dt_bias"]].float().contiguous()
        self.gain = (tensors[n["norm"]].float() * self.scale).contiguous()

    def input_projection(self):
        return self.proj

    def take_projection(self) -> torch.Tensor:
        w, self.proj = self.proj.weight, None
        return w

    def from_projection(self, proj, batch, cache, owns_cache: bool = True):
        if not owns_cache:
            raise ops.KernelError("gated delta rule: a run cannot read another run's state")
        memory, inputs = cache
        at = self.columns
        gates = (proj, None, at["b"], self.heads, None) if self.channel_decay else (proj, at["a"], at["b"], self.A, self.dt_bias)
        qkv, g, beta = ops.short_conv(proj, self.conv, None, inputs.state, batch, self.segments, UNIT_EPS, gates=gates)
        gate, gate_off = (None, 0) if self.lowrank_gate else (proj, at["g"])
        second = []                                  # the second halves of what goes through a small inner size
        if self.channel_decay:
            second.append((at["a1"], self.a2, ops.LOWRANK_DECAY, self.A, self.dt_bias))
        if self.lowrank_gate:
            second.append((at["g1"], self.g2, ops.LOWRANK_SIGMOID, None, None))
        if second:
            made = ops.lowrank_gates(proj, second)
            g = made[0] if self.channel_decay else g
            gate = made[-1] if self.lowrank_gate else gate
        rep = self.heads // self.kv_heads
        if self.ctx.dtype == torch.bfloat16 and batch.T > batch.R:      # portions: a chunk of tokens at a time
            o = ops.chunk_scan(True, qkv, 0, self.K, 2 * self.K, g, beta, batch, memory.state, self.heads, rep, self.dk, self.dv)
        else:
            o = ops.delta_scan(qkv, 0, self.K, 2 * self.K, g, beta, batch, memory.state, self.heads, rep, self.dk, self.dv)
        return ops.gla_gate(o, gate, gate_off, self.gain, self.heads, self.dv, self.eps, self.ctx.dtype, ready=self.lowrank_gate)

    def forward(self, x, residual, batch, cache, owns_cache: bool = True, accumulate: bool = True) -> None:
        y = self.from_projection(self.proj(x, out_dtype=torch.float32), batch, cache, owns_cache)
        if accumulate:
            self.o.add_to(y, residual)
        elif accumulate is None:
            self.o.write_to(y, residual)
        else:
            self.o(y, out=residual)


register_mixer("gated_delta", GatedDeltaRule)
