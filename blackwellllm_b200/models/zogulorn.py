"""Zogulorn: config.json -> :class:`ModelConfig`.

A decoder whose layers are listed one by one (config ``layers``: each with ``type``, the mixer; ``mixer``, its sizes; ``mlp``, its
feed-forward or null).  What sets the design apart:

* its norm is a dynamic tanh, ``tanh(alpha x) * w + b``, without any statistic of the row;
* a layer is pre-norm with a scale per channel on each sublayer's output: ``x += ls1 * mixer(norm1(x))``, ``x += ls2 * ffn(norm2(x))``;
* mixer ``parallel``: two mixers side by side on the same input (``parts/side_by_side.py``), their outputs added with a factor each:
  left, grouped-query attention with rotary positions on pairs of neighbouring channels, kept inside blocks of ``mask.size``
  positions, with an output gate per head; right, the gated delta rule with a decay per key channel and a low-rank output gate
  (``parts/gated_delta.py``);
* mixer ``attention``: differential attention without positions (``parts/diff_attention.py``), with short convolutions on queries,
  keys and values, blocks of positions and a gate per head; with ``kv_from`` it reads an earlier such layer's keys and values;
* feed-forward ``dense``: down(gelu_tanh(gate x) * up x); ``moe``: the ``top`` experts by router logit, weighted by the softmax over
  those logits, each down(max(up x, 0)^2);
* the embedding's rows are multiplied by ``embedding.scale``; logits = head(final norm(x)).

Tensors: ``embed``, ``l<i>.norm1|norm2`` with ``.alpha`` and ``.b``, ``l<i>.ls1|ls2``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``, ``head``;
below ``mix.left`` ``q|k|v|g|o``, below ``mix.right`` ``q|k|v`` with ``.conv``, ``b|A_log|dt_bias|a1|a2|g1|g2|norm|o``, below the other
mixer ``q|k|v`` with ``.conv``, ``lq1|lk1|lq2|lk2|g|o``; below ``mlp`` ``gate|up|down`` or ``router`` and ``e<n>.up|down``.

``mixer.right.decay_rank`` and ``gate_rank`` are taken where a model with random weights is to be written; a stored model gives the
inner sizes by its tensors' shapes.

This module only describes the model.  It builds nothing and owns no tensor.
"""
from __future__ import annotations

from typing import Any, Mapping

from ..config.registry import ConfigError, register_architecture
from ..config.specs import (AttentionSpec, DifferentialAttentionSpec, DynamicTanhSpec, GatedDeltaSpec, LayerSpec, ModelConfig,
                            RopeSpec, RoutedFFNSpec, ScheduleEntry, SideBySideSpec, SwiGLUSpec)

_ATTENTION_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("g", "g"))
_DELTA_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("b", "b"), ("a1", "a1"), ("a2", "a2"), ("g1", "g1"), ("g2", "g2"), ("o", "o"),
                ("norm", "norm"), ("q_conv", "q.conv"), ("k_conv", "k.conv"), ("v_conv", "v.conv"), ("A_log", "A_log"),
                ("dt_bias", "dt_bias"))
_DIFF_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("q_conv", "q.conv"), ("k_conv", "k.conv"), ("v_conv", "v.conv"), ("lq1", "lq1"),
               ("lk1", "lk1"), ("lq2", "lq2"), ("lk2", "lk2"), ("g", "g"), ("o", "o"))


def _get(d: Mapping[str, Any], key: str, where: str, kind=None):
    if not isinstance(d, Mapping) or key not in d:
        raise ConfigError(f"config.json: {where} lacks {key!r}")
    v = d[key]
    if kind is int and (isinstance(v, bool) or not isinstance(v, int) or v <= 0):
        raise ConfigError(f"config.json: {where}.{key} must be a positive integer, got {v!r}")
    if kind is float:
        if isinstance(v, bool) or not isinstance(v, (int, float)):
            raise ConfigError(f"config.json: {where}.{key} must be a number, got {v!r}")
        v = float(v)
    return v


def _positive(d, key, where) -> float:
    v = _get(d, key, where, float)
    if not v > 0:
        raise ConfigError(f"config.json: {where}.{key} must be > 0, got {v!r}")
    return v


def _heads(m, w) -> tuple:
    a, b = _get(m, "heads", w, int), _get(m, "kv_heads", w, int)
    if a % b:
        raise ConfigError(f"config.json: {w}: heads ({a}) is not a multiple of kv_heads ({b})")
    return a, b


def _block_size(m: Mapping[str, Any], w: str):
    mask = m.get("mask")
    return None if mask is None else _get(mask, "size", w + ".mask", int)


def _attention(m: Mapping[str, Any], w: str, factor: float) -> AttentionSpec:
    heads, kv = _heads(m, w)
    dim, vdim = _get(m, "dim", w, int), _get(m, "vdim", w, int)
    rot = _get(m, "rot", w)
    dims = _get(rot, "dims", w + ".rot", int)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {w}.rot.dims ({dims}) must be even and at most dim ({dim})")
    return AttentionSpec(num_heads=heads, num_kv_heads=kv, head_dim=dim, qkv_bias=False,
                         position=RopeSpec(theta=_positive(rot, "base", w + ".rot"), rotary_dim=dims, interleaved=True),
                         chunk=_block_size(m, w), softmax_scale=_positive(m, "scale", w), v_head_dim=vdim if vdim != dim else None,
                         names=_ATTENTION_NAMES, output_gate=True, gate_per_head=True, output_scale=factor)


def _delta(m: Mapping[str, Any], w: str, eps: float, factor: float) -> GatedDeltaSpec:
    heads, kv = _heads(m, w)
    rank = lambda key: None if m.get(key) is None else _get(m, key, w, int)
    return GatedDeltaSpec(num_heads=heads, num_kv_heads=kv, key_dim=_get(m, "dim", w, int), value_dim=_get(m, "vdim", w, int),
                          conv_taps=_get(m, "conv", w, int), norm_eps=eps, output_scale=factor, names=_DELTA_NAMES,
                          channel_decay=True, lowrank_gate=True, decay_rank=rank("decay_rank"), gate_rank=rank("gate_rank"))


def _parallel(m: Mapping[str, Any], w: str, eps: float, index: int, raw_layers) -> SideBySideSpec:
    left, right = _get(m, "left_scale", w, float), _get(m, "right_scale", w, float)
    return SideBySideSpec(left=_attention(_get(m, "left", w), w + ".left", left),
                          right=_delta(_get(m, "right", w), w + ".right", eps, right), combine="sum")


def _differential(m: Mapping[str, Any], w: str, eps: float, index: int, raw_layers) -> DifferentialAttentionSpec:
    heads, kv = _heads(m, w)
    dim, vdim = _get(m, "dim", w, int), _get(m, "vdim", w, int)
    src = m.get("kv_from")
    if src is not None:
        if isinstance(src, bool) or not isinstance(src, int) or not 0 <= src < index:
            raise ConfigError(f"config.json: {w}.kv_from must name an earlier layer, got {src!r}")
        layer = raw_layers[src]
        other = layer.get("mixer", {})
        if layer.get("type") != "attention" or other.get("kv_from") is not None:
            raise ConfigError(f"config.json: {w}.kv_from names layer {src}, which has no such keys and values of its own")
        if (other.get("kv_heads"), other.get("dim"), other.get("vdim")) != (kv, dim, vdim):
            raise ConfigError(f"config.json: {w}.kv_from names layer {src}, whose kv_heads, dim or vdim differ")
    return DifferentialAttentionSpec(num_heads=heads, num_kv_heads=kv, head_dim=dim, v_head_dim=vdim,
                                     conv_taps=_get(m, "conv", w, int), diff=_get(m, "diff", w, float), norm_eps=eps,
                                     softmax_scale=_positive(m, "scale", w), chunk=_block_size(m, w), gate_per_head=True,
                                     shares_kv=src is not None, names=_DIFF_NAMES)


_MIXERS = {"parallel": _parallel, "attention": _differential}


def _mixer(layer: Mapping[str, Any], where: str, eps: float, index: int, raw_layers):
    kind = _get(layer, "type", where)
    if kind not in _MIXERS:
        raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design ({sorted(_MIXERS)})")
    return _MIXERS[kind](_get(layer, "mixer", where), where + ".mixer", eps, index, raw_layers)


def _ffn(layer: Mapping[str, Any], where: str):
    f = layer.get("mlp")
    if f is None:
        return None
    w = where + ".mlp"
    kind = _get(f, "kind", w)
    if kind == "dense":
        return SwiGLUSpec(intermediate_size=_get(f, "ff", w, int), activation="gelu_tanh", names=("gate", "up", "down"))
    if kind != "moe":
        raise ConfigError(f"config.json: {w}.kind {kind!r} is not a feed-forward of this design ('dense', 'moe')")
    router = _get(f, "router", w)
    experts, top = _get(router, "experts", w + ".router", int), _get(router, "top", w + ".router", int)
    if top > experts:
        raise ConfigError(f"config.json: {w}.router.top ({top}) exceeds the experts ({experts})")
    return RoutedFFNSpec(num_experts=experts, top_k=top, expert_size=_get(_get(f, "expert", w), "ff", w + ".expert", int),
                         score="softmax_chosen", renormalize=True, activation="relu2")


def parse_zogulorn(raw: Mapping[str, Any]) -> ModelConfig:
    width, vocab = _get(raw, "width", "the top level", int), _get(raw, "vocab", "the top level", int)
    eps = _positive(_get(raw, "norm", "the top level"), "eps", "norm")
    scale = _get(_get(raw, "embedding", "the top level"), "scale", "embedding", float)
    raw_layers = _get(raw, "layers", "the top level")
    if not isinstance(raw_layers, list) or not raw_layers:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    norm = lambda name: DynamicTanhSpec(param=name, alpha_param=name + ".alpha", bias_param=name + ".b")
    layers, schedule = [], []
    for i, layer in enumerate(raw_layers):
        where = f"layers[{i}]"
        layers.append(LayerSpec(
            mixer=_mixer(layer, where, eps, i, raw_layers), ffn=_ffn(layer, where), block="prenorm", mixer_norm=norm("norm1"),
            ffn_norm=norm("norm2"), mixer_prefix="mix.", ffn_prefix="mlp.", mixer_norm_prefix="", ffn_norm_prefix="",
            layer_scale=("ls1", "ls2")))
        schedule.append(ScheduleEntry(layer=i, cache_of=layer["mixer"].get("kv_from") if layer["type"] == "attention" else None))
    eos = raw.get("eos_token_id")
    eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(int(e) for e in eos))
    return ModelConfig(
        architecture="Zogulorn", hidden_size=width, vocab_size=vocab, layers=tuple(layers), schedule=tuple(schedule),
        final_norm=norm("norm"), tie_word_embeddings=False, max_position_embeddings=0, weight_prefix="", layer_prefix="l{i}.",
        embed_name="embed", final_norm_prefix="final.", head_name="head", embedding_multiplier=scale, eos_token_ids=eos_ids,
        stored_dtype=str(raw.get("torch_dtype", "bfloat16")), raw=dict(raw))


register_architecture("Zogulorn", parse_zogulorn, model_type="zogulorn")
