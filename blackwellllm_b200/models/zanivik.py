"""Zanivik: config.json -> :class:`ModelConfig`.

A decoder whose layers are listed one by one (config ``layers``: each with ``type``, the mixer; ``mixer``, its sizes;
``mlp``, its feed-forward or null).  What sets the design apart:

* a layer has a layer norm before and after each sublayer, a scale per channel on what the second norm returns, and the
  constant ``residual_mult`` on both: ``x += m ls1 * norm1b(mixer(norm1(x)))``, ``x += m ls2 * norm2b(ffn(norm2(x)))``;
* a mixer is two mixers side by side on the same input (``parts/side_by_side.py``), an attention with a sliding window
  (``mask.size``) on the left and a recurrence on the right:

  - ``parallel``: left, grouped-query attention with rotary positions (frequencies by wavelength bands where
    ``rot.scaling`` is given), queries and keys divided by their root mean square after the rotation, a learned sink per
    head and an output gate; right, the gated delta rule (``parts/gated_delta.py``); the two outputs added, times
    ``left_scale`` and ``right_scale``;
  - ``parallel_2``: left, attention whose values are the key projection, per-head norms with gains before the rotation and a
    learned factor per head on the scores; right, a state-space mixer (``parts/state_space.py``); half the sum of the two
    outputs, each RMS-normed over the width with a gain;

* feed-forward ``dense``: down(gelu(up x)), the gelu with the error function;
* logits = head(final layer norm(x)).

Tensors: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b|ls1|ls2``, ``l<i>.mix.left.*``, ``l<i>.mix.right.*``,
``l<i>.mlp.up|down``, ``final.norm``, ``head``; below ``left`` ``q|k|v|sink|g|o`` or ``q|k|q.norm|k.norm|temp|o`` (and
``out``), below ``right`` ``q|q.conv|k|k.conv|v|v.conv|b|a|A_log|dt_bias|g|norm|o`` or
``in|conv|conv.b|dt_bias|A_log|D|norm|o`` (and ``out``).

This module only describes the model.  It builds nothing and owns no tensor.
"""
from __future__ import annotations

from typing import Any, Mapping

from ..config.registry import ConfigError, register_architecture
from ..config.specs import (AttentionSpec, DenseMLPSpec, GatedDeltaSpec, LayerNormSpec, LayerSpec, Llama3RopeScaling,
                            ModelConfig, RopeSpec, ScheduleEntry, SideBySideSpec, StateSpaceSpec)

_ATTENTION_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("o", "o"), ("q_norm", "q.norm"), ("k_norm", "k.norm"),
                    ("sink", "sink"), ("g", "g"), ("temp", "temp"))
_DELTA_NAMES = (("q", "q"), ("k", "k"), ("v", "v"), ("g", "g"), ("b", "b"), ("a", "a"), ("o", "o"), ("norm", "norm"),
                ("q_conv", "q.conv"), ("k_conv", "k.conv"), ("v_conv", "v.conv"), ("A_log", "A_log"), ("dt_bias", "dt_bias"))
_SPACE_NAMES = (("in", "in"), ("conv", "conv"), ("conv_bias", "conv.b"), ("dt_bias", "dt_bias"), ("A_log", "A_log"),
                ("D", "D"), ("norm", "norm"), ("o", "o"))


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


def _divides(m, w, whole, part) -> tuple:
    a, b = _get(m, whole, w, int), _get(m, part, w, int)
    if a % b:
        raise ConfigError(f"config.json: {w}: {whole} ({a}) is not a multiple of {part} ({b})")
    return a, b


def _rotation(m: Mapping[str, Any], w: str, dim: int) -> RopeSpec:
    rot = _get(m, "rot", w)
    w += ".rot"
    dims = _get(rot, "dims", w, int)
    if dims % 2 or dims > dim:
        raise ConfigError(f"config.json: {w}.dims ({dims}) must be even and at most dim ({dim})")
    scaling = rot.get("scaling")
    if scaling is not None:
        ws = w + ".scaling"
        scaling = Llama3RopeScaling(factor=_positive(scaling, "factor", ws), low_freq_factor=_positive(scaling, "low", ws),
                                    high_freq_factor=_positive(scaling, "high", ws),
                                    original_max_position_embeddings=_positive(scaling, "original", ws))
        if not scaling.high_freq_factor > scaling.low_freq_factor:
            raise ConfigError(f"config.json: {ws}.high must be larger than low")
    return RopeSpec(theta=_positive(rot, "base", w), rotary_dim=dims, scaling=scaling, interleaved=False)


def _window(m: Mapping[str, Any], w: str):
    mask = m.get("mask")
    return None if mask is None else _get(mask, "size", w + ".mask", int)


def _sink_attention(m: Mapping[str, Any], w: str, eps: float, scale: float) -> AttentionSpec:
    heads, kv = _divides(m, w, "heads", "kv_heads")
    dim, vdim = _get(m, "dim", w, int), _get(m, "vdim", w, int)
    return AttentionSpec(num_heads=heads, num_kv_heads=kv, head_dim=dim, qkv_bias=False, position=_rotation(m, w, dim),
                         window=_window(m, w), softmax_scale=_get(m, "scale", w, float),
                         v_head_dim=vdim if vdim != dim else None, qk_norm_eps=eps, qk_norm="unit", names=_ATTENTION_NAMES,
                         sink=True, output_gate=True, output_scale=scale)


def _shared_kv_attention(m: Mapping[str, Any], w: str, eps: float) -> AttentionSpec:
    heads, kv = _divides(m, w, "heads", "kv_heads")
    dim = _get(m, "dim", w, int)
    if m.get("vdim", dim) != dim:
        raise ConfigError(f"config.json: {w}.vdim ({m['vdim']!r}) must be dim ({dim}): the values are the keys")
    return AttentionSpec(num_heads=heads, num_kv_heads=kv, head_dim=dim, qkv_bias=False, position=_rotation(m, w, dim),
                         window=_window(m, w), softmax_scale=_get(m, "scale", w, float), qk_norm_eps=eps, qk_norm="head",
                         names=_ATTENTION_NAMES, values_from_keys=True, head_temperature=True)


def _delta(m: Mapping[str, Any], w: str, eps: float, scale: float) -> GatedDeltaSpec:
    heads, kv = _divides(m, w, "heads", "kv_heads")
    return GatedDeltaSpec(num_heads=heads, num_kv_heads=kv, key_dim=_get(m, "dim", w, int), value_dim=_get(m, "vdim", w, int),
                          conv_taps=_get(m, "conv", w, int), norm_eps=eps, output_scale=scale, names=_DELTA_NAMES)


def _space(m: Mapping[str, Any], w: str, eps: float) -> StateSpaceSpec:
    heads, groups = _divides(m, w, "heads", "groups")
    vdim, parts = _get(m, "vdim", w, int), _get(m, "norm_groups", w, int)
    if heads * vdim % parts:
        raise ConfigError(f"config.json: {w}: heads * vdim ({heads * vdim}) is not a multiple of norm_groups ({parts})")
    return StateSpaceSpec(num_heads=heads, value_dim=vdim, state_dim=_get(m, "state", w, int), groups=groups,
                          conv_taps=_get(m, "conv", w, int), norm_groups=parts, norm_eps=eps, names=_SPACE_NAMES)


def _parallel(m: Mapping[str, Any], w: str, eps: float) -> SideBySideSpec:
    left, right = _get(m, "left_scale", w, float), _get(m, "right_scale", w, float)
    return SideBySideSpec(left=_sink_attention(_get(m, "left", w), w + ".left", eps, left),
                          right=_delta(_get(m, "right", w), w + ".right", eps, right), combine="sum")


def _parallel_2(m: Mapping[str, Any], w: str, eps: float) -> SideBySideSpec:
    return SideBySideSpec(left=_shared_kv_attention(_get(m, "left", w), w + ".left", eps),
                          right=_space(_get(m, "right", w), w + ".right", eps), combine="norm_mean", norm_eps=eps)


_MIXERS = {"parallel": _parallel, "parallel_2": _parallel_2}


def _mixer(layer: Mapping[str, Any], where: str, eps: float):
    kind = _get(layer, "type", where)
    if kind not in _MIXERS:
        raise ConfigError(f"config.json: {where}.type {kind!r} is not a mixer of this design ({sorted(_MIXERS)})")
    return _MIXERS[kind](_get(layer, "mixer", where), where + ".mixer", eps)


def _ffn(layer: Mapping[str, Any], where: str):
    f = layer.get("mlp")
    if f is None:
        return None
    kind = _get(f, "kind", where + ".mlp")
    if kind != "dense":
        raise ConfigError(f"config.json: {where}.mlp.kind {kind!r} is not a feed-forward of this design ('dense')")
    return DenseMLPSpec(intermediate_size=_get(f, "ff", where + ".mlp", int), activation="gelu", names=("up", "down"))


def parse_zanivik(raw: Mapping[str, Any]) -> ModelConfig:
    width, vocab = _get(raw, "width", "the top level", int), _get(raw, "vocab", "the top level", int)
    eps = _positive(_get(raw, "norm", "the top level"), "eps", "norm")
    mult = _get(raw, "residual_mult", "the top level", float)
    raw_layers = _get(raw, "layers", "the top level")
    if not isinstance(raw_layers, list) or not raw_layers:
        raise ConfigError("config.json: 'layers' must be a non-empty list")
    layers = []
    for i, layer in enumerate(raw_layers):
        where = f"layers[{i}]"
        layers.append(LayerSpec(
            mixer=_mixer(layer, where, eps), ffn=_ffn(layer, where), block="sandwich",
            mixer_norm=LayerNormSpec(eps=eps, param="norm1"), ffn_norm=LayerNormSpec(eps=eps, param="norm2"),
            mixer_post_norm=LayerNormSpec(eps=eps, param="norm1b"), ffn_post_norm=LayerNormSpec(eps=eps, param="norm2b"),
            mixer_prefix="mix.", ffn_prefix="mlp.", mixer_norm_prefix="", ffn_norm_prefix="", layer_scale=("ls1", "ls2"),
            residual_mult=mult))
    eos = raw.get("eos_token_id")
    eos_ids = () if eos is None else ((eos,) if isinstance(eos, int) else tuple(int(e) for e in eos))
    return ModelConfig(
        architecture="Zanivik", hidden_size=width, vocab_size=vocab, layers=tuple(layers),
        schedule=tuple(ScheduleEntry(layer=i) for i in range(len(layers))),
        final_norm=LayerNormSpec(eps=eps, param="norm"), tie_word_embeddings=False, max_position_embeddings=0,
        weight_prefix="", layer_prefix="l{i}.", embed_name="embed", final_norm_prefix="final.", head_name="head",
        eos_token_ids=eos_ids, stored_dtype=str(raw.get("torch_dtype", "bfloat16")), raw=dict(raw))


register_architecture("Zanivik", parse_zanivik, model_type="zanivik")
