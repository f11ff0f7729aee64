"""Tiny Zanivik configurations for the tests, and their random weights.

They differ from one another in every size and option: the order of the two mixers (each of them first somewhere); layers
without a feed-forward; query heads per kv head (1, 2, 3, 4, 20); key and value sizes that are equal or differ either way,
multiples of 16 and not; rotations of all or part of a head, with and without wavelength bands (bands that keep, mix and
divide frequencies); windows shorter and longer than a page, windows that differ between layers, none; score scales that
are not the usual root; convolutions of 1 to 6 taps; recurrences whose query/key heads (or groups) are shared by 1, 2 or 3
heads; state sizes on both sides of 32, 64 and 128, value sizes that leave the last block of columns ragged; norm parts that
are one head, several heads or cut across heads; widths that are no multiple of 8 or of 4; factors that are 1, 0 or
negative.  Sinks, temperatures, layer scales, D and gains are not close to 1 or 0, so that one that is left out or read
from the wrong place shows.
"""
import json
import os

import torch

from blackwellllm_b200.weights.random_init import model_param_specs, random_tensors
from blackwellllm_b200.weights.safetensors_io import write_file


def _attn(heads, kv, dim, vdim, scale, size, base, dims=None, scaling=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
         "rot": {"base": base, "dims": dim if dims is None else dims}}
    if size is not None:
        m["mask"] = {"size": size}
    if scaling is not None:
        m["rot"]["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    return m


def _one(left, delta, scales, ff):
    """A layer of type 'parallel'; delta = (heads, kv_heads, dim, vdim, taps)."""
    m = {"left": left, "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), delta)),
         "left_scale": scales[0], "right_scale": scales[1]}
    return {"type": "parallel", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _two(left, space, ff):
    """A layer of type 'parallel_2'; space = (heads, vdim, state, groups, taps, norm_groups)."""
    m = {"left": left, "right": dict(zip(("heads", "vdim", "state", "groups", "conv", "norm_groups"), space))}
    return {"type": "parallel_2", "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def _model(vocab, width, eps, mult, layers):
    return {"architecture": "Zanivik", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


# the delta rule first; windows 24 and 9 with pages of 8; head sizes 32/16 and 16
MIXED = _model(210, 64, 1e-5, 0.6, [
    _one(_attn(6, 2, 32, 16, 0.4, 24, 500.0, dims=16, scaling=(4.0, 1.0, 4.0, 40)), (4, 2, 16, 24, 3), (0.9, -0.4), 96),
    _two(_attn(4, 2, 16, 16, 0.25, 9, 10000.0), (6, 8, 24, 3, 4, 2), 80),
    _one(_attn(3, 3, 16, 48, 1.1, 17, 100.0), (3, 1, 40, 12, 2), (1.0, 1.0), None),
    _two(_attn(2, 1, 32, 32, 0.2, 40, 3000.0, dims=8), (4, 20, 33, 1, 5, 5), 64),
])
# head sizes the tcgen05 prompt kernel takes; state sizes above 128; a window longer than a page
TENSOR = _model(300, 96, 1e-6, 1.0, [
    _two(_attn(4, 1, 64, 64, 0.125, 50, 10000.0, scaling=(8.0, 1.0, 3.0, 200)), (4, 32, 160, 2, 4, 1), 128),
    _one(_attn(8, 2, 64, 64, 0.3, 33, 1e6, dims=32), (2, 2, 160, 40, 4), (0.5, 0.8), 160),
    _one(_attn(2, 2, 128, 64, 0.09, 70, 20000.0, scaling=(2.0, 2.0, 8.0, 64)), (6, 2, 64, 16, 6), (1.3, 0.2), None),
])
# sizes that no fast kernel takes (a width that is no multiple of 4, head sizes 24/40 and 10, odd feed-forward sizes);
# 20 query heads on one kv head; one tap; no window in one layer
OPEN = _model(77, 50, 3e-5, 0.35, [
    _two(_attn(3, 1, 10, 10, 0.5, 16, 1000.0, dims=6), (3, 7, 5, 3, 1, 3), 45),
    _one(_attn(3, 3, 24, 40, 0.21, None, 700.0, dims=22), (5, 5, 12, 33, 4), (0.0, 1.5), 30),
    _one(_attn(20, 1, 8, 8, 0.6, 16, 50.0), (2, 1, 70, 9, 3), (0.7, 0.6), None),
    _two(_attn(2, 2, 12, 12, 0.35, 5, 1e5, scaling=(16.0, 0.5, 1.5, 30)), (2, 9, 66, 2, 3, 6), 53),
])
# one layer of each; head size 128; a window of one page exactly
BROAD = _model(400, 128, 1e-6, 0.8, [
    _one(_attn(2, 1, 128, 128, 0.09, 64, 250.0), (2, 1, 128, 64, 4), (0.8, 0.9), 256),
    _two(_attn(4, 2, 64, 64, 0.2, 65, 50000.0, dims=32), (8, 16, 128, 2, 4, 2), 200),
])

# name -> (config, page size)
CONFIGS = {"mixed": (MIXED, 8), "tensor": (TENSOR, 16), "open": (OPEN, 32), "broad": (BROAD, 64)}


def make_tensors(raw, seed, std=0.1, bias_std=0.3, dtype=torch.bfloat16):
    """Random weights by their checkpoint names, rounded to ``dtype``.  Gains and layer scales 1 + noise; sinks N(0, 1);
    temperatures in [0.5, 1.5]; decays from fast to slow (A_log in [-5, 1])."""
    specs = model_param_specs(raw)
    tensors = random_tensors(specs, seed, std, bias_std, dtype=torch.float32, skip_optional=False)
    g = torch.Generator().manual_seed(seed + 99)
    for name, spec in specs.items():
        if spec.role == "gain" and spec.init == "ones":
            tensors[name] = 1.0 + 0.4 * torch.randn(spec.shape, generator=g)
        if name.endswith(".sink"):
            tensors[name] = torch.randn(spec.shape, generator=g)
        if name.endswith(".temp"):
            tensors[name] = 0.5 + torch.rand(spec.shape, generator=g)
        if name.endswith(".A_log"):
            tensors[name] = -5.0 + 6.0 * torch.rand(spec.shape, generator=g)
        if name.endswith(".D"):
            tensors[name] = 0.5 + torch.randn(spec.shape, generator=g)
        if name.endswith(".dt_bias"):
            tensors[name] = torch.randn(spec.shape, generator=g)
        if name.endswith(".conv"):
            tensors[name] = 0.5 * torch.randn(spec.shape, generator=g)
        if name.endswith((".right.a", ".right.b")):
            tensors[name] = tensors[name] * 3.0        # gates that move with the token
        if name == "embed":
            tensors[name] = 0.5 * torch.randn(spec.shape, generator=g)
    return {k: v.to(dtype) for k, v in tensors.items()}


def make_folder(name, dtype, root, seed=5):
    raw, _ = CONFIGS[name]
    d = os.path.join(root, f"zanivik-{name}-{dtype}")
    if not os.path.isdir(d):
        os.makedirs(d)
        tensors = make_tensors(raw, seed, dtype={"float32": torch.float32, "bfloat16": torch.bfloat16}[dtype])
        with open(os.path.join(d, "config.json"), "w") as f:
            json.dump(raw, f)
        write_file(os.path.join(d, "model.safetensors"), tensors, metadata={"format": "pt"})
    return d


def prompt(n, vocab, seed):
    g = torch.Generator().manual_seed(seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()
