"""Tiny Zogulorn configurations for the tests, and their random weights.

They differ from one another in every size and option: the order of the mixers (each of them first somewhere); layers without a
feed-forward; layers that read an earlier layer's keys and values, next to it or further on, with another number of query heads'
maps to merge, another block of positions and other taps; query heads per kv head (1, 2, 3, 4, 10); key and value sizes that are
equal or differ either way, multiples of 16 and not; rotations of all or part of a head; blocks of positions shorter and longer than a
page, that differ between layers, and none; score scales that are not the usual root; convolutions of 1 to 6 taps; recurrences
whose query/key heads are shared by 1, 2 or 3 heads; state sizes on both sides of 32, 64 and 128; inner sizes that are no multiple of 8;
one expert, all experts, expert sizes that no fast kernel takes; widths that are no multiple of 8 or of 4; factors that are 1, 0 or
negative; two maps whose weights cancel (diff far from and close to 1).  Layer scales, gains, alphas and biases are not close to 1
or 0, so that one that is left out or read from the wrong place shows.
"""
import json
import os

import torch

from blackwellllm_b200.weights.random_init import model_param_specs, random_tensors
from blackwellllm_b200.weights.safetensors_io import write_file


def _rot(heads, kv, dim, vdim, scale, size, base, dims=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale,
         "rot": {"base": base, "dims": dim if dims is None else dims}}
    if size is not None:
        m["mask"] = {"size": size}
    return m


def _par(left, delta, ranks, scales, mlp):
    """A layer of type 'parallel'; delta = (heads, kv_heads, dim, vdim, taps), ranks = inner sizes of decay and gate."""
    right = dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), delta), decay_rank=ranks[0], gate_rank=ranks[1])
    return {"type": "parallel", "mixer": {"left": left, "right": right, "left_scale": scales[0], "right_scale": scales[1]}, "mlp": mlp}


def _dif(heads, kv, dim, vdim, scale, size, taps, diff, mlp, kv_from=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale, "conv": taps, "diff": diff}
    if size is not None:
        m["mask"] = {"size": size}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def _model(vocab, width, eps, scale, layers):
    return {"architecture": "Zogulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "layers": layers}


# the differential attention first; blocks of 24 and 9 positions on pages of 8; a layer that reads keys from two layers back
MIXED = _model(210, 64, 1e-5, 1.5, [
    _dif(4, 2, 16, 24, 0.35, 24, 3, 0.3, dense(96)),
    _par(_rot(6, 2, 32, 16, 0.2, 9, 500.0, dims=16), (4, 2, 16, 24, 4), (8, 16), (0.9, -0.6), moe(6, 2, 32)),
    _dif(6, 2, 16, 24, 0.5, 17, 2, 0.7, None, kv_from=0),
    _par(_rot(3, 3, 16, 48, 0.4, 40, 100.0), (3, 1, 40, 12, 2), (5, 3), (1.0, 1.0), dense(80)),
])
# head sizes the tcgen05 prompt kernel takes; state sizes above 128; blocks longer than a page; a lender between two readers
TENSOR = _model(300, 96, 1e-6, 2.0, [
    _par(_rot(4, 1, 64, 64, 0.125, 50, 10000.0, dims=32), (2, 2, 160, 40, 4), (24, 8), (0.5, 0.8), dense(128)),
    _dif(4, 2, 32, 64, 0.25, 33, 4, 0.5, moe(5, 1, 48)),
    _dif(2, 1, 64, 128, 0.15, None, 4, 0.2, dense(64)),
    _dif(8, 2, 32, 64, 0.2, 70, 3, 0.9, moe(4, 4, 40), kv_from=1),
    _par(_rot(8, 2, 128, 128, 0.09, 33, 1e6), (6, 2, 64, 16, 3), (16, 40), (1.3, 0.2), None),
])
# sizes that no fast kernel takes (a width that is no multiple of 4, odd head, expert and feed-forward sizes); 20 maps on one
# kv head; one tap; no block of positions in one layer
OPEN = _model(77, 50, 3e-5, 0.8, [
    _par(_rot(3, 3, 10, 7, 0.5, 16, 1000.0, dims=6), (5, 5, 12, 33, 1), (3, 7), (0.8, 1.5), dense(45)),
    _dif(10, 1, 5, 9, 0.6, None, 1, 0.4, moe(3, 2, 21)),
    _dif(3, 1, 5, 9, 0.9, 5, 6, 0.55, dense(30), kv_from=1),
    _par(_rot(20, 1, 8, 12, 0.3, 16, 50.0, dims=2), (2, 1, 70, 9, 6), (1, 2), (0.7, 0.0), None),
    _dif(2, 2, 9, 5, 0.35, 3, 2, 0.1, None),
])
# one layer of each; head size 128; a block of one page exactly
BROAD = _model(400, 128, 1e-6, 1.0, [
    _par(_rot(2, 1, 128, 128, 0.09, 64, 250.0, dims=64), (2, 1, 128, 64, 4), (32, 64), (0.8, 0.9), moe(8, 3, 64)),
    _dif(4, 4, 64, 96, 0.2, 65, 4, 0.35, dense(200)),
])

# name -> (config, page size)
CONFIGS = {"mixed": (MIXED, 8), "tensor": (TENSOR, 16), "open": (OPEN, 32), "broad": (BROAD, 64)}


def make_tensors(raw, seed, std=0.1, bias_std=0.3, dtype=torch.bfloat16):
    """Random weights by their checkpoint names, rounded to ``dtype``.  Gains and layer scales 1 + noise; alphas in [0.4, 1]; decays
    from fast to slow (A_log in [-5, 1]); router rows long enough that two experts are seldom close."""
    specs = model_param_specs(raw)
    tensors = random_tensors(specs, seed, std, bias_std, dtype=torch.float32, skip_optional=False)
    g = torch.Generator().manual_seed(seed + 99)
    for name in sorted(specs):
        spec = specs[name]
        if spec.role == "gain" and spec.init == "ones":
            tensors[name] = 1.0 + 0.4 * torch.randn(spec.shape, generator=g)
        if name.endswith(".alpha"):
            tensors[name] = 0.4 + 0.6 * torch.rand(spec.shape, generator=g)
        if name.endswith(".A_log"):
            tensors[name] = -5.0 + 6.0 * torch.rand(spec.shape, generator=g)
        if name.endswith(".dt_bias"):
            tensors[name] = torch.randn(spec.shape, generator=g)
        if name.endswith(".conv"):
            tensors[name] = 0.5 * torch.randn(spec.shape, generator=g)
        if name.endswith((".right.b", ".a1", ".a2", ".g1", ".g2", ".mix.g", ".left.g")):
            tensors[name] = tensors[name] * 3.0        # gates that move with the token
        if name.endswith(".router"):
            tensors[name] = tensors[name] * 10.0
        if name == "embed":
            tensors[name] = 0.5 * torch.randn(spec.shape, generator=g)
    return {k: v.to(dtype) for k, v in tensors.items()}


def make_folder(name, dtype, root, seed=5):
    raw, _ = CONFIGS[name]
    d = os.path.join(root, f"zogulorn-{name}-{dtype}")
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
