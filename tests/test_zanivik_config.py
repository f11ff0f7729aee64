"""The Zanivik design without a GPU: what a configuration turns into (layer descriptions, what each layer asks of the
cache manager, names and shapes of the tensors), refusals, and properties of the plain implementation itself."""
import copy
import math

import pytest
import torch

import plain_zanivik as plain
import tiny_zanivik as tz
from blackwellllm_b200.config.registry import ConfigError, parse_config
from blackwellllm_b200.weights.random_init import model_param_specs

F64 = torch.float64


def test_registered_under_its_name_and_model_type():
    cfg = parse_config(tz.MIXED)
    assert cfg.architecture == "Zanivik" and not cfg.tie_word_embeddings and cfg.final_norm.kind == "layernorm"
    assert (cfg.embedding_multiplier, cfg.logit_scale, cfg.logit_softcap) == (1.0, 1.0, None)
    raw = {k: v for k, v in tz.MIXED.items() if k != "architecture"}
    raw["model_type"] = "zanivik"
    assert parse_config(raw).architecture == "Zanivik"


@pytest.mark.parametrize("name", list(tz.CONFIGS))
def test_layers(name):
    raw, _ = tz.CONFIGS[name]
    cfg = parse_config(raw)
    eps = raw["norm"]["eps"]
    assert len(cfg.layers) == len(raw["layers"]) == len(cfg.schedule)
    for layer, spec in zip(raw["layers"], cfg.layers):
        m, s = layer["mixer"], spec.mixer
        assert spec.block == "sandwich" and spec.layer_scale == ("ls1", "ls2") and spec.residual_mult == raw["residual_mult"]
        assert [n.param for n in (spec.mixer_norm, spec.mixer_post_norm, spec.ffn_norm, spec.ffn_post_norm)] == \
            ["norm1", "norm1b", "norm2", "norm2b"]
        assert all(n.kind == "layernorm" and n.eps == eps for n in (spec.mixer_norm, spec.mixer_post_norm, spec.ffn_norm, spec.ffn_post_norm))
        assert s.kind == "side_by_side"
        a, l = s.left, m["left"]
        assert (a.num_heads, a.num_kv_heads, a.head_dim, a.v_head_dim or a.head_dim) == (l["heads"], l["kv_heads"], l["dim"], l["vdim"])
        assert a.window == (l.get("mask") or {}).get("size") and a.softmax_scale == l["scale"] and a.qk_norm_eps == eps
        assert a.position.theta == l["rot"]["base"] and a.position.rotary_dim == l["rot"]["dims"] and not a.position.interleaved
        sc = l["rot"].get("scaling")
        if sc:
            p = a.position.scaling
            assert (p.factor, p.low_freq_factor, p.high_freq_factor, p.original_max_position_embeddings) == \
                (sc["factor"], sc["low"], sc["high"], sc["original"])
        else:
            assert a.position.scaling is None
        r, rr = s.right, m["right"]
        if layer["type"] == "parallel":
            assert s.combine == "sum" and a.qk_norm == "unit" and a.sink and a.output_gate and not a.values_from_keys
            assert (a.output_scale, r.output_scale) == (m["left_scale"], m["right_scale"])
            assert (r.kind, r.num_heads, r.num_kv_heads, r.key_dim, r.value_dim, r.conv_taps, r.norm_eps) == \
                ("gated_delta", rr["heads"], rr["kv_heads"], rr["dim"], rr["vdim"], rr["conv"], eps)
        else:
            assert s.combine == "norm_mean" and s.norm_eps == eps and a.qk_norm == "head" and a.values_from_keys and a.head_temperature
            assert not a.sink and not a.output_gate and a.output_scale == 1.0
            assert (r.kind, r.num_heads, r.value_dim, r.state_dim, r.groups, r.conv_taps, r.norm_groups, r.norm_eps) == \
                ("state_space", rr["heads"], rr["vdim"], rr["state"], rr["groups"], rr["conv"], rr["norm_groups"], eps)
        if layer["mlp"] is None:
            assert spec.ffn is None
        else:
            assert spec.ffn.kind == "dense_mlp" and spec.ffn.activation == "gelu" and spec.ffn.intermediate_size == layer["mlp"]["ff"]


def test_tensor_names_and_shapes():
    specs = model_param_specs(tz.MIXED)
    W = 64
    want = {"embed": (210, W), "head": (210, W), "final.norm": (W,), "l0.norm1": (W,), "l0.norm1b": (W,), "l0.norm2": (W,),
            "l0.norm2b": (W,), "l0.ls1": (W,), "l0.ls2": (W,), "l0.mlp.up": (96, W), "l0.mlp.down": (W, 96),
            "l0.mix.left.q": (192, W), "l0.mix.left.k": (64, W), "l0.mix.left.v": (32, W), "l0.mix.left.sink": (6,),
            "l0.mix.left.g": (96, W), "l0.mix.left.o": (W, 96),
            "l0.mix.right.q": (32, W), "l0.mix.right.q.conv": (32, 3), "l0.mix.right.k": (32, W), "l0.mix.right.k.conv": (32, 3),
            "l0.mix.right.v": (96, W), "l0.mix.right.v.conv": (96, 3), "l0.mix.right.b": (4, W), "l0.mix.right.a": (4, W),
            "l0.mix.right.A_log": (4,), "l0.mix.right.dt_bias": (4,), "l0.mix.right.g": (96, W), "l0.mix.right.norm": (24,),
            "l0.mix.right.o": (W, 96),
            "l1.mix.left.q": (64, W), "l1.mix.left.k": (32, W), "l1.mix.left.q.norm": (16,), "l1.mix.left.k.norm": (16,),
            "l1.mix.left.temp": (4,), "l1.mix.left.o": (W, 64), "l1.mix.left.out": (W,), "l1.mix.right.out": (W,),
            "l1.mix.right.in": (48 + 48 + 2 * 72 + 6, W), "l1.mix.right.conv": (48 + 144, 4), "l1.mix.right.conv.b": (192,),
            "l1.mix.right.dt_bias": (6,), "l1.mix.right.A_log": (6,), "l1.mix.right.D": (6,), "l1.mix.right.norm": (48,),
            "l1.mix.right.o": (W, 48)}
    for name, shape in want.items():
        assert name in specs and tuple(specs[name].shape) == shape, (name, specs.get(name))
    for absent in ("l0.mix.left.q.norm", "l0.mix.left.temp", "l0.mix.left.out", "l1.mix.left.v", "l1.mix.left.sink", "l1.mix.left.g"):
        assert absent not in specs
    # a layer without a feed-forward has none of its tensors; its second norms and scale are taken if stored
    assert not any(k.startswith("l2.mlp.") for k in specs)
    assert specs["l2.norm2"].optional and specs["l2.norm2b"].optional and specs["l2.ls2"].optional and not specs["l2.ls1"].optional


def test_what_the_layers_ask_of_the_cache():
    from blackwellllm_b200.models.decoder import DecoderModel
    from blackwellllm_b200.parts import BuildContext, FixedStateRequest, PagedKVRequest
    model = DecoderModel(parse_config(tz.MIXED), BuildContext(torch.device("cpu"), torch.float32))
    rq = model.cache_requests()
    assert rq[0] == (PagedKVRequest(2, 32, 24, 0), FixedStateRequest((4, 16, 24), torch.float32), FixedStateRequest((3, 160), torch.float32))
    assert rq[1] == (PagedKVRequest(2, 16, 9, 0), FixedStateRequest((6, 24, 8), torch.float32), FixedStateRequest((4, 192), torch.float32))
    assert rq[2][0] == PagedKVRequest(3, 48, 17, 0)
    model16 = DecoderModel(parse_config(tz.OPEN), BuildContext(torch.device("cpu"), torch.bfloat16))
    # bfloat16 pads head sizes to what the kernels take: 10 -> 16, 24/40 -> 48; the recurrent state stays float32
    assert model16.cache_requests()[0][0] == PagedKVRequest(1, 16, 16, 0) and model16.cache_requests()[1][0] == PagedKVRequest(3, 48, None, 0)
    assert all(r.dtype == torch.float32 for e in model16.cache_requests() for r in e[1:])


@pytest.mark.parametrize("edit,text", [
    (lambda r: r["layers"][0].__setitem__("type", "conv"), "not a mixer"),
    (lambda r: r["layers"][0]["mlp"].__setitem__("kind", "moe"), "not a feed-forward"),
    (lambda r: r["layers"][0]["mixer"]["left"].__setitem__("kv_heads", 4), "multiple"),
    (lambda r: r["layers"][0]["mixer"]["right"].__setitem__("kv_heads", 3), "multiple"),
    (lambda r: r["layers"][1]["mixer"]["right"].__setitem__("groups", 4), "multiple"),
    (lambda r: r["layers"][1]["mixer"]["right"].__setitem__("norm_groups", 7), "multiple"),
    (lambda r: r["layers"][1]["mixer"]["left"].__setitem__("vdim", 32), "the values are the keys"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 34), "at most dim"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"].__setitem__("dims", 7), "even"),
    (lambda r: r["layers"][0]["mixer"]["left"]["rot"]["scaling"].__setitem__("high", 1.0), "larger than low"),
    (lambda r: r["layers"][0]["mixer"].pop("left_scale"), "left_scale"),
    (lambda r: r["layers"][0]["mixer"]["right"].__setitem__("conv", 0), "positive integer"),
    (lambda r: r.pop("residual_mult"), "residual_mult"),
    (lambda r: r["norm"].__setitem__("eps", 0), "eps"),
    (lambda r: r.__setitem__("layers", []), "non-empty"),
])
def test_refusals(edit, text):
    raw = copy.deepcopy(tz.MIXED)
    edit(raw)
    with pytest.raises(ConfigError, match=text):
        parse_config(raw)


def test_specs_that_do_not_go_together():
    from blackwellllm_b200.config.specs import AttentionSpec, RopeSpec, SideBySideSpec, YarnRopeScaling
    from blackwellllm_b200.parts import BuildContext, build_mixer
    ctx = BuildContext(torch.device("cpu"), torch.float32)

    def attn(**kw):
        base = dict(num_heads=2, num_kv_heads=1, head_dim=16, qkv_bias=False, position=RopeSpec(theta=100.0, rotary_dim=16))
        base.update(kw)
        return AttentionSpec(**base)
    for bad in (dict(values_from_keys=True, v_head_dim=8), dict(values_from_keys=True, qkv_bias=True), dict(qk_norm="unit"),
                dict(shares_kv=True, output_scale=0.5), dict(qk_norm="other"),
                dict(qk_norm="unit", qk_norm_eps=1e-6, position=RopeSpec(theta=100.0, rotary_dim=16, scaling=YarnRopeScaling(4.0, 64, 8.0, 1.0)))):
        with pytest.raises(ValueError):
            build_mixer(attn(**bad), 32, ctx)
    with pytest.raises(ValueError):
        build_mixer(SideBySideSpec(left=attn(), right=attn(), combine="product"), 32, ctx)


# ------------------------------------------------------------------ the plain implementation itself

def test_plain_frequency_bands():
    rot = {"base": 10000.0, "dims": 32, "scaling": {"factor": 6.0, "low": 1.5, "high": 5.0, "original": 700}}
    f = plain.frequencies(rot)
    plain_f = plain.frequencies({"base": 10000.0, "dims": 32})
    kept = mixed = divided = 0
    for a, b in zip(f, plain_f):
        wave = 2 * math.pi / b
        if wave < 140:
            assert a == b
            kept += 1
        elif wave > 700 / 1.5:
            assert abs(a - b / 6) < 1e-15
            divided += 1
        else:
            assert b / 6 < a < b
            mixed += 1
    assert kept and mixed and divided


def test_plain_rotation_is_relative_and_keeps_lengths():
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(1, 1, 6, generator=g, dtype=F64).expand(9, 1, 6), torch.randn(1, 1, 6, generator=g, dtype=F64).expand(9, 1, 6)
    rot = {"base": 50.0, "dims": 4}
    a, b = plain.rotate_halves(q, rot)[:, 0], plain.rotate_halves(k, rot)[:, 0]
    s = a @ b.T
    assert abs(float(s[5, 3] - s[8, 6])) < 1e-12 and abs(float(s[2, 2] - q[0, 0] @ k[0, 0])) < 1e-12
    assert torch.equal(a[:, 4:], q[:, 0, 4:]) and float((a.norm(dim=-1) - q[0, 0].norm()).abs().max()) < 1e-12


def test_plain_sink_takes_its_share():
    q, k = torch.zeros(4, 2, 3, dtype=F64), torch.zeros(4, 1, 3, dtype=F64)
    v = torch.ones(4, 1, 2, dtype=F64)
    o = plain.attend(q, k, v, 1.0, plain.window_mask(4, 2), sink=torch.tensor([0.0, math.log(2.0)], dtype=F64))
    assert torch.allclose(o[0], torch.tensor([1 / 2, 1 / 2, 1 / 3, 1 / 3], dtype=F64))
    assert torch.allclose(o[3], torch.tensor([2 / 3, 2 / 3, 1 / 2, 1 / 2], dtype=F64))
    assert plain.window_mask(5, 2)[4].tolist() == [False, False, False, True, True]


def test_plain_delta_rule_replaces_what_a_key_holds():
    """With beta 1 and no decay a key written twice returns its second value, and another key's value is untouched."""
    e = torch.eye(3, dtype=F64).view(3, 1, 3)
    k = torch.stack([e[0], e[1], e[0]])
    v = torch.tensor([[[1.0, 2.0]], [[3.0, 4.0]], [[5.0, 6.0]]], dtype=F64)
    ones = torch.ones(3, 1, dtype=F64)
    assert torch.equal(plain.delta_rule(k, k, v, ones, ones)[2, 0], v[2, 0])
    q = torch.stack([e[0], e[0], e[1]])
    assert torch.equal(plain.delta_rule(q, k, v, ones, ones)[2, 0], v[1, 0])


def test_plain_state_space_equals_its_sum():
    g = torch.Generator().manual_seed(4)
    T, H, P, N = 9, 2, 3, 4
    x, B, C = (torch.randn(T, H, n, generator=g, dtype=F64) for n in (P, N, N))
    dt, A, D = torch.rand(T, H, generator=g, dtype=F64), -torch.rand(H, generator=g, dtype=F64), torch.randn(H, generator=g, dtype=F64)
    y = plain.state_space(x, B, C, dt, A, D)
    for t in range(T):
        for h in range(H):
            want = D[h] * x[t, h]
            for s in range(t + 1):
                want = want + math.exp(float(A[h] * dt[s + 1:t + 1, h].sum())) * dt[s, h] * (B[s, h] @ C[t, h]) * x[s, h]
            assert float((y[t, h] - want).abs().max()) < 1e-12


def test_plain_convolution_and_gelu():
    x = torch.arange(1.0, 5.0, dtype=F64).view(4, 1)
    out = plain.short_conv(x, torch.tensor([[100.0, 10.0, 1.0]], dtype=F64), torch.tensor([0.5], dtype=F64))
    assert out.view(-1).tolist() == [1.5, 12.5, 123.5, 234.5]
    z = torch.linspace(-4, 4, 33, dtype=F64)
    assert torch.allclose(plain.gelu(z), torch.nn.functional.gelu(z), atol=1e-14)
