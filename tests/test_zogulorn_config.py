"""The Zogulorn design without a GPU: what a configuration turns into (layer descriptions, what each run asks of the cache manager,
names and shapes of the tensors), refusals, and properties of the plain implementation itself."""
import copy
import math

import pytest
import torch

import plain_zogulorn as plain
import tiny_zogulorn as tz
from blackwellllm_b200.config.registry import ConfigError, parse_config
from blackwellllm_b200.weights.random_init import model_param_specs

F64 = torch.float64


def test_registered_under_its_name_and_model_type():
    cfg = parse_config(tz.MIXED)
    assert cfg.architecture == "Zogulorn" and not cfg.tie_word_embeddings and cfg.final_norm.kind == "dynamic_tanh"
    assert (cfg.embedding_multiplier, cfg.logit_scale, cfg.logit_softcap) == (1.5, 1.0, None)
    raw = {k: v for k, v in tz.MIXED.items() if k != "architecture"}
    raw["model_type"] = "zogulorn"
    assert parse_config(raw).architecture == "Zogulorn"


@pytest.mark.parametrize("name", list(tz.CONFIGS))
def test_layers(name):
    raw, _ = tz.CONFIGS[name]
    cfg = parse_config(raw)
    eps = raw["norm"]["eps"]
    assert len(cfg.layers) == len(raw["layers"]) == len(cfg.schedule)
    for layer, spec, run in zip(raw["layers"], cfg.layers, cfg.schedule):
        m, s, f = layer["mixer"], spec.mixer, layer["mlp"]
        assert spec.block == "prenorm" and spec.layer_scale == ("ls1", "ls2")
        for norm, n in ((spec.mixer_norm, "norm1"), (spec.ffn_norm, "norm2")):
            assert (norm.kind, norm.param, norm.alpha_param, norm.bias_param) == ("dynamic_tanh", n, n + ".alpha", n + ".b")
        if layer["type"] == "parallel":
            a, l, r, rr = s.left, m["left"], s.right, m["right"]
            assert s.kind == "side_by_side" and s.combine == "sum" and run.cache_of is None
            assert (a.num_heads, a.num_kv_heads, a.head_dim, a.v_head_dim or a.head_dim) == (l["heads"], l["kv_heads"], l["dim"], l["vdim"])
            assert a.chunk == (l.get("mask") or {}).get("size") and a.window is None and a.softmax_scale == l["scale"]
            assert a.position.theta == l["rot"]["base"] and a.position.rotary_dim == l["rot"]["dims"] and a.position.interleaved
            assert a.output_gate and a.gate_per_head and a.qk_norm_eps is None and not a.sink
            assert (a.output_scale, r.output_scale) == (m["left_scale"], m["right_scale"])
            assert (r.kind, r.num_heads, r.num_kv_heads, r.key_dim, r.value_dim, r.conv_taps, r.norm_eps) == \
                ("gated_delta", rr["heads"], rr["kv_heads"], rr["dim"], rr["vdim"], rr["conv"], eps)
            assert r.channel_decay and r.lowrank_gate and (r.decay_rank, r.gate_rank) == (rr["decay_rank"], rr["gate_rank"])
        else:
            assert (s.kind, s.num_heads, s.num_kv_heads, s.head_dim, s.v_head_dim, s.conv_taps, s.diff, s.norm_eps, s.softmax_scale) == \
                ("differential_attention", m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"], m["diff"], eps, m["scale"])
            assert s.chunk == (m.get("mask") or {}).get("size") and s.gate_per_head
            assert s.shares_kv == ("kv_from" in m) and run.cache_of == m.get("kv_from")
        if f is None:
            assert spec.ffn is None
        elif f["kind"] == "dense":
            assert (spec.ffn.kind, spec.ffn.activation, spec.ffn.intermediate_size) == ("swiglu", "gelu_tanh", f["ff"])
        else:
            e = spec.ffn
            assert (e.kind, e.num_experts, e.top_k, e.expert_size, e.score, e.activation) == \
                ("routed_ffn", f["router"]["experts"], f["router"]["top"], f["expert"]["ff"], "softmax_chosen", "relu2")


def test_tensor_names_and_shapes():
    specs = model_param_specs(tz.MIXED)
    W = 64
    want = {"embed": (210, W), "head": (210, W), "final.norm": (W,), "final.norm.b": (W,), "final.norm.alpha": (),
            "l0.norm1": (W,), "l0.norm1.b": (W,), "l0.norm1.alpha": (), "l0.norm2": (W,), "l0.ls1": (W,), "l0.ls2": (W,),
            "l0.mix.q": (128, W), "l0.mix.k": (64, W), "l0.mix.v": (48, W), "l0.mix.q.conv": (128, 3), "l0.mix.k.conv": (64, 3),
            "l0.mix.v.conv": (48, 3), "l0.mix.lq1": (16,), "l0.mix.lk2": (16,), "l0.mix.g": (4, W), "l0.mix.o": (W, 96),
            "l0.mlp.gate": (96, W), "l0.mlp.up": (96, W), "l0.mlp.down": (W, 96),
            "l1.mix.left.q": (192, W), "l1.mix.left.k": (64, W), "l1.mix.left.v": (32, W), "l1.mix.left.g": (6, W),
            "l1.mix.left.o": (W, 96), "l1.mix.right.q": (32, W), "l1.mix.right.q.conv": (32, 4), "l1.mix.right.k": (32, W),
            "l1.mix.right.v": (96, W), "l1.mix.right.v.conv": (96, 4), "l1.mix.right.b": (4, W), "l1.mix.right.A_log": (4,),
            "l1.mix.right.dt_bias": (64,), "l1.mix.right.a1": (8, W), "l1.mix.right.a2": (64, 8), "l1.mix.right.g1": (16, W),
            "l1.mix.right.g2": (96, 16), "l1.mix.right.norm": (24,), "l1.mix.right.o": (W, 96),
            "l1.mlp.router": (6, W), "l1.mlp.e5.up": (32, W), "l1.mlp.e5.down": (W, 32),
            "l2.mix.q": (192, W), "l2.mix.q.conv": (192, 2), "l2.mix.g": (6, W), "l2.mix.o": (W, 144)}
    for name, shape in want.items():
        assert name in specs and tuple(specs[name].shape) == shape, (name, specs.get(name))
    for absent in ("l2.mix.k", "l2.mix.v", "l2.mix.k.conv", "l2.mix.v.conv", "l1.mlp.e0.gate", "l1.mix.right.a", "l1.mix.right.g"):
        assert absent not in specs
    # a layer without a feed-forward has none of its tensors; its second norm and scale are taken if stored
    assert not any(k.startswith("l2.mlp.") for k in specs)
    assert all(specs[n].optional for n in ("l2.norm2", "l2.norm2.alpha", "l2.norm2.b", "l2.ls2")) and not specs["l2.ls1"].optional
    # inner sizes that the configuration does not state are the stored tensors'
    raw = copy.deepcopy(tz.MIXED)
    for key in ("decay_rank", "gate_rank"):
        del raw["layers"][1]["mixer"]["right"][key]
    open_specs = model_param_specs(raw)
    assert tuple(open_specs["l1.mix.right.a1"].shape) == (-1, W) and tuple(open_specs["l1.mix.right.g2"].shape) == (96, -1)


def test_what_the_runs_ask_of_the_cache():
    from blackwellllm_b200.models.decoder import DecoderModel
    from blackwellllm_b200.parts import BuildContext, FixedStateRequest, PagedKVRequest
    state = lambda *shape: FixedStateRequest(shape, torch.float32)
    model = DecoderModel(parse_config(tz.MIXED), BuildContext(torch.device("cpu"), torch.float32))
    rq = model.cache_requests()
    assert rq[0] == (PagedKVRequest(2, 32), state(3, 128 + 64 + 48))
    assert rq[1] == (PagedKVRequest(2, 32), state(4, 16, 24), state(4, 160))
    assert rq[2] == state(2, 192)          # keys and values of layer 0; its own queries' earlier inputs
    assert rq[3] == (PagedKVRequest(3, 48), state(3, 40, 12), state(2, 116))
    # bfloat16 pads rows to what the kernels take: a key row holds both maps
    model16 = DecoderModel(parse_config(tz.OPEN), BuildContext(torch.device("cpu"), torch.bfloat16))
    assert [e[0] for e in model16.cache_requests() if isinstance(e, tuple)] == \
        [PagedKVRequest(3, 16), PagedKVRequest(1, 16), PagedKVRequest(1, 16), PagedKVRequest(2, 32)]


@pytest.mark.parametrize("edit,text", [
    (lambda r: r["layers"][0].__setitem__("type", "conv"), "not a mixer"),
    (lambda r: r["layers"][0]["mlp"].__setitem__("kind", "glu"), "not a feed-forward"),
    (lambda r: r["layers"][0]["mixer"].__setitem__("kv_heads", 3), "multiple"),
    (lambda r: r["layers"][1]["mixer"]["left"].__setitem__("kv_heads", 4), "multiple"),
    (lambda r: r["layers"][1]["mixer"]["right"].__setitem__("kv_heads", 3), "multiple"),
    (lambda r: r["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 34), "at most dim"),
    (lambda r: r["layers"][1]["mixer"]["left"]["rot"].__setitem__("dims", 7), "even"),
    (lambda r: r["layers"][1]["mixer"].pop("left_scale"), "left_scale"),
    (lambda r: r["layers"][1]["mlp"]["router"].__setitem__("top", 7), "exceeds"),
    (lambda r: r["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda r: r["layers"][0]["mixer"].__setitem__("conv", 0), "positive integer"),
    (lambda r: r["layers"][0]["mixer"].__setitem__("scale", -1.0), "> 0"),
    (lambda r: r["layers"][0]["mixer"].__setitem__("kv_from", 0), "earlier layer"),
    (lambda r: r["layers"][2]["mixer"].__setitem__("kv_from", 1), "no such keys"),
    (lambda r: r["layers"][2]["mixer"].__setitem__("vdim", 32), "differ"),
    (lambda r: r.pop("embedding"), "embedding"),
    (lambda r: r["norm"].__setitem__("eps", 0), "eps"),
    (lambda r: r.__setitem__("layers", []), "non-empty"),
])
def test_refusals(edit, text):
    raw = copy.deepcopy(tz.MIXED)
    edit(raw)
    with pytest.raises(ConfigError, match=text):
        parse_config(raw)


def test_parts_that_do_not_go_together():
    from blackwellllm_b200.config.specs import LayerSpec, DynamicTanhSpec, NoPositionSpec, AttentionSpec, RMSNormSpec, RoutedFFNSpec
    from blackwellllm_b200.parts import BuildContext, build_block, build_ffn
    ctx = BuildContext(torch.device("cpu"), torch.float32)
    with pytest.raises(ValueError, match="chosen logits"):
        build_ffn(RoutedFFNSpec(4, 2, 16, score="softmax_chosen", choice_bias="bias"), 32, ctx)
    with pytest.raises(ValueError, match="router score"):
        build_ffn(RoutedFFNSpec(4, 2, 16, score="argmax"), 32, ctx)
    e = build_ffn(RoutedFFNSpec(4, 2, 16, activation="relu2"), 32, ctx)
    assert sorted({p.name.split(".")[-1] for p in e.param_specs()}) == ["down", "router", "up"]
    att = AttentionSpec(2, 1, 16, qkv_bias=False, position=NoPositionSpec())
    with pytest.raises(ValueError, match="add_to"):      # a dynamic tanh cannot follow a sublayer
        build_block(LayerSpec(mixer=att, ffn=None, mixer_norm=RMSNormSpec(1e-5), ffn_norm=None, block="sandwich",
                              mixer_post_norm=DynamicTanhSpec()), 32, ctx)


# ------------------------------------------------------------------ the plain implementation itself

def test_plain_rotation_is_relative_and_keeps_lengths():
    g = torch.Generator().manual_seed(2)
    q, k = torch.randn(1, 1, 6, generator=g, dtype=F64).expand(9, 1, 6), torch.randn(1, 1, 6, generator=g, dtype=F64).expand(9, 1, 6)
    a, b = plain.rotate_pairs(q, 50.0, 4)[:, 0], plain.rotate_pairs(k, 50.0, 4)[:, 0]
    s = a @ b.T
    assert abs(float(s[5, 3] - s[8, 6])) < 1e-12 and abs(float(s[2, 2] - q[0, 0] @ k[0, 0])) < 1e-12
    assert torch.equal(a[:, 4:], q[:, 0, 4:]) and float((a.norm(dim=-1) - q[0, 0].norm()).abs().max()) < 1e-12
    assert abs(float(a[1, 0] - (q[0, 0, 0] * math.cos(1) - q[0, 0, 1] * math.sin(1)))) < 1e-12


def test_plain_blocks_of_positions():
    m = plain.block_mask(7, 3)
    assert m[2].tolist() == [True, True, True, False, False, False, False]
    assert m[3].tolist() == [False, False, False, True, False, False, False]
    assert m[5].tolist() == [False, False, False, True, True, True, False]
    assert plain.block_mask(4, None)[3].all()


def test_plain_channel_decay_forgets_channel_by_channel():
    """Orthogonal keys with step size 1: what channel 0 holds fades by its own decay, channel 1 keeps its value."""
    k = torch.zeros(4, 1, 2, dtype=F64)
    k[0, 0, 0] = k[1, 0, 1] = 1.0
    q = k.clone()
    q[2, 0, 0] = q[3, 0, 1] = 1.0
    v = torch.tensor([[[4.0]], [[6.0]], [[9.0]], [[9.0]]], dtype=F64)
    g = torch.tensor([0.5, 1.0], dtype=F64).expand(4, 1, 2)
    beta = torch.tensor([[1.0], [1.0], [0.0], [0.0]], dtype=F64)
    o = plain.channel_delta_rule(q, k, v, g, beta)
    assert o.view(-1).tolist() == [4.0, 6.0, 1.0, 6.0]


def test_plain_difference_of_equal_maps_is_a_norm_of_one():
    a = torch.randn(3, 2, 8, generator=torch.Generator().manual_seed(1), dtype=F64)
    z = torch.zeros(4, dtype=F64)
    w = {n: z for n in ("lq1", "lk1", "lq2", "lk2")}          # lambda = diff
    o = plain.difference(a, a, w, {"diff": 0.25}, 1e-12)
    assert torch.allclose(o, 0.75 * plain.rms_unit(a, 1e-12), atol=1e-9)


def test_plain_convolution_gelu_and_router():
    x = torch.arange(1.0, 5.0, dtype=F64).view(4, 1)
    assert plain.short_conv(x, torch.tensor([[100.0, 10.0, 1.0]], dtype=F64)).view(-1).tolist() == [1.0, 12.0, 123.0, 234.0]
    z = torch.linspace(-4, 4, 33, dtype=F64)
    assert torch.allclose(plain.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"), atol=1e-14)
    # two experts with equal logits halve their outputs; the third, far below, is not chosen
    w = {"router": torch.tensor([[1.0], [1.0], [-50.0]], dtype=F64)}
    for e, up in enumerate((1.0, 2.0, 100.0)):
        w[f"e{e}.up"], w[f"e{e}.down"] = torch.tensor([[up]], dtype=F64), torch.ones(1, 1, dtype=F64)
    out = plain.routed_ffn(torch.tensor([[1.0], [-1.0]], dtype=F64), w, {"router": {"top": 2}})
    assert float(out[0]) == 0.5 * 1.0 + 0.5 * 4.0 and float(out[1]) == 0.0
