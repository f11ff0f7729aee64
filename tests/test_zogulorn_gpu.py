"""The Zogulorn design on the GPU against its plain implementation (tests/plain_zogulorn.py): each mechanism's kernels alone, then
whole models through Engine.step in every way of cutting and batching, through the scheduler's generate(), the command line and
bin/trace_run."""
import math

import pytest
import torch

import plain_zogulorn as plain
import replay
import tiny_zogulorn as tz

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
# of the largest logit of the compared request.  The sharp comparison is the float32 one; every bfloat16 kernel has
# its own tight test below.
TOL = {"float32": 1e-4, "bfloat16": 6e-2}
F64 = torch.float64
_DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


@pytest.fixture(scope="module")
def ops():
    from blackwellllm_b200.kernels import ops as o
    return o


def rnd(*shape, seed=0, scale=1.0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed)) * scale


def d(t):
    return t.to(DEV).contiguous()


def rel_err(got, want):
    return float((got.double().cpu() - want.double()).abs().max()) / max(float(want.abs().max()), 1e-30)


class Rows:
    """A step's batch as the row kernels see it: requests' portions, their positions and state slots."""

    def __init__(self, q_lens, starts, slots):
        from test_kernels_gpu import FakeBatch
        fb = FakeBatch(q_lens, [s + q for s, q in zip(starts, q_lens)])
        self.__dict__.update(fb.__dict__)
        self.state_slot = torch.tensor(slots, dtype=torch.int32, device=DEV)


def walk(cuts, lens):
    """Steps of (request, start, length) from each request's list of portions; requests run side by side."""
    at = [0] * len(lens)
    step = 0
    while any(a < n for a, n in zip(at, lens)):
        part = []
        for r in range(len(lens)):
            if step < len(cuts[r]):
                part.append((r, at[r], cuts[r][step]))
                at[r] += cuts[r][step]
        step += 1
        yield part


# =============================================================================== mechanisms alone

@pytest.mark.parametrize("T,H", [(1, 64), (7, 50), (5, 1028), (3, 2048), (2, 4100), (2, 4099), (200, 256)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_tanh_norm_in_the_seam(ops, T, H, out_dtype):
    """The scaled sum into the stream and tanh(alpha x) w + b of the new rows: with and without a sublayer's output, all rows or
    some; saturated and tiny values; an alpha that is negative."""
    tol = 3e-6 if out_dtype == torch.float32 else 6e-3
    x0, y = 4.0 * rnd(T, H, seed=1), 2.0 * rnd(T, H, seed=2)
    x0[:, ::5] *= 1e-4
    ls, w, b = (1.0 + 0.5 * rnd(H, seed=s) for s in (3, 4, 5))
    for alpha in (0.6, -1.7):
        for branch in (False, True):
            stream = d(x0.clone())
            got = ops.row_step(stream, d(y) if branch else None, (ops.NORM_NONE, d(ls), 0.0) if branch else None,
                               (ops.NORM_TANH, d(w), alpha, d(b)), out_dtype=out_dtype)
            want_x = x0.double() + (ls.double() * y.double() if branch else 0.0)
            params = {"n": w.double(), "n.b": b.double(), "n.alpha": torch.tensor(alpha, dtype=F64)}
            want = plain.dynamic_tanh(want_x, params, "n")
            assert rel_err(stream, want_x) < 1e-6 and rel_err(got, want) < tol
            rows = torch.tensor([T - 1, 0], dtype=torch.int32)
            stream = d(x0.clone())
            got = ops.row_step(stream, d(y) if branch else None, (ops.NORM_NONE, d(ls), 0.0) if branch else None,
                               (ops.NORM_TANH, d(w), alpha, d(b)), rows=d(rows), out_dtype=out_dtype)
            assert torch.equal(stream.cpu(), x0) and rel_err(got, want[rows.long()]) < tol


@pytest.mark.parametrize("w_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("T,ra,rg,heads,dk,V", [(1, 3, 7, 5, 12, 165), (9, 24, 24, 4, 32, 128), (70, 128, 128, 2, 128, 256), (130, 16, 72, 3, 40, 9),
                                                (8, 1, 2, 2, 70, 18), (65, 200, 8, 1, 64, 64)])
def test_second_halves_of_low_rank_projections(ops, w_dtype, T, ra, rg, heads, dk, V):
    """Decay per key channel and sigmoid gate from columns of a wider product, at aligned and odd columns; slow and fast decays
    (softplus on both sides of zero); each part alone too."""
    a2, g2 = rnd(heads * dk, ra, seed=1).to(w_dtype), rnd(V, rg, seed=2).to(w_dtype)
    A, bias = -torch.exp(rnd(heads, seed=3) * 2), 4.0 * rnd(heads * dk, seed=4)
    for extra in (0, 3):
        proj = rnd(T, 8 + ra + rg + 13 + extra, seed=5 + extra)
        ca, cg = 8 + extra, 8 + extra + ra
        za, zg = proj[:, ca:ca + ra].double() @ a2.double().T, proj[:, cg:cg + rg].double() @ g2.double().T
        want_a = torch.exp(A.double().repeat_interleave(dk) * plain.softplus(za + bias.double()))
        want_g = torch.sigmoid(zg)
        pa, pg = (ca, d(a2), ops.LOWRANK_DECAY, d(A), d(bias)), (cg, d(g2), ops.LOWRANK_SIGMOID, None, None)
        got = ops.lowrank_gates(d(proj), [pa, pg])
        for g, w in zip(got, (want_a, want_g)):
            assert float((g.double().cpu() - w).abs().max()) < (2e-5 if w_dtype == torch.float32 else 1e-4)
        assert torch.equal(ops.lowrank_gates(d(proj), [pg])[0], got[1]) and torch.equal(ops.lowrank_gates(d(proj), [pa])[0], got[0])
        assert torch.equal(ops.lowrank_gates(d(proj)[T - 1:], [pa])[0][0], got[0][T - 1])      # a row does not depend on the others


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("nq,d_,maps,nkv,dv,page", [(8, 16, 2, 2, 24, 8), (4, 64, 2, 1, 128, 16), (6, 5, 2, 1, 9, 8), (20, 5, 2, 1, 9, 16), (4, 32, 1, 2, 32, 64),
                                                    (2, 150, 2, 1, 20, 16), (8, 64, 2, 4, 96, 32)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_convolution_of_the_heads(ops, taps, nq, d_, maps, nkv, dv, page, dtype):
    """Queries in their map's place, keys and values on the pages of their positions, zeros around them; three requests in slots out
    of order in portions down to one token; a reader of another layer's keys convolves its queries alone."""
    lens, slots = [60, 9, 131], [2, 0, 3]
    cuts = [[33, 2, 1, 1, 20, 1, 2], [1] * 9, [1, 1, 64, 33, 2, 30]]
    dk = maps * d_
    step = 16 if dtype == torch.bfloat16 else 2
    dpad = -(-max(dk, dv) // step) * step
    tol = 2e-6 if dtype == torch.float32 else 6e-3
    g = torch.Generator().manual_seed(taps)
    blocks = [-(-L // page) for L in lens]
    ids = torch.randperm(sum(blocks) + 2, generator=g).tolist()
    own = [[ids.pop() for _ in range(b)] for b in blocks]
    for has_kv in (True, False):
        C = nq * d_ + (nkv * (dk + dv) if has_kv else 0)
        w = rnd(C, taps, seed=1)
        for pad in (0, 4, 5):
            data = [rnd(L, C + pad + 3, seed=10 + r) for r, L in enumerate(lens)]
            ref = [plain.short_conv(x[:, pad:pad + C].double(), w.double()) for x in data]
            state = torch.full((4, taps, C), float("nan"), device=DEV)
            kp = torch.full((sum(blocks) + 2, nkv, page, dpad), float("nan"), dtype=dtype, device=DEV)
            vp = kp.clone()
            for part in walk(cuts, lens):
                rows = Rows([n for _, _, n in part], [a for _, a, _ in part], [slots[r] for r, _, _ in part])
                table = torch.full((len(part), max(blocks)), -1, dtype=torch.int32)
                for i, (r, _, _) in enumerate(part):
                    table[i, :blocks[r]] = torch.tensor(own[r], dtype=torch.int32)
                x = d(torch.cat([data[r][a:a + n] for r, a, n in part]))
                q = ops.conv_heads(x[:, pad:], d(w.t()), state, rows, d(table), kp, vp, nq, d_, maps, nkv, dv, has_kv=has_kv)
                q = q.view(-1, nq, dpad).double().cpu()
                o = 0
                for r, a, n in part:
                    want = torch.zeros(n, nq, dpad, dtype=F64)
                    for h in range(nq):
                        off = h % maps * d_
                        want[:, h, off:off + d_] = ref[r][a:a + n, h * d_:(h + 1) * d_]
                    assert rel_err(q[o:o + n], want) < tol and torch.equal(q[o:o + n] == 0, want == 0)
                    o += n
            if not has_kv:
                assert torch.isnan(kp.float()).all() and torch.isnan(vp.float()).all()
                continue
            for r, L in enumerate(lens):
                for p in range(L):
                    for pool, c0, n in ((kp, nq * d_, dk), (vp, nq * d_ + nkv * dk, dv)):
                        got = pool[own[r][p // page], :, p % page].double().cpu()
                        want = ref[r][p, c0:c0 + nkv * n].view(nkv, n)
                        assert float((got[:, :n] - want).abs().max()) <= tol * float(ref[r].abs().max()), (r, p)
                        assert float(got[:, n:].abs().sum()) == 0.0
            if pad == 0:
                held = (kp.float() == kp.float()).all(-1).sum().item()
                assert held == sum(lens) * nkv         # nothing was written outside the requests' positions
            if taps > 4 and pad:
                break


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("heads,rep,dk,dv", [(80, 2, 36, 20), (4, 2, 16, 24), (2, 1, 160, 40), (3, 3, 12, 33), (2, 1, 128, 64), (4, 4, 40, 72), (1, 1, 256, 17), (2, 2, 64, 128), (40, 1, 128, 64), (5, 5, 30, 7)])
def test_channel_delta_rule_across_steps_and_slots(ops, heads, rep, dk, dv, chunked):
    """Portions of several sizes down to single tokens, slots out of order; decays per key channel that are 0 and 1 for some tokens
    and channels, step sizes 0 and 1; token by token and in chunks of tokens."""
    lens, slots = [70, 9, 131], [2, 0, 3]
    cuts = [[33, 2, 1, 1, 20, 13], [9], [1, 1, 64, 33, 2, 30]]
    K, V = heads // rep * dk, heads * dv
    data, want = [], []
    for r, L in enumerate(lens):
        x = rnd(L, 2 * K + V + 2, seed=20 + r)
        q, k = x[:, 2:2 + K].view(L, -1, dk), x[:, 2 + K:2 + 2 * K].view(L, -1, dk)
        q /= q.norm(dim=-1, keepdim=True)
        k /= k.norm(dim=-1, keepdim=True)
        gen = torch.Generator().manual_seed(r)
        g = 1.0 - 0.4 * torch.rand(L, heads, dk, generator=gen)
        b = torch.rand(L, heads, generator=gen)
        g[::17], g[3::5] = 0.0, 1.0
        g[1::6, :, ::3] = 0.0
        b[4::7], b[5::11] = 0.0, 1.0
        data.append((x, g.reshape(L, -1), b))
        want.append(plain.channel_delta_rule(q.double().repeat_interleave(rep, 1), k.double().repeat_interleave(rep, 1),
                                             x[:, 2 + 2 * K:].double().view(L, heads, dv), g.double(), b.double()).reshape(L, V))
    state = torch.zeros(4, heads, dk, dv, device=DEV)
    state[1] = float("nan")
    for part in walk(cuts, lens):
        rows = Rows([n for _, _, n in part], [a for _, a, _ in part], [slots[r] for r, _, _ in part])
        x, g, b = (d(torch.cat([data[r][i][a:a + n] for r, a, n in part])) for i in range(3))
        args = (x, 2, 2 + K, 2 + 2 * K, g, b, rows, state, heads, rep, dk, dv)
        got = ops.chunk_scan(True, *args) if chunked else ops.delta_scan(*args)
        o = 0
        for r, a, n in part:
            assert rel_err(got[o:o + n], want[r][a:a + n]) < 3e-5, (r, a, n)
            o += n


@pytest.mark.parametrize("chunked", [False, True])
def test_channel_decay_forgets_one_channel_and_keeps_another(ops, chunked):
    """Values written 400 tokens back along two channels: the one whose channel was closed once in between reads as nothing, the
    other in full; one that faded by a known factor reads faded."""
    dk, dv, L = 16, 8, 420
    for case, want in (("kept", 5.0), ("closed", 0.0), ("faded", 5.0 * 0.999 ** 409)):
        x = torch.zeros(L, 2 * dk + dv)
        x[:, dk + 1] = 1.0                      # every token writes along channel 1 ...
        x[:, 2 * dk:] = 1.0
        x[10, dk:2 * dk] = 0.0                  # ... token 10 along channel 0, value 5
        x[10, dk] = 1.0
        x[10, 2 * dk:] = 5.0
        g, b = torch.ones(L, dk), torch.ones(L, 1)
        g[:, 1] = 0.9
        if case == "closed":
            g[200, 0] = 0.0
        if case == "kept":
            g[200, 1] = 0.0                     # the other channel's
        if case == "faded":
            g[:, 0] = 0.999
        x[-1, 0] = 1.0                          # the last query asks for channel 0
        state = torch.zeros(1, 1, dk, dv, device=DEV)
        for lens in ([L], [211, 2, 200, 1, 6]):
            state.zero_()
            at = 0
            for n in lens:
                args = (d(x[at:at + n]), 0, dk, 2 * dk, d(g[at:at + n]), d(b[at:at + n]), Rows([n], [at], [0]), state, 1, 1, dk, dv)
                o = ops.chunk_scan(True, *args) if chunked else ops.delta_scan(*args)
                at += n
            assert float((o[-1].cpu() - want).abs().max()) < 2e-5 * max(1.0, want), (case, lens)


@pytest.mark.parametrize("heads,dv,dpad", [(3, 24, 32), (4, 128, 128), (2, 9, 16), (5, 7, 12), (1, 300, 304)])
@pytest.mark.parametrize("a_dtype,out_dtype", [(torch.float32, torch.float32), (torch.bfloat16, torch.bfloat16), (torch.float32, torch.bfloat16)])
def test_two_maps_become_one(ops, heads, dv, dpad, a_dtype, out_dtype):
    T, eps = 37, 1e-3
    a = torch.zeros(T, heads, 2, dpad)
    a[..., :dv] = rnd(T, heads, 2, dv, seed=1)
    a = a.to(a_dtype)
    gate = rnd(T, heads + 6, seed=2, scale=2.0)
    for g in (None, gate[:, 3:3 + heads]):
        lam = torch.tensor([0.37])
        got = ops.diff_combine(d(a.view(T, -1)), heads, dv, d(lam), eps, 0.6, None if g is None else gate.to(DEV)[:, 3:3 + heads], out_dtype)
        o = 0.6 * plain.rms_unit(a[:, :, 0, :dv].double() - float(lam) * a[:, :, 1, :dv].double(), eps)
        if g is not None:
            o = o * torch.sigmoid(g.double()).unsqueeze(-1)
        got = got.view(T, heads, dpad).cpu()
        assert rel_err(got[..., :dv], o) < (2e-6 if out_dtype == torch.float32 else 5e-3) and float(got[..., dv:].abs().sum()) == 0.0


@pytest.mark.parametrize("E,top", [(6, 2), (5, 1), (4, 4), (40, 3)])
def test_router_weights_are_a_softmax_over_the_chosen(ops, E, top):
    """Also where the logits lie so far apart that a softmax over all of them has only zeros beyond the first."""
    for T in (3, 60):
        z = rnd(T, E, seed=E, scale=3.0)
        z[0] = torch.arange(E).float() * -200.0
        z[1] = z[1] - 5000.0
        sel, wt = ops.moe_route(d(z), top, 2, True)
        best = torch.topk(z.double(), top)
        assert torch.equal(sel.cpu().long(), best.indices) and float((wt.cpu().double() - torch.softmax(best.values, -1)).abs().max()) < 1e-6
    with pytest.raises(ops.KernelError):
        ops.moe_route(d(z), top, 2, False)
    with pytest.raises(ops.KernelError):
        ops.moe_route(d(z), top, 2, True, bias=d(torch.zeros(E)))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("W,ff,experts,top", [(64, 32, 6, 2), (96, 200, 5, 1), (50, 21, 3, 3), (128, 136, 4, 2), (256, 64, 12, 3)])
def test_experts_without_a_gate(ops, dtype, W, ff, experts, top):
    """Few tokens (one kernel routes and regroups) and many; each token's result does not depend on the others."""
    from blackwellllm_b200.config.specs import RoutedFFNSpec
    from blackwellllm_b200.parts import BuildContext, build_ffn
    part = build_ffn(RoutedFFNSpec(experts, top, ff, score="softmax_chosen", activation="relu2"), W, BuildContext(DEV, _DT[dtype]))
    t = {p.name: rnd(*p.shape, seed=i, scale=1.0 if p.name == "router" else 0.2).to(_DT[dtype]) for i, p in enumerate(part.param_specs())}
    part.bind({k: d(v) for k, v in t.items()})
    assert part.tc == (dtype == "bfloat16" and W % 8 == 0 and ff % 8 == 0)
    for T in (1, 7, 150):
        x = rnd(T, W, seed=T).to(_DT[dtype])
        want = plain.routed_ffn(x.double(), {k: v.double() for k, v in t.items()}, {"router": {"top": top}})
        out = torch.full((T, W), float("nan"), device=DEV)
        part.forward(d(x), out, None, accumulate=None)
        assert rel_err(out, want) < (1e-5 if dtype == "float32" else 1e-2)
        base = rnd(T, W, seed=3)
        res = d(base.clone())
        part.forward(d(x), res, None)
        assert rel_err(res, base.double() + want) < (1e-5 if dtype == "float32" else 1e-2)


def test_gated_gelu_feed_forward(ops):
    from blackwellllm_b200.config.specs import SwiGLUSpec
    from blackwellllm_b200.parts import BuildContext, build_ffn
    for dtype in ("float32", "bfloat16"):
        part = build_ffn(SwiGLUSpec(80, activation="gelu_tanh", names=("gate", "up", "down")), 64, BuildContext(DEV, _DT[dtype]))
        t = {p.name: rnd(*p.shape, seed=i, scale=0.3).to(_DT[dtype]) for i, p in enumerate(part.param_specs())}
        part.bind({k: d(v) for k, v in t.items()})
        x = rnd(9, 64, seed=9).to(_DT[dtype])
        out = torch.zeros(9, 64, device=DEV)
        part.forward(d(x), out, None, accumulate=False)
        assert rel_err(out, plain.dense_ffn(x.double(), {k: v.double() for k, v in t.items()})) < (1e-5 if dtype == "float32" else 1e-2)


@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,dq,dv,rd", [(6, 3, 48, 48, 48), (4, 2, 32, 16, 16), (3, 1, 10, 7, 6), (2, 1, 128, 128, 64), (4, 4, 64, 96, 62),
                                             (20, 1, 8, 12, 2), (2, 2, 256, 40, 256), (4, 2, 12, 12, 4)])
def test_rotation_of_neighbouring_channels(ops, out_dtype, nh, nkv, dq, dv, rd):
    """Pairs (2i, 2i + 1) of queries and keys turned, the rest passed, values scaled, with a gate's columns behind; aligned and odd
    rows, with and without norms in front; positions far from 0."""
    from blackwellllm_b200.parts.rope import rotary_inv_freq
    from test_kernels_gpu import FakeBatch
    page, T, L = 8, 19, 700
    cols = nh * dq + nkv * (dq + dv)
    dpad = -(-max(dq, dv) // 16) * 16
    tol = 6e-6 if out_dtype == torch.float32 else 8e-3
    blocks = -(-L // page)
    pages = torch.randperm(blocks, generator=torch.Generator().manual_seed(1)).tolist()
    batch, table = FakeBatch([T], [L]), torch.tensor([pages], dtype=torch.int32, device=DEV)
    cs = ops.rope_table(batch.positions, rotary_inv_freq(300.0, rd).to(DEV), rd)
    gq, gk = 1.0 + 0.4 * rnd(dq, seed=3), 1.0 + 0.4 * rnd(dq, seed=4)
    for extra in (nh, 8 - cols % 8, 5):
        qkv = rnd(T, cols + extra, seed=dq + extra)
        x = torch.zeros(L, cols, dtype=F64)
        x[L - T:] = qkv[:, :cols].double()
        for normed in (False, True):
            q, k, v = x[:, :nh * dq].view(L, nh, dq), x[:, nh * dq:(nh + nkv) * dq].view(L, nkv, dq), 0.7 * x[L - T:, (nh + nkv) * dq:].view(T, nkv, dv)
            if normed:
                q, k = plain.rms_unit(q, 1e-3) * gq.double(), plain.rms_unit(k, 1e-3) * gk.double()
            q, k = plain.rotate_pairs(q, 300.0, rd)[L - T:], plain.rotate_pairs(k, 300.0, rd)[L - T:]
            kp = torch.full((blocks, nkv, page, dpad), float("nan"), dtype=out_dtype, device=DEV)
            vp = kp.clone()
            gains = (d(gq), d(gk)) if normed else (None, None)
            got = ops.head_norm_rope_append(d(qkv), batch, table, cs, rd, True, gains[0], gains[1], 1e-3, kp, vp, nh, nkv, dq, dv, v_scale=0.7)
            got = got.view(T, nh, dpad).double().cpu()
            assert rel_err(got[..., :dq], q) < tol * 10 and (dpad == dq or float(got[..., dq:].abs().max()) == 0.0)
            for t in range(T):
                p = L - T + t
                kt, vt = kp[pages[p // page], :, p % page].double().cpu(), vp[pages[p // page], :, p % page].double().cpu()
                assert float((kt[:, :dq] - k[t]).abs().max()) <= tol * 10 * float(k.abs().max())
                assert float((vt[:, :dv] - v[t]).abs().max()) <= tol * float(v.abs().max())
                assert float(kt[:, dq:].abs().sum()) == 0.0 and float(vt[:, dv:].abs().sum()) == 0.0


def step_batch(cm, part, at, group=0):
    """The batch of a step of (request, tokens) on a cache manager, after the requests were grown."""
    from test_kernels_gpu import FakeBatch
    batch = FakeBatch([n for _, n in part], [at[r] + n for r, n in part])
    batch.state_slot = torch.tensor([cm.slot(r) for r, _ in part], dtype=torch.int32, device=DEV)
    batch.block_tables = {}
    for g in range(len(cm.groups)):
        width = max(cm.num_blocks(r, g) for r, _ in part)
        table = torch.full((len(part), width), -1, dtype=torch.int32)
        for i, (r, _) in enumerate(part):
            row = cm.block_table(r, g)
            table[i, :len(row)] = torch.tensor(row, dtype=torch.int32)
        batch.block_tables[g] = d(table)
    return batch


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("dim,vdim", [(16, 24), (32, 64), (64, 128)])
@pytest.mark.parametrize("which", [0, 1])
def test_one_loud_key_at_the_edge_of_a_block_of_positions(ops, dtype, dim, vdim, which):
    """Differential attention whose scores are all 0 but one key's in one of its maps.  The row's value turns with that key just
    inside its block of positions and does not just outside it or hundreds of tokens back; in portions (also of two tokens) and
    decoded, at page borders."""
    from blackwellllm_b200.cache.manager import CacheManager
    from blackwellllm_b200.config.specs import DifferentialAttentionSpec
    from blackwellllm_b200.parts import BuildContext, build_mixer
    W, H, G, size, L, page, taps = 64, 2, 1, 96, 500, 16, 3
    spec = DifferentialAttentionSpec(H, G, dim, vdim, taps, 0.3, 1e-6, 1.0, chunk=size,
                                     names=tuple((r, r) for r in ("q", "k", "v", "lq1", "lk1", "lq2", "lk2", "o", "q_conv", "k_conv", "v_conv")))
    t = {n: torch.zeros(s.shape) for n, s in ((p.name, p) for p in build_mixer(spec, W, BuildContext(torch.device("cpu"), torch.float32)).param_specs())}
    for c in ("q_conv", "k_conv", "v_conv"):
        t[c][:, -1] = 1.0                                  # the convolution passes the current token
    for h in range(H):
        t["q"][(2 * h + which) * dim, 0] = 4.0             # every token asks along channel 0 of one map
        t["o"][h, h * vdim] = 1.0
        t["o"][8 + h, h * vdim + 1] = 1.0
    t["k"][which * dim, 1] = 4.0                           # only a loud token answers
    t["v"][0, 0] = 1.0                                     # quiet tokens: value along channel 0, loud: channel 1
    t["v"][1, 1] = 1.0
    edge = (L - 1) // size * size
    mixer = build_mixer(spec, W, BuildContext(DEV, _DT[dtype]))
    mixer.bind({k: d(v.to(_DT[dtype])) for k, v in t.items()})
    m = {"heads": H, "kv_heads": G, "dim": dim, "vdim": vdim, "scale": 1.0, "diff": 0.3, "mask": {"size": size}}
    w = {k.replace("_", "."): v.to(_DT[dtype]).double() for k, v in t.items()}
    w["g"] = torch.full((H, W), 0.0, dtype=F64)
    results = {}
    for loud in (edge, edge - 1, L - 1, 3, edge - size):
        x = torch.zeros(L, W)
        x[:, 0] = 1.0
        x[loud, 1] = 1.0
        h = x.double()
        want = 2.0 * plain.differential_attention(h, w, m, 1e-6, plain.keys_values(h, w, m))      # (a gate of one half)
        for cuts in ([L], [edge - 1, 2, L - edge - 1], [edge + 2] + [1] * (L - edge - 2), [L - 2, 2]):
            cm = CacheManager([mixer.cache_request()], page, 40, 1, dtype=_DT[dtype], device=DEV)
            cm.add_request(0)
            at, got = {0: 0}, []
            for n in cuts:
                cm.append(0, n)
                batch = step_batch(cm, [(0, n)], at)
                res = torch.zeros(n, W, device=DEV)
                mixer.forward(d(x[at[0]:at[0] + n].to(_DT[dtype])), res, batch, cm.views[0], accumulate=False)
                got.append(res.double().cpu())
                at[0] += n
            got = torch.cat(got)
            assert rel_err(got[-40:], want[-40:]) < (1e-4 if dtype == "float32" else 2e-2), (loud, cuts[:3])
        results[loud] = want[-1]
    # the oracle itself tells the cases apart
    assert float((results[edge] - results[edge - 1]).abs().max()) > 0.3 and float((results[edge - 1] - results[3]).abs().max()) < 1e-9


@pytest.mark.parametrize("hd,nh,nkv,page", [(48, 4, 2, 16), (64, 4, 1, 8), (64, 32, 4, 16), (128, 8, 4, 16), (192, 4, 2, 32), (256, 4, 1, 64), (16, 16, 1, 8),
                                            (80, 6, 3, 16), (64, 16, 1, 5), (128, 16, 1, 16), (64, 40, 2, 16), (272, 4, 2, 16)])
@pytest.mark.parametrize("q_lens,kv_lens", [([1, 1], [700, 33]), ([1], [2500]), ([50, 1, 3], [400, 90, 3]), ([130], [131]), ([1] * 9, [70] * 9)])
def test_pairs_of_heads_become_one_in_the_attention_kernels(ops, hd, nh, nkv, page, q_lens, kv_lens):
    """bfloat16, every kernel's epilogue (prompt tiles on either tensor path, one key slice, few and many slices): a1 - lambda a2 in
    float32 before anything is rounded, over the channels that are values, times the gate of the head.  (Maps that nearly cancel:
    outputs rounded one by one would be off by far more than the bound.)"""
    from test_kernels_gpu import FakeBatch, paged_case
    dv = hd - hd // 8
    chunk, eps, factor = 200, 1e-6, 0.7

    def spike(r, q, k, v):
        v[..., dv:] = 0
        q[:, 1::2] = q[:, 0::2] + 0.1 * q[:, 1::2]
    q, kp, vp, table, refs = paged_case(q_lens, kv_lens, nh, nkv, hd, page, torch.bfloat16, seed=hd, spike=spike)
    T, H = sum(q_lens), nh // 2
    lam = torch.tensor([0.9])
    gate = rnd(T, H + 3, seed=1)
    batch = FakeBatch(q_lens, kv_lens)
    scale = 0.5 * hd ** -0.5
    out = ops.paged_attention(q, kp, vp, batch, table, nh, None, scale, chunk, gate=(gate.to(DEV)[:, 2:2 + H], dv, "head"),
                              diff=(d(lam), eps, factor, dv)).view(T, H, hd).double().cpu()
    want = []
    for q_, k_, v_, start in refs:
        L = q_.shape[0]
        seen = plain.block_mask(L, chunk)[start:]
        maps = [plain.softmax_rows(q_[start:, h].double() @ k_[:, h // (nh // nkv)].double().T * scale, seen) @ v_[:, h // (nh // nkv), :dv].double()
                for h in range(nh)]
        want.append(torch.stack([plain.rms_unit(maps[2 * h] - float(lam) * maps[2 * h + 1], eps) * factor for h in range(H)], 1))
    want = torch.cat(want) * torch.sigmoid(gate[:, 2:2 + H].double()).unsqueeze(-1)
    assert float(out[..., dv:].abs().sum()) == 0.0
    # (the CUDA-core kernel, for sizes the others do not take, rounds its outputs first; attention weights are bfloat16 in P V)
    err = float((out[..., :dv] - want).abs().max()) / float(want.abs().max())
    assert err < (0.2 if nh // nkv > 16 or hd > 256 else 0.06), err


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("hd", [48, 64])
@pytest.mark.parametrize("q_len", [1, 2, 50])
def test_one_loud_key_in_blocks_with_a_gate_per_head(ops, dtype, hd, q_len):
    """All scores of the last query are 0 but one key's: seen from the block's first position on, not one token before; the gate
    per head multiplies."""
    from test_kernels_gpu import FakeBatch, paged_case
    nh, nkv, page, size, L = 4, 2, 16, 36, 700
    last, first = L - 1, (L - 1) // 36 * 36
    g = torch.zeros(q_len, nh + 2)
    g[:, 1:1 + nh] = torch.tensor([0.0, math.log(3.0), -50.0, 50.0])
    share = torch.tensor([0.5, 0.75, 0.0, 1.0]).view(nh, 1)
    for loud, seen in [(first, True), (first - 1, False), (last, True), (0, False), (last - 63, False)]:
        def spike(r, q, k, v):
            k[:] = 0
            k[loud, :, 0] = 8.0
            q[-1] = 0
            q[-1, :, 0] = 5.0
            v[:] = 1.0
            v[loud] = 5.0
        q, kp, vp, table, _ = paged_case([q_len], [L], nh, nkv, hd, page, _DT[dtype], seed=2, spike=spike)
        out = ops.paged_attention(q, kp, vp, FakeBatch([q_len], [L]), table, nh, None, 1.0, chunk=size, gate=(d(g)[:, 1:1 + nh], hd, "head"))
        row = out[-1].float().cpu().view(nh, hd)
        want = share * (5.0 if seen else 1.0)
        assert float((row - want).abs().max()) < 0.03, (loud, seen)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,layer", [("mixed", 0), ("mixed", 1), ("mixed", 2), ("mixed", 3), ("tensor", 0), ("tensor", 1), ("tensor", 2), ("tensor", 3),
                                        ("open", 0), ("open", 1), ("open", 2), ("open", 3), ("open", 4), ("broad", 0), ("broad", 1)])
def test_mixer_alone(ops, dtype, name, layer):
    """Each mixer against the plain functions: portions and then single tokens, next to another request; in a tensor of its own, added
    to one that holds something, and as the open form a block takes.  A reader of another layer's keys runs behind that layer."""
    from blackwellllm_b200.cache.manager import CacheManager
    from blackwellllm_b200.config.registry import parse_config
    from blackwellllm_b200.parts import BorrowedCache, BuildContext, build_mixer
    raw, page = tz.CONFIGS[name]
    W, eps, entry = raw["width"], raw["norm"]["eps"], raw["layers"][layer]
    m = entry["mixer"]
    src = m.get("kv_from")
    cfg, tensors = parse_config(raw), tz.make_tensors(raw, seed=11, dtype=_DT[dtype])
    ctx = BuildContext(DEV, _DT[dtype])

    def bound(i):
        part = build_mixer(cfg.layers[i].mixer, W, ctx)
        t = plain.sub(tensors, f"l{i}.mix.")
        part.bind({k: d(v) for k, v in t.items()})
        return part, {k: v.double() for k, v in t.items()}
    mixer, w = bound(layer)
    lender, w_lender = bound(src) if src is not None else (None, None)
    L = {0: 75, 1: 30}
    xs = {r: rnd(n, W, seed=60 + r).to(_DT[dtype]) for r, n in L.items()}
    other = {r: rnd(n, W, seed=70 + r).to(_DT[dtype]) for r, n in L.items()}       # what the lender reads
    want = {}
    for r, x in xs.items():
        h = x.double()
        if entry["type"] == "parallel":
            want[r] = (m["left_scale"] * plain.rotary_attention(h, plain.sub(w, "left."), m["left"])
                       + m["right_scale"] * plain.channel_delta(h, plain.sub(w, "right."), m["right"], eps))
        else:
            kv = plain.keys_values(h, w, m) if src is None else plain.keys_values(other[r].double(), w_lender, raw["layers"][src]["mixer"])
            want[r] = plain.differential_attention(h, w, m, eps, kv)
    tol = 3e-5 if dtype == "float32" else 5e-2
    for form in ("write", "add", "open"):
        requests = [mixer.cache_request()] if src is None else [lender.cache_request(), mixer.borrower_request()]
        cm = CacheManager(requests, page, 16, 3, dtype=_DT[dtype], device=DEV)
        for r in (1, 0):
            cm.add_request(r)
        at, got = {0: 0, 1: 0}, {0: [], 1: []}
        for step in [[(0, 33), (1, 2)], [(1, 1), (0, 30)]] + [[(0, 1), (1, 1)] for _ in range(12)]:
            for r, n in step:
                cm.append(r, n)
            batch = step_batch(cm, step, at)
            x = d(torch.cat([xs[r][at[r]:at[r] + n] for r, n in step]))
            cache = cm.views[0]
            if src is not None:
                scratch = torch.zeros(x.shape[0], W, device=DEV)
                lender.forward(d(torch.cat([other[r][at[r]:at[r] + n] for r, n in step])), scratch, batch, cm.views[0], accumulate=False)
                cache = BorrowedCache(cm.views[0], cm.views[1])
            res = d(rnd(x.shape[0], W, seed=5))
            base = res.clone()
            if form == "open":
                if hasattr(mixer, "forward_open"):
                    y = mixer.forward_open(x, batch, cache)
                else:
                    y = torch.full_like(res, float("nan"))
                    mixer.forward(x, y, batch, cache, src is None, accumulate=None)
                ops.row_step(res, y)
            else:
                mixer.forward(x, res, batch, cache, src is None, accumulate=form == "add")
                ops.resolve_pending()
            if form != "write":
                res = res - base
            o = 0
            for r, n in step:
                got[r].append(res[o:o + n].cpu().double())
                o += n
                at[r] += n
        for r in (0, 1):
            g = torch.cat(got[r])
            assert rel_err(g, want[r][:g.shape[0]]) <= tol, (form, r)


# =============================================================================== whole models through the engine

_models = {}


def plain_logits(raw, tensors, ids, streams=None):
    return plain.forward(raw, {k: v.double() for k, v in tensors.items()}, ids, streams)


def model(name, dtype):
    key = (name, dtype)
    if key not in _models:
        raw, page = tz.CONFIGS[name]
        tensors = tz.make_tensors(raw, seed=7, dtype=_DT[dtype])
        reqs = {f"r{i}": tz.prompt(n, raw["vocab"], 50 + i) for i, n in enumerate([70, 33, 131, 2, 90])}
        ref = {rid: plain_logits(raw, tensors, ids) for rid, ids in reqs.items()}
        _models[key] = (raw, page, tensors, reqs, ref)
    return _models[key]


def engine_for(name, dtype, **kw):
    from blackwellllm_b200.engine.engine import Engine
    raw, page, tensors, _, _ = model(name, dtype)
    opts = dict(dtype=dtype, page_size=page, num_pages=64, max_requests=4, max_batch_tokens=1 << 16)
    opts.update(kw)
    return Engine.from_tensors(raw, tensors, **opts)


def check_rows(rows, ref, dtype, what):
    """rows {(rid, pos): logits}: every row within the bound.  (bfloat16: a router's close call may take another expert at one place
    in fifty; such a place differs by an expert's output, not by orders.)"""
    errs = {key: float((row.double().cpu() - ref[key[0]][key[1]]).abs().max()) / float(ref[key[0]].abs().max()) for key, row in rows.items()}
    over = {key: e for key, e in errs.items() if not e <= TOL[dtype]}
    allowed = 0 if dtype == "float32" else len(errs) // 50
    assert len(over) <= allowed and all(e <= 0.5 for e in over.values()), (what, over)


def run_steps(eng, steps):
    """steps: [[(rid, tokens, start)]]: every position's logits by (rid, position)."""
    from blackwellllm_b200.engine.engine import StepEntry
    rows = {}
    for step in steps:
        out = eng.step([StepEntry(rid, toks, list(range(len(toks)))) for rid, toks, _ in step]).cpu()
        at = 0
        for rid, toks, start in step:
            for i in range(len(toks)):
                rows[(rid, start + i)] = out[at + i].clone()
            at += len(toks)
    return rows


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tz.CONFIGS))
def test_whole_prompts_and_the_stream_after_every_layer(name, dtype):
    raw, _, tensors, reqs, ref = model(name, dtype)
    eng = engine_for(name, dtype)
    streams, want_streams = [], []
    plain_logits(raw, tensors, reqs["r0"], want_streams)
    eng.model.stream_hook = lambda pos, h: streams.append(h.double().cpu().clone())
    rows = run_steps(eng, [[("r0", reqs["r0"], 0)]])
    eng.model.stream_hook = None
    assert len(streams) == len(want_streams) == len(raw["layers"])
    if dtype == "float32":
        for i, (got, want) in enumerate(zip(streams, want_streams)):
            assert float((got - want).abs().max()) <= 2e-5 * float(want.abs().max()), f"layer {i}"
    eng.end_request("r0")
    for rid in ("r1", "r2", "r3", "r4"):
        rows.update(run_steps(eng, [[(rid, reqs[rid], 0)]]))
        eng.end_request(rid)
    check_rows(rows, ref, dtype, "whole")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tz.CONFIGS))
def test_token_by_token_from_the_first_token(name, dtype):
    """Decoding from position 0 (the first tokens of a sequence, every page border, the blocks' edges passing over decoded tokens,
    recurrences and convolutions from their zero states), long enough that the decode steps are replayed from a CUDA graph."""
    _, _, _, reqs, ref = model(name, dtype)
    eng = engine_for(name, dtype)
    ids = reqs["r2"]
    rows = run_steps(eng, [[("r2", [t], i)] for i, t in enumerate(ids)])
    check_rows(rows, ref, dtype, "token by token")
    assert eng.graph_kernel_count(1) > 0


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tz.CONFIGS))
@pytest.mark.parametrize("sizes", [(2,), (7, 2, 13, 3, 5, 2, 16, 17, 4, 31, 2), (64, 1, 1, 1, 40, 1)])
def test_portions(name, dtype, sizes):
    _, _, _, reqs, ref = model(name, dtype)
    eng = engine_for(name, dtype)
    rows = {}
    for rid in ("r0", "r2", "r4"):
        ids, at, k, steps = reqs[rid], 0, 0, []
        while at < len(ids):
            n = min(sizes[k % len(sizes)], len(ids) - at)
            steps.append([(rid, ids[at:at + n], at)])
            at, k = at + n, k + 1
        rows.update(run_steps(eng, steps))
        eng.end_request(rid)
    check_rows(rows, ref, dtype, f"portions {sizes}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(tz.CONFIGS))
def test_unequal_requests_together_and_pages_used_again(name, dtype):
    """A pool that holds two requests: five pass through, portions of one beside single tokens of another; every later request gets a
    slot (with the states of its layers in it) and pages that an earlier one gave back."""
    raw, page, _, reqs, ref = model(name, dtype)
    eng = engine_for(name, dtype, num_pages=-(-(131 + 90) // page) + 2, max_requests=2)
    waiting = list(reqs.items())
    live, rows = {}, {}
    g = torch.Generator().manual_seed(3)
    while waiting or live:
        while waiting and len(live) < 2:
            rid, ids = waiting.pop(0)
            live[rid] = 0
        step = []
        for rid in list(live):
            ids, at = reqs[rid], live[rid]
            if at >= len(ids) - 6:
                n = 1
            else:
                n = min(int(torch.randint(2, 30, (1,), generator=g)), len(ids) - 6 - at)
            step.append((rid, ids[at:at + n], at))
            live[rid] = at + n
        rows.update(run_steps(eng, [step]))
        for rid in list(live):
            if live[rid] == len(reqs[rid]):
                eng.end_request(rid)
                del live[rid]
    check_rows(rows, ref, dtype, "mixed")
    eng.cache.check_invariants()
    assert eng.cache.slots.num_free == 2


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["mixed", "tensor"])
def test_a_long_request_in_portions_then_decoded(name, dtype):
    """700 tokens: dozens of blocks of positions, the recurrences have run 700 steps; prompt portions that start and end inside
    pages, then 40 tokens one by one."""
    raw, page, tensors, _, _ = model(name, dtype)
    ids = tz.prompt(700, raw["vocab"], 999)
    ref = {"long": plain_logits(raw, tensors, ids)}
    eng = engine_for(name, dtype, num_pages=-(-700 // page) + 1, max_requests=1)
    steps, at = [], 0
    for n in (333, 2, 190, 135):
        steps.append([("long", ids[at:at + n], at)])
        at += n
    steps += [[("long", [ids[i]], i)] for i in range(at, 700)]
    check_rows(run_steps(eng, steps), ref, dtype, "long")


@pytest.mark.parametrize("name", list(tz.CONFIGS))
def test_a_batch_changes_no_bit_of_a_request(name):
    """float32: a request's logits beside other requests equal its logits alone, bit for bit."""
    _, _, _, reqs, _ = model(name, "float32")
    alone = engine_for(name, "float32")
    a = run_steps(alone, [[("r1", reqs["r1"][:20], 0)], [("r1", reqs["r1"][20:21], 20)]])
    both = engine_for(name, "float32")
    b = run_steps(both, [[("r4", reqs["r4"][:9], 0), ("r1", reqs["r1"][:20], 0), ("r0", reqs["r0"][:3], 0)],
                         [("r0", reqs["r0"][3:4], 3), ("r1", reqs["r1"][20:21], 20), ("r4", reqs["r4"][9:40], 9)]])
    for key, row in a.items():
        assert torch.equal(row, b[key]), key


def test_a_request_left_out_of_steps_goes_on_where_it_was():
    """A request that sits out some steps finds its states and its keys as it left them, while another request in the neighbouring
    slot runs on."""
    _, _, _, reqs, ref = model("mixed", "float32")
    eng = engine_for("mixed", "float32")
    a, b = reqs["r0"], reqs["r4"]
    steps = [[("r0", a[:10], 0), ("r4", b[:3], 0)], [("r4", b[3:50], 3)], [("r4", b[50:51], 50)],
             [("r0", a[10:11], 10), ("r4", b[51:52], 51)], [("r0", a[11:70], 11)], [("r4", b[52:90], 52)]]
    check_rows(run_steps(eng, steps), ref, "float32", "left out")


@pytest.mark.parametrize("name", list(tz.CONFIGS))
def test_greedy_generation_through_the_entry_point(name, tmp_path):
    """generate() (scheduler, sampling, continuous batching) gives the plain implementation's greedy tokens."""
    import os
    from safetensors.torch import load_file
    from blackwellllm_b200 import BlackwellEngine, InferenceConfig, SamplingParams
    raw, page = tz.CONFIGS[name]
    folder = tz.make_folder(name, "float32", str(tmp_path))
    W = {k: v.double() for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}
    prompts = [tz.prompt(n, raw["vocab"], 80 + n) for n in (5, 40, 1)]
    steps = 12
    llm = BlackwellEngine(folder, InferenceConfig(max_context_length=128, max_batch_size=3), dtype="float32")
    got = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=steps))
    for p, g in zip(prompts, got):
        assert list(g.token_ids) == plain.greedy(raw, W, p, steps)


def test_command_line_and_position_addressed_calls(tmp_path, capsys):
    import os
    from safetensors.torch import load_file
    from blackwellllm_b200 import BlackwellEngine, InferenceConfig, cli
    name = "mixed"
    raw, _ = tz.CONFIGS[name]
    folder = tz.make_folder(name, "float32", str(tmp_path))
    W = {k: v.double() for k, v in load_file(os.path.join(folder, "model.safetensors")).items()}
    prompt = tz.prompt(9, raw["vocab"], 4)
    want = plain.greedy(raw, W, prompt, 6)
    rc = cli.main(["-m", folder, "--dtype", "float32", "--ctx", "128", "--temperature", "0", "--max-new-tokens", "6",
                   "--prompt-ids", ",".join(map(str, prompt))])
    out = capsys.readouterr().out
    assert rc == 0 and [int(t) for t in out.strip().splitlines()[0].split()] == want
    llm = BlackwellEngine(folder, InferenceConfig(max_context_length=128, max_batch_size=2), dtype="float32")
    nxt = llm.prefill(prompt, start_pos=0, temperature=0.0, seq_id=0)
    got = [nxt]
    for i in range(5):
        nxt = llm.forward(nxt, pos=len(prompt) + i, temperature=0.0, seq_id=0)
        got.append(nxt)
    assert got == want


def test_an_inner_size_that_the_configuration_does_not_state(tmp_path):
    """The low-rank projections' inner sizes come from the stored tensors."""
    import copy
    raw, page, tensors, reqs, ref = model("mixed", "float32")
    open_raw = copy.deepcopy(raw)
    for layer in open_raw["layers"]:
        for key in ("decay_rank", "gate_rank"):
            layer["mixer"].get("right", {}).pop(key, None)
    from blackwellllm_b200.engine.engine import Engine
    eng = Engine.from_tensors(open_raw, tensors, dtype="float32", page_size=page, num_pages=40, max_requests=1)
    check_rows(run_steps(eng, [[("r1", reqs["r1"], 0)]]), ref, "float32", "open sizes")
    bad = dict(tensors)
    bad["l1.mix.right.a1"] = bad["l1.mix.right.a1"][:-1]
    with pytest.raises(ValueError, match="a1"):
        Engine.from_tensors(open_raw, bad, dtype="float32", page_size=page, num_pages=40, max_requests=1)


# =============================================================================== bin/trace_run

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("family", ["tail", "portions", "mixed"])
def test_replay(tmp_path_factory, dtype, family):
    import os
    from safetensors.torch import load_file
    name = "mixed"
    raw, page = tz.CONFIGS[name]
    folder = tz.make_folder(name, dtype, str(tmp_path_factory.mktemp("zogulorn")))
    W = load_file(os.path.join(folder, "model.safetensors"))
    reqs = {f"q{i}": tz.prompt(n, raw["vocab"], 200 + i) for i, n in enumerate([40, 97, 50, 70, 130, 65])}
    ref = {rid: plain_logits(raw, W, ids) for rid, ids in reqs.items()}
    if family == "tail":
        steps, max_tokens = replay.trace_tail(reqs)
    elif family == "portions":
        steps, max_tokens = replay.trace_portions(reqs)
    else:
        max_tokens = 384
        steps = replay.trace_mixed(reqs, max_tokens, seed=3)
    rows = replay.run_trace(folder, dtype, steps, max_tokens, raw["vocab"], page_size=page)
    check_rows(rows, ref, dtype, f"replay {family}")


# =============================================================================== random configurations

def _random_configuration(rng):
    def pick(*xs):
        return xs[int(torch.randint(0, len(xs), (1,), generator=rng))]

    def mlp():
        return pick(None, tz.dense(pick(24, 41)), tz.moe(3, pick(1, 2, 3), pick(16, 19)), tz.moe(7, 2, 24))
    layers, lenders = [], []
    for i in range(pick(2, 3, 4)):
        if pick(0, 1):
            kv, dim, rk = pick(1, 2, 3), pick(6, 8, 12, 20), pick(1, 2)
            layers.append(tz._par(tz._rot(kv * pick(1, 2, 3), kv, dim, pick(4, dim, 24), pick(0.2, 0.9), pick(None, 1, 3, 11, 40), pick(50.0, 10000.0), pick(2, 4, dim)),
                                  (rk * pick(1, 2, 3), rk, pick(4, 20, 40), pick(4, 31, 32), pick(1, 2, 4, 7)), (pick(3, 8), pick(2, 16)),
                                  (pick(0.3, 1.0, -1.2), pick(0.4, 1.0)), mlp()))
            continue
        src = lenders[int(torch.randint(0, len(lenders), (1,), generator=rng))] if lenders and pick(0, 1) else None
        kv, dim, vdim = (pick(1, 2, 3), pick(5, 8, 16), pick(8, 10, 33)) if src is None else \
            tuple(layers[src]["mixer"][k] for k in ("kv_heads", "dim", "vdim"))
        layers.append(tz._dif(kv * pick(1, 2, 3), kv, dim, vdim, pick(0.2, 0.9), pick(None, 1, 3, 11, 40), pick(1, 2, 4, 7), pick(0.1, 0.5, 0.8), mlp(), src))
        if src is None:
            lenders.append(i)
    return tz._model(pick(60, 130), pick(40, 48, 71), pick(1e-6, 1e-3), pick(0.5, 1.0, 3.0), layers), pick(8, 16)


@pytest.mark.parametrize("seed", range(12))
def test_random_configurations_float32(seed):
    from blackwellllm_b200.engine.engine import Engine
    rng = torch.Generator().manual_seed(3000 + seed)
    raw, page = _random_configuration(rng)
    tensors = tz.make_tensors(raw, seed=seed, dtype=torch.float32)
    ids = tz.prompt(90, raw["vocab"], seed)
    ref = {"a": plain_logits(raw, tensors, ids)}
    eng = Engine.from_tensors(raw, tensors, dtype="float32", page_size=page, num_pages=24, max_requests=2)
    check_rows(run_steps(eng, [[("a", ids, 0)]]), ref, "float32", "whole")
    eng.end_request("a")
    steps, at = [], 0
    while at < 90:
        n = min(int(torch.randint(1, 25, (1,), generator=rng)), 90 - at)
        steps.append([("a", ids[at:at + n], at)])
        at += n
    check_rows(run_steps(eng, steps), ref, "float32", "portions")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_blocks_of_other_kinds_after_an_open_seam(dtype):
    """A stack of this design's layers between plain pre-norm ones (no layer scale): the seam left open is made before the other kind
    of block reads the stream, and a sum the other kind leaves open before this kind does."""
    import dataclasses
    from blackwellllm_b200.config.registry import parse_config
    from blackwellllm_b200.engine.engine import Engine, EngineOptions
    from blackwellllm_b200.weights.loader import bind_tensors
    raw, page = tz.CONFIGS["broad"]
    cfg = parse_config(raw)
    bare = [dataclasses.replace(ls, layer_scale=None) for ls in cfg.layers]
    mixed = dataclasses.replace(cfg, layers=(bare[1], cfg.layers[0], bare[0], cfg.layers[1]),
                                schedule=tuple(dataclasses.replace(cfg.schedule[0], layer=i) for i in range(4)))
    tensors = tz.make_tensors(raw, seed=2, dtype=_DT[dtype])
    src = [1, 0, 0, 1]
    named = {k: v for k, v in tensors.items() if not k.startswith(("l0.", "l1."))}
    for i, s in enumerate(src):
        named.update({f"l{i}." + k[3:]: v for k, v in tensors.items() if k.startswith(f"l{s}.")})
    options = EngineOptions(dtype=dtype, page_size=page, num_pages=8, max_requests=2)
    model_, ctx = Engine._build(mixed, options)
    specs = model_.param_specs()
    model_.bind(bind_tensors({k: v for k, v in named.items() if k in specs}, specs, ctx.dtype, ctx.device))
    eng = Engine(mixed, model_, options)
    ids = tz.prompt(40, raw["vocab"], 3)
    order = {"architecture": "Zogulorn", "norm": raw["norm"], "embedding": raw["embedding"], "layers": [raw["layers"][s] for s in src]}
    oracle = {k: v.double() for k, v in named.items()}
    for i in (0, 2):
        oracle[f"l{i}.ls1"], oracle[f"l{i}.ls2"] = (torch.ones(raw["width"], dtype=F64) for _ in range(2))
    ref = {"a": plain.forward(order, oracle, ids)}
    rows = run_steps(eng, [[("a", ids[:30], 0)]] + [[("a", [ids[i]], i)] for i in range(30, 40)])
    check_rows(rows, ref, dtype, "other blocks")
