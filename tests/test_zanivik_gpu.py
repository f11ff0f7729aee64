"""The Zanivik design on the GPU against its plain implementation (tests/plain_zanivik.py): each mechanism's kernels
alone, then whole models through Engine.step in every way of cutting and batching, through the scheduler's
generate(), the command line and bin/trace_run."""
import math

import pytest
import torch

import plain_zanivik as plain
import replay
import tiny_zanivik as tz

pytestmark = pytest.mark.gpu
DEV = torch.device("cuda:0")
# of the largest logit of the compared request.  The sharp comparison is the float32 one; every bfloat16 kernel has
# its own tight test below.
TOL = {"float32": 1e-4, "bfloat16": 6e-2}
F64 = torch.float64


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

KINDS = {0: lambda x, g, eps: x if g is None else x * g, 1: lambda x, g, eps: plain.rms_unit(x, eps) * (1.0 if g is None else g),
         2: lambda x, g, eps: plain.layer_norm(x, 1.0 if g is None else g, eps)}


@pytest.mark.parametrize("T,H", [(1, 64), (7, 50), (5, 1028), (3, 2048), (2, 4100), (3, 9000), (2, 4099), (200, 256)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
def test_seam_between_sublayers(ops, T, H, out_dtype):
    """The sum into the stream and the next norm: every kind of norm on either side, one branch or a pair of normed ones,
    all rows or some; rows with a large mean (a layer norm that forgets it, or its variance's, shows)."""
    tol = 3e-6 if out_dtype == torch.float32 else 6e-3
    x0, y, z = rnd(T, H, seed=1) + 3.0, 2.0 * rnd(T, H, seed=2) - 5.0, rnd(T, H, seed=3) + 1.0
    gp, gn, gy, gz = (1.0 + 0.5 * rnd(H, seed=s) for s in (4, 5, 6, 7))
    pair_ref = 0.5 * (plain.rms_unit(y.double(), 1e-2) * gy.double() + plain.rms_unit(z.double(), 1e-2) * gz.double())
    for post, nxt in ((2, 2), (1, 2), (0, 1), (2, 0), (2, None), (None, 2)):
        for pair in (False, True):
            branch = None if post is None else (ops.NormedPair(d(y), d(gy), d(z), d(gz), 1e-2) if pair else d(y))
            xs = d(x0.clone())
            got = ops.row_step(xs, branch, None if post is None else (post, d(gp), 1e-3), None if nxt is None else (nxt, d(gn), 1e-5),
                               out_dtype=out_dtype)
            want_x = x0.double() + (0.0 if post is None else KINDS[post](pair_ref if pair else y.double(), gp.double(), 1e-3))
            assert rel_err(xs, want_x) < 3e-6, (post, nxt, pair)
            if nxt is None:
                assert got is None
                continue
            want = KINDS[nxt](want_x, gn.double(), 1e-5)
            assert rel_err(got, want) < tol, (post, nxt, pair)
            rows = torch.tensor([T - 1, 0, T - 1], dtype=torch.int32)
            branch = None if post is None else (ops.NormedPair(d(y), d(gy), d(z), d(gz), 1e-2) if pair else d(y))
            xs = d(x0.clone())
            got = ops.row_step(xs, branch, None if post is None else (post, d(gp), 1e-3), (nxt, d(gn), 1e-5), rows=d(rows), out_dtype=out_dtype)
            assert torch.equal(xs.cpu(), x0) and rel_err(got, want[rows.long()]) < tol


@pytest.mark.parametrize("T,K,H", [(4, 512, 192), (16, 2048, 256), (40, 1024, 128)])
def test_seam_takes_open_sums(ops, T, K, H):
    """A branch whose product is still in planes, written or written and then added to; a pair of two sets of planes."""
    from blackwellllm_b200.parts.linear import Linear
    a, b = d(rnd(T, K, seed=1, scale=0.1).bfloat16()), d(rnd(T, K, seed=2, scale=0.1).bfloat16())
    wa, wb = Linear(d(rnd(H, K, seed=3).bfloat16())), Linear(d(rnd(H, K, seed=4).bfloat16()))
    ya, yb = a.double().cpu() @ wa.weight.double().cpu().T, b.double().cpu() @ wb.weight.double().cpu().T
    gain = 1.0 + 0.3 * rnd(H, seed=5)
    x0 = rnd(T, H, seed=6)
    for two in (False, True):
        buf, xs = torch.full((T, H), float("nan"), device=DEV), d(x0.clone())
        wa.write_to(a, buf)
        if two:
            wb.add_to(b, buf)
        ops.row_step(xs, buf, (2, d(gain), 1e-5))
        assert rel_err(xs, x0.double() + plain.layer_norm(ya + yb if two else ya, gain.double(), 1e-5)) < 1e-4
    y = wa.planes(a)
    z = wb.planes(b, behind=y)
    assert y.dim() == 3 and z.dim() == 3
    xs = d(x0.clone())
    ops.row_step(xs, ops.NormedPair(y, d(gain), z, d(gain), 1e-5))
    want = x0.double() + 0.5 * (plain.rms_unit(ya, 1e-5) + plain.rms_unit(yb, 1e-5)) * gain.double()
    assert rel_err(xs, want) < 1e-4
    pair = ops.NormedPair(wa.planes(a), d(gain), wb.planes(b), d(gain), 1e-5)    # the second product wrote over the first's planes
    wa.planes(a)
    with pytest.raises(ops.KernelError):
        ops.row_step(xs, pair)


@pytest.mark.parametrize("taps", [1, 2, 3, 4, 6])
@pytest.mark.parametrize("dims", [((2, 16), (2, 16), (4, 24)), ((1, 160), (1, 160), (3, 40)), ((3, 7), (3, 7), (5, 33)), ((2, 128), (2, 128), (2, 128))])
def test_short_convolution_unit_norms_and_gates(ops, taps, dims):
    """Three requests in slots out of order in portions down to one token beside longer ones; the state holds what the next
    step's first tokens look back on, also where a portion is shorter than the look-back; an unowned slot holds NaN."""
    lens, slots = [60, 9, 131], [2, 0, 3]
    cuts = [[33, 2, 1, 1, 20, 1, 2], [1] * 9, [1, 1, 64, 33, 2, 30]]
    C = sum(n * s for n, s in dims)
    heads = 5
    segs = [(dims[0][0], dims[0][1], 0.3), (dims[1][0], dims[1][1], 1.0), (dims[2][0], dims[2][1], None)]
    w, bias = rnd(C, taps, seed=1), rnd(C, seed=2)
    A, dtb = -torch.exp(rnd(heads, seed=3)), rnd(heads, seed=4)
    pad = 3
    data = [rnd(L, pad + C + 2 * heads, seed=10 + r) for r, L in enumerate(lens)]

    def want(x):
        u = plain.silu(plain.short_conv(x[:, pad:pad + C].double(), w.double(), bias.double()))
        out, c = [], 0
        for n, s, scale in segs:
            v = u[:, c:c + n * s].view(-1, n, s)
            out.append((v if scale is None else v / torch.sqrt((v * v).sum(-1, keepdim=True) + 1e-6) * scale).reshape(-1, n * s))
            c += n * s
        z = x[:, pad + C:].double()
        dt = plain.softplus(z[:, :heads] + dtb.double())
        return torch.cat(out, 1), torch.exp(A.double() * dt), dt, torch.sigmoid(z[:, heads:])
    ref = [want(x) for x in data]
    for second in (True, False):
        state = torch.full((4, taps, C), float("nan"), device=DEV)
        for part in walk(cuts, lens):
            rows = Rows([n for _, _, n in part], [a for _, a, _ in part], [slots[r] for r, _, _ in part])
            x = d(torch.cat([data[r][a:a + n] for r, a, n in part]))
            got, g, other = ops.short_conv(x[:, pad:], d(w.t()), d(bias), state, rows, segs, 1e-6,
                                           gates=(x, pad + C, pad + C + heads if second else None, d(A), d(dtb)))
            o = 0
            for r, a, n in part:
                assert rel_err(got[o:o + n], ref[r][0][a:a + n]) < 1e-5, (r, a, n)
                assert rel_err(g[o:o + n], ref[r][1][a:a + n]) < 1e-5
                assert rel_err(other[o:o + n], ref[r][3 if second else 2][a:a + n]) < 1e-5
                o += n


@pytest.mark.parametrize("chunked", [False, True])
@pytest.mark.parametrize("heads,rep,dk,dv", [(80, 2, 36, 20), (4, 2, 16, 24), (2, 1, 160, 40), (3, 3, 12, 33), (2, 1, 128, 64), (4, 4, 40, 72), (1, 1, 256, 17), (2, 2, 64, 128)])
def test_delta_rule_across_steps_and_slots(ops, heads, rep, dk, dv, chunked):
    """Portions of several sizes down to single tokens, slots out of order; decays that are 0 and 1, step sizes 0 and 1;
    token by token and in chunks of tokens."""
    lens, slots = [70, 9, 131], [2, 0, 3]
    cuts = [[33, 2, 1, 1, 20, 13], [9], [1, 1, 64, 33, 2, 30]]
    K, V = heads // rep * dk, heads * dv
    data, want = [], []
    for r, L in enumerate(lens):
        x = rnd(L, 2 * K + V + 2, seed=20 + r)
        q, k = x[:, 2:2 + K].view(L, -1, dk), x[:, 2 + K:2 + 2 * K].view(L, -1, dk)
        q /= q.norm(dim=-1, keepdim=True)
        k /= k.norm(dim=-1, keepdim=True)
        g, b = torch.rand(L, heads, generator=torch.Generator().manual_seed(r)), torch.rand(L, heads, generator=torch.Generator().manual_seed(9 + r))
        g = 1.0 - 0.3 * g
        g[::17], g[3::5], b[4::7], b[5::11] = 0.0, 1.0, 0.0, 1.0
        data.append((x, g, b))
        want.append(plain.delta_rule(q.double().repeat_interleave(rep, 1), k.double().repeat_interleave(rep, 1),
                                     x[:, 2 + 2 * K:].double().view(L, heads, dv), g.double(), b.double()).reshape(L, V))
    state = torch.zeros(4, heads, dk, dv, device=DEV)
    state[1] = float("nan")
    for part in walk(cuts, lens):
        rows = Rows([n for _, _, n in part], [a for _, a, _ in part], [slots[r] for r, _, _ in part])
        x, g, b = (d(torch.cat([data[r][i][a:a + n] for r, a, n in part])) for i in range(3))
        if chunked:
            got = ops.chunk_scan(True, x, 2, 2 + K, 2 + 2 * K, g, b, rows, state, heads, rep, dk, dv)
        else:
            got = ops.delta_scan(x, 2, 2 + K, 2 + 2 * K, g, b, rows, state, heads, rep, dk, dv)
        o = 0
        for r, a, n in part:
            assert rel_err(got[o:o + n], want[r][a:a + n]) < 3e-5, (r, a, n)
            o += n


@pytest.mark.parametrize("chunked", [False, True])
def test_delta_rule_keeps_and_replaces_a_far_token(ops, chunked):
    """No decay, orthogonal keys: a value written 400 tokens back is read in full, unless its key was written again
    since (the second value is read) or the state was closed once in between (nothing is read)."""
    dk, dv, L = 16, 8, 420
    for case in ("kept", "replaced", "closed"):
        x = torch.zeros(L, 2 * dk + dv)
        x[:, dk + 1] = 1.0                      # every token writes along channel 1 ...
        x[:, 2 * dk:] = 1.0
        x[10, dk:2 * dk] = 0.0                  # ... token 10 along channel 0, value 5
        x[10, dk] = 1.0
        x[10, 2 * dk:] = 5.0
        g, b = torch.ones(L, 1), torch.ones(L, 1)
        if case == "replaced":
            x[300, dk:2 * dk] = 0.0
            x[300, dk] = 1.0
            x[300, 2 * dk:] = -2.0
        if case == "closed":
            g[200] = 0.0
        x[-1, 0] = 1.0                          # the last query asks for channel 0
        state = torch.zeros(1, 1, dk, dv, device=DEV)
        for lens in ([L], [211, 2, 200, 1, 6]):
            state.zero_()
            at = 0
            for n in lens:
                args = (d(x[at:at + n]), 0, dk, 2 * dk, d(g[at:at + n]), d(b[at:at + n]), Rows([n], [at], [0]), state, 1, 1, dk, dv)
                o = ops.chunk_scan(True, *args) if chunked else ops.delta_scan(*args)
                at += n
            want = {"kept": 5.0, "replaced": -2.0, "closed": 0.0}[case]
            assert float((o[-1].cpu() - want).abs().max()) < 1e-5, (case, lens)


@pytest.mark.parametrize("heads,groups,P,N,parts", [(4, 2, 32, 32, 2), (6, 3, 8, 24, 2), (4, 1, 20, 33, 5), (3, 3, 7, 5, 3), (4, 2, 32, 160, 1),
                                                    (2, 2, 9, 66, 6), (8, 2, 64, 128, 8), (2, 1, 16, 256, 4), (60, 3, 48, 40, 5)])
@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("chunked", [False, True])
def test_state_space_across_steps_and_slots(ops, heads, groups, P, N, parts, out_dtype, chunked):
    """Scan and output kernels: heads that share a group's B and C, norm parts that cut across heads, D, the gate before
    the norm."""
    lens, slots = [70, 9, 131], [2, 0, 3]
    cuts = [[33, 2, 1, 1, 20, 13], [9], [1, 1, 64, 33, 2, 30]]
    I, GN = heads * P, groups * N
    A, D, gain = -torch.exp(rnd(heads, seed=1)), 0.5 + rnd(heads, seed=2), 1.0 + 0.3 * rnd(I, seed=3)
    data, want = [], []
    for r, L in enumerate(lens):
        x, z = rnd(L, I + 2 * GN, seed=30 + r), rnd(L, I + 3, seed=40 + r)
        dt = plain.softplus(rnd(L, heads, seed=50 + r, scale=2.0))
        data.append((x, z, torch.exp(A * dt), dt))
        xd = x.double()
        B, C = (xd[:, I + i * GN:I + (i + 1) * GN].view(L, groups, N).repeat_interleave(heads // groups, 1) for i in range(2))
        y = plain.state_space(xd[:, :I].view(L, heads, P), B, C, dt.double(), A.double(), D.double()).reshape(L, I)
        y = y * plain.silu(z[:, 3:].double())
        want.append(plain.rms_unit(y.view(L, parts, -1), 1e-5).reshape(L, I) * gain.double())
    state = torch.zeros(4, heads, N, -(-P // 4) * 4, device=DEV)
    state[1] = float("nan")
    for part in walk(cuts, lens):
        rows = Rows([n for _, _, n in part], [a for _, a, _ in part], [slots[r] for r, _, _ in part])
        x, z, a_, dt = (d(torch.cat([data[r][i][a:a + n] for r, a, n in part])) for i in range(4))
        if chunked:
            y = ops.chunk_scan(False, x, I + GN, I, 0, a_, dt, rows, state, heads, heads // groups, N, P)
        else:
            y = ops.gla_scan(x, I + GN, I, 0, a_, rows, state, heads, N, P, 1.0, k_scale=dt, scalar_decay=True, qk_rep=heads // groups)
        got = ops.ssd_out(y, x, z[:, 3:], d(D), d(gain), P, parts, 1e-5, out_dtype)
        o = 0
        for r, a, n in part:
            assert rel_err(got[o:o + n], want[r][a:a + n]) < (5e-5 if out_dtype == torch.float32 else 6e-3), (r, a, n)
            o += n


@pytest.mark.parametrize("out_dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("nh,nkv,dq,dv,rd", [(4, 2, 32, 16, 32), (3, 1, 24, 40, 22), (2, 2, 64, 64, 32), (6, 3, 10, 10, 6), (4, 1, 128, 128, 128),
                                             (2, 1, 256, 256, 200), (4, 2, 96, 48, 96), (3, 3, 12, 12, 4)])
def test_norms_around_the_rotation_shared_values_head_factors(ops, out_dtype, nh, nkv, dq, dv, rd):
    """Queries and keys as they reach the attention: normed after the rotation without gains (values scaled), or before it
    with gains, a factor per query head and the key projection as the value; rows inside a wider product."""
    from blackwellllm_b200.parts.rope import rotary_inv_freq
    from test_kernels_gpu import FakeBatch
    page, T = 8, 19
    rot = {"base": 300.0, "dims": rd}
    cols = nh * dq + nkv * (dq + dv)
    dpad = -(-max(dq, dv) // 16) * 16
    tol = 4e-6 if out_dtype == torch.float32 else 8e-3
    pages = [2, 0, 3, 1]
    batch, table = FakeBatch([T], [T]), torch.tensor([pages], dtype=torch.int32, device=DEV)
    cs = ops.rope_table(batch.positions, rotary_inv_freq(300.0, rd).to(DEV), rd)
    gq, gk, mult = 1.0 + 0.4 * rnd(dq, seed=3), 1.0 + 0.4 * rnd(dq, seed=4), 0.5 + rnd(nh, seed=5)
    for shared in (False, True):
        if shared and dv != dq:
            continue
        for extra in (0, 4, 5):                  # 16-byte, 16-byte and odd row strides
            qkv = rnd(T, cols + extra, seed=dq + extra)
            x = qkv.double()
            q, k = x[:, :nh * dq].view(T, nh, dq), x[:, nh * dq:(nh + nkv) * dq].view(T, nkv, dq)
            if shared:
                v = k
                q = plain.rotate_halves(plain.rms_unit(q, 1e-3) * gq.double(), rot) * mult.double().view(1, nh, 1)
                k = plain.rotate_halves(plain.rms_unit(k, 1e-3) * gk.double(), rot)
                kw = dict(q_head_mult=d(mult), kv_shared=True)
                gains = (d(gq), d(gk))
            else:
                v = 0.7 * x[:, (nh + nkv) * dq:cols].view(T, nkv, dv)
                q, k = plain.rms_unit(plain.rotate_halves(q, rot), 1e-3), plain.rms_unit(plain.rotate_halves(k, rot), 1e-3)
                kw = dict(v_scale=0.7)
                gains = (d(torch.ones(dq)),) * 2
            kp = torch.full((4, nkv, page, dpad), float("nan"), dtype=out_dtype, device=DEV)
            vp = kp.clone()
            got = ops.head_norm_rope_append(d(qkv), batch, table, cs, rd, False, gains[0], gains[1], 1e-3, kp, vp, nh, nkv, dq, dv, **kw)
            got = got.view(T, nh, dpad).double().cpu()
            assert rel_err(got[..., :dq], q) < tol and (dpad == dq or float(got[..., dq:].abs().max()) == 0.0)
            for t in range(T):
                kt, vt = kp[pages[t // page], :, t % page].double().cpu(), vp[pages[t // page], :, t % page].double().cpu()
                assert float((kt[:, :dq] - k[t]).abs().max()) <= tol * float(k.abs().max())
                assert float((vt[:, :dv] - v[t]).abs().max()) <= tol * float(v.abs().max())
                assert float(kt[:, dq:].abs().sum()) == 0.0 and float(vt[:, dv:].abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("hd", [48, 64])
@pytest.mark.parametrize("q_len", [1, 2, 50])
def test_one_loud_key_at_the_window_edge_with_sink_and_gate(ops, dtype, hd, q_len):
    """All scores of the last query are 0 but one key's.  Just inside the window the row returns that key's value times
    the gate; just outside it, the mean share the sink (a part of 3 in window + 3) leaves to the others; hundreds of
    positions back, and at page borders."""
    from test_kernels_gpu import FakeBatch, paged_case
    nh, nkv, page, window, L = 4, 2, 16, 36, 700
    last = L - 1
    sink = torch.full((nh,), math.log(3.0))
    g = torch.zeros(q_len, nh * hd)                 # the gate's sigmoid: one half
    for loud, seen in [(last - window + 1, True), (last - window, False), (last, True), (last - 1, True), (0, False), (last - 63, False)]:
        def spike(r, q, k, v):
            k[:] = 0
            k[loud, :, 0] = 8.0
            q[-1] = 0
            q[-1, :, 0] = 5.0
            v[:] = 1.0
            v[loud] = 5.0
        q, kp, vp, table, _ = paged_case([q_len], [L], nh, nkv, hd, page, dtype, seed=2, spike=spike)
        out = ops.paged_attention(q, kp, vp, FakeBatch([q_len], [L]), table, nh, window, 1.0, sink=d(sink), gate=(d(g), hd))
        row = out[-1].float().cpu().view(nh, hd)
        want = 0.5 * (5.0 if seen else window / (window + 3.0))
        assert float((row - want).abs().max()) < 0.02, (loud, seen, float(row.mean()))


def test_gelu(ops):
    """The error function's gelu: to float32 rounding alone, within bfloat16 rounding in the tensor-core epilogue."""
    x = torch.cat([torch.linspace(-9, 9, 4001), torch.tensor([0.0, -0.0, 1e-20, -1e-20, 30.0, -30.0])])
    got = ops.unary_act(d(x), ops.ACT_GELU).cpu()
    assert float((got.double() - plain.gelu(x.double())).abs().max()) < 1e-6
    for M in (1, 5, 40, 300):
        a, w = rnd(M, 64, seed=M).bfloat16(), rnd(96, 64, seed=2, scale=0.3).bfloat16()
        out = ops.gemm_tc(d(a), d(w), act=ops.ACT_GELU)
        want = plain.gelu(a.double() @ w.double().T)
        assert float((out.double().cpu() - want).abs().max()) <= 5e-3 * float(want.abs().max())
        f32 = ops.gemm_tc(d(a), d(w), act=ops.ACT_GELU, out_dtype=torch.float32)
        assert float((f32.double().cpu() - want).abs().max()) <= 2e-5 * float(want.abs().max())


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name,layer", [("mixed", 0), ("mixed", 1), ("mixed", 2), ("tensor", 0), ("tensor", 2), ("open", 1), ("open", 2), ("open", 3), ("broad", 0), ("broad", 1)])
def test_mixer_alone(ops, dtype, name, layer):
    """Two mixers side by side against the plain functions: portions and then single tokens, next to another request; in a
    tensor of its own, added to one that holds something, and as the open form a block takes."""
    from blackwellllm_b200.cache.manager import CacheManager
    from blackwellllm_b200.config.registry import parse_config
    from blackwellllm_b200.parts import BuildContext, build_mixer
    from test_kernels_gpu import FakeBatch
    raw, page = tz.CONFIGS[name]
    W, eps, entry = raw["width"], raw["norm"]["eps"], raw["layers"][layer]
    mixer = build_mixer(parse_config(raw).layers[layer].mixer, W, BuildContext(DEV, dtype))
    t = plain.sub(tz.make_tensors(raw, seed=11, dtype=dtype), f"l{layer}.mix.")
    mixer.bind({k: d(v) for k, v in t.items()})
    L = {0: 75, 1: 30}
    xs = {r: rnd(n, W, seed=60 + r).to(dtype) for r, n in L.items()}
    want = {r: plain.mixer(entry["type"], x.double(), {k: v.double() for k, v in t.items()}, entry["mixer"], eps) for r, x in xs.items()}
    tol = 3e-5 if dtype == torch.float32 else 5e-2
    for form in ("write", "add", "open"):
        cm = CacheManager([mixer.cache_request()], page, 16, 3, dtype=dtype, device=DEV)
        for r in (1, 0):
            cm.add_request(r)
        at, got = {0: 0, 1: 0}, {0: [], 1: []}
        for step in [[(0, 33), (1, 2)], [(1, 1), (0, 30)]] + [[(0, 1), (1, 1)] for _ in range(12)]:
            for r, n in step:
                cm.append(r, n)
            batch = FakeBatch([n for _, n in step], [at[r] + n for r, n in step])
            batch.state_slot = torch.tensor([cm.slot(r) for r, _ in step], dtype=torch.int32, device=DEV)
            width = max(cm.num_blocks(r, 0) for r, _ in step)
            table = torch.full((len(step), width), -1, dtype=torch.int32)
            for i, (r, _) in enumerate(step):
                row = cm.block_table(r, 0)
                table[i, :len(row)] = torch.tensor(row, dtype=torch.int32)
            batch.block_tables = {0: d(table)}
            x = d(torch.cat([xs[r][at[r]:at[r] + n] for r, n in step]))
            base = d(rnd(x.shape[0], W, seed=5))
            if form == "open":
                res = base.clone()
                ops.row_step(res, mixer.forward_open(x, batch, cm.views[0]))
                res = res - base
            else:
                res = base.clone()
                mixer.forward(x, res, batch, cm.views[0], accumulate=form == "add")
                ops.resolve_pending()
                if form == "add":
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
_DT = {"float32": torch.float32, "bfloat16": torch.bfloat16}


def plain_logits(raw, tensors, ids, streams=None):
    return plain.forward(raw, {k: v.double() for k, v in tensors.items()}, ids, streams)


def model(name, dtype):
    key = (name, dtype)
    if key not in _models:
        raw, page = tz.CONFIGS[name]
        # (a seed whose model amplifies the rounding of 16-bit operands at no place of these requests)
        tensors = tz.make_tensors(raw, seed=9 if name == "open" else 7, dtype=_DT[dtype])
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
    """rows {(rid, pos): logits}: every row within the bound."""
    for (rid, p), row in rows.items():
        err = float((row.double().cpu() - ref[rid][p]).abs().max()) / float(ref[rid].abs().max())
        assert err <= TOL[dtype], (what, rid, p, err)


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
    """Decoding from position 0 (the first tokens of a sequence, every page border, the windows' edges passing
    over decoded tokens, the recurrences and convolutions from their zero states), long enough that the decode steps are replayed
    from a CUDA graph."""
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
    """A pool that holds two requests: five pass through, portions of one beside single tokens of another; every
    later request gets a slot (with the states of its layers in it) and pages that an earlier one gave back."""
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
    """700 tokens: the windows have passed dozens of pages (given back meanwhile), the recurrences have run 700 steps; prompt portions that start
    and end inside pages, then 40 tokens one by one."""
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
    # the windows gave pages back on the way: the groups with a window hold far fewer than 700 tokens' worth now
    held = [sum(1 for p in eng.cache.block_table("long", g) if p >= 0) for g in range(len(eng.cache.groups))]
    assert all(h * page < 300 for h, grp in zip(held, eng.cache.groups) if grp.request.window), held


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
    """A request that sits out some steps finds its states and its keys as it left them, while another request in the
    neighbouring slot runs on."""
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
    W = load_file(os.path.join(folder, "model.safetensors"))
    prompts = [tz.prompt(n, raw["vocab"], 80 + n) for n in (5, 40, 1)]
    steps = 12
    llm = BlackwellEngine(folder, InferenceConfig(max_context_length=128, max_batch_size=3), dtype="float32")
    got = llm.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=steps))
    for p, g in zip(prompts, got):
        ids = list(p)
        for _ in range(steps):
            ids.append(int(torch.argmax(plain_logits(raw, W, ids)[-1])))
        assert list(g.token_ids) == ids[len(p):]


def test_command_line_and_position_addressed_calls(tmp_path, capsys):
    import os
    from safetensors.torch import load_file
    from blackwellllm_b200 import BlackwellEngine, InferenceConfig, cli
    name = "mixed"
    raw, _ = tz.CONFIGS[name]
    folder = tz.make_folder(name, "float32", str(tmp_path))
    W = load_file(os.path.join(folder, "model.safetensors"))
    prompt = tz.prompt(9, raw["vocab"], 4)
    ids = list(prompt)
    for _ in range(6):
        ids.append(int(torch.argmax(plain_logits(raw, W, ids)[-1])))
    want = ids[len(prompt):]
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


# =============================================================================== bin/trace_run

@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("family", ["tail", "portions", "mixed"])
def test_replay(tmp_path_factory, dtype, family):
    import os
    from safetensors.torch import load_file
    name = "mixed"
    raw, page = tz.CONFIGS[name]
    folder = tz.make_folder(name, dtype, str(tmp_path_factory.mktemp("zanivik")))
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
    layers = []
    for _ in range(pick(1, 2, 3, 4)):
        kv, dim = pick(1, 2, 3), pick(6, 8, 12, 20)
        scaling = pick(None, (pick(2.0, 8.0), pick(0.5, 1.0), pick(2.0, 4.0), pick(20, 60)))
        size, base, dims, ff = pick(None, 1, 3, 11, 40), pick(50.0, 10000.0), pick(2, 4, dim), pick(None, 24, 41)
        if pick(0, 1):
            rk = pick(1, 2)
            layers.append(tz._one(tz._attn(kv * pick(1, 2, 3), kv, dim, pick(4, dim, 24), pick(0.2, 1.5), size, base, dims, scaling),
                                  (rk * pick(1, 2, 3), rk, pick(4, 20, 40), pick(4, 31, 32), pick(1, 2, 4, 7)), (pick(0.3, 1.0, -1.2), pick(0.4, 1.0)), ff))
        else:
            groups, per, vdim = pick(1, 2), pick(1, 3), pick(4, 10, 36)
            layers.append(tz._two(tz._attn(kv * pick(1, 2, 3), kv, dim, dim, pick(0.2, 0.5), size, base, dims, scaling),
                                  (groups * per, vdim, pick(3, 16, 40), groups, pick(1, 2, 4, 7), pick(1, groups * per, 2)), ff))
    raw = tz._model(pick(60, 130), pick(40, 48, 71), pick(1e-6, 1e-3), pick(0.2, 1.0, 1.4), layers)
    return raw, pick(8, 16)


@pytest.mark.parametrize("seed", range(10))
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
    """A stack of this design's layers between pre-norm ones: the seam left open is made before the other kind of block
    reads the stream, and a sum the other kind leaves open before this kind does."""
    import dataclasses
    from blackwellllm_b200.config.registry import parse_config
    from blackwellllm_b200.engine.engine import Engine, EngineOptions, StepEntry
    from blackwellllm_b200.weights.loader import bind_tensors
    raw, page = tz.CONFIGS["broad"]
    cfg = parse_config(raw)
    pre = [dataclasses.replace(ls, block="prenorm", layer_scale=None, residual_mult=1.0) for ls in cfg.layers]
    mixed = dataclasses.replace(cfg, layers=(pre[1], cfg.layers[0], pre[0], cfg.layers[1]),
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
    x = tensors["embed"].double()[torch.tensor(ids)]
    eps, mult = raw["norm"]["eps"], raw["residual_mult"]
    for i, s in enumerate(src):
        t, layer = {k: v.double() for k, v in plain.sub(tensors, f"l{s}.").items()}, raw["layers"][s]
        own = i in (1, 3)
        for n, nb, ls, f in (("norm1", "norm1b", "ls1", lambda h: plain.mixer(layer["type"], h, plain.sub(t, "mix."), layer["mixer"], eps)),
                             ("norm2", "norm2b", "ls2", lambda h: plain.dense_ffn(h, plain.sub(t, "mlp.")))):
            y = f(plain.layer_norm(x, t[n], eps))
            x = x + (mult * plain.layer_norm(y, t[nb], eps) * t[ls] if own else y)
    ref = {"a": plain.layer_norm(x, tensors["final.norm"].double(), eps) @ tensors["head"].double().T}
    rows = run_steps(eng, [[("a", ids[:30], 0)]] + [[("a", [ids[i]], i)] for i in range(30, 40)])
    check_rows(rows, ref, dtype, "other blocks")
