// Gated linear attention: a recurrent mixer with a matrix state per head and a decay per key channel.
//
//   S_t = diag(a_t) S_(t-1) + k_t v_t^T        S: [dk, dv] per head, float32, one per request
//   o_t = S_t^T q_t                            q scaled by q_scale
//   a_t = sigmoid(z_t) ^ (1 / tau) = exp(log_sigmoid(z_t) / tau),   z_t = W2 (W1 x_t) + b
//
// Everything but the projections that make q, k, v, z is float32 here: the decay and its logarithm,
// the state, the products that enter and leave it, and the norm of the head's output.
//
// gla_scan_kernel walks the tokens of one request's segment in order (a single decoded token and a
// portion of a prompt are the same case), from the state the steps before left in the request's slot,
// and leaves the new state there.  A block owns (request, head, COLS value columns); its state lies in registers, a tile of
// rows x columns per lane (common.cuh), two rows per packed instruction.  A token's S^T q is summed over a warp's row groups
// by shuffles that nothing waits for, the warps' parts go to shared memory and are added, in warp order, after a chunk of tokens.
// The order of all sums depends on dk alone, never on how the tokens were cut into steps or on the batch.  The scan keeps
// float32 throughout (as the design asks): it is bound by the issue of its packed multiply-adds and the shared-memory reads
// that feed them, and its parallelism is requests x heads x columns / COLS.
//
// gla_decay_kernel makes a_t from the first projection's result (W2 has a small inner size: float32 FMAs).
// gla_gate_kernel: per token and head, o / rms(o) * gain * silu(g) -> the output projection's operand.
#include "common.cuh"

using bf16 = __nv_bfloat16;

namespace {

#ifndef SCAN_NARROW_BELOW
#define SCAN_NARROW_BELOW 3     // quarters of the SM count: with fewer 32-column blocks than that they become 16 columns wide
#endif
constexpr int MAX_DK = 256;

struct ScanParams {
    const float* qkv;      // [T, ld]: q at q_off, k at k_off, v at v_off (head-major within each)
    const float* decay;    // [T, heads * dk]: a_t, already in (0, 1)
    const int* cu_q;       // [R + 1]
    const int* state_slot; // [R]
    float* state;          // [slots, heads, dk, dv]
    float* o;              // [T, heads * dv]
    long long ld;
    int q_off, k_off, v_off;
    int heads, dk, dv;
    float q_scale;
    // The same recurrence serves a matrix memory with ONE decay per head and token and a normaliser:
    // scalar_decay != 0: decay is [T, heads] (a_t of the head, used for every key channel);
    // k_scale != null: [T, heads], the token's keys count times it (an input gate);
    // ones_col != 0: the head's last value column (dv - 1) is the constant 1 and v holds dv - 1 columns a head, so that
    // column of the state is n_t = a_t n_(t-1) + k_t and the last output column is n_t . q_t.
    const float* k_scale;
    int scalar_decay, ones_col;
    int sld;               // floats between the state's rows (>= dv; columns from dv on stay zero)
    int single;            // every request has one token
    int rep;               // head h reads query/key head h / rep (heads / rep of them; the plain form has rep == 1)
};

__device__ __forceinline__ float log_sigmoid(float z) {
    // log(1 / (1 + exp(-z))) without overflow on either side
    return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

// a[t, c] = sigmoid(z)^(1 / tau) with z = sum_r x[t, r] w[c, r] + b[c]: the decay's second projection (its inner
// size is small), the sigmoid's logarithm, the division by tau and the exponential, all float32.
// x: float32 [T, ldx] at column x_off; w: [C, rank] (float32 or bfloat16); one thread per (t, c).
template <typename WT>
__global__ void __launch_bounds__(256)
gla_decay_kernel(const float* __restrict__ x, long long ldx, int x_off, const WT* __restrict__ w,
                 const WT* __restrict__ b, float* __restrict__ a, int T, int C, int rank, float inv_tau) {
    BW_PDL_TRIGGER();
    BW_PDL_WAIT();
    const long long idx = (long long)blockIdx.x * blockDim.x + threadIdx.x;
    if (idx >= (long long)T * C) return;
    const int t = (int)(idx / C), c = (int)(idx - (long long)t * C);
    const float* xr = x + (size_t)t * ldx + x_off;
    const WT* wr = w + (size_t)c * rank;
    float z = 0.f;
    for (int r = 0; r < rank; ++r) z = fmaf(xr[r], bw::to_f32(wr[r]), z);
    z += bw::to_f32(b[c]);
    a[idx] = expf(log_sigmoid(z) * inv_tau);
}

// NW warps of 32 state rows: dk <= DKP = 32 NW.  CPT value columns a lane: COLS = 8 CPT.  TOK_CHUNK tokens are staged in shared
// memory at a time: 16, or 1 in steps of single tokens (fewer registers, more blocks side by side).  In shared memory a token's q, k
// (and a) are padded with zeros to DKP channels (a padded channel stays at zero and adds nothing), so the inner loop has no
// bounds.
// MEM: the form for a matrix memory (ScanParams: one decay per head, keys times k_scale, the column of ones, query/key
// heads shared by several heads); the plain form's code does not know of it.  What a fetch loads is not touched before it
// is staged: a thread never waits for a load inside the fetch.  The key's scale multiplies the token's value instead, which is
// the same product.
template <int NW, int CPT, bool MEM, int TOK_CHUNK>
struct ScanSmem {
    static constexpr int DKP = NW * bw::TILE_WARP_ROWS, COLS = bw::TILE_CG * CPT;
    static constexpr int floats = (MEM ? 2 : 3) * TOK_CHUNK * DKP + TOK_CHUNK * COLS + 2 * TOK_CHUNK + TOK_CHUNK * NW * COLS;
};

template <int NW, int CPT, bool MEM, int TOK_CHUNK>
__global__ void __launch_bounds__(32 * NW)
gla_scan_kernel(ScanParams p) {
    BW_PDL_TRIGGER();
    constexpr int THREADS = 32 * NW, DKP = NW * bw::TILE_WARP_ROWS, COLS = bw::TILE_CG * CPT, RP = bw::TILE_ROWS / 2;
    extern __shared__ __align__(16) float sm[];
    float* qs = sm;                                      // [TOK_CHUNK][DKP]
    float* ks = qs + TOK_CHUNK * DKP;
    float* as = ks + TOK_CHUNK * DKP;                    // plain form: [TOK_CHUNK][DKP]
    float* vs = as + (MEM ? 0 : TOK_CHUNK * DKP);        // [TOK_CHUNK][COLS]
    float* gs = vs + TOK_CHUNK * COLS;                   // MEM: [TOK_CHUNK] decays, [TOK_CHUNK] scales of the keys
    float* part = gs + 2 * TOK_CHUNK;                    // [TOK_CHUNK][NW][COLS]
    constexpr int NST = (TOK_CHUNK * DKP + THREADS - 1) / THREADS;       // staged values of q, k, a per thread
    constexpr int NSV = (TOK_CHUNK * COLS + THREADS - 1) / THREADS;
    const int r = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int rg = lane >> 3, cg = lane & 7;
    const int row0 = warp * bw::TILE_WARP_ROWS + rg * bw::TILE_ROWS;
    const int t0 = p.cu_q[r], t1 = p.cu_q[r + 1];
    const int hk = MEM ? h / p.rep : h;
    float* S = p.state + (((size_t)p.state_slot[r] * p.heads + h) * p.dk) * p.sld;
    BW_PDL_WAIT();
    bw::f32x2 s[RP][CPT];
    bw::tile_load<CPT>(s, S, row0, p.dk, p.sld, c0 + cg * CPT, p.dv);
    // The next chunk's values travel from memory into registers while this chunk is worked on from shared
    // memory, so that their latency is not added to the chain through the tokens.
    float rq[NST], rk[NST], ra[MEM ? 1 : NST], rv[NSV], rg_ = 0.f, rs = 1.f;
    const int dv_in = p.dv - ((MEM && p.ones_col) ? 1 : 0);   // value columns a head has in memory
    auto fetch = [&](int tb, int n) {
#pragma unroll
        for (int u = 0; u < NST; ++u) {
            const int idx = threadIdx.x + u * THREADS;
            const int tt = idx / DKP, i = idx % DKP;
            rq[u] = rk[u] = 0.f;
            if constexpr (!MEM) ra[u] = 0.f;
            if (tt < n && i < p.dk) {
                const float* row = p.qkv + (size_t)(tb + tt) * p.ld;
                rq[u] = row[p.q_off + hk * p.dk + i];
                rk[u] = row[p.k_off + hk * p.dk + i];
                if constexpr (!MEM) ra[u] = p.decay[(size_t)(tb + tt) * p.heads * p.dk + h * p.dk + i];
            }
        }
#pragma unroll
        for (int u = 0; u < NSV; ++u) {
            const int idx = threadIdx.x + u * THREADS;
            const int tt = idx / COLS, cc = idx % COLS;
            rv[u] = (tt < n && c0 + cc < dv_in) ? p.qkv[(size_t)(tb + tt) * p.ld + p.v_off + h * dv_in + c0 + cc]
                                                : ((MEM && tt < n && p.ones_col && c0 + cc == dv_in) ? 1.f : 0.f);
        }
        if constexpr (MEM) {
            if (threadIdx.x < TOK_CHUNK && (int)threadIdx.x < n) {
                rg_ = p.decay[(size_t)(tb + threadIdx.x) * p.heads + h];
                if (p.k_scale) rs = p.k_scale[(size_t)(tb + threadIdx.x) * p.heads + h];
            }
        }
    };
    if (t0 < t1) fetch(t0, min(TOK_CHUNK, t1 - t0));
    const ulonglong2* q2 = reinterpret_cast<const ulonglong2*>(qs + row0);
    const ulonglong2* k2 = reinterpret_cast<const ulonglong2*>(ks + row0);
    const ulonglong2* a2 = reinterpret_cast<const ulonglong2*>(as + row0);
    // the column whose sum ends in this lane, and whether this lane stores it
    const int my_col = cg * CPT + (CPT == 4 ? ((lane & 16) ? 2 : 0) + ((lane & 8) ? 1 : 0) : ((lane & 16) ? 1 : 0));
    const bool mine = CPT == 4 || (lane & 8) == 0;
    for (int tb = t0; tb < t1; tb += TOK_CHUNK) {
        const int n = min(TOK_CHUNK, t1 - tb);
        __syncthreads();                      // the chunk before has been read
#pragma unroll
        for (int u = 0; u < NST; ++u) {
            const int idx = threadIdx.x + u * THREADS;
            qs[idx] = rq[u] * p.q_scale;
            ks[idx] = rk[u];
            if constexpr (!MEM) as[idx] = ra[u];
        }
#pragma unroll
        for (int u = 0; u < NSV; ++u) {
            const int idx = threadIdx.x + u * THREADS;
            if (TOK_CHUNK * COLS % THREADS == 0 || idx < TOK_CHUNK * COLS) vs[idx] = rv[u];
        }
        if constexpr (MEM) { if (threadIdx.x < TOK_CHUNK) { gs[threadIdx.x] = rg_; gs[TOK_CHUNK + threadIdx.x] = rs; } }
        __syncthreads();
        if (tb + TOK_CHUNK < t1) fetch(tb + TOK_CHUNK, min(TOK_CHUNK, t1 - tb - TOK_CHUNK));
#pragma unroll 2
        for (int tt = 0; tt < n; ++tt) {
            bw::f32x2 v[CPT], g = 0;
            bw::tile_values<CPT>(v, vs + tt * COLS + cg * CPT, MEM ? gs[TOK_CHUNK + tt] : 1.f);
            if constexpr (MEM) { const float g1 = gs[tt]; g = bw::pack2(g1, g1); }
            bw::f32x2 acc[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) acc[c] = 0;     // (two zeros)
#pragma unroll
            for (int j = 0; j < RP / 2; ++j) {
                const ulonglong2 k = k2[tt * (DKP / 4) + j], q = q2[tt * (DKP / 4) + j];
                ulonglong2 a;
                if constexpr (MEM) { a.x = g; a.y = g; } else a = a2[tt * (DKP / 4) + j];
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    s[2 * j][c] = bw::fma2(a.x, s[2 * j][c], bw::mul2(k.x, v[c]));
                    s[2 * j + 1][c] = bw::fma2(a.y, s[2 * j + 1][c], bw::mul2(k.y, v[c]));
                    acc[c] = bw::fma2(s[2 * j][c], q.x, acc[c]);
                    acc[c] = bw::fma2(s[2 * j + 1][c], q.y, acc[c]);
                }
            }
            float sum;
            if constexpr (CPT == 4) sum = bw::tile_sum4(bw::sum2(acc[0]), bw::sum2(acc[1]), bw::sum2(acc[2]), bw::sum2(acc[3]));
            else sum = bw::tile_sum2(bw::sum2(acc[0]), bw::sum2(acc[1]));
            if (mine) part[(tt * NW + warp) * COLS + my_col] = sum;
        }
        __syncthreads();
        for (int idx = threadIdx.x; idx < n * COLS; idx += THREADS) {
            const int tt = idx / COLS, cc = idx % COLS;
            float o = 0.f;
#pragma unroll
            for (int w = 0; w < NW; ++w) o += part[(tt * NW + w) * COLS + cc];
            if (c0 + cc < p.dv) p.o[(size_t)(tb + tt) * p.heads * p.dv + h * p.dv + c0 + cc] = o;
        }
    }
    bw::tile_store<CPT>(s, S, row0, p.dk, p.sld, c0 + cg * CPT, p.dv);
}

template <int NW, int CPT, bool MEM, int TOK_CHUNK>
int launch_scan(const ScanParams& p, int R, cudaStream_t s) {
    constexpr int smem = ScanSmem<NW, CPT, MEM, TOK_CHUNK>::floats * (int)sizeof(float), COLS = bw::TILE_CG * CPT;
    static bool raised[bw::MAX_DEVICES] = {};
    if (smem > 48 * 1024)
        if (bw::allow_dynamic_smem(gla_scan_kernel<NW, CPT, MEM, TOK_CHUNK>, smem, raised) != cudaSuccess) return BW_ERR_DRIVER;
    bw::launch((gla_scan_kernel<NW, CPT, MEM, TOK_CHUNK>), dim3(R, p.heads, (p.dv + COLS - 1) / COLS), dim3(32 * NW), smem, s, p);
    BW_LAUNCH_CHECK();
    return 0;
}

// few blocks: narrower ones, so that more SMs work
inline bool scan_narrow(int R, int heads, int dv) { return (long long)R * heads * ((dv + 31) / 32) < (long long)bw::num_sms() * SCAN_NARROW_BELOW / 4; }

template <int NW, bool MEM>
int launch_scan_any(const ScanParams& p, int R, cudaStream_t s) {
    if (p.single) return launch_scan<NW, 4, MEM, 1>(p, R, s);
    return scan_narrow(R, p.heads, p.dv) ? launch_scan<NW, 2, MEM, 16>(p, R, s) : launch_scan<NW, 4, MEM, 16>(p, R, s);
}

// one warp per (token, head): o / sqrt(mean(o^2) + eps) * gain[c] * silu(g[c]); ready != 0: times g[c] as it is
template <typename OT>
__global__ void __launch_bounds__(128)
gla_gate_kernel(const float* __restrict__ o, const float* __restrict__ g, long long g_ld, int g_off,
                const float* __restrict__ gain, OT* __restrict__ out, int T, int heads, int dv, float eps, int ready) {
    BW_PDL_TRIGGER();
    BW_PDL_WAIT();
    const int item = blockIdx.x * 4 + (threadIdx.x >> 5);
    const int lane = threadIdx.x & 31;
    if (item >= T * heads) return;
    const int t = item / heads, h = item - t * heads;
    const float* orow = o + (size_t)t * heads * dv + (size_t)h * dv;
    const float* grow = g + (size_t)t * g_ld + g_off + (size_t)h * dv;
    float ss = 0.f;
    for (int c = lane; c < dv; c += 32) { const float v = orow[c]; ss = fmaf(v, v, ss); }
    ss = bw::warp_sum(ss);
    const float r = rsqrtf(ss / (float)dv + eps);
    OT* dst = out + (size_t)t * heads * dv + (size_t)h * dv;
    for (int c = lane; c < dv; c += 32) {
        const float gv = grow[c];
        const float sg = ready ? gv : gv / (1.f + expf(-gv));
        dst[c] = bw::from_f32<OT>(orow[c] * r * gain[c] * sg);
    }
}

}  // namespace

// decay: float32 [T, heads * dk] from bw_gla_decay; with scalar_decay [T, heads].  k_scale: float32 [T, heads] or null.
// ones_col != 0: dv counts a last column of ones that v does not hold (state [slots, heads, dk, state_ld], o [T, heads * dv]).
// state_ld: floats between the state's rows (0: dv); columns from dv on stay zero.
// qk_rep: head h uses query/key head h / qk_rep (1: every head has its own).  single != 0: one token per request.
BW_EXPORT int bw_gla_scan(const float* qkv, long long ld, int q_off, int k_off, int v_off, const float* decay,
                          const int* cu_q, const int* state_slot, float* state, float* o, int R, int heads, int dk,
                          int dv, float q_scale, const float* k_scale, int scalar_decay, int ones_col, int state_ld,
                          int qk_rep, int single, void* stream) {
    if (R <= 0) return 0;
    if (heads <= 0 || dk <= 0 || dv <= 0 || (ones_col && dv < 2) || (state_ld != 0 && state_ld < dv) ||
        qk_rep <= 0 || heads % qk_rep)
        return BW_ERR_BAD_ARG;
    if (dk > MAX_DK) return BW_ERR_UNSUPPORTED;
    ScanParams p;
    p.qkv = qkv; p.decay = decay; p.cu_q = cu_q; p.state_slot = state_slot; p.state = state; p.o = o; p.ld = ld;
    p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.heads = heads; p.dk = dk; p.dv = dv;
    p.q_scale = q_scale;
    p.k_scale = k_scale; p.scalar_decay = scalar_decay; p.ones_col = ones_col; p.sld = state_ld ? state_ld : dv;
    p.rep = qk_rep; p.single = single;
    cudaStream_t s = (cudaStream_t)stream;
    const bool mem = k_scale || scalar_decay || ones_col || qk_rep > 1;
    if (mem && !scalar_decay) return BW_ERR_UNSUPPORTED;     // the memory's form has one decay per head
    if (dk <= 32) return mem ? launch_scan_any<1, true>(p, R, s) : launch_scan_any<1, false>(p, R, s);
    if (dk <= 64) return mem ? launch_scan_any<2, true>(p, R, s) : launch_scan_any<2, false>(p, R, s);
    if (dk <= 128) return mem ? launch_scan_any<4, true>(p, R, s) : launch_scan_any<4, false>(p, R, s);
    return mem ? launch_scan_any<8, true>(p, R, s) : launch_scan_any<8, false>(p, R, s);
}

// x: float32 [T, ldx], the decay's first projection at column x_off; w [C, rank] and b [C] of w_type.
BW_EXPORT int bw_gla_decay(const float* x, long long ldx, int x_off, const void* w, const void* b, int w_type, float* a,
                           int T, int C, int rank, float tau, void* stream) {
    if (T <= 0) return 0;
    if (C <= 0 || rank <= 0 || !(tau > 0.f)) return BW_ERR_BAD_ARG;
    const long long total = (long long)T * C;
    const dim3 grid((unsigned)((total + 255) / 256));
    cudaStream_t s = (cudaStream_t)stream;
    if (w_type == BW_F32) bw::launch((gla_decay_kernel<float>), grid, dim3(256), 0, s, x, ldx, x_off, (const float*)w, (const float*)b, a, T, C, rank, 1.f / tau);
    else if (w_type == BW_BF16) bw::launch((gla_decay_kernel<bf16>), grid, dim3(256), 0, s, x, ldx, x_off, (const bf16*)w, (const bf16*)b, a, T, C, rank, 1.f / tau);
    else return BW_ERR_BAD_ARG;
    BW_LAUNCH_CHECK();
    return 0;
}

// ready != 0: g holds the gate itself (whatever activation it has is in it already); 0: its silu is taken here.
BW_EXPORT int bw_gla_gate(const float* o, const float* g, long long g_ld, int g_off, const float* gain, void* out,
                          int out_type, int T, int heads, int dv, float eps, int ready, void* stream) {
    if (T <= 0) return 0;
    if (heads <= 0 || dv <= 0) return BW_ERR_BAD_ARG;
    const int items = T * heads;
    cudaStream_t s = (cudaStream_t)stream;
    if (out_type == BW_F32)
        bw::launch((gla_gate_kernel<float>), dim3((items + 3) / 4), dim3(128), 0, s, o, g, g_ld, g_off, gain, (float*)out, T, heads, dv, eps, ready);
    else if (out_type == BW_BF16)
        bw::launch((gla_gate_kernel<bf16>), dim3((items + 3) / 4), dim3(128), 0, s, o, g, g_ld, g_off, gain, (bf16*)out, T, heads, dv, eps, ready);
    else return BW_ERR_BAD_ARG;
    BW_LAUNCH_CHECK();
    return 0;
}
