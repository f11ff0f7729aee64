// The gated delta rule: a recurrent mixer whose state S [dk, dv] per head decays by one number per token, then takes in the
// part of the token's value that it does not yet return for the token's key:
//
//   S <- g_t S        u = beta_t (v_t - S^T k_t)        S <- S + k_t u^T        o_t = S^T q_t
//
// delta_scan_kernel walks the tokens of one request's portion in order (a single decoded token and a portion of a prompt
// are the same case), from the state the steps before left in the request's slot, and leaves the new state there.  A block
// owns (request, head, COLS value columns); LPC neighbouring lanes own one column, its dk state rows spread over them, in
// registers, two rows per packed instruction.  The chain through the tokens is one product with k, a sum over LPC lanes and
// the update; the sum for q of the token before rides in the same shuffles.  The order of all sums depends on dk alone, never on how the tokens were
// cut into steps or on the batch.  Everything is float32.  A second form has one decay per head and KEY CHANNEL: row c of the
// state decays by g_t[c]; a token's decays are staged beside its q and k.
#include "common.cuh"

using bf16 = __nv_bfloat16;

namespace {

constexpr int THREADS = 128;
constexpr int MAX_DK = 256;

struct DeltaParams {
    const float* qkv; long long ld;        // rows of q, k, v (already convolved, q and k unit vectors, q scaled)
    int q_off, k_off, v_off;
    const float *decay, *beta;             // [T, heads]; with a decay per key channel: decay [T, heads * dk]
    const int *cu_q, *state_slot;
    float* state;                          // [slots, heads, dk, dv]
    float* o;                              // [T, heads * dv]
    int heads, rep, dk, dv;                // head h uses query/key head h / rep
};

// LPC lanes per column, RPL rows per lane (a multiple of 4): dk <= LPC * RPL.  Lane l of a column holds rows
// (j * LPC + l) * 4 + e (j < RPL / 4, e < 4); in shared memory a token's q and k are padded with zeros to LPC * RPL rows.  TOK
// tokens are staged at a time: 16, or 1 in steps of single tokens.
// CH: a decay per key channel.
template <int LPC, int RPL, int TOK, bool CH>
__global__ void __launch_bounds__(THREADS)
delta_scan_kernel(DeltaParams p) {
    BW_PDL_TRIGGER();
    constexpr int DKP = LPC * RPL, COLS = THREADS / LPC;
    constexpr int NST = (TOK * DKP + THREADS - 1) / THREADS, NSV = (TOK * COLS + THREADS - 1) / THREADS;
    __shared__ __align__(16) float qs[TOK * DKP], ks[TOK * DKP];
    __shared__ __align__(16) float gs[CH ? TOK * DKP : TOK];
    __shared__ float vs[TOK * COLS], bs[TOK];
    const int r = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS;
    const int l = threadIdx.x % LPC, cc = threadIdx.x / LPC, col = c0 + cc;
    const int t0 = p.cu_q[r], t1 = p.cu_q[r + 1];
    const int hk = h / p.rep;
    float* S = p.state + ((size_t)p.state_slot[r] * p.heads + h) * (size_t)p.dk * p.dv;
    BW_PDL_WAIT();
    bw::f32x2 s[RPL / 2];
#pragma unroll
    for (int j = 0; j < RPL / 2; ++j) {
        const int i = ((j >> 1) * LPC + l) * 4 + (j & 1) * 2;
        s[j] = bw::pack2((i < p.dk && col < p.dv) ? S[(size_t)i * p.dv + col] : 0.f,
                         (i + 1 < p.dk && col < p.dv) ? S[(size_t)(i + 1) * p.dv + col] : 0.f);
    }
    // the next chunk's values travel into registers while this chunk is worked on from shared memory
    float rq[NST], rk[NST], rv[NSV], rc[CH ? NST : 1], rg = 0.f, rb = 0.f;
    auto fetch = [&](int tb, int n) {
#pragma unroll
        for (int u = 0; u < NST; ++u) {
            const int idx = threadIdx.x + u * THREADS;
            const int tt = idx / DKP, i = idx % DKP;
            rq[u] = rk[u] = 0.f;
            if constexpr (CH) rc[u] = 0.f;
            if (tt < n && i < p.dk) {
                const float* row = p.qkv + (size_t)(tb + tt) * p.ld + hk * p.dk + i;
                rq[u] = row[p.q_off];
                rk[u] = row[p.k_off];
                if constexpr (CH) rc[u] = p.decay[((size_t)(tb + tt) * p.heads + h) * p.dk + i];
            }
        }
#pragma unroll
        for (int u = 0; u < NSV; ++u) {
            const int idx = threadIdx.x + u * THREADS;
            const int tt = idx / COLS, c = idx % COLS;
            rv[u] = (tt < n && c0 + c < p.dv) ? p.qkv[(size_t)(tb + tt) * p.ld + p.v_off + h * p.dv + c0 + c] : 0.f;
        }
        if (threadIdx.x < TOK && (int)threadIdx.x < n) {
            if constexpr (!CH) rg = p.decay[(size_t)(tb + threadIdx.x) * p.heads + h];
            rb = p.beta[(size_t)(tb + threadIdx.x) * p.heads + h];
        }
    };
    if (t0 < t1) fetch(t0, min(TOK, t1 - t0));
    const ulonglong2* q4 = reinterpret_cast<const ulonglong2*>(qs);
    const ulonglong2* k4 = reinterpret_cast<const ulonglong2*>(ks);
    const ulonglong2* g4 = reinterpret_cast<const ulonglong2*>(gs);
    const bool writes = l == 0 && col < p.dv;
    float* orow = p.o + (size_t)h * p.dv + col;          // + token * heads * dv
    const size_t o_ld = (size_t)p.heads * p.dv;
    float pq = 0.f;                                      // this lane's part of the last token's S^T q
    for (int tb = t0; tb < t1; tb += TOK) {
        const int n = min(TOK, t1 - tb);
        __syncthreads();                                 // the chunk before has been read
#pragma unroll
        for (int u = 0; u < NST; ++u) {
            const int idx = threadIdx.x + u * THREADS;
            if (TOK * DKP % THREADS == 0 || idx < TOK * DKP) {
                qs[idx] = rq[u]; ks[idx] = rk[u];
                if constexpr (CH) gs[idx] = rc[u];
            }
        }
#pragma unroll
        for (int u = 0; u < NSV; ++u) {
            const int idx = threadIdx.x + u * THREADS;
            if (TOK * COLS % THREADS == 0 || idx < TOK * COLS) vs[idx] = rv[u];
        }
        if (threadIdx.x < TOK) { if constexpr (!CH) gs[threadIdx.x] = rg; bs[threadIdx.x] = rb; }
        __syncthreads();
        if (tb + TOK < t1) fetch(tb + TOK, min(TOK, t1 - tb - TOK));
#pragma unroll 2
        for (int tt = 0; tt < n; ++tt) {
            const int base = tt * (DKP / 4) + l;
            const float g = CH ? 1.f : gs[tt], beta = bs[tt], v = vs[tt * COLS + cc];
            const bw::f32x2 g2 = bw::pack2(g, g);
            bw::f32x2 a0 = 0, a1 = 0;          // (pairs of zeros)
            ulonglong2 kk[RPL / 4];
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j) {
                kk[j] = k4[base + j * LPC];
                ulonglong2 gg;
                if constexpr (CH) gg = g4[base + j * LPC]; else { gg.x = g2; gg.y = g2; }
                s[2 * j] = bw::mul2(s[2 * j], gg.x);
                s[2 * j + 1] = bw::mul2(s[2 * j + 1], gg.y);
                a0 = bw::fma2(s[2 * j], kk[j].x, a0);
                a1 = bw::fma2(s[2 * j + 1], kk[j].y, a1);
            }
            float pk = bw::sum2(a0) + bw::sum2(a1);
#pragma unroll
            for (int d = LPC / 2; d > 0; d >>= 1) {
                pk += __shfl_xor_sync(0xffffffffu, pk, d);
                pq += __shfl_xor_sync(0xffffffffu, pq, d);
            }
            if (writes && tb + tt > t0) orow[(size_t)(tb + tt - 1) * o_ld] = pq;
            const float u = beta * (v - pk);
            const bw::f32x2 u2 = bw::pack2(u, u);
            bw::f32x2 b0 = 0, b1 = 0;
#pragma unroll
            for (int j = 0; j < RPL / 4; ++j) {
                const ulonglong2 q = q4[base + j * LPC];
                s[2 * j] = bw::fma2(kk[j].x, u2, s[2 * j]);
                s[2 * j + 1] = bw::fma2(kk[j].y, u2, s[2 * j + 1]);
                b0 = bw::fma2(s[2 * j], q.x, b0);
                b1 = bw::fma2(s[2 * j + 1], q.y, b1);
            }
            pq = bw::sum2(b0) + bw::sum2(b1);
        }
    }
#pragma unroll
    for (int d = LPC / 2; d > 0; d >>= 1) pq += __shfl_xor_sync(0xffffffffu, pq, d);
    if (writes && t1 > t0) orow[(size_t)(t1 - 1) * o_ld] = pq;
#pragma unroll
    for (int j = 0; j < RPL / 2; ++j) {
        const int i = ((j >> 1) * LPC + l) * 4 + (j & 1) * 2;
        float lo, hi;
        bw::unpack2(s[j], lo, hi);
        if (i < p.dk && col < p.dv) S[(size_t)i * p.dv + col] = lo;
        if (i + 1 < p.dk && col < p.dv) S[(size_t)(i + 1) * p.dv + col] = hi;
    }
}

}  // namespace

// qkv: float32 rows `ld` apart with q and k (heads / rep heads of dk channels) and v (heads of dv) at the given columns;
// decay, beta float32 [T, heads]; state [slots, heads, dk, dv]; o [T, heads * dv].  single != 0: one token per request.
// channel != 0: decay is float32 [T, heads * dk], one number per key channel.
BW_EXPORT int bw_delta_scan(const float* qkv, long long ld, int q_off, int k_off, int v_off, const float* decay,
                            const float* beta, const int* cu_q, const int* state_slot, float* state, float* o, int R,
                            int heads, int rep, int dk, int dv, int channel, int single, void* stream) {
    if (R <= 0) return 0;
    if (heads <= 0 || rep <= 0 || heads % rep || dk <= 0 || dv <= 0) return BW_ERR_BAD_ARG;
    if (dk > MAX_DK) return BW_ERR_UNSUPPORTED;
    DeltaParams p;
    p.qkv = qkv; p.ld = ld; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.decay = decay; p.beta = beta;
    p.cu_q = cu_q; p.state_slot = state_slot; p.state = state; p.o = o; p.heads = heads; p.rep = rep; p.dk = dk; p.dv = dv;
    cudaStream_t s = (cudaStream_t)stream;
#define BW_DELTA(LPC, RPL) do { const dim3 grid(R, heads, (dv + THREADS / LPC - 1) / (THREADS / LPC)); \
        if (channel && single) bw::launch((delta_scan_kernel<LPC, RPL, 1, true>), grid, dim3(THREADS), 0, s, p); \
        else if (channel) bw::launch((delta_scan_kernel<LPC, RPL, (LPC * RPL > 128 ? 8 : 16), true>), grid, dim3(THREADS), 0, s, p); \
        else if (single) bw::launch((delta_scan_kernel<LPC, RPL, 1, false>), grid, dim3(THREADS), 0, s, p); \
        else bw::launch((delta_scan_kernel<LPC, RPL, 16, false>), grid, dim3(THREADS), 0, s, p); } while (0)
    if (dk <= 32) BW_DELTA(8, 4);
    else if (dk <= 64) BW_DELTA(8, 8);
    else if (dk <= 128) BW_DELTA(8, 16);
    else BW_DELTA(16, 16);
#undef BW_DELTA
    BW_LAUNCH_CHECK();
    return 0;
}
