// Recurrences with one decay per head and token (the delta rule also with one per key channel), for portions of prompts, 32 tokens at a time on the tensor cores with
// compensated products.  Two forms over a state S [dk, dv] per head:
//
//   linear   S <- g_t S + c_t k_t v_t^T                                          o_t = S^T q_t
//   delta    S <- g_t S;  u_t = beta_t (v_t - S^T k_t);  S <- S + k_t u_t^T      o_t = S^T q_t
//
// With S0 the state before a chunk, G_t the product of its decays up to t, R_t of those after t and D_ts that of the decays
// after s up to t (products, never quotients: a decay may be zero):
//
//   delta:   U = T B,  B_t = beta_t (v_t - G_t S0^T k_t),  T = (I + L)^-1,  L_ts = beta_t D_ts k_s . k_t  (s < t)
//   linear:  U = V, and c_s multiplies k_s below
//   o_t = G_t S0^T q_t + sum_{s<=t} M_ts u_s,    M_ts = D_ts k_s . q_t           S = G S0 + sum_s R_s k_s u_s^T
//
// A third form is the delta rule with a decay per KEY CHANNEL, S <- diag(g_t) S in place of g_t S.  Then D_ts is a vector inside
// the dot products, L_ts = beta_t sum_c k_s[c] D_ts[c] k_t[c] and M_ts likewise with q_t; G_t and R_t multiply q_t and k_t channel by
// channel, and the chunk's G is a vector over the state's rows.  Since U = T beta V - (T beta (G o K)) S0, the part of U that does not
// know S0 and the rows W = T beta (G o K) are made beforehand too, so that the walk needs no T: U = U0 - W S0.
// chunk_rows_channel_kernel makes all of that, again with products of decays only: the vector D_ts o k_s is carried along t in
// registers.
//
// chunk_rows_kernel makes the rows of T and M and the numbers G, R for every token and head, in parallel over the chunks, with
// float32 FMAs.  chunk_scan_kernel walks the chunks of one request's portion: a block owns (request, head, 16 value columns)
// and keeps S^T in mma accumulators, [16, 32] per warp, the warps splitting dk; only two small exchanges per chunk cross
// warps.  State, decays and sums are float32; every product a b of the mma's is made as a_lo b_hi + a_hi b_lo + a_hi b_hi with
// a_hi the value rounded to 11 bits of mantissa and a_lo the rest, of which the tensor core reads the leading 11 bits; that leaves
// an error of about 2^-21 of a product (float32's own rounding is 2^-24), and the sums are float32.  The 32-bit path does not come here: it walks token by
// token (delta.cu, gla.cu), as do steps of single tokens.
#include "common.cuh"

namespace {

constexpr int C = 32;             // tokens of a chunk
constexpr int ROW_DELTA = 68;     // floats per (token, head): T row, M row, G, R, beta, 0
constexpr int ROW_LINEAR = 36;    // M row (with c_s in it), G, c R, 0, 0
constexpr int ROW_CHANNEL = 32;   // M row
constexpr int TS = 40;            // floats between rows of 32 in shared memory: 8-byte reads of (row g, column 2 t) hit 32 banks
constexpr int VS = 20;            // floats between tokens' 16 values
constexpr int COLS = 16;

struct ChunkParams {
    const float* qkv; long long ld; int q_off, k_off, v_off;
    const float *decay, *second;           // [T, heads]: g; beta (delta) or c (linear)
    const int *cu_q, *state_slot;
    float* rows;                           // [T, heads, ROW]
    float* state; int sld;                 // [slots, heads, dk, sld]
    float* o;                              // [T, heads * dv]
    int T, R, heads, rep, dk, dv, vec;     // vec: 16-byte copies of q and k rows (1), of the values (2)
    // the form with a decay per key channel: decay [T, heads, dk], and two more scratches
    float* chan;                           // [T, heads, 3, dk]: W, G o q, R o k
    float* u0;                             // [T, heads, dv]: U0
    float* gend;                           // [T / C + R, heads, dk]: the product of a chunk's decays (chunk_index)
};

// The number of request r's i-th chunk among all chunks of a step, a its first token: distinct for all chunks, below T / C + R.
__device__ __forceinline__ int chunk_index(int r, int a, int i) { return a / C + r + i; }

// The chunk of this block: its first token (< 0: none), its tokens and chunk_index; `number` counts the chunks of all requests.
__device__ __forceinline__ void find_chunk(const ChunkParams& p, int number, int& t0, int& n, int& index) {
    const int lane = threadIdx.x & 31;
    t0 = -1; n = 0; index = 0;
    for (int r0 = 0, before = 0; r0 < p.R; r0 += 32) {
        const int r = r0 + lane;
        const int a = r < p.R ? p.cu_q[r] : 0, len = r < p.R ? p.cu_q[r + 1] - a : 0;
        int upto = (len + C - 1) / C;
#pragma unroll
        for (int d = 1; d < 32; d <<= 1) {
            const int v = __shfl_up_sync(0xffffffffu, upto, d);
            if (lane >= d) upto += v;
        }
        const unsigned has = __ballot_sync(0xffffffffu, before + upto > number);
        if (has) {
            const int l = __ffs(has) - 1;                  // the first request whose chunks reach past this one
            const int first = number - (before + (l ? __shfl_sync(0xffffffffu, upto, l - 1) : 0));
            const int start = __shfl_sync(0xffffffffu, a, l);
            t0 = start + first * C;
            n = min(C, __shfl_sync(0xffffffffu, a + len, l) - t0);
            index = chunk_index(r0 + l, start, first);
            return;
        }
        before += __shfl_sync(0xffffffffu, upto, 31);
    }
}

// ------------------------------------------------------------------ the chunks' small matrices
// One block per (chunk, query/key head); the grid has room for as many chunks as the requests can have, blocks behind the last
// one leave.
template <bool DELTA, int DKP>
__global__ void __launch_bounds__(128)
chunk_rows_kernel(ChunkParams p) {
    BW_PDL_TRIGGER();
    const int hk = blockIdx.y;
    int t0, n, index;
    find_chunk(p, blockIdx.x, t0, n, index);
    if (t0 < 0) return;
    extern __shared__ __align__(16) float sm[];
    constexpr int lds = DKP + 4;
    float* ks = sm;                        // [C][lds]
    float* qs = ks + C * lds;              // [C][lds]
    float* kk = qs + C * lds;              // [C][C + 1] each
    float* kq = kk + C * (C + 1);
    float* Ls = kq + C * (C + 1);          // [4][C][C + 4]
    BW_PDL_WAIT();
    if (p.vec & 1) {
#pragma unroll 4
        for (int idx = threadIdx.x; idx < C * DKP / 4; idx += 128) {
            const int t = idx / (DKP / 4), i = (idx % (DKP / 4)) * 4;
            const bool in = t < n && i < p.dk;
            const float* src = p.qkv + (size_t)(t0 + t) * p.ld + hk * p.dk + i;
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
            *reinterpret_cast<float4*>(ks + t * lds + i) = in ? *reinterpret_cast<const float4*>(src + p.k_off) : zero;
            *reinterpret_cast<float4*>(qs + t * lds + i) = in ? *reinterpret_cast<const float4*>(src + p.q_off) : zero;
        }
    } else {
#pragma unroll 4
        for (int idx = threadIdx.x; idx < C * DKP; idx += 128) {
            const int t = idx / DKP, i = idx % DKP;
            const bool in = t < n && i < p.dk;
            const float* src = p.qkv + (size_t)(t0 + t) * p.ld + hk * p.dk + i;
            ks[t * lds + i] = in ? src[p.k_off] : 0.f;
            qs[t * lds + i] = in ? src[p.q_off] : 0.f;
        }
    }
    __syncthreads();
    {
        const int t = threadIdx.x >> 2, sg = threadIdx.x & 3;      // s = sg, sg + 4, ..
        float x[8], y[8];
#pragma unroll
        for (int j = 0; j < 8; ++j) x[j] = y[j] = 0.f;
        for (int i = 0; i < DKP; i += 4) {
            const float4 kt = *reinterpret_cast<const float4*>(ks + t * lds + i), qt = *reinterpret_cast<const float4*>(qs + t * lds + i);
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const float4 k = *reinterpret_cast<const float4*>(ks + (sg + 4 * j) * lds + i);
                if constexpr (DELTA) { x[j] = fmaf(k.x, kt.x, x[j]); x[j] = fmaf(k.y, kt.y, x[j]); x[j] = fmaf(k.z, kt.z, x[j]); x[j] = fmaf(k.w, kt.w, x[j]); }
                y[j] = fmaf(k.x, qt.x, y[j]); y[j] = fmaf(k.y, qt.y, y[j]); y[j] = fmaf(k.z, qt.z, y[j]); y[j] = fmaf(k.w, qt.w, y[j]);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if constexpr (DELTA) kk[t * (C + 1) + sg + 4 * j] = x[j];
            kq[t * (C + 1) + sg + 4 * j] = y[j];
        }
    }
    __syncthreads();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    constexpr int ROW = DELTA ? ROW_DELTA : ROW_LINEAR, M0 = DELTA ? C : 0;
    float* L = Ls + warp * C * (C + 4);
    for (int h = hk * p.rep + warp; h < (hk + 1) * p.rep; h += 4) {
        const float g = lane < n ? p.decay[(size_t)(t0 + lane) * p.heads + h] : 1.f;
        const float c = lane < n ? p.second[(size_t)(t0 + lane) * p.heads + h] : 0.f;
        float G = g, R = g;                // products over the tokens up to this lane's; from this lane's on
#pragma unroll
        for (int d = 1; d < 32; d <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, G, d), down = __shfl_down_sync(0xffffffffu, R, d);
            if (lane >= d) G *= up;
            if (lane + d < 32) R *= down;
        }
        R = __shfl_down_sync(0xffffffffu, R, 1);
        if (lane == 31) R = 1.f;
        float* base = p.rows + ((size_t)t0 * p.heads + h) * ROW;
        const size_t step = (size_t)p.heads * ROW;
        float D = 1.f;                     // lane s: D_ts, t rising
        for (int t = 0; t < n; ++t) {
            const float gt = __shfl_sync(0xffffffffu, g, t), ct = __shfl_sync(0xffffffffu, c, t);
            if (t > lane) D *= gt;
            const float m = t >= lane ? D * kq[t * (C + 1) + lane] : 0.f;
            base[t * step + M0 + lane] = DELTA ? m : m * c;
            if constexpr (DELTA) L[t * (C + 4) + lane] = t > lane ? ct * D * kk[t * (C + 1) + lane] : 0.f;
        }
        if (lane < n) {
            float* sc = base + lane * step + M0 + C;
            sc[0] = G; sc[1] = DELTA ? R : R * c; sc[2] = DELTA ? c : 0.f; sc[3] = 0.f;
        }
        if constexpr (DELTA) {
            for (int t = n; t < C; ++t) L[t * (C + 4) + lane] = 0.f;
            __syncwarp();
            float x[C];                    // lane s: column s of T, row by row
#pragma unroll
            for (int t = 0; t < C; ++t) {
                float s0 = t == lane ? 1.f : 0.f, s1 = 0.f;
#pragma unroll
                for (int j = 0; j < t; j += 4) {
                    const float4 l = *reinterpret_cast<const float4*>(L + t * (C + 4) + j);
                    s0 = fmaf(-l.x, x[j], s0);
                    if (j + 1 < t) s1 = fmaf(-l.y, x[j + 1], s1);
                    if (j + 2 < t) s0 = fmaf(-l.z, x[j + 2], s0);
                    if (j + 3 < t) s1 = fmaf(-l.w, x[j + 3], s1);
                }
                x[t] = s0 + s1;
                if (t < n) base[t * step + lane] = x[t];
            }
            __syncwarp();
        }
    }
}

// The same for a decay per key channel.  One block per (chunk, head).  DKP: dk up to a multiple of 32.
template <int DKP>
__global__ void __launch_bounds__(128, DKP <= 128 ? 4 : 1)
chunk_rows_channel_kernel(ChunkParams p) {
    BW_PDL_TRIGGER();
    constexpr int lds = DKP;
    const int h = blockIdx.y, hk = h / p.rep;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    int t0, n, index;
    find_chunk(p, blockIdx.x, t0, n, index);
    if (t0 < 0) return;
    extern __shared__ __align__(16) float sm[];
    float* ks = sm;                        // [C][lds] each
    float* qs = ks + C * lds;
    float* gs = qs + C * lds;
    float* kk = gs + C * lds;              // [C][C + 4]: sum_c k_s D_ts k_t, turned into L and then into T beta in place
    float* m_rows = p.rows + ((size_t)t0 * p.heads + h) * ROW_CHANNEL;      // M: what the walk reads of it (8 x 8 blocks up to the diagonal's)
    const size_t m_step = (size_t)p.heads * ROW_CHANNEL;
    BW_PDL_WAIT();
    if (p.vec & 1) {
#pragma unroll 4
        for (int idx = threadIdx.x; idx < C * DKP / 4; idx += 128) {
            const int t = idx / (DKP / 4), i = (idx % (DKP / 4)) * 4;
            const bool in = t < n && i < p.dk;
            const float* src = p.qkv + (size_t)(t0 + t) * p.ld + hk * p.dk + i;
            const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
            *reinterpret_cast<float4*>(ks + t * lds + i) = in ? *reinterpret_cast<const float4*>(src + p.k_off) : zero;
            *reinterpret_cast<float4*>(qs + t * lds + i) = in ? *reinterpret_cast<const float4*>(src + p.q_off) : zero;
            *reinterpret_cast<float4*>(gs + t * lds + i) = in ? *reinterpret_cast<const float4*>(p.decay + ((size_t)(t0 + t) * p.heads + h) * p.dk + i) : zero;
        }
    } else {
#pragma unroll 4
        for (int idx = threadIdx.x; idx < C * DKP; idx += 128) {
            const int t = idx / DKP, i = idx % DKP;
            const bool in = t < n && i < p.dk;
            const float* src = p.qkv + (size_t)(t0 + t) * p.ld + hk * p.dk + i;
            ks[t * lds + i] = in ? src[p.k_off] : 0.f;
            qs[t * lds + i] = in ? src[p.q_off] : 0.f;
            gs[t * lds + i] = in ? p.decay[((size_t)(t0 + t) * p.heads + h) * p.dk + i] : 0.f;
        }
    }
    __syncthreads();
    {
        // Warp w has the tokens s = 8 w .. 8 w + 7, lane = NG sl + cg the NS of them from 8 w + NS sl on, on the channels
        // (NG j + cg) 4 + e; z = D_ts o k_s goes along t, zero before s.
        constexpr int NG = DKP >= 64 ? 16 : 8, NS = NG / 4, CH = DKP / NG;
        const int cg = lane % NG, s0 = 8 * warp + NS * (lane / NG);
        bw::f32x2 z[NS][CH / 2];
#pragma unroll
        for (int u = 0; u < NS; ++u)
#pragma unroll
            for (int j = 0; j < CH / 2; ++j) z[u][j] = 0;              // (pairs of zeros)
        for (int idx = threadIdx.x; idx < C * (C + 4); idx += 128) kk[idx] = 0.f;
        __syncthreads();
        const ulonglong2 *k4 = reinterpret_cast<const ulonglong2*>(ks) + cg, *q4 = reinterpret_cast<const ulonglong2*>(qs) + cg,
                         *g4 = reinterpret_cast<const ulonglong2*>(gs) + cg;
        for (int t = 8 * warp; t < n; ++t) {
            bw::f32x2 a[2 * NS];                                       // sums with k_t, then with q_t
#pragma unroll
            for (int u = 0; u < 2 * NS; ++u) a[u] = 0;
            const bool near = t < 8 * warp + 8;                        // (uniform over the warp)
#pragma unroll
            for (int j = 0; j < CH / 4; ++j) {
                const int at = t * (lds / 4) + NG * j;
                const ulonglong2 k = k4[at], q = q4[at], g = g4[at];
#pragma unroll
                for (int u = 0; u < NS; ++u) {
                    z[u][2 * j] = bw::mul2(z[u][2 * j], g.x);
                    z[u][2 * j + 1] = bw::mul2(z[u][2 * j + 1], g.y);
                    if (near && t == s0 + u) { z[u][2 * j] = k.x; z[u][2 * j + 1] = k.y; }
                    a[u] = bw::fma2(z[u][2 * j], k.x, a[u]);
                    a[u] = bw::fma2(z[u][2 * j + 1], k.y, a[u]);
                    a[NS + u] = bw::fma2(z[u][2 * j], q.x, a[NS + u]);
                    a[NS + u] = bw::fma2(z[u][2 * j + 1], q.y, a[NS + u]);
                }
            }
            // 2 NS sums over the NG lanes of a group of tokens: at every step a lane keeps half of its sums and gives the other half
            // away; it ends with the one that its bits from NG / 2 down to 2 name
            float v[2 * NS];
#pragma unroll
            for (int u = 0; u < 2 * NS; ++u) v[u] = bw::sum2(a[u]);
#pragma unroll
            for (int m = NG / 2, w = NS; m >= 2; m >>= 1, w >>= 1) {
                const bool hi = lane & m;
#pragma unroll
                for (int u = 0; u < w; ++u) v[u] = (hi ? v[w + u] : v[u]) + __shfl_xor_sync(0xffffffffu, hi ? v[u] : v[w + u], m);
            }
            v[0] += __shfl_xor_sync(0xffffffffu, v[0], 1);
            if (!(lane & 1)) *((lane & (NG / 2)) ? m_rows + t * m_step + s0 + ((lane & (NG / 2 - 1)) >> 1)
                                                 : kk + t * (C + 4) + s0 + ((lane & (NG / 2 - 1)) >> 1)) = v[0];
        }
    }
    __syncthreads();
    if (warp == 0) {
        const float beta = lane < n ? p.second[(size_t)(t0 + lane) * p.heads + h] : 0.f;
        for (int t = 0; t < n; ++t) {
            const float bt = __shfl_sync(0xffffffffu, beta, t);
            kk[t * (C + 4) + lane] = t > lane ? bt * kk[t * (C + 4) + lane] : 0.f;
        }
        __syncwarp();
        float x[C];                        // lane s: column s of T, row by row (rows of kk from n on are zeros)
#pragma unroll
        for (int t = 0; t < C; ++t) {
            float u0 = t == lane ? 1.f : 0.f, u1 = 0.f;
#pragma unroll
            for (int j = 0; j < t; j += 4) {
                const float4 l = *reinterpret_cast<const float4*>(kk + t * (C + 4) + j);
                u0 = fmaf(-l.x, x[j], u0);
                if (j + 1 < t) u1 = fmaf(-l.y, x[j + 1], u1);
                if (j + 2 < t) u0 = fmaf(-l.z, x[j + 2], u0);
                if (j + 3 < t) u1 = fmaf(-l.w, x[j + 3], u1);
            }
            x[t] = u0 + u1;
        }
        __syncwarp();
#pragma unroll
        for (int t = 0; t < C; ++t) kk[t * (C + 4) + lane] = x[t] * beta;        // T beta in place of L (zero columns from n on)
    } else {
        // meanwhile the other warps: the rows with the decays in them; G o k stays here
        const size_t step = (size_t)p.heads * 3 * p.dk;
        for (int c = threadIdx.x - 32; c < p.dk; c += 96) {
            float* dst = p.chan + ((size_t)t0 * p.heads + h) * 3 * p.dk + c;
            float R = 1.f;
            for (int t = n - 1; t >= 0; --t) {
                dst[t * step + 2 * p.dk] = R * ks[t * lds + c];
                R *= gs[t * lds + c];
            }
            float G = 1.f;
            for (int t = 0; t < n; ++t) {
                G *= gs[t * lds + c];
                ks[t * lds + c] *= G;
                dst[t * step + p.dk] = G * qs[t * lds + c];
            }
            p.gend[((size_t)index * p.heads + h) * p.dk + c] = G;
        }
    }
    __syncthreads();
    // W = T beta (G o K) and U0 = T beta V: two columns a thread, which it keeps in registers
    const int cols = p.dk + p.dv;
    for (int c0 = threadIdx.x; c0 < cols; c0 += 256) {
        float x[2][C];
        float* dst[2];
        size_t step[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            const int c = c0 + 128 * u;
            const bool is_k = c < p.dk, there = c < cols;
            const float* v = p.qkv + (size_t)t0 * p.ld + p.v_off + h * p.dv + (c - p.dk);
            dst[u] = is_k ? p.chan + ((size_t)t0 * p.heads + h) * 3 * p.dk + c : (there ? p.u0 + ((size_t)t0 * p.heads + h) * p.dv + (c - p.dk) : nullptr);
            step[u] = (size_t)p.heads * (is_k ? 3 * p.dk : p.dv);
#pragma unroll
            for (int t = 0; t < C; ++t) x[u][t] = is_k ? ks[t * lds + c] : (there && t < n ? v[(size_t)t * p.ld] : 0.f);
        }
#pragma unroll
        for (int t = 0; t < C; ++t) {
            asm volatile("" ::: "memory");        // (rows of T beta are not fetched ahead: there are no registers for that)
            float a[2][2] = {{0.f, 0.f}, {0.f, 0.f}};
#pragma unroll
            for (int j = 0; j <= t; j += 4) {
                const float4 m = *reinterpret_cast<const float4*>(kk + t * (C + 4) + j);     // (zeros above the diagonal)
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    a[u][0] = fmaf(m.x, x[u][j], a[u][0]);
                    a[u][1] = fmaf(m.y, x[u][j + 1], a[u][1]);
                    a[u][0] = fmaf(m.z, x[u][j + 2], a[u][0]);
                    a[u][1] = fmaf(m.w, x[u][j + 3], a[u][1]);
                }
            }
            if (t < n) {
                dst[0][t * step[0]] = a[0][0] + a[0][1];
                if (dst[1]) dst[1][t * step[1]] = a[1][0] + a[1][1];
            }
        }
    }
}

// ------------------------------------------------------------------ the walk through the chunks
struct Split { uint32_t hi, lo; };
__device__ __forceinline__ Split split(float x) {
    Split s;
    s.hi = (__float_as_uint(x) + 0x1000u) & 0xffffe000u;                  // x rounded to the operand's 11 bits of mantissa
    s.lo = __float_as_uint(x - __uint_as_float(s.hi));                    // exact; the tensor core reads its leading 11 bits
    return s;
}
__device__ __forceinline__ void mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
struct SplitA { uint32_t hi[4], lo[4]; };
__device__ __forceinline__ SplitA split_a(float a0, float a1, float a2, float a3) {
    SplitA r;
    const float v[4] = {a0, a1, a2, a3};
#pragma unroll
    for (int i = 0; i < 4; ++i) { const Split s = split(v[i]); r.hi[i] = s.hi; r.lo[i] = s.lo; }
    return r;
}
// c[i] += a b[i] for N operands b with everything split: the two cross terms, then the leading one; N sums side by side, so
// that an instruction does not wait for the one before
template <int N>
__device__ __forceinline__ void mma3(float (&c)[N][4], const SplitA& a, const float (&b)[N][2]) {
    Split x[N], y[N];
#pragma unroll
    for (int i = 0; i < N; ++i) { x[i] = split(b[i][0]); y[i] = split(b[i][1]); }
#pragma unroll
    for (int i = 0; i < N; ++i) mma(c[i], a.lo, x[i].hi, y[i].hi);
#pragma unroll
    for (int i = 0; i < N; ++i) mma(c[i], a.hi, x[i].lo, y[i].lo);
#pragma unroll
    for (int i = 0; i < N; ++i) mma(c[i], a.hi, x[i].hi, y[i].hi);
}
// asynchronous copies into shared memory; in == false writes zeros and reads nothing
__device__ __forceinline__ void copy16(float* dst, const float* src, bool in) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    const int n = in ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" :: "r"(d), "l"(src), "r"(n) : "memory");
}
__device__ __forceinline__ void copy4(float* dst, const float* src, bool in) {
    const uint32_t d = (uint32_t)__cvta_generic_to_shared(dst);
    const int n = in ? 4 : 0;
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" :: "r"(d), "l"(src), "r"(n) : "memory");
}

// NW warps split dk (8 NB state rows each: dk <= DKP = 8 NB NW), MT groups of NW warps take 16 value columns each.
// CHAN: a decay per key channel (delta only).  The next chunk is fetched while this one is worked on where two fit.
template <bool DELTA, bool CHAN, int NW, int NB, int MT>
struct ChunkSmem {
    static constexpr int LDK = 8 * NB * NW + 4;                 // a token's q or k
    static constexpr int LDV = MT == 1 ? VS : 36;           // a token's values (twice it is 8 modulo 32)
    static constexpr int k0 = 0, q0 = k0 + C * LDK, v0 = q0 + C * LDK, m0 = v0 + C * LDV, t0 = m0 + C * TS, s0 = t0 + (DELTA && !CHAN ? C * TS : 0);
    static constexpr int r0 = s0 + (CHAN ? 0 : C * 4), g0 = r0 + (CHAN ? C * LDK : 0);
    static constexpr int buffer = g0 + (CHAN ? 8 * NB * NW : 0);
    static constexpr int part = (DELTA ? 2 : 1) * COLS * TS;            // one warp's parts of S0^T q (and S0^T k)
    static constexpr int tail = NW * MT * part + (DELTA ? MT * COLS * TS : 0);
    static constexpr int buffers = (2 * buffer + tail) * 4 <= 227 * 1024 ? 2 : 1;
    static constexpr int floats = buffers * buffer + tail;
};

template <bool DELTA, bool CHAN, int NW, int NB, int MT>
__global__ void __launch_bounds__(32 * NW * MT)
chunk_scan_kernel(ChunkParams p) {
    BW_PDL_TRIGGER();
    using L = ChunkSmem<DELTA, CHAN, NW, NB, MT>;
    constexpr int THREADS = 32 * NW * MT, DKP = 8 * NB * NW, LDK = L::LDK, LDV = L::LDV;
    constexpr int ROW = CHAN ? ROW_CHANNEL : (DELTA ? ROW_DELTA : ROW_LINEAR);
    extern __shared__ __align__(16) float sm[];
    float* part = sm + L::buffers * L::buffer;
    const int r = blockIdx.x, h = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, kw = warp % NW, mt = warp / NW;
    const int g = lane >> 2, t4 = lane & 3, pg = (g >> 1) + (g & 1) * 4;
    const int cb = blockIdx.z * COLS * MT, c0 = cb + mt * COLS;     // first value column of the block, of this warp
    const int k0 = kw * 8 * NB;                                          // first state row of this warp
    const int ta = p.cu_q[r], te = p.cu_q[r + 1], hk = h / p.rep;
    float* S = p.state + ((size_t)p.state_slot[r] * p.heads + h) * (size_t)p.dk * p.sld;
    float* my = part + (size_t)warp * L::part;
    float* us = part + (size_t)NW * MT * L::part + mt * COLS * TS;
    BW_PDL_WAIT();

    auto fetch = [&](int tb, int buf) {
        float* b = sm + buf * L::buffer;
        const int n = min(C, te - tb);
        const float* src = p.qkv + (size_t)tb * p.ld;
        if constexpr (CHAN) {
            const float* rows = p.chan + ((size_t)tb * p.heads + h) * 3 * p.dk;
            const size_t step = (size_t)p.heads * 3 * p.dk;
            const float* end = p.gend + ((size_t)chunk_index(r, ta, (tb - ta) / C) * p.heads + h) * p.dk;
            if (p.vec & 1) {
                for (int idx = threadIdx.x; idx < C * (DKP / 4); idx += THREADS) {
                    const int t = idx / (DKP / 4), i = (idx % (DKP / 4)) * 4;
                    const bool in = t < n && i < p.dk;
                    const float* s = in ? rows + t * step + i : rows;
                    copy16(b + L::k0 + t * LDK + i, s, in);
                    copy16(b + L::q0 + t * LDK + i, in ? s + p.dk : rows, in);
                    copy16(b + L::r0 + t * LDK + i, in ? s + 2 * p.dk : rows, in);
                }
            } else {
                for (int idx = threadIdx.x; idx < C * DKP; idx += THREADS) {
                    const int t = idx / DKP, i = idx % DKP;
                    const bool in = t < n && i < p.dk;
                    const float* s = in ? rows + t * step + i : rows;
                    copy4(b + L::k0 + t * LDK + i, s, in);
                    copy4(b + L::q0 + t * LDK + i, in ? s + p.dk : rows, in);
                    copy4(b + L::r0 + t * LDK + i, in ? s + 2 * p.dk : rows, in);
                }
            }
            for (int i = threadIdx.x; i < DKP; i += THREADS) copy4(b + L::g0 + i, i < p.dk ? end + i : end, i < p.dk);
        } else if (p.vec & 1) {
            for (int idx = threadIdx.x; idx < C * (DKP / 4); idx += THREADS) {
                const int t = idx / (DKP / 4), i = (idx % (DKP / 4)) * 4;
                const bool in = t < n && i < p.dk;
                const float* s = in ? src + (size_t)t * p.ld + hk * p.dk + i : src;
                copy16(b + L::k0 + t * LDK + i, in ? s + p.k_off : src, in);
                copy16(b + L::q0 + t * LDK + i, in ? s + p.q_off : src, in);
            }
        } else {
            for (int idx = threadIdx.x; idx < C * DKP; idx += THREADS) {
                const int t = idx / DKP, i = idx % DKP;
                const bool in = t < n && i < p.dk;
                const float* s = in ? src + (size_t)t * p.ld + hk * p.dk + i : src;
                copy4(b + L::k0 + t * LDK + i, in ? s + p.k_off : src, in);
                copy4(b + L::q0 + t * LDK + i, in ? s + p.q_off : src, in);
            }
        }
        const float* vals = CHAN ? p.u0 + ((size_t)tb * p.heads + h) * p.dv + cb : src + p.v_off + h * p.dv + cb;
        const size_t v_step = CHAN ? (size_t)p.heads * p.dv : (size_t)p.ld;
        if (p.vec & 2) {
            for (int idx = threadIdx.x; idx < C * 4 * MT; idx += THREADS) {
                const int t = idx / (4 * MT), c = (idx % (4 * MT)) * 4;
                const bool in = t < n && cb + c < p.dv;
                copy16(b + L::v0 + t * LDV + c, in ? vals + t * v_step + c : src, in);
            }
        } else {
            for (int idx = threadIdx.x; idx < C * COLS * MT; idx += THREADS) {
                const int t = idx / (COLS * MT), c = idx % (COLS * MT);
                const bool in = t < n && cb + c < p.dv;
                copy4(b + L::v0 + t * LDV + c, in ? vals + t * v_step + c : src, in);
            }
        }
        for (int idx = threadIdx.x; idx < C * (ROW / 4); idx += THREADS) {
            const int t = idx / (ROW / 4), u = idx % (ROW / 4);
            const bool in = t < n;
            const float* s = in ? p.rows + ((size_t)(tb + t) * p.heads + h) * ROW + u * 4 : p.rows;
            float* dst;
            if constexpr (CHAN) dst = b + L::m0 + t * TS + u * 4;
            else if constexpr (DELTA) dst = u < 8 ? b + L::t0 + t * TS + u * 4 : (u < 16 ? b + L::m0 + t * TS + (u - 8) * 4 : b + L::s0 + t * 4);
            else dst = u < 8 ? b + L::m0 + t * TS + u * 4 : b + L::s0 + t * 4;
            copy16(dst, s, in);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };

    // S^T: s[nb] is the accumulator of state rows k0 + 8 nb + (t4, t4 + 4) for columns c0 + (g, g + 8)
    float s[NB][4];
#pragma unroll
    for (int nb = 0; nb < NB; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = k0 + 8 * nb + t4 + (e & 1) * 4, c = c0 + g + (e >> 1) * 8;
            s[nb][e] = (i < p.dk && c < p.dv) ? S[(size_t)i * p.sld + c] : 0.f;
        }
    if (ta < te) fetch(ta, 0);
    int buf = 0;
    for (int tb = ta; tb < te; tb += C, buf ^= L::buffers - 1) {
        const int n = min(C, te - tb);
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                   // this chunk has arrived, the one before has been read
        if (L::buffers == 2 && tb + C < te) fetch(tb + C, buf ^ 1);
        const float* b = sm + buf * L::buffer;
        const float *ks = b + L::k0, *qs = b + L::q0, *vs = b + L::v0 + mt * COLS, *ms = b + L::m0, *ts = b + L::t0, *sc = b + L::s0;
        {   // this warp's rows of S0^T q_t (and S0^T k_t), all tokens side by side
            float x[4][4], y[4][4];
#pragma unroll
            for (int tk = 0; tk < 4; ++tk)
#pragma unroll
                for (int e = 0; e < 4; ++e) x[tk][e] = y[tk][e] = 0.f;
#pragma unroll
            for (int nb = 0; nb < NB; ++nb) {
                const SplitA a = split_a(s[nb][0], s[nb][2], s[nb][1], s[nb][3]);
                const int at = g * LDK + k0 + 8 * nb + t4;
                float q[4][2], k[4][2];
#pragma unroll
                for (int tk = 0; tk < 4; ++tk) {
                    q[tk][0] = qs[at + 8 * tk * LDK]; q[tk][1] = qs[at + 8 * tk * LDK + 4];
                    if constexpr (DELTA) { k[tk][0] = ks[at + 8 * tk * LDK]; k[tk][1] = ks[at + 8 * tk * LDK + 4]; }
                }
                mma3<4>(x, a, q);
                if constexpr (DELTA) mma3<4>(y, a, k);
            }
#pragma unroll
            for (int tk = 0; tk < 4; ++tk) {
                *reinterpret_cast<float2*>(my + g * TS + 8 * tk + 2 * t4) = make_float2(x[tk][0], x[tk][1]);
                *reinterpret_cast<float2*>(my + (g + 8) * TS + 8 * tk + 2 * t4) = make_float2(x[tk][2], x[tk][3]);
                if constexpr (DELTA) {
                    *reinterpret_cast<float2*>(my + (COLS + g) * TS + 8 * tk + 2 * t4) = make_float2(y[tk][0], y[tk][1]);
                    *reinterpret_cast<float2*>(my + (COLS + g + 8) * TS + 8 * tk + 2 * t4) = make_float2(y[tk][2], y[tk][3]);
                }
            }
        }
        __syncthreads();
        // the sum over the warps of this column group of a part's entries (row, tokens 8 kb + 2 t4 and + 1)
        const float* group = part + (size_t)mt * NW * L::part;
        auto total = [&](int row, int kb) {
            float2 v = make_float2(0.f, 0.f);
#pragma unroll
            for (int w = 0; w < NW; ++w) {
                const float2 e = *reinterpret_cast<const float2*>(group + (size_t)w * L::part + row * TS + 8 * kb + 2 * t4);
                v.x += e.x; v.y += e.y;
            }
            return v;
        };
        if constexpr (CHAN) {
            // U = U0 - W S0, a thread per column and pair of tokens (zeros behind the portion's end)
            for (int i = threadIdx.x % (32 * NW); i < COLS * (C / 2); i += 32 * NW) {
                const int row = i / (C / 2), t = i % (C / 2) * 2;
                float2 y = make_float2(0.f, 0.f);
#pragma unroll
                for (int w = 0; w < NW; ++w) {
                    const float2 e = *reinterpret_cast<const float2*>(group + (size_t)w * L::part + (COLS + row) * TS + t);
                    y.x += e.x; y.y += e.y;
                }
                *reinterpret_cast<float2*>(us + row * TS + t) = make_float2(vs[t * LDV + row] - y.x, vs[(t + 1) * LDV + row] - y.y);
            }
            __syncthreads();
        } else if constexpr (DELTA) {
            for (int tk = kw; 8 * tk < n; tk += NW) {          // U of this warp's eight tokens
                float u[1][4] = {{0.f, 0.f, 0.f, 0.f}};
                for (int kb = 0; kb <= tk; ++kb) {
                    const int t = 8 * kb + 2 * t4;
                    const float2 w0 = total(COLS + g, kb), w1 = total(COLS + g + 8, kb);
                    const float G0 = sc[t * 4], G1 = sc[t * 4 + 4], B0 = sc[t * 4 + 2], B1 = sc[t * 4 + 6];
                    // (a token behind the portion's end has beta 0, and its part may never have been written)
                    const bool in0 = t < n, in1 = t + 1 < n;
                    const SplitA a = split_a(in0 ? B0 * (vs[t * LDV + g] - G0 * w0.x) : 0.f, in0 ? B0 * (vs[t * LDV + g + 8] - G0 * w1.x) : 0.f,
                                             in1 ? B1 * (vs[(t + 1) * LDV + g] - G1 * w0.y) : 0.f, in1 ? B1 * (vs[(t + 1) * LDV + g + 8] - G1 * w1.y) : 0.f);
                    const float2 m = *reinterpret_cast<const float2*>(ts + (8 * tk + g) * TS + t);
                    const float mm[1][2] = {{m.x, m.y}};
                    mma3<1>(u, a, mm);
                }
                *reinterpret_cast<float2*>(us + g * TS + 8 * tk + 2 * t4) = make_float2(u[0][0], u[0][1]);
                *reinterpret_cast<float2*>(us + (g + 8) * TS + 8 * tk + 2 * t4) = make_float2(u[0][2], u[0][3]);
            }
            __syncthreads();
        }
        // U of all tokens as operand A: u[kb] = (column g, token 8 kb + 2 t4), (g + 8, same), (g, + 1), (g + 8, + 1)
        float u[4][4];
#pragma unroll
        for (int kb = 0; kb < 4; ++kb) {
            const int t = 8 * kb + 2 * t4;
            if (8 * kb >= n) {
#pragma unroll
                for (int e = 0; e < 4; ++e) u[kb][e] = 0.f;
            } else if constexpr (DELTA) {
                const float2 x = *reinterpret_cast<const float2*>(us + g * TS + t), y = *reinterpret_cast<const float2*>(us + (g + 8) * TS + t);
                u[kb][0] = x.x; u[kb][1] = y.x; u[kb][2] = x.y; u[kb][3] = y.y;
            } else {
                u[kb][0] = vs[t * LDV + g]; u[kb][1] = vs[t * LDV + g + 8]; u[kb][2] = vs[(t + 1) * LDV + g]; u[kb][3] = vs[(t + 1) * LDV + g + 8];
            }
        }
        for (int tk = kw; 8 * tk < n; tk += NW) {              // o of this warp's eight tokens
            float o[1][4] = {{0.f, 0.f, 0.f, 0.f}};
#pragma unroll
            for (int kb = 0; kb < 4; ++kb) {
                if (kb > tk) break;
                const float2 m = *reinterpret_cast<const float2*>(ms + (8 * tk + g) * TS + 8 * kb + 2 * t4);
                const float mm[1][2] = {{m.x, m.y}};
                mma3<1>(o, split_a(u[kb][0], u[kb][1], u[kb][2], u[kb][3]), mm);
            }
            const int t = 8 * tk + 2 * t4;
            const float2 p0 = total(g, tk), p1 = total(g + 8, tk);
            const float G0 = CHAN ? 1.f : sc[t * 4], G1 = CHAN ? 1.f : sc[t * 4 + 4];
            float* dst = p.o + ((size_t)(tb + t) * p.heads + h) * p.dv + c0 + g;
            const size_t ldo = (size_t)p.heads * p.dv;
            if (t < n) {
                if (c0 + g < p.dv) dst[0] = fmaf(G0, p0.x, o[0][0]);
                if (c0 + g + 8 < p.dv) dst[8] = fmaf(G0, p1.x, o[0][2]);
            }
            if (t + 1 < n) {
                if (c0 + g < p.dv) dst[ldo] = fmaf(G1, p0.y, o[0][1]);
                if (c0 + g + 8 < p.dv) dst[ldo + 8] = fmaf(G1, p1.y, o[0][3]);
            }
        }
        {   // the state after the chunk
            const float G = CHAN ? 1.f : sc[(n - 1) * 4];
            const float *ge = b + L::g0 + k0 + t4, *ku = CHAN ? b + L::r0 : ks;       // the keys that take the decays after them in
#pragma unroll
            for (int nb = 0; nb < NB; ++nb)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[nb][e] *= CHAN ? ge[8 * nb + (e & 1) * 4] : G;
#pragma unroll
            for (int kb = 0; kb < 4; ++kb) {
                if (8 * kb >= n) break;
                const int t = 8 * kb + 2 * t4;
                const float R0 = CHAN ? 1.f : sc[t * 4 + 1], R1 = CHAN ? 1.f : sc[t * 4 + 5];
                const SplitA a = split_a(u[kb][0] * R0, u[kb][1] * R0, u[kb][2] * R1, u[kb][3] * R1);
                float k[NB][2];
#pragma unroll
                for (int nb = 0; nb < NB; ++nb) { k[nb][0] = ku[t * LDK + k0 + 8 * nb + pg]; k[nb][1] = ku[(t + 1) * LDK + k0 + 8 * nb + pg]; }
                mma3<NB>(s, a, k);
            }
        }
        if (L::buffers == 1 && tb + C < te) {
            __syncthreads();               // the one buffer has been read
            fetch(tb + C, 0);
        }
    }
#pragma unroll
    for (int nb = 0; nb < NB; ++nb)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = k0 + 8 * nb + t4 + (e & 1) * 4, c = c0 + g + (e >> 1) * 8;
            if (i < p.dk && c < p.dv) S[(size_t)i * p.sld + c] = s[nb][e];
        }
}

template <bool DELTA, int DKP>
int launch_rows(const ChunkParams& p, cudaStream_t s) {
    constexpr int smem = (2 * C * (DKP + 4) + 2 * C * (C + 1) + (DELTA ? 4 * C * (C + 4) : 0)) * (int)sizeof(float);
    static bool raised[bw::MAX_DEVICES] = {};
    if (bw::allow_dynamic_smem(chunk_rows_kernel<DELTA, DKP>, smem, raised) != cudaSuccess) return BW_ERR_DRIVER;
    bw::launch((chunk_rows_kernel<DELTA, DKP>), dim3(p.T / C + p.R, p.heads / p.rep), dim3(128), smem, s, p);
    BW_LAUNCH_CHECK();
    return 0;
}

template <int DKP>
int launch_rows_channel(const ChunkParams& p, cudaStream_t s) {
    constexpr int smem = (3 * C * DKP + C * (C + 4)) * (int)sizeof(float);
    static bool raised[bw::MAX_DEVICES] = {};
    if (bw::allow_dynamic_smem(chunk_rows_channel_kernel<DKP>, smem, raised) != cudaSuccess) return BW_ERR_DRIVER;
    bw::launch((chunk_rows_channel_kernel<DKP>), dim3(p.T / C + p.R, p.heads), dim3(128), smem, s, p);
    BW_LAUNCH_CHECK();
    return 0;
}

template <bool DELTA, bool CHAN, int NW, int NB, int MT>
int launch_scan(const ChunkParams& p, int R, cudaStream_t s) {
    constexpr int smem = ChunkSmem<DELTA, CHAN, NW, NB, MT>::floats * (int)sizeof(float);
    static_assert(smem <= 227 * 1024, "shared memory budget");
    static bool raised[bw::MAX_DEVICES] = {};
    if (bw::allow_dynamic_smem(chunk_scan_kernel<DELTA, CHAN, NW, NB, MT>, smem, raised) != cudaSuccess) return BW_ERR_DRIVER;
    const int cols = COLS * MT;
    bw::launch((chunk_scan_kernel<DELTA, CHAN, NW, NB, MT>), dim3(R, p.heads, (p.dv + cols - 1) / cols), dim3(32 * NW * MT), smem, s, p);
    BW_LAUNCH_CHECK();
    return 0;
}

template <bool DELTA, bool CHAN>
int run(const ChunkParams& p, int R, cudaStream_t s) {
    const int nw = p.dk <= 32 ? 1 : (p.dk <= 64 ? 2 : (p.dk <= 128 ? 4 : 8));
    int rc;
    if constexpr (CHAN)
        rc = nw == 1 ? launch_rows_channel<32>(p, s) : (nw == 2 ? launch_rows_channel<64>(p, s)
           : (nw == 4 ? launch_rows_channel<128>(p, s) : launch_rows_channel<256>(p, s)));
    else
        rc = nw == 1 ? launch_rows<DELTA, 32>(p, s) : (nw == 2 ? launch_rows<DELTA, 64>(p, s)
           : (nw == 4 ? launch_rows<DELTA, 128>(p, s) : launch_rows<DELTA, 256>(p, s)));
    if (rc) return rc;
    // more blocks than fit side by side: two column groups share a block, its keys and its matrices
    const bool wide = (long long)R * p.heads * ((p.dv + COLS - 1) / COLS) > (long long)bw::num_sms() * (DELTA ? 1 : 2);
    switch (nw) {
        case 1: return wide ? launch_scan<DELTA, CHAN, 2, 2, 2>(p, R, s) : launch_scan<DELTA, CHAN, 2, 2, 1>(p, R, s);
        case 2: return wide ? launch_scan<DELTA, CHAN, 4, 2, 2>(p, R, s) : launch_scan<DELTA, CHAN, 4, 2, 1>(p, R, s);
        case 4: return wide ? launch_scan<DELTA, CHAN, 4, 4, 2>(p, R, s) : (DELTA ? launch_scan<DELTA, CHAN, 8, 2, 1>(p, R, s) : launch_scan<DELTA, CHAN, 4, 4, 1>(p, R, s));
        default: return launch_scan<DELTA, CHAN, 8, 4, 1>(p, R, s);
    }
}

}  // namespace

// floats per (token, head) of the scratch that bw_chunk_scan takes
BW_EXPORT int bw_chunk_row_floats(int delta) { return delta == 2 ? ROW_CHANNEL : (delta ? ROW_DELTA : ROW_LINEAR); }

// qkv: float32 rows `ld` apart with q and k (heads / rep heads of dk channels) and v (heads of dv) at the given columns;
// decay [T, heads]; second [T, heads]: beta (delta != 0) or the keys' factor; rows: scratch float32
// [T, heads, bw_chunk_row_floats(delta)], 16-byte aligned; state [slots, heads, dk, sld]; o [T, heads * dv].
// delta == 2: the delta rule with decay [T, heads * dk]; scratches float32, 16-byte aligned (otherwise null): chan [T, heads, 3, dk],
// u0 [T, heads, dv], gend [T / 32 + R, heads, dk].
BW_EXPORT int bw_chunk_scan(int delta, const float* qkv, long long ld, int q_off, int k_off, int v_off, const float* decay,
                            const float* second, const int* cu_q, const int* state_slot, float* rows,
                            float* chan, float* u0, float* gend, float* state, float* o, int T, int R, int heads, int rep, int dk, int dv,
                            int sld, void* stream) {
    if (T <= 0 || R <= 0) return 0;
    if (heads <= 0 || rep <= 0 || heads % rep || dk <= 0 || dv <= 0 || sld < dv || !rows || ((uintptr_t)rows & 15)) return BW_ERR_BAD_ARG;
    if (dk > 256) return BW_ERR_UNSUPPORTED;
    if (delta == 2 && (!chan || !u0 || !gend || (((uintptr_t)chan | (uintptr_t)u0 | (uintptr_t)gend) & 15))) return BW_ERR_BAD_ARG;
    ChunkParams p;
    p.chan = chan; p.u0 = u0; p.gend = gend;
    p.qkv = qkv; p.ld = ld; p.q_off = q_off; p.k_off = k_off; p.v_off = v_off; p.decay = decay; p.second = second; p.cu_q = cu_q;
    p.state_slot = state_slot; p.rows = rows; p.state = state; p.sld = sld; p.o = o;
    p.T = T; p.R = R; p.heads = heads; p.rep = rep; p.dk = dk; p.dv = dv;
    const bool base = ((uintptr_t)qkv & 15) == 0 && (ld & 3) == 0;
    p.vec = (base && (dk & 3) == 0 && (q_off & 3) == 0 && (k_off & 3) == 0 ? 1 : 0) | (base && (dv & 3) == 0 && (v_off & 3) == 0 ? 2 : 0);
    if (delta == 2) p.vec = (((uintptr_t)decay & 15) ? p.vec & ~1 : p.vec) & ~2;
    if (delta == 2 && (dv & 3) == 0) p.vec |= 2;           // (the values come from the scratch)
    if (delta == 2) return run<true, true>(p, R, (cudaStream_t)stream);
    return delta ? run<true, false>(p, R, (cudaStream_t)stream) : run<false, false>(p, R, (cudaStream_t)stream);
}
