// The second halves of projections through a small inner size, W2 (W1 x), and what a recurrent mixer makes of them:
//
//   decay   g[t, c] = exp(A[c / per] * softplus(z + bias[c])),  A = -exp(A_log), one per `per` neighbouring channels (a head)
//   gate    s[t, c] = sigmoid(z)
//
// with z = sum_r x[t, r] W2[c, r], x being `rank` columns of the first halves' float32 result.  Several such parts share a
// launch (blockIdx.z).  Everything is float32.  bfloat16 weights: mma.sync m16n8k16 with x split into two bfloat16 halves
// (x = hi + lo up to 2^-17 of it) and float32 sums, the weights as they are; float32 weights: float32 multiply-adds.  The
// order of the sums depends on the inner size alone.
#include "common.cuh"

using bf16 = __nv_bfloat16;

namespace {

constexpr int MAX_PARTS = 2;
enum { PART_DECAY = 0, PART_SIGMOID = 1 };

struct Part {
    const void* w;               // [n_out, rank]
    const float *A, *bias;       // decay: [n_out / per], [n_out]
    float* out;                  // [T, n_out]
    int x_off, rank, n_out, per, kind;
};
struct LowRankParams {
    const float* x; long long ld;
    int T, vec;
    Part part[MAX_PARTS];
};

__device__ __forceinline__ float sigmoid(float z) { return __fdividef(1.f, 1.f + expf(-z)); }   // (a quotient flushed to zero is the sigmoid's)
__device__ __forceinline__ float decay(float A, float z) { return expf(A * (fmaxf(z, 0.f) + log1pf(expf(-fabsf(z))))); }
__device__ __forceinline__ float finish(const Part& q, int c, float z) {
    return q.kind == PART_SIGMOID ? sigmoid(z) : decay(q.A[c / q.per], z + q.bias[c]);
}

// float32 weights: 32 tokens x 64 outputs a block, 32 inner values at a time
constexpr int FT = 32, FO = 64, FK = 32;
__global__ void __launch_bounds__(256)
lowrank_f32_kernel(LowRankParams p) {
    BW_PDL_TRIGGER();
    const Part q = p.part[blockIdx.z];
    const int t0 = blockIdx.x * FT, o0 = blockIdx.y * FO;
    if (o0 >= q.n_out) return;
    __shared__ float xs[FT][FK + 1], ws[FO][FK + 1];
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    const float* w = (const float*)q.w;
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    BW_PDL_WAIT();
    for (int k0 = 0; k0 < q.rank; k0 += FK) {
        for (int idx = threadIdx.x; idx < FT * FK; idx += 256) {
            const int t = t0 + idx / FK, k = k0 + idx % FK;
            xs[idx / FK][idx % FK] = (t < p.T && k < q.rank) ? p.x[(size_t)t * p.ld + q.x_off + k] : 0.f;
        }
        for (int idx = threadIdx.x; idx < FO * FK; idx += 256) {
            const int o = o0 + idx / FK, k = k0 + idx % FK;
            ws[idx / FK][idx % FK] = (o < q.n_out && k < q.rank) ? w[(size_t)o * q.rank + k] : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < FK; ++k) {
            const float a0 = xs[ty * 2][k], a1 = xs[ty * 2 + 1][k];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float b = ws[tx + 16 * j][k];
                acc[0][j] = fmaf(a0, b, acc[0][j]);
                acc[1][j] = fmaf(a1, b, acc[1][j]);
            }
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int t = t0 + ty * 2 + i;
        if (t >= p.T) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int o = o0 + tx + 16 * j;
            if (o < q.n_out) q.out[(size_t)t * q.n_out + o] = finish(q, o, acc[i][j]);
        }
    }
}

// bfloat16 weights.  Both forms add, per 16 inner values in rising order, the low half's product and then the high half's, so a row's
// result is the same in either.
__device__ __forceinline__ uint32_t smem_addr(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
// two neighbouring values as bfloat16 pairs: the rounded values, and what the rounding left
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = bw::pack_bf16x2(a - __low2float(h), b - __high2float(h));
}
__device__ __forceinline__ void store_pair(const Part& q, int row, int c, float z0, float z1) {
    float* dst = q.out + (size_t)row * q.n_out;
    if (c + 1 < q.n_out && (((uintptr_t)(dst + c)) & 7) == 0)
        *reinterpret_cast<float2*>(dst + c) = make_float2(finish(q, c, z0), finish(q, c + 1, z1));
    else {
        if (c < q.n_out) dst[c] = finish(q, c, z0);
        if (c + 1 < q.n_out) dst[c + 1] = finish(q, c + 1, z1);
    }
}

// Up to 16 tokens: a warp makes 8 outputs, operands straight into registers, no barrier; the weights are requested before the wait
// for the kernels before.
constexpr int FEW = 16, KR = 128;      // inner values at a time
__global__ void __launch_bounds__(128)
lowrank_few_kernel(LowRankParams p) {
    BW_PDL_TRIGGER();
    const Part q = p.part[blockIdx.z];
    const int lane = threadIdx.x & 31, o0 = (blockIdx.x * 4 + (threadIdx.x >> 5)) * 8;
    if (o0 >= q.n_out) return;
    const bf16* w = (const bf16*)q.w;
    const int o = o0 + (lane >> 2), k = 2 * (lane & 3);
    const bool vec = (p.vec >> blockIdx.z) & 1;
    float acc[1][4] = {{0.f, 0.f, 0.f, 0.f}};
    for (int k0 = 0; k0 < q.rank; k0 += KR) {
        uint32_t b[KR / 16][2];
#pragma unroll
        for (int ks = 0; ks < KR / 16; ++ks)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int kk = k0 + ks * 16 + e * 8 + k;
                const bf16* src = w + (size_t)o * q.rank + kk;
                if (vec) b[ks][e] = (o < q.n_out && kk < q.rank) ? __ldg(reinterpret_cast<const uint32_t*>(src)) : 0u;
                else {
                    const float lo = (o < q.n_out && kk < q.rank) ? __bfloat162float(src[0]) : 0.f;
                    const float hi = (o < q.n_out && kk + 1 < q.rank) ? __bfloat162float(src[1]) : 0.f;
                    b[ks][e] = bw::pack_bf16x2(lo, hi);
                }
            }
        if (k0 == 0) BW_PDL_WAIT();
        float2 x[KR / 16][4];
#pragma unroll
        for (int ks = 0; ks < KR / 16; ++ks)
#pragma unroll
            for (int e = 0; e < 4; ++e) {       // rows lane / 4 (and + 8), inner values k (and + 8)
                const int t = (lane >> 2) + 8 * (e & 1), kk = k0 + ks * 16 + 8 * (e >> 1) + k;
                const float* src = p.x + (size_t)t * p.ld + q.x_off + kk;
                x[ks][e] = make_float2(0.f, 0.f);
                if (t < p.T) {
                    if (vec) { if (kk < q.rank) x[ks][e] = *reinterpret_cast<const float2*>(src); }
                    else {
                        if (kk < q.rank) x[ks][e].x = src[0];
                        if (kk + 1 < q.rank) x[ks][e].y = src[1];
                    }
                }
            }
#pragma unroll
        for (int ks = 0; ks < KR / 16; ++ks) {
            if (k0 + ks * 16 >= q.rank) break;
            uint32_t ah[4], al[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) split2(x[ks][e].x, x[ks][e].y, ah[e], al[e]);
            mma_bf16(acc[0], al, b[ks][0], b[ks][1]);
            mma_bf16(acc[0], ah, b[ks][0], b[ks][1]);
        }
    }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int row = (lane >> 2) + 8 * half;
        if (row < p.T) store_pair(q, row, o0 + k, acc[0][2 * half], acc[0][2 * half + 1]);
    }
}

// Many tokens: a block of 8 warps makes 64 tokens x 128 outputs, each warp 16 tokens x two stretches of 32 outputs; 128 inner values at
// a time; the weights are requested before the wait for the kernels before.  Rows of shared memory are padded to 272 bytes, so that
// the 8 rows of an ldmatrix fall into different banks.
constexpr int MT = 64, MO = 128, MROW = (KR + 8) * 2;
constexpr int SMEM_MMA = (2 * MT + MO) * MROW;

__global__ void __launch_bounds__(256, 3)
lowrank_mma_kernel(LowRankParams p) {
    BW_PDL_TRIGGER();
    const Part q = p.part[blockIdx.z];
    const int t0 = blockIdx.x * MT, o0 = blockIdx.y * MO;
    if (o0 >= q.n_out) return;
    extern __shared__ __align__(16) uint8_t smem[];
    uint8_t *xh = smem, *xl = smem + MT * MROW, *ws = smem + 2 * MT * MROW;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, wm = warp & 3, wn = warp >> 2;
    const bf16* w = (const bf16*)q.w;
    float acc[2][4][4];
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) { acc[i][j][0] = acc[i][j][1] = acc[i][j][2] = acc[i][j][3] = 0.f; }
    const bool vec = (p.vec >> blockIdx.z) & 1;
    for (int k0 = 0; k0 < q.rank; k0 += KR) {
        // eight inner values of a weight row, then of a token row, per step of a thread
#pragma unroll
        for (int i = 0; i < MO * (KR / 8) / 256; ++i) {
            const int idx = threadIdx.x + i * 256, r = idx / (KR / 8), c = idx % (KR / 8) * 8, o = o0 + r;
            uint8_t* dst = ws + r * MROW + c * 2;
            const bf16* src = w + (size_t)(o < q.n_out ? o : 0) * q.rank + k0 + c;
            if (vec) {           // (the inner size is a multiple of 8: a stretch of eight is inside or outside)
                const bool in = o < q.n_out && k0 + c < q.rank;
                const int n = in ? 16 : 0;
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" :: "r"(smem_addr(dst)), "l"(in ? src : w), "r"(n) : "memory");
            } else {
                bf16 e[8];
#pragma unroll
                for (int j = 0; j < 8; ++j) e[j] = (o < q.n_out && k0 + c + j < q.rank) ? src[j] : __float2bfloat16_rn(0.f);
                *reinterpret_cast<uint4*>(dst) = *reinterpret_cast<const uint4*>(e);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
        if (k0 == 0) BW_PDL_WAIT();
#pragma unroll
        for (int i = 0; i < MT * (KR / 8) / 256; ++i) {
            const int idx = threadIdx.x + i * 256, r = idx / (KR / 8), c = idx % (KR / 8) * 8, t = t0 + r;
            const float* src = p.x + (size_t)(t < p.T ? t : 0) * p.ld + q.x_off + k0 + c;
            float v[8];
            if (vec) {
                const bool in = t < p.T && k0 + c < q.rank;
                const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
                const float4 a = in ? *reinterpret_cast<const float4*>(src) : zero, b = in ? *reinterpret_cast<const float4*>(src + 4) : zero;
                v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
            } else {
#pragma unroll
                for (int j = 0; j < 8; ++j) v[j] = (t < p.T && k0 + c + j < q.rank) ? src[j] : 0.f;
            }
            uint4 hi, lo;
            split2(v[0], v[1], hi.x, lo.x); split2(v[2], v[3], hi.y, lo.y); split2(v[4], v[5], hi.z, lo.z); split2(v[6], v[7], hi.w, lo.w);
            *reinterpret_cast<uint4*>(xh + r * MROW + c * 2) = hi;
            *reinterpret_cast<uint4*>(xl + r * MROW + c * 2) = lo;
        }
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();
#pragma unroll
        for (int ks = 0; ks < KR / 16; ++ks) {
            if (k0 + ks * 16 >= q.rank) break;
            uint32_t ah[4], al[4];
            const int at = (wm * 16 + (lane & 7) + 8 * ((lane >> 3) & 1)) * MROW + 16 * (lane >> 4) + ks * 32;
            ldsm_x4(smem_addr(xh) + at, ah);
            ldsm_x4(smem_addr(xl) + at, al);
#pragma unroll
            for (int i = 0; i < 2; ++i)
#pragma unroll
                for (int nb = 0; nb < 2; ++nb) {
                    uint32_t b[4];
                    ldsm_x4(smem_addr(ws) + (i * 64 + wn * 32 + nb * 16 + (lane & 7) + 8 * (lane >> 4)) * MROW + 16 * ((lane >> 3) & 1) + ks * 32, b);
                    mma_bf16(acc[i][2 * nb], al, b[0], b[1]);
                    mma_bf16(acc[i][2 * nb + 1], al, b[2], b[3]);
                    mma_bf16(acc[i][2 * nb], ah, b[0], b[1]);
                    mma_bf16(acc[i][2 * nb + 1], ah, b[2], b[3]);
                }
        }
        if (k0 + KR < q.rank) __syncthreads();
    }
    // the sums change places through shared memory: a thread finishes four neighbouring columns of every eighth row (few
    // instructions for the many results, whole sectors for the stores)
    constexpr int ZS = MO + 4;
    static_assert(MT * ZS * 4 <= SMEM_MMA, "the sums take the operands' place");
    float* zs = reinterpret_cast<float*>(smem);
    __syncthreads();
#pragma unroll
    for (int i = 0; i < 2; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int half = 0; half < 2; ++half)
                *reinterpret_cast<float2*>(zs + (wm * 16 + (lane >> 2) + 8 * half) * ZS + i * 64 + wn * 32 + j * 8 + 2 * (lane & 3)) =
                    make_float2(acc[i][j][2 * half], acc[i][j][2 * half + 1]);
    __syncthreads();
    const int c = o0 + lane * 4, n = min(4, q.n_out - c);
    if (n <= 0) return;
    const bool dec = q.kind == PART_DECAY, quads = (q.n_out & 3) == 0 && ((uintptr_t)q.out & 15) == 0;
    float A[4] = {0.f, 0.f, 0.f, 0.f}, bias[4] = {0.f, 0.f, 0.f, 0.f};
    if (dec)
        for (int e = 0; e < n; ++e) { A[e] = q.A[(c + e) / q.per]; bias[e] = q.bias[c + e]; }
#pragma unroll 1
    for (int r = warp; r < MT && t0 + r < p.T; r += 8) {
        const float4 z = *reinterpret_cast<const float4*>(zs + r * ZS + lane * 4);
        float v[4] = {z.x, z.y, z.z, z.w};
        if (dec) {
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = decay(A[e], v[e] + bias[e]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) v[e] = sigmoid(v[e]);
        }
        float* dst = q.out + (size_t)(t0 + r) * q.n_out + c;
        if (quads) *reinterpret_cast<float4*>(dst) = make_float4(v[0], v[1], v[2], v[3]);
        else
            for (int e = 0; e < n; ++e) dst[e] = v[e];
    }
}

}  // namespace

// x: float32 [T, .], rows `ld` apart.  n parts (1 or 2), each: the column x_off of its inner values, rank, w [n_out, rank] of
// w_type, kind (0 decay, 1 sigmoid), A [n_out / per] and bias [n_out] float32 (decay), out float32 [T, n_out].
BW_EXPORT int bw_lowrank_gates(const float* x, long long ld, int w_type, int T, int n, const int* x_off, const int* rank,
                               const int* n_out, const int* kind, const int* per, const void* const* w,
                               const float* const* A, const float* const* bias, float* const* out, void* stream) {
    if (T <= 0) return 0;
    if (n < 1 || n > MAX_PARTS) return BW_ERR_BAD_ARG;
    LowRankParams p;
    p.x = x; p.ld = ld; p.T = T; p.vec = 0;
    int widest = 0;
    for (int i = 0; i < n; ++i) {
        Part& q = p.part[i];
        q.w = w[i]; q.A = A[i]; q.bias = bias[i]; q.out = out[i];
        q.x_off = x_off[i]; q.rank = rank[i]; q.n_out = n_out[i]; q.per = per[i]; q.kind = kind[i];
        if (q.rank <= 0 || q.n_out <= 0 || q.x_off < 0 || !q.w || !q.out || q.kind < 0 || q.kind > PART_SIGMOID || ld < q.x_off + q.rank ||
            (q.kind == PART_DECAY && (!q.A || !q.bias || q.per <= 0 || q.n_out % q.per)))
            return BW_ERR_BAD_ARG;
        if (q.rank % 8 == 0 && ld % 4 == 0 && (((uintptr_t)(x + q.x_off) | (uintptr_t)q.w) & 15) == 0) p.vec |= 1 << i;
        if (q.n_out > widest) widest = q.n_out;
    }
    for (int i = n; i < MAX_PARTS; ++i) p.part[i] = p.part[0];
    cudaStream_t s = (cudaStream_t)stream;
    if (w_type == BW_F32)
        bw::launch((lowrank_f32_kernel), dim3((T + FT - 1) / FT, (widest + FO - 1) / FO, n), dim3(256), 0, s, p);
    else if (w_type == BW_BF16)
    {
        static bool raised[bw::MAX_DEVICES] = {};
        if (T <= FEW) bw::launch((lowrank_few_kernel), dim3((widest + 31) / 32, 1, n), dim3(128), 0, s, p);
        else {
            if (bw::allow_dynamic_smem(lowrank_mma_kernel, SMEM_MMA, raised) != cudaSuccess) return BW_ERR_DRIVER;
            bw::launch((lowrank_mma_kernel), dim3((T + MT - 1) / MT, (widest + MO - 1) / MO, n), dim3(256), SMEM_MMA, s, p);
        }
    }
    else return BW_ERR_BAD_ARG;
    BW_LAUNCH_CHECK();
    return 0;
}
