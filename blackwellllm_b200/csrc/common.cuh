// Shared helpers for the sm_100a kernels of this engine.
//
// Every launcher is an extern "C" function over raw device pointers and a stream,
// returns 0 on success or a negative BW_ERR_* / positive cudaError_t code, and
// never allocates.  Python binds them with ctypes (kernels/ops.py).
#pragma once
#include <cuda_runtime.h>
#include <cuda_bf16.h>
#include <stdint.h>

#define BW_EXPORT extern "C" __attribute__((visibility("default")))

// error codes returned by launchers (negative: ours; positive: cudaError_t)
#define BW_ERR_BAD_ARG   (-1)
#define BW_ERR_UNSUPPORTED (-2)
#define BW_ERR_DRIVER    (-3)

// element type codes used across the C interface
#define BW_F32  0
#define BW_BF16 1

// activations of feed-forwards (the codes cross the C interface)
//   BW_ACT_SILU           gated:  silu(g) * u
//   BW_ACT_CLAMPED_SWISH  gated:  g' = min(g, limit), u' = clamp(u, -limit, limit):  g' sigmoid(alpha g') (u' + 1)
//   BW_ACT_RELU2          no gate: max(x, 0)^2
//   BW_ACT_GELU_TANH      gated:  0.5 g (1 + tanh(sqrt(2 / pi) (g + 0.044715 g^3))) * u
//   BW_ACT_GELU           no gate: 0.5 x (1 + erf(x / sqrt(2)))
#define BW_ACT_SILU 0
#define BW_ACT_CLAMPED_SWISH 1
#define BW_ACT_RELU2 2
#define BW_ACT_GELU_TANH 3
#define BW_ACT_GELU 4

// Programmatic dependent launch: a kernel launched through bw::launch may start while the kernel
// before it in the stream is still draining.  Such a kernel calls BW_PDL_TRIGGER() early (the next
// kernel may start launching) and BW_PDL_WAIT() before its first access to memory that an earlier
// kernel may write (everything but weights); the wait returns once all earlier kernels are
// complete and their writes visible.  Both are no-ops for ordinary launches.  BW_PDL=0 in the
// environment turns the early launch off.
#define BW_PDL_TRIGGER() asm volatile("griddepcontrol.launch_dependents;" ::: "memory")
#define BW_PDL_WAIT() asm volatile("griddepcontrol.wait;" ::: "memory")

#define BW_LAUNCH_CHECK() do { cudaError_t e__ = cudaGetLastError(); if (e__ != cudaSuccess) return (int)e__; } while (0)

#include <stdlib.h>
#include <utility>

namespace bw {

inline bool pdl_enabled() {
    static int v = -1;
    if (v < 0) { const char* e = getenv("BW_PDL"); v = (e && e[0] == '0') ? 0 : 1; }
    return v != 0;
}

// overlap == false: an ordinary launch (the kernel starts when everything before it is complete)
template <typename... KArgs, typename... Args>
inline cudaError_t launch_opt(bool overlap, void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem,
                              cudaStream_t stream, Args&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = stream;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr; cfg.numAttrs = (overlap && pdl_enabled()) ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}

// the same for a kernel whose CTAs come in clusters of two (grid.x even)
template <typename... KArgs, typename... Args>
inline cudaError_t launch_pairs(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                                Args&&... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = stream;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 2; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr; cfg.numAttrs = pdl_enabled() ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, kernel, std::forward<Args>(args)...);
}

// The current device's number (0 where none can be asked: host-only use of a planner) and its number of SMs
// (148, the B200's, where none can be asked), looked up once per device.
constexpr int MAX_DEVICES = 64;
inline int current_device() {
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= MAX_DEVICES) { cudaGetLastError(); return 0; }
    return dev;
}
inline int num_sms() {
    static int cached[MAX_DEVICES] = {0};
    const int dev = current_device();
    if (cached[dev] <= 0) {
        int n = 0;
        if (cudaDeviceGetAttribute(&n, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || n <= 0) { cudaGetLastError(); n = 148; }
        cached[dev] = n;
    }
    return cached[dev];
}
// Raises a kernel's dynamic shared-memory limit once per device (`done`: one flag per device, zero-initialised).
template <typename K>
inline cudaError_t allow_dynamic_smem(K kernel, int bytes, bool (&done)[MAX_DEVICES]) {
    const int dev = current_device();
    if (done[dev]) return cudaSuccess;
    const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
    if (e == cudaSuccess) done[dev] = true;
    return e;
}

template <typename... KArgs, typename... Args>
inline cudaError_t launch(void (*kernel)(KArgs...), dim3 grid, dim3 block, size_t smem, cudaStream_t stream,
                          Args&&... args) {
    return launch_opt(true, kernel, grid, block, smem, stream, std::forward<Args>(args)...);
}

// The first key position a query at q_pos may see: a sliding window of `window` keys (0: none) and / or
// blocks of `chunk` positions, counted from position 0, that a query does not look out of (0: none).
__host__ __device__ __forceinline__ int first_visible(int q_pos, int window, int chunk) {
    int lo = (window > 0 && q_pos - window + 1 > 0) ? q_pos - window + 1 : 0;
    if (chunk > 0) { const int c0 = q_pos - q_pos % chunk; if (c0 > lo) lo = c0; }
    return lo;
}

// What a query at q_pos sees of the key at k_pos <= q_pos: the keys from first_visible(...) on, and the first
// `keep_first` keys of the sequence whatever the window says (0: none are kept).
__host__ __device__ __forceinline__ bool key_visible(int k_pos, int lo, int keep_first) {
    return k_pos >= lo || k_pos < keep_first;
}

// The distance bias that is taken off a score: r1 ln(1 + r2 (q_pos - k_pos)), r1 and r2 numbers of the query head.
__device__ __forceinline__ float distance_bias(float r1, float r2, int dist) {
    return r1 * log1pf(r2 * (float)dist);
}

// A soft cap on a score: cap * tanh(s / cap).  soft_cap: the library's tanh (the 32-bit path).  soft_cap_fast: tanh as
// 1 - 2 / (2^(2 x log2 e) + 1) with the fast exponential and division; its error is a few ulps of 1, so a few 1e-7 * cap.
__device__ __forceinline__ float soft_cap(float s, float cap) { return cap * tanhf(s / cap); }
__device__ __forceinline__ float soft_cap_fast(float s, float cap, float inv_cap) {
    const float e = exp2f(s * inv_cap * 2.8853900817779268f);
    return cap * (1.f - __fdividef(2.f, e + 1.f));
}

// tanh(x) / x for |x| <= 1 as a polynomial of degree 5 in x^2 (six coefficients fitted over [0, 1]; the error of x * p is
// below 6e-7): five FMAs in place of two special-function instructions.
__device__ __forceinline__ float tanh_over_x_poly(float x2) {
    float p = -0.0030804092530161142f;
    p = fmaf(p, x2, 0.01677677594125271f);
    p = fmaf(p, x2, -0.05163545906543732f);
    p = fmaf(p, x2, 0.13282513618469238f);
    p = fmaf(p, x2, -0.33329179883003235f);
    return fmaf(p, x2, 0.999999463558197f);
}

// A learned bias per (query head, distance): table float32 [heads][len], the last entry standing for every distance
// from len - 1 on.
__device__ __forceinline__ float table_bias(const float* __restrict__ head_row, int len, int dist) {
    return head_row[dist < len ? dist : len - 1];
}

__device__ __forceinline__ uint32_t pack_bf16x2(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);   // lo in the low half
    return *reinterpret_cast<const uint32_t*>(&v);
}

__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }

template <typename T> __device__ __forceinline__ T from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float glu(int act, float g, float u, float limit, float alpha) {
    if (act == BW_ACT_CLAMPED_SWISH) {
        g = fminf(g, limit);
        u = fminf(fmaxf(u, -limit), limit);
        return g / (1.f + expf(-alpha * g)) * (u + 1.f);
    }
    if (act == BW_ACT_GELU_TANH) return 0.5f * g * (1.f + tanhf(0.7978845608028654f * (g + 0.044715f * g * g * g))) * u;
    return g / (1.f + expf(-g)) * u;
}
__device__ __forceinline__ float unary_act(int act, float x) {
    if (act == BW_ACT_RELU2) { const float r = fmaxf(x, 0.f); return r * r; }
    if (act == BW_ACT_GELU) return 0.5f * x * (1.f + erff(x * 0.70710678118654752f));
    return x;
}
// The same gelu for results that are rounded to 16 bits: erf by formula 7.1.26 of Abramowitz and Stegun, Handbook of
// Mathematical Functions (absolute error below 1.5e-7): erf(z) = 1 - (a1 t + .. + a5 t^5) exp(-z^2), t = 1 / (1 + 0.3275911 z).
__device__ __forceinline__ float gelu_fast(float x) {
    const float z = fabsf(x) * 0.70710678118654752f;
    const float t = __fdividef(1.f, fmaf(0.3275911f, z, 1.f));
    float q = fmaf(1.061405429f, t, -1.453152027f);
    q = fmaf(q, t, 1.421413741f);
    q = fmaf(q, t, -0.284496736f);
    q = fmaf(q, t, 0.254829592f);
    const float tail = q * t * __expf(-z * z);        // 1 - erf(z)
    return 0.5f * x * (x >= 0.f ? 2.f - tail : tail);
}

// The output gate of an attention mixer: sigmoid(gate[token, head * dv + c]) for c < dv, 0 for the pad channels beyond
// dv, 1 without a gate.  gate: float32 rows `ld` apart.  dv < 0: the gate has ONE number per head, gate[token, head],
// for the head's first -dv channels.
__device__ __forceinline__ float out_gate(const float* __restrict__ gate, long long ld, int dv, size_t token, int head, int c) {
    if (!gate) return 1.f;
    if (dv < 0) return c < -dv ? 1.f / (1.f + expf(-gate[token * (size_t)ld + (size_t)head])) : 0.f;
    if (c >= dv) return 0.f;
    return 1.f / (1.f + expf(-gate[token * (size_t)ld + (size_t)head * dv + c]));
}

// Differential attention in the attention kernels' epilogues: query heads 2 h and 2 h + 1 are the two maps a1, a2 of head h, and what is
// written is  o / sqrt(mean(o^2) + eps) * scale * gate_h,  o = a1 - *lam a2,  over dv channels (those beyond are zeros), as head h of
// half as many heads.  lam == null: every query head is written by itself.
struct DiffHeads {
    const float* lam;
    float eps, scale;
    int dv;
};
// What map `which` of a pair counts with, `inv` the inverse of its softmax's denominator.
__device__ __forceinline__ float diff_weight(const DiffHeads& d, int which, float inv) { return which ? -__ldg(d.lam) * inv : inv; }
// The factor of a head's o from its sum of squares; the gate: one number per head, or none.
__device__ __forceinline__ float diff_factor(const DiffHeads& d, float ss, const float* __restrict__ gate, long long ld, size_t token, int head) {
    float f = rsqrtf(ss / (float)d.dv + d.eps) * d.scale;
    if (gate) f *= 1.f / (1.f + expf(-gate[token * (size_t)ld + (size_t)head]));
    return f;
}

// Two float32 operations in one instruction (sm_100: the packed form of fma and mul); a pair is a 64-bit register, the first
// value in the low half.
typedef unsigned long long f32x2;
__device__ __forceinline__ f32x2 pack2(float lo, float hi) {
    f32x2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
__device__ __forceinline__ void unpack2(f32x2 v, float& lo, float& hi) { asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v)); }
__device__ __forceinline__ float sum2(f32x2 v) { float a, b; unpack2(v, a, b); return a + b; }
__device__ __forceinline__ f32x2 fma2(f32x2 a, f32x2 b, f32x2 c) {
    f32x2 d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ f32x2 mul2(f32x2 a, f32x2 b) {
    f32x2 d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

// The register tiles of the recurrent scans (gla.cu, delta.cu): lane = 8 * rg + cg; a lane holds TILE_ROWS state rows of its
// row group rg (4 groups a warp) and a few neighbouring value columns of its column group cg (8 groups).  What a lane reads
// of a token from shared memory (its rows' key and query channels, its columns' values) then serves rows x columns elements.
constexpr int TILE_ROWS = 8, TILE_RG = 4, TILE_CG = 8, TILE_WARP_ROWS = TILE_ROWS * TILE_RG;

// Sums over the row groups (lane bits 3 and 4).  Four values per lane: the lane gets the sum of value 2 b4 + b3 (b4, b3: its
// bits 4 and 3); two values: of value b4 (in both lanes of bit 3).
__device__ __forceinline__ float tile_sum4(float a0, float a1, float a2, float a3) {
    const bool hi16 = threadIdx.x & 16, hi8 = threadIdx.x & 8;
    const float g0 = __shfl_xor_sync(0xffffffffu, hi16 ? a0 : a2, 16);
    const float g1 = __shfl_xor_sync(0xffffffffu, hi16 ? a1 : a3, 16);
    const float b0 = (hi16 ? a2 : a0) + g0, b1 = (hi16 ? a3 : a1) + g1;
    return (hi8 ? b1 : b0) + __shfl_xor_sync(0xffffffffu, hi8 ? b0 : b1, 8);
}
__device__ __forceinline__ float tile_sum2(float a0, float a1) {
    const bool hi16 = threadIdx.x & 16;
    const float b = (hi16 ? a1 : a0) + __shfl_xor_sync(0xffffffffu, hi16 ? a0 : a1, 16);
    return b + __shfl_xor_sync(0xffffffffu, b, 8);
}

// A lane's tile of a state [rows, ld] in memory, row0 its first row, col0 its first column; rows from `rows` on and columns
// from `cols` on count as zeros and are not written.  s[j][c]: rows row0 + 2 j and + 1 of column col0 + c.
template <int CPT>
__device__ __forceinline__ void tile_load(f32x2 (&s)[TILE_ROWS / 2][CPT], const float* __restrict__ S, int row0, int rows, int ld,
                                          int col0, int cols) {
    const bool vec = (ld % CPT) == 0 && col0 + CPT <= ld && ((uintptr_t)S & (4 * CPT - 1)) == 0;
#pragma unroll
    for (int j = 0; j < TILE_ROWS / 2; ++j) {
        float v[2][CPT];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = row0 + 2 * j + e;
            const float* src = S + (size_t)i * ld + col0;
            if (vec && i < rows) {
                if constexpr (CPT == 4) {
                    const float4 t = *reinterpret_cast<const float4*>(src);
                    v[e][0] = t.x; v[e][1] = t.y; v[e][2] = t.z; v[e][3] = t.w;
                } else {
                    const float2 t = *reinterpret_cast<const float2*>(src);
                    v[e][0] = t.x; v[e][1] = t.y;
                }
            } else {
#pragma unroll
                for (int c = 0; c < CPT; ++c) v[e][c] = (i < rows && col0 + c < cols) ? src[c] : 0.f;
            }
        }
#pragma unroll
        for (int c = 0; c < CPT; ++c) s[j][c] = pack2(v[0][c], v[1][c]);
    }
}
template <int CPT>
__device__ __forceinline__ void tile_store(const f32x2 (&s)[TILE_ROWS / 2][CPT], float* __restrict__ S, int row0, int rows, int ld,
                                           int col0, int cols) {
    const bool vec = (ld % CPT) == 0 && col0 + CPT <= ld && ((uintptr_t)S & (4 * CPT - 1)) == 0;
#pragma unroll
    for (int j = 0; j < TILE_ROWS / 2; ++j) {
        float v[2][CPT];
#pragma unroll
        for (int c = 0; c < CPT; ++c) unpack2(s[j][c], v[0][c], v[1][c]);
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int i = row0 + 2 * j + e;
            if (i >= rows) continue;
            float* dst = S + (size_t)i * ld + col0;
            if (vec) {
                if constexpr (CPT == 4) *reinterpret_cast<float4*>(dst) = make_float4(v[e][0], v[e][1], v[e][2], v[e][3]);
                else *reinterpret_cast<float2*>(dst) = make_float2(v[e][0], v[e][1]);
            } else {
#pragma unroll
                for (int c = 0; c < CPT; ++c)
                    if (col0 + c < cols) dst[c] = v[e][c];
            }
        }
    }
}
// CPT neighbouring floats from shared memory, each as a pair of itself twice
template <int CPT>
__device__ __forceinline__ void tile_values(f32x2 (&v)[CPT], const float* src, float scale) {
    if constexpr (CPT == 4) {
        const float4 t = *reinterpret_cast<const float4*>(src);
        v[0] = pack2(t.x * scale, t.x * scale); v[1] = pack2(t.y * scale, t.y * scale);
        v[2] = pack2(t.z * scale, t.z * scale); v[3] = pack2(t.w * scale, t.w * scale);
    } else {
        const float2 t = *reinterpret_cast<const float2*>(src);
        v[0] = pack2(t.x * scale, t.x * scale); v[1] = pack2(t.y * scale, t.y * scale);
    }
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}

// Block-wide sum in a fixed order (lane tree, then warp 0 over the warp sums), so
// the result for a row never depends on which other rows are in the launch.
// `scratch` holds at least 32 floats.  All threads get the result.
__device__ __forceinline__ float block_sum(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float r = (lane < nwarps) ? scratch[lane] : 0.f;
    r = warp_sum(r);
    return r;
}
__device__ __forceinline__ float block_max(float v, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int nwarps = (blockDim.x + 31) >> 5;
    v = warp_max(v);
    __syncthreads();
    if (lane == 0) scratch[warp] = v;
    __syncthreads();
    float r = (lane < nwarps) ? scratch[lane] : -INFINITY;
    r = warp_max(r);
    return r;
}

}  // namespace bw
