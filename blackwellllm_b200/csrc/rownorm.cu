// The seam between two sublayers of a block that norms a sublayer's output before it joins the stream:
//
//   y   = what the sublayer left: one float32 row, or the mean of two rows that are RMS-normed with a gain each
//   x  += post(y) * gp                    post: layer norm, RMS norm or nothing; gp may hold further constants
//   h   = next(x) * gn                    next: the norm before the next sublayer (or none), which may also be
//                                         tanh(alpha x) * gn + bn, a norm without any statistic of the row
//
// in one pass over the stream.  A row of y may come as planes of a matrix product that its kernel left unsummed; they are
// added (in plane order) while they are read.  One block per row; a row's values stay in registers from the first load to
// the last store, and every sum runs over the row in an order that depends on H alone.  All arithmetic is float32.
#include "common.cuh"

using bf16 = __nv_bfloat16;

namespace {

// what a norm does to a row: 0 nothing, 1 x / sqrt(mean(x^2) + eps), 2 (x - mean) / sqrt(mean((x - mean)^2) + eps), 3 (only as the
// next norm) tanh(alpha x), with a bias after the gain
enum { NORM_NONE = 0, NORM_RMS = 1, NORM_LAYER = 2, NORM_TANH = 3 };

struct RowParams {
    float* x;                // the stream [T, H]
    const float* y;          // [T, H] (null with planes that are all of it); y_planes of them behind one another if y_n > 0
    const float* y_planes; long long y_stride; int y_n;
    const float* z;          // the second row of a pair, the same way; pair != 0
    const float* z_planes; long long z_stride; int z_n;
    const float *gy, *gz;    // the pair's gains [H]
    float pair_eps;
    int pair, has_y;
    const float* gp; float post_eps; int post;
    const float* gn; float next_eps; int next;
    const float* bn; float alpha;   // NORM_TANH: the bias after the gain [H] or null, the factor inside the tanh
    const int* rows;         // only these rows, and x stays as it is
    void* out; int H;
};

__device__ __forceinline__ void st(float* p, float v) { *p = v; }
__device__ __forceinline__ void st(bf16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void st4(float* p, const float* v) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void st4(bf16* p, const float* v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(bw::pack_bf16x2(v[0], v[1]), bw::pack_bf16x2(v[2], v[3]));
}
template <int W> __device__ __forceinline__ void ld(const float* p, float* v) {
    if constexpr (W == 4) {
        const float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    } else v[0] = *p;
}

// both values summed over the block, in a fixed order
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    a = bw::warp_sum(a); b = bw::warp_sum(b);
    __syncthreads();
    if (lane == 0) scratch[warp] = make_float2(a, b);
    __syncthreads();
    const float2 v = lane < nw ? scratch[lane] : make_float2(0.f, 0.f);
    return make_float2(bw::warp_sum(v.x), bw::warp_sum(v.y));
}

// a row of a sublayer's output: base (if there is one) plus its planes in order, eight loads in flight
template <int W>
__device__ __forceinline__ void row_of(const float* base, const float* planes, long long stride, int n, size_t at, float* v) {
    if (base) ld<W>(base + at, v);
    else {
#pragma unroll
        for (int e = 0; e < W; ++e) v[e] = 0.f;
    }
    for (int p0 = 0; p0 < n; p0 += 8) {
        float t[8][W];
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            if (p0 + j < n) ld<W>(planes + (size_t)(p0 + j) * stride + at, t[j]);
            else {
#pragma unroll
                for (int e = 0; e < W; ++e) t[j][e] = 0.f;
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < W; ++e) v[e] += t[j][e];
    }
}

// W: values per access (4: 16-byte aligned rows, H a multiple of 4); NV: accesses per thread
template <typename OT, int W, int NV>
__global__ void __launch_bounds__(1024)
row_step_kernel(RowParams p) {
    BW_PDL_TRIGGER();
    __shared__ float2 scratch[32];
    const int H = p.H, step = blockDim.x * W;
    const float inv_h = 1.f / (float)H;
    BW_PDL_WAIT();
    const size_t row = (size_t)(p.rows ? p.rows[blockIdx.x] : (int)blockIdx.x) * H;
    float x[NV][W];
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = i * step + threadIdx.x * W;
        if (c < H) ld<W>(p.x + row + c, x[i]);
        else {
#pragma unroll
            for (int e = 0; e < W; ++e) x[i][e] = 0.f;
        }
    }
    if (p.has_y) {
        float y[NV][W];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = i * step + threadIdx.x * W;
            if (c < H) row_of<W>(p.y, p.y_planes, p.y_stride, p.y_n, row + c, y[i]);
            else {
#pragma unroll
                for (int e = 0; e < W; ++e) y[i][e] = 0.f;
            }
        }
        if (p.pair) {
            float z[NV][W];
            float sy = 0.f, sz = 0.f;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = i * step + threadIdx.x * W;
                if (c < H) row_of<W>(p.z, p.z_planes, p.z_stride, p.z_n, row + c, z[i]);
                else {
#pragma unroll
                    for (int e = 0; e < W; ++e) z[i][e] = 0.f;
                }
#pragma unroll
                for (int e = 0; e < W; ++e) { sy = fmaf(y[i][e], y[i][e], sy); sz = fmaf(z[i][e], z[i][e], sz); }
            }
            const float2 s = block_sum2(sy, sz, scratch);
            const float ry = rsqrtf(s.x * inv_h + p.pair_eps), rz = rsqrtf(s.y * inv_h + p.pair_eps);
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = i * step + threadIdx.x * W;
                if (c < H) {
                    float gy[W], gz[W];
                    ld<W>(p.gy + c, gy); ld<W>(p.gz + c, gz);
#pragma unroll
                    for (int e = 0; e < W; ++e) y[i][e] = 0.5f * (y[i][e] * ry * gy[e] + z[i][e] * rz * gz[e]);
                }
            }
        }
        float mean = 0.f, r = 1.f;
        if (p.post == NORM_LAYER) {
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < NV; ++i)
#pragma unroll
                for (int e = 0; e < W; ++e) s += y[i][e];
            mean = block_sum2(s, 0.f, scratch).x * inv_h;
        }
        if (p.post != NORM_NONE) {
            float s = 0.f;
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const int c = i * step + threadIdx.x * W;
#pragma unroll
                for (int e = 0; e < W; ++e) { const float d = c < H ? y[i][e] - mean : 0.f; s = fmaf(d, d, s); }
            }
            r = rsqrtf(block_sum2(s, 0.f, scratch).x * inv_h + p.post_eps);
        }
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = i * step + threadIdx.x * W;
            if (c < H) {
                float g[W];
                if (p.gp) ld<W>(p.gp + c, g);
#pragma unroll
                for (int e = 0; e < W; ++e) {
                    float v = (y[i][e] - mean) * r;
                    if (p.gp) v *= g[e];
                    x[i][e] += v;
                }
                if (!p.rows) {
                    if constexpr (W == 4) st4(p.x + row + c, x[i]);
                    else st(p.x + row + c, x[i][0]);
                }
            }
        }
    }
    if (!p.out) return;
    float mean = 0.f, r = 1.f;
    if (p.next == NORM_LAYER) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i)
#pragma unroll
            for (int e = 0; e < W; ++e) s += x[i][e];
        mean = block_sum2(s, 0.f, scratch).x * inv_h;
    }
    if (p.next == NORM_RMS || p.next == NORM_LAYER) {
        float s = 0.f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const int c = i * step + threadIdx.x * W;
#pragma unroll
            for (int e = 0; e < W; ++e) { const float d = c < H ? x[i][e] - mean : 0.f; s = fmaf(d, d, s); }
        }
        r = rsqrtf(block_sum2(s, 0.f, scratch).x * inv_h + p.next_eps);
    }
    OT* out = (OT*)p.out + (size_t)blockIdx.x * H;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = i * step + threadIdx.x * W;
        if (c < H) {
            float g[W], o[W];
            if (p.gn) ld<W>(p.gn + c, g);
            if (p.next == NORM_TANH) {
                float b[W];
#pragma unroll
                for (int e = 0; e < W; ++e) b[e] = 0.f;
                if (p.bn) ld<W>(p.bn + c, b);
#pragma unroll
                for (int e = 0; e < W; ++e) o[e] = fmaf(tanhf(p.alpha * x[i][e]), p.gn ? g[e] : 1.f, b[e]);
            } else {
#pragma unroll
                for (int e = 0; e < W; ++e) { o[e] = (x[i][e] - mean) * r; if (p.gn) o[e] *= g[e]; }
            }
            if constexpr (W == 4) st4(out + c, o);
            else st(out + c, o[0]);
        }
    }
}

template <typename OT, int W>
int run(const RowParams& p, int n, cudaStream_t s) {
    const int units = (p.H + W - 1) / W;
    // (few rows: as many loads in flight per row as can be; many rows: smaller blocks)
    const int nv = units <= (n <= 64 ? 1024 : 256) ? 1 : (units <= 2048 ? 2 : (units <= 4096 ? 4 : (units <= 8192 ? 8 : (units <= 16384 ? 16 : 0))));
    if (!nv) return BW_ERR_UNSUPPORTED;
    const int threads = ((units + nv - 1) / nv + 31) / 32 * 32;
    switch (nv) {
        case 1: bw::launch((row_step_kernel<OT, W, 1>), dim3(n), dim3(threads), 0, s, p); break;
        case 2: bw::launch((row_step_kernel<OT, W, 2>), dim3(n), dim3(threads), 0, s, p); break;
        case 4: bw::launch((row_step_kernel<OT, W, 4>), dim3(n), dim3(threads), 0, s, p); break;
        case 8: bw::launch((row_step_kernel<OT, W, 8>), dim3(n), dim3(threads), 0, s, p); break;
        default:
            if constexpr (W == 1) { bw::launch((row_step_kernel<OT, 1, 16>), dim3(n), dim3(threads), 0, s, p); break; }
            return BW_ERR_UNSUPPORTED;
    }
    BW_LAUNCH_CHECK();
    return 0;
}

}  // namespace

// x: float32 [T, H], updated in place unless `rows` names the rows to make (then out is dense [n, H]).  has_y == 0: no
// sublayer output, only the next norm.  y / z: float32 [T, H] or null where the planes are all of it; planes: n of them,
// `stride` floats apart, each [T, H].  pair: z counts, both rows are RMS-normed (pair_eps) times gy / gz and averaged.
// post / next: 0 none, 1 RMS norm, 2 layer norm, next also 3 tanh(alpha x); gp / gn: float32 [H] or null; bn: float32 [H] or null,
// added after gn where next is 3.  out: null, or the next norm's result.
BW_EXPORT int bw_row_step(float* x, int has_y, const float* y, const float* y_planes, long long y_stride, int y_n,
                          int pair, const float* z, const float* z_planes, long long z_stride, int z_n,
                          const float* gy, const float* gz, float pair_eps, int post, const float* gp, float post_eps,
                          int next, const float* gn, float next_eps, const float* bn, float alpha, const int* rows, void* out, int out_type, int n, int H,
                          void* stream) {
    if (n <= 0) return 0;
    if (H <= 0 || post < 0 || post > 2 || next < 0 || next > 3 || (bn && next != 3) || (pair && (!gy || !gz || !has_y)) || y_n < 0 || z_n < 0 ||
        (has_y && !y && y_n == 0) || (pair && !z && z_n == 0) || (y_n && !y_planes) || (z_n && !z_planes))
        return BW_ERR_BAD_ARG;
    RowParams p;
    p.x = x; p.has_y = has_y; p.y = y; p.y_planes = y_planes; p.y_stride = y_stride; p.y_n = y_n;
    p.pair = pair; p.z = z; p.z_planes = z_planes; p.z_stride = z_stride; p.z_n = z_n;
    p.gy = gy; p.gz = gz; p.pair_eps = pair_eps; p.post = post; p.gp = gp; p.post_eps = post_eps;
    p.next = next; p.gn = gn; p.next_eps = next_eps; p.bn = bn; p.alpha = alpha; p.rows = rows; p.out = out; p.H = H;
    const uintptr_t all = (uintptr_t)x | (uintptr_t)y | (uintptr_t)y_planes | (uintptr_t)z | (uintptr_t)z_planes | (uintptr_t)gy |
                          (uintptr_t)gz | (uintptr_t)gp | (uintptr_t)gn | (uintptr_t)bn | (uintptr_t)out;
    const bool vec = (H & 3) == 0 && (all & 15) == 0 && (y_stride & 3) == 0 && (z_stride & 3) == 0;
    cudaStream_t s = (cudaStream_t)stream;
    if (out_type == BW_F32) return vec ? run<float, 4>(p, n, s) : run<float, 1>(p, n, s);
    if (out_type == BW_BF16) return vec ? run<bf16, 4>(p, n, s) : run<bf16, 1>(p, n, s);
    return BW_ERR_BAD_ARG;
}
