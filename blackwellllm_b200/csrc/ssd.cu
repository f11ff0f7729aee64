// The output of a state-space mixer with one decay per head (Mamba-2): from the recurrence's read-out y, the convolved
// inputs x and the gate's projection z,
//
//   u = (y + D_h x) * silu(z)          per channel, D one number per head
//   out = u / rms(u over the channel's part) * gain        `parts` equal parts of all the heads' channels
//
// in float32.  One block per (token, part).  Parts of up to 4,096 channels with aligned rows stay in registers, four channels
// an access; of others every value is made twice rather than kept.
#include "common.cuh"

using bf16 = __nv_bfloat16;

namespace {

template <typename OT>
__global__ void __launch_bounds__(256)
ssd_out_kernel(const float* __restrict__ y, const float* __restrict__ x, long long x_ld, const float* __restrict__ z,
               long long z_ld, const float* __restrict__ D, const float* __restrict__ gain, OT* __restrict__ out, int inner,
               int vdim, int part, float eps) {
    BW_PDL_TRIGGER();
    BW_PDL_WAIT();
    __shared__ float scratch[32];
    const size_t t = blockIdx.x;
    const int c0 = blockIdx.y * part, c1 = c0 + part;
    const float* yr = y + t * inner;
    const float* xr = x + t * x_ld;
    const float* zr = z + t * z_ld;
    auto at = [&](int c) {
        const float zv = zr[c];
        return (yr[c] + D[c / vdim] * xr[c]) * (zv / (1.f + expf(-zv)));
    };
    float ss = 0.f;
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) { const float u = at(c); ss = fmaf(u, u, ss); }
    const float r = rsqrtf(bw::block_sum(ss, scratch) / (float)part + eps);
    for (int c = c0 + threadIdx.x; c < c1; c += blockDim.x) out[t * inner + c] = bw::from_f32<OT>(at(c) * r * gain[c]);
}

__device__ __forceinline__ void put4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void put4(bf16* p, float4 v) {
    *reinterpret_cast<uint2*>(p) = make_uint2(bw::pack_bf16x2(v.x, v.y), bw::pack_bf16x2(v.z, v.w));
}

// NV accesses of four channels a thread: part <= NV * 1024, vdim and part multiples of 4
template <typename OT, int NV>
__global__ void __launch_bounds__(256)
ssd_out_vec_kernel(const float* __restrict__ y, const float* __restrict__ x, long long x_ld, const float* __restrict__ z,
                   long long z_ld, const float* __restrict__ D, const float* __restrict__ gain, OT* __restrict__ out, int inner,
                   int vdim, int part, float eps) {
    BW_PDL_TRIGGER();
    BW_PDL_WAIT();
    __shared__ float scratch[32];
    const size_t t = blockIdx.x;
    const int c0 = blockIdx.y * part, c1 = c0 + part;
    float4 u[NV];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = c0 + (i * blockDim.x + threadIdx.x) * 4;
        u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < c1) {
            const float4 a = *reinterpret_cast<const float4*>(y + t * inner + c), b = *reinterpret_cast<const float4*>(x + t * x_ld + c),
                         g = *reinterpret_cast<const float4*>(z + t * z_ld + c);
            const float d = D[c / vdim];
            u[i].x = (a.x + d * b.x) * (g.x / (1.f + expf(-g.x))); u[i].y = (a.y + d * b.y) * (g.y / (1.f + expf(-g.y)));
            u[i].z = (a.z + d * b.z) * (g.z / (1.f + expf(-g.z))); u[i].w = (a.w + d * b.w) * (g.w / (1.f + expf(-g.w)));
        }
        ss = fmaf(u[i].x, u[i].x, ss); ss = fmaf(u[i].y, u[i].y, ss); ss = fmaf(u[i].z, u[i].z, ss); ss = fmaf(u[i].w, u[i].w, ss);
    }
    const float r = rsqrtf(bw::block_sum(ss, scratch) / (float)part + eps);
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const int c = c0 + (i * blockDim.x + threadIdx.x) * 4;
        if (c < c1) {
            const float4 g = *reinterpret_cast<const float4*>(gain + c);
            put4(out + t * inner + c, make_float4(u[i].x * r * g.x, u[i].y * r * g.y, u[i].z * r * g.z, u[i].w * r * g.w));
        }
    }
}

template <typename OT>
void launch_out(const float* y, const float* x, long long x_ld, const float* z, long long z_ld, const float* D, const float* gain,
                OT* out, int T, int inner, int vdim, int parts, float eps, cudaStream_t s) {
    const int part = inner / parts;
    const dim3 grid(T, parts);
    const bool vec = (vdim & 3) == 0 && (part & 3) == 0 && (x_ld & 3) == 0 && (z_ld & 3) == 0 && part <= 4096 &&
                     (((uintptr_t)y | (uintptr_t)x | (uintptr_t)z | (uintptr_t)gain | (uintptr_t)out) & 15) == 0;
    if (vec) {
        const int threads = part >= 1024 ? 256 : (part / 4 + 31) / 32 * 32;
        if (part <= 1024) bw::launch((ssd_out_vec_kernel<OT, 1>), grid, dim3(threads), 0, s, y, x, x_ld, z, z_ld, D, gain, out, inner, vdim, part, eps);
        else if (part <= 2048) bw::launch((ssd_out_vec_kernel<OT, 2>), grid, dim3(threads), 0, s, y, x, x_ld, z, z_ld, D, gain, out, inner, vdim, part, eps);
        else bw::launch((ssd_out_vec_kernel<OT, 4>), grid, dim3(threads), 0, s, y, x, x_ld, z, z_ld, D, gain, out, inner, vdim, part, eps);
    } else {
        const int threads = part >= 256 ? 256 : (part + 31) / 32 * 32;
        bw::launch((ssd_out_kernel<OT>), grid, dim3(threads), 0, s, y, x, x_ld, z, z_ld, D, gain, out, inner, vdim, part, eps);
    }
}

}  // namespace

// y [T, inner], x rows x_ld apart (the convolved inputs, inner channels), z rows z_ld apart: float32; D [inner / vdim];
// gain [inner]; inner a multiple of `parts`.
BW_EXPORT int bw_ssd_out(const float* y, const float* x, long long x_ld, const float* z, long long z_ld, const float* D,
                         const float* gain, void* out, int out_type, int T, int inner, int vdim, int parts, float eps,
                         void* stream) {
    if (T <= 0) return 0;
    if (inner <= 0 || vdim <= 0 || inner % vdim || parts <= 0 || inner % parts) return BW_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    if (out_type == BW_F32) launch_out<float>(y, x, x_ld, z, z_ld, D, gain, (float*)out, T, inner, vdim, parts, eps, s);
    else if (out_type == BW_BF16) launch_out<bf16>(y, x, x_ld, z, z_ld, D, gain, (bf16*)out, T, inner, vdim, parts, eps, s);
    else return BW_ERR_BAD_ARG;
    BW_LAUNCH_CHECK();
    return 0;
}
