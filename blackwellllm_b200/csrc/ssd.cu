// The output of a state-space mixer with one decay per head (Mamba-2): from the recurrence's read-out y, the convolved
// inputs x and the gate's projection z,
//
//   u = (y + D_h x) * silu(z)          per channel, D one number per head
//   out = u / rms(u over the channel's part) * gain        `parts` equal parts of all the heads' channels
//
// in float32.  One block per (token, part); a part's values are made twice rather than kept.
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

}  // namespace

// y [T, inner], x rows x_ld apart (the convolved inputs, inner channels), z rows z_ld apart: float32; D [inner / vdim];
// gain [inner]; inner a multiple of `parts`.
BW_EXPORT int bw_ssd_out(const float* y, const float* x, long long x_ld, const float* z, long long z_ld, const float* D,
                         const float* gain, void* out, int out_type, int T, int inner, int vdim, int parts, float eps,
                         void* stream) {
    if (T <= 0) return 0;
    if (inner <= 0 || vdim <= 0 || inner % vdim || parts <= 0 || inner % parts) return BW_ERR_BAD_ARG;
    const int part = inner / parts;
    const int threads = part >= 256 ? 256 : (part + 31) / 32 * 32;
    const dim3 grid(T, parts);
    cudaStream_t s = (cudaStream_t)stream;
    if (out_type == BW_F32) bw::launch((ssd_out_kernel<float>), grid, dim3(threads), 0, s, y, x, x_ld, z, z_ld, D, gain, (float*)out, inner, vdim, part, eps);
    else if (out_type == BW_BF16) bw::launch((ssd_out_kernel<bf16>), grid, dim3(threads), 0, s, y, x, x_ld, z, z_ld, D, gain, (bf16*)out, inner, vdim, part, eps);
    else return BW_ERR_BAD_ARG;
    BW_LAUNCH_CHECK();
    return 0;
}
