// Differential attention: the two maps' outputs of a head become one.
//
//   o = a1 - lambda a2       o <- o / sqrt(mean(o^2) + eps) * scale * sigmoid(gate)        per token and head
//
// a: [T, 2 heads, dpad], the maps of head h at 2 h and 2 h + 1; channels from dv on are padding (zeros) and stay zeros.  lambda is
// one number on the device; the gate is one number per head, or there is none.  Float32 arithmetic, one warp per (token, head).
#include "common.cuh"

using bf16 = __nv_bfloat16;

namespace {

__device__ __forceinline__ float2 get2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 get2(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void put2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void put2(bf16* p, float a, float b) { *reinterpret_cast<uint32_t*>(p) = bw::pack_bf16x2(a, b); }

template <typename AT, typename OT>
__global__ void __launch_bounds__(128)
diff_combine_kernel(const AT* __restrict__ a, OT* __restrict__ out, int T, int heads, int dv, int dpad, const float* __restrict__ lam,
                    float eps, float scale, const float* __restrict__ gate, long long g_ld) {
    BW_PDL_TRIGGER();
    BW_PDL_WAIT();
    const int item = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (item >= T * heads) return;
    const int t = item / heads, h = item - t * heads;
    const AT* a1 = a + ((size_t)t * heads + h) * 2 * dpad;
    const AT* a2 = a1 + dpad;
    OT* dst = out + ((size_t)t * heads + h) * dpad;
    const float l = *lam;
    float ss = 0.f;
    const bool even = (dpad & 1) == 0;
    if (even) {
        for (int c = lane * 2; c < dpad; c += 64) {
            const float2 u = get2(a1 + c), v = get2(a2 + c);
            const float x = c < dv ? fmaf(-l, v.x, u.x) : 0.f, y = c + 1 < dv ? fmaf(-l, v.y, u.y) : 0.f;
            ss = fmaf(x, x, ss); ss = fmaf(y, y, ss);
        }
    } else {
        for (int c = lane; c < dv; c += 32) { const float x = fmaf(-l, bw::to_f32(a2[c]), bw::to_f32(a1[c])); ss = fmaf(x, x, ss); }
    }
    float f = rsqrtf(bw::warp_sum(ss) / (float)dv + eps) * scale;
    if (gate) f *= 1.f / (1.f + expf(-gate[(size_t)t * g_ld + h]));
    if (even) {
        for (int c = lane * 2; c < dpad; c += 64) {
            const float2 u = get2(a1 + c), v = get2(a2 + c);
            put2(dst + c, c < dv ? fmaf(-l, v.x, u.x) * f : 0.f, c + 1 < dv ? fmaf(-l, v.y, u.y) * f : 0.f);
        }
    } else {
        for (int c = lane; c < dpad; c += 32)
            dst[c] = bw::from_f32<OT>(c < dv ? fmaf(-l, bw::to_f32(a2[c]), bw::to_f32(a1[c])) * f : 0.f);
    }
}

}  // namespace

// a [T, 2 heads, dpad] of a_type, out [T, heads, dpad] of out_type; lam: one float32 on the device; gate: float32 rows g_ld apart
// with one number per head, or null.
BW_EXPORT int bw_diff_combine(const void* a, int a_type, void* out, int out_type, int T, int heads, int dv, int dpad, const float* lam,
                              float eps, float scale, const float* gate, long long g_ld, void* stream) {
    if (T <= 0) return 0;
    if (heads <= 0 || dv <= 0 || dpad < dv || !lam || (((uintptr_t)a | (uintptr_t)out) & 7)) return BW_ERR_BAD_ARG;
    const dim3 grid(((unsigned)T * heads + 3) / 4);
    cudaStream_t s = (cudaStream_t)stream;
#define BW_DC(AT, OT) bw::launch((diff_combine_kernel<AT, OT>), grid, dim3(128), 0, s, (const AT*)a, (OT*)out, T, heads, dv, dpad, lam, eps, scale, gate, g_ld)
    if (a_type == BW_F32 && out_type == BW_F32) BW_DC(float, float);
    else if (a_type == BW_F32 && out_type == BW_BF16) BW_DC(float, bf16);
    else if (a_type == BW_BF16 && out_type == BW_BF16) BW_DC(bf16, bf16);
    else return BW_ERR_BAD_ARG;
#undef BW_DC
    BW_LAUNCH_CHECK();
    return 0;
}
