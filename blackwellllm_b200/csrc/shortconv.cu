// What stands between a recurrent mixer's projections and its recurrence:
//
//   short_conv   a causal convolution over time per channel with `taps` columns (the last one is the current token's),
//                an optional bias, silu, and for the channels that ask for it the unit norm of each head:
//                u / sqrt(sum(u^2) + unit_eps) * scale
//   step_gates   per head: d = softplus(z + dt_bias), decay = exp(A d) with A = -exp(A_log), and either the step size d
//                itself or a second gate sigmoid(z2)
//
//   conv_heads   the same convolution without silu on the queries, keys and values of an attention mixer: its results go
//                straight to the attention's queries and to the cache pages
//
// Each is one kernel.  The convolution's earlier inputs of a request are part of its state: `state` [slots, taps, channels]
// float32 holds the input of position p at entry p mod taps.  A token at position p reads the entries of p - 1 ..
// p - (taps - 1) where they lie before the step's own tokens, so a step of one token per request may write the entry of p
// at once; a step with longer portions writes the last taps - 1 inputs with a kernel of its own afterwards (another block
// may still read the entries it replaces).  Positions before the sequence's start count as zeros and are never read.
// All arithmetic is float32.
#include "common.cuh"

using bf16 = __nv_bfloat16;

namespace {

constexpr int MAX_SEGS = 3;
constexpr int CHUNK = 128;      // channels of a warp's piece where a segment has no norm

struct Seg {
    int c0;            // first channel
    int pieces;        // warps: heads of a normed segment, stretches of CHUNK channels otherwise
    int size;          // channels of a piece
    int channels;      // channels of the segment
    int unit;          // 1: every piece is a head that becomes a unit vector times scale
    float scale;
};

struct ConvParams {
    const float* x; long long ld;          // the projections' rows; channel c of the convolution is column c
    const float* w;                        // [taps, C]
    const float* bias;                     // [C] or null
    float* state;                          // [slots, taps, C]
    const int *positions, *req_of_token, *cu_q, *state_slot;
    float* out;                            // [T, C]
    int T, C, taps, single;                // single: one token per request, the state is written here
    int nseg; Seg seg[MAX_SEGS];
    float unit_eps;
    // gates: z at column z_off of zx (rows zld apart; < 0: no decay is made), z2 at z2_off (< 0: none, the step size is written
    // instead)
    const float* zx; long long zld; int z_off, z2_off, heads;
    const float *A, *dt_bias;              // [heads]: -exp(A_log), dt_bias
    float *decay, *second;                 // [T, heads]
};

constexpr int TILE = 8;        // tokens of a warp, one after another (their rows overlap in the cache)
constexpr int WARPS = 8;

__device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + log1pf(expf(-fabsf(x))); }
__device__ __forceinline__ float silu(float x) { return x / (1.f + expf(-x)); }

// TAPS > 0: the number of columns at compile time (all loads of a token in flight at once); 0: p.taps
template <int TAPS>
__device__ __forceinline__ float conv_at(const ConvParams& p, int t, int local, int pos, const float* st, int c) {
    const int taps = TAPS > 0 ? TAPS : p.taps;
    float acc = p.bias ? p.bias[c] : 0.f;
#pragma unroll
    for (int j = taps - 1; j >= 0; --j) {            // j tokens back, the oldest first
        if (j > pos) continue;                        // before the sequence's start
        const float v = j <= local ? p.x[(size_t)(t - j) * p.ld + c] : st[(size_t)((pos - j) % taps) * p.C + c];
        acc = fmaf(p.w[(size_t)(taps - 1 - j) * p.C + c], v, acc);
    }
    return acc;
}

// NR: channels a lane holds of a piece (pieces of up to 32 * NR channels)
template <int NR, int TAPS>
__global__ void __launch_bounds__(32 * WARPS)
short_conv_kernel(ConvParams p) {
    BW_PDL_TRIGGER();
    BW_PDL_WAIT();
    const int lane = threadIdx.x & 31;
    int item = blockIdx.y * WARPS + (threadIdx.x >> 5);
    const int tile = p.single ? 1 : TILE;
    const int t0 = blockIdx.x * tile, t1 = min(p.T, t0 + tile);
    int s = 0;
    while (s < p.nseg && item >= p.seg[s].pieces) { item -= p.seg[s].pieces; ++s; }
    if (s == p.nseg) {
        // the gates: the pieces behind the last segment, 32 heads each
        const int h = item * 32 + lane;
        if (h >= p.heads) return;
        const bool decays = p.z_off >= 0;
        const float A = decays ? p.A[h] : 0.f, b = decays ? p.dt_bias[h] : 0.f;
        for (int t = t0; t < t1; ++t) {
            const float* z = p.zx + (size_t)t * p.zld;
            if (!decays) {
                p.second[(size_t)t * p.heads + h] = 1.f / (1.f + expf(-z[p.z2_off + h]));
                continue;
            }
            const float d = softplus(z[p.z_off + h] + b);
            p.decay[(size_t)t * p.heads + h] = expf(A * d);
            p.second[(size_t)t * p.heads + h] = p.z2_off >= 0 ? 1.f / (1.f + expf(-z[p.z2_off + h])) : d;
        }
        return;
    }
    const Seg sg = p.seg[s];
    const int first = sg.c0 + item * sg.size;
    const int n = min(sg.size, sg.channels - item * sg.size);
    const int r0 = p.req_of_token[t0], local0 = t0 - p.cu_q[r0];
    if (TAPS > 0 && t1 - t0 == TILE && local0 >= TAPS - 1 && t0 + TILE <= p.cu_q[r0 + 1]) {
        // the whole tile and the tokens before it belong to one portion: every row is read once, all loads side by side
        float u[TILE][NR];
#pragma unroll
        for (int k = 0; k < NR; ++k) {
            const int c = first + k * 32 + lane;
            const bool in = k * 32 + lane < n;
            float v[TILE + TAPS - 1], w[TAPS > 0 ? TAPS : 1];
            const float* src = p.x + (size_t)(t0 - (TAPS - 1)) * p.ld + c;
#pragma unroll
            for (int j = 0; j < TILE + TAPS - 1; ++j) v[j] = in ? src[(size_t)j * p.ld] : 0.f;
#pragma unroll
            for (int j = 0; j < TAPS; ++j) w[j] = in ? p.w[(size_t)j * p.C + c] : 0.f;
            const float b = (in && p.bias) ? p.bias[c] : 0.f;
#pragma unroll
            for (int i = 0; i < TILE; ++i) {
                float acc = b;
#pragma unroll
                for (int j = 0; j < TAPS; ++j) acc = fmaf(w[j], v[i + j], acc);
                u[i][k] = silu(acc);
            }
        }
        float f[TILE];
#pragma unroll
        for (int i = 0; i < TILE; ++i) {
            f[i] = 1.f;
            if (sg.unit) {
                float ss = 0.f;
#pragma unroll
                for (int k = 0; k < NR; ++k) ss = fmaf(u[i][k], u[i][k], ss);
                f[i] = sg.scale * rsqrtf(bw::warp_sum(ss) + p.unit_eps);
            }
        }
#pragma unroll
        for (int i = 0; i < TILE; ++i)
#pragma unroll
            for (int k = 0; k < NR; ++k)
                if (k * 32 + lane < n) p.out[(size_t)(t0 + i) * p.C + first + k * 32 + lane] = u[i][k] * f[i];
        return;
    }
    for (int t = t0; t < t1; ++t) {
        const int r = p.req_of_token[t], local = t - p.cu_q[r], pos = p.positions[t];
        float* st = p.state + (size_t)p.state_slot[r] * p.taps * p.C;
        float* dst = p.out + (size_t)t * p.C;
        float u[NR];
        float ss = 0.f;
#pragma unroll
        for (int k = 0; k < NR; ++k) {
            const int c = k * 32 + lane;
            u[k] = c < n ? silu(conv_at<TAPS>(p, t, local, pos, st, first + c)) : 0.f;
            ss = fmaf(u[k], u[k], ss);
        }
        const float f = sg.unit ? sg.scale * rsqrtf(bw::warp_sum(ss) + p.unit_eps) : 1.f;
#pragma unroll
        for (int k = 0; k < NR; ++k) {
            const int c = k * 32 + lane;
            if (c < n) {
                dst[first + c] = u[k] * f;
                if (p.single) st[(size_t)(pos % p.taps) * p.C + first + c] = p.x[(size_t)t * p.ld + first + c];
            }
        }
    }
}

// the last taps - 1 inputs of every request's portion to its state
__global__ void __launch_bounds__(256)
conv_state_kernel(const float* __restrict__ x, long long ld, float* __restrict__ state, const int* __restrict__ cu_q,
                  const int* __restrict__ positions, const int* __restrict__ state_slot, int C, int taps) {
    BW_PDL_TRIGGER();
    BW_PDL_WAIT();
    const int r = blockIdx.x;
    const int a = cu_q[r], e = cu_q[r + 1];
    const int from = max(a, e - (taps - 1));
    float* st = state + (size_t)state_slot[r] * taps * C;
    for (int t = from; t < e; ++t)
        for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x)
            st[(size_t)(positions[t] % taps) * C + c] = x[(size_t)t * ld + c];
}

// ---------------------------------------------------------------- convolution of an attention's heads
// Channels: nq query heads of d, then nkv key heads of dk = maps * d and nkv value heads of dv (has_kv), or queries only.  A query
// head's d channels stand at offset (head % maps) * d of its row of dpad, zeros around them: with maps > 1 the heads
// head .. head + maps - 1 are maps of one head, each of which meets its own part of the key row in a plain product.  Keys and
// values go to the page of the token's position, zeros up to dpad.
struct HeadConvParams {
    const float* x; long long ld;
    const float* w;                        // [taps, C]
    float* state;                          // [slots, taps, C]
    const int *positions, *req_of_token, *cu_q, *state_slot, *block_table;
    void *q_out, *k_pages, *v_pages;       // [T, nq, dpad]; [num_pages, nkv, page_size, dpad]
    int T, C, taps, single, max_blocks, page_size, num_pages;
    int nq, d, maps, nkv, dk, dv, dpad, has_kv;
};

template <int W> __device__ __forceinline__ void load(const float* p, float (&v)[W]) {
    if constexpr (W == 2) { const float2 t = *reinterpret_cast<const float2*>(p); v[0] = t.x; v[1] = t.y; }
    else v[0] = *p;
}
template <int W> __device__ __forceinline__ void put(float* p, const float (&v)[W]) {
    if constexpr (W == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[1]);
    else *p = v[0];
}
template <int W> __device__ __forceinline__ void put(bf16* p, const float (&v)[W]) {
    if constexpr (W == 2) *reinterpret_cast<uint32_t*>(p) = bw::pack_bf16x2(v[0], v[1]);
    else *p = __float2bfloat16_rn(v[0]);
}

// A warp makes one head of up to TILE tokens; a lane W neighbouring channels at a time.
template <typename OT, int TAPS, int W>
__global__ void __launch_bounds__(32 * WARPS)
conv_heads_kernel(HeadConvParams p) {
    BW_PDL_TRIGGER();
    const int lane = threadIdx.x & 31;
    const int item = blockIdx.y * WARPS + (threadIdx.x >> 5);
    const int tile = p.single ? 1 : TILE;
    const int t0 = blockIdx.x * tile, t1 = min(p.T, t0 + tile);
    if (item >= p.nq + (p.has_kv ? 2 * p.nkv : 0)) return;
    const bool is_q = item < p.nq, is_v = item >= p.nq + p.nkv;
    const int head = is_q ? item : item - p.nq - (is_v ? p.nkv : 0);
    const int n = is_q ? p.d : (is_v ? p.dv : p.dk);                       // channels of the head
    const int at = is_q ? head % p.maps * p.d : 0;                         // where they stand in its row
    const int first = is_q ? head * p.d : p.nq * p.d + (is_v ? p.nkv * p.dk : 0) + head * n;   // the head's first column
    const int taps = TAPS > 0 ? TAPS : p.taps;
    BW_PDL_WAIT();
    // where each token's row goes (lane i: token t0 + i); null: nowhere
    OT* row = nullptr;
    if (lane < t1 - t0) {
        const int t = t0 + lane;
        if (is_q) row = (OT*)p.q_out + ((size_t)t * p.nq + head) * p.dpad;
        else {
            const int pos = p.positions[t], page = p.block_table[(size_t)p.req_of_token[t] * p.max_blocks + pos / p.page_size];
            if (page >= 0 && page < p.num_pages)
                row = (OT*)(is_v ? p.v_pages : p.k_pages) + (((size_t)page * p.nkv + head) * p.page_size + pos % p.page_size) * p.dpad;
        }
    }
    auto row_of = [&](int i) { return reinterpret_cast<OT*>(__shfl_sync(0xffffffffu, reinterpret_cast<unsigned long long>(row), i)); };
    const int r0 = p.req_of_token[t0], local0 = t0 - p.cu_q[r0];
    const bool whole = TAPS > 0 && t1 - t0 == TILE && local0 >= TAPS - 1 && t0 + TILE <= p.cu_q[r0 + 1];
    for (int base = 0; base < p.dpad; base += 32 * W) {
        const int o = base + lane * W, c = o - at;                         // column of the row; channel of the head
        const bool there = o < p.dpad, in = there && c >= 0 && c < n;
        if constexpr (TAPS > 0) {
            if (whole) {       // the tile and the tokens before it belong to one portion: every row is read once
                float v[TILE + TAPS - 1][W], w[TAPS][W];
                const float* src = p.x + (size_t)(t0 - (TAPS - 1)) * p.ld + first + c;
#pragma unroll
                for (int j = 0; j < TILE + TAPS - 1; ++j) {
                    if (in) load<W>(src + (size_t)j * p.ld, v[j]);
                    else {
#pragma unroll
                        for (int e = 0; e < W; ++e) v[j][e] = 0.f;
                    }
                }
#pragma unroll
                for (int j = 0; j < TAPS; ++j) {
                    if (in) load<W>(p.w + (size_t)j * p.C + first + c, w[j]);
                    else {
#pragma unroll
                        for (int e = 0; e < W; ++e) w[j][e] = 0.f;
                    }
                }
#pragma unroll
                for (int i = 0; i < TILE; ++i) {
                    float u[W];
#pragma unroll
                    for (int e = 0; e < W; ++e) {
                        u[e] = 0.f;
#pragma unroll
                        for (int j = 0; j < TAPS; ++j) u[e] = fmaf(w[j][e], v[i + j][e], u[e]);
                    }
                    OT* dst = row_of(i);
                    if (there && dst) put<W>(dst + o, u);
                }
                continue;
            }
        }
        for (int t = t0; t < t1; ++t) {
            const int r = p.req_of_token[t], local = t - p.cu_q[r], pos = p.positions[t];
            float* st = p.state + (size_t)p.state_slot[r] * p.taps * p.C;
            float u[W], x[W];
#pragma unroll
            for (int e = 0; e < W; ++e) u[e] = x[e] = 0.f;
            if (in) {
#pragma unroll
                for (int j = taps - 1; j >= 0; --j) {        // j tokens back, the oldest first; none before the sequence's start
                    if (j > pos) continue;
                    float w[W];
                    load<W>(j <= local ? p.x + (size_t)(t - j) * p.ld + first + c : st + (size_t)((pos - j) % taps) * p.C + first + c, x);
                    load<W>(p.w + (size_t)(taps - 1 - j) * p.C + first + c, w);
#pragma unroll
                    for (int e = 0; e < W; ++e) u[e] = fmaf(w[e], x[e], u[e]);
                }
                if (p.single) put<W>(st + (size_t)(pos % taps) * p.C + first + c, x);      // (x: the token's own input, read last)
            }
            OT* dst = row_of(t - t0);
            if (there && dst) put<W>(dst + o, u);
        }
    }
}

}  // namespace

// x: float32 rows `ld` apart, the convolution's C channels side by side (segments in order: n heads of `size` channels,
// unit != 0: unit vectors times scale).  w: float32 [taps, C] (oldest tap first).  single: one token per request.  Gates
// (heads > 0): see ConvParams.  max piece of a unit segment: 256 channels.
BW_EXPORT int bw_short_conv(const float* x, long long ld, const float* w, const float* bias, float* state,
                            const int* positions, const int* req_of_token, const int* cu_q, const int* state_slot,
                            float* out, int T, int R, int C, int taps, int single, int nseg, const int* seg_heads,
                            const int* seg_size, const int* seg_unit, const float* seg_scale, float unit_eps,
                            const float* zx, long long zld, int z_off, int z2_off, int heads, const float* A,
                            const float* dt_bias, float* decay, float* second, void* stream) {
    if (T <= 0) return 0;
    if (C <= 0 || taps <= 0 || nseg <= 0 || nseg > MAX_SEGS || R <= 0 || (single && T != R) || ld < C ||
        (heads > 0 && (!second || !zx || (z_off >= 0 ? (!A || !dt_bias || !decay) : z2_off < 0))))
        return BW_ERR_BAD_ARG;
    ConvParams p;
    p.x = x; p.ld = ld; p.w = w; p.bias = bias; p.state = state; p.positions = positions; p.req_of_token = req_of_token;
    p.cu_q = cu_q; p.state_slot = state_slot; p.out = out; p.T = T; p.C = C; p.taps = taps; p.single = single;
    p.nseg = nseg; p.unit_eps = unit_eps;
    p.zx = zx; p.zld = zld; p.z_off = z_off; p.z2_off = z2_off; p.heads = heads; p.A = A; p.dt_bias = dt_bias;
    p.decay = decay; p.second = second;
    int c0 = 0, pieces = 0, widest = 0;
    for (int s = 0; s < nseg; ++s) {
        Seg& g = p.seg[s];
        if (seg_heads[s] <= 0 || seg_size[s] <= 0) return BW_ERR_BAD_ARG;
        g.c0 = c0; g.channels = seg_heads[s] * seg_size[s]; g.unit = seg_unit[s]; g.scale = seg_scale[s];
        g.size = g.unit ? seg_size[s] : CHUNK;
        g.pieces = (g.channels + g.size - 1) / g.size;
        if (g.unit && g.size > widest) widest = g.size;
        c0 += g.channels; pieces += g.pieces;
    }
    if (c0 != C) return BW_ERR_BAD_ARG;
    if (widest > 256) return BW_ERR_UNSUPPORTED;
    pieces += (heads + 31) / 32;
    const int tile = single ? 1 : TILE;
    const dim3 grid((T + tile - 1) / tile, (pieces + WARPS - 1) / WARPS);
    cudaStream_t s = (cudaStream_t)stream;
#define BW_CONV(NR) switch (taps) { \
        case 2: bw::launch((short_conv_kernel<NR, 2>), grid, dim3(32 * WARPS), 0, s, p); break; \
        case 3: bw::launch((short_conv_kernel<NR, 3>), grid, dim3(32 * WARPS), 0, s, p); break; \
        case 4: bw::launch((short_conv_kernel<NR, 4>), grid, dim3(32 * WARPS), 0, s, p); break; \
        default: bw::launch((short_conv_kernel<NR, 0>), grid, dim3(32 * WARPS), 0, s, p); }
    if (widest <= 128) { BW_CONV(4) } else { BW_CONV(8) }
#undef BW_CONV
    BW_LAUNCH_CHECK();
    if (!single && taps > 1) {
        const int blocks = (C + 255) / 256;
        bw::launch((conv_state_kernel), dim3(R, blocks < 32 ? blocks : 32), dim3(256), 0, s, x, ld, state, cu_q, positions, state_slot, C, taps);
        BW_LAUNCH_CHECK();
    }
    return 0;
}

// See HeadConvParams.  w: float32 [taps, C], C = nq * d (+ nkv * (maps * d + dv) with has_kv).  type: element type of q_out and the
// pages.  single: one token per request, the state is written by the same kernel.
BW_EXPORT int bw_conv_heads(const float* x, long long ld, const float* w, float* state, const int* positions,
                            const int* req_of_token, const int* cu_q, const int* state_slot, const int* block_table, int max_blocks,
                            void* q_out, void* k_pages, void* v_pages, int type, int T, int R, int taps, int single, int nq, int d,
                            int maps, int nkv, int dv, int dpad, int has_kv, int page_size, int num_pages, void* stream) {
    if (T <= 0) return 0;
    if (R <= 0 || taps <= 0 || nq <= 0 || d <= 0 || maps <= 0 || nq % maps || dpad < maps * d || (single && T != R) || page_size <= 0 ||
        (has_kv && (nkv <= 0 || dv <= 0 || dpad < dv || !k_pages || !v_pages || !block_table)))
        return BW_ERR_BAD_ARG;
    HeadConvParams p;
    p.x = x; p.ld = ld; p.w = w; p.state = state; p.positions = positions; p.req_of_token = req_of_token; p.cu_q = cu_q;
    p.state_slot = state_slot; p.block_table = block_table; p.q_out = q_out; p.k_pages = k_pages; p.v_pages = v_pages;
    p.T = T; p.taps = taps; p.single = single; p.max_blocks = max_blocks; p.page_size = page_size; p.num_pages = num_pages;
    p.nq = nq; p.d = d; p.maps = maps; p.nkv = has_kv ? nkv : 0; p.dk = maps * d; p.dv = dv; p.dpad = dpad; p.has_kv = has_kv;
    p.C = nq * d + p.nkv * (p.dk + dv);
    if (ld < p.C) return BW_ERR_BAD_ARG;
    const int items = nq + 2 * p.nkv, tile = single ? 1 : TILE;
    const dim3 grid((T + tile - 1) / tile, (items + WARPS - 1) / WARPS);
    cudaStream_t s = (cudaStream_t)stream;
    // two channels a lane where every head begins at an even column of aligned rows
    const bool two = (d & 1) == 0 && (dv & 1) == 0 && (dpad & 1) == 0 && (ld & 1) == 0 &&
                     (((uintptr_t)x | (uintptr_t)w | (uintptr_t)state) & 7) == 0 && (((uintptr_t)q_out | (uintptr_t)k_pages | (uintptr_t)v_pages) & 7) == 0;
#define BW_CH(OT, W) switch (taps) { \
        case 2: bw::launch((conv_heads_kernel<OT, 2, W>), grid, dim3(32 * WARPS), 0, s, p); break; \
        case 3: bw::launch((conv_heads_kernel<OT, 3, W>), grid, dim3(32 * WARPS), 0, s, p); break; \
        case 4: bw::launch((conv_heads_kernel<OT, 4, W>), grid, dim3(32 * WARPS), 0, s, p); break; \
        default: bw::launch((conv_heads_kernel<OT, 0, W>), grid, dim3(32 * WARPS), 0, s, p); }
    if (type == BW_F32) { if (two) BW_CH(float, 2) else BW_CH(float, 1) }
    else if (type == BW_BF16) { if (two) BW_CH(bf16, 2) else BW_CH(bf16, 1) }
    else return BW_ERR_BAD_ARG;
#undef BW_CH
    BW_LAUNCH_CHECK();
    if (!single && taps > 1) {
        const int blocks = (p.C + 255) / 256;
        bw::launch((conv_state_kernel), dim3(R, blocks < 32 ? blocks : 32), dim3(256), 0, s, x, ld, state, cu_q, positions, state_slot, p.C, taps);
        BW_LAUNCH_CHECK();
    }
    return 0;
}
