// Row kernels of layers whose sublayers stand side by side on one norm: the residual update of the layer before,
// the norm, and the token-shift mixes of a recurrence, in one pass over the rows.
//
// x' = x + (rms(left) w_l + rms(right) w_r) / 2 + feed-forward;  h = rms(x') w;  m_s = h + (h_before - h) mu_s.
// The residual, every norm and every mix are f32; what the products read is written once as bf16 (or f32) planes.
// A CTA takes rpc consecutive rows and the one ahead of them (whose h the mixes of the first need), W warps each, so no CTA
// waits for another; the rows of h meet in shared memory.
//
// Bound: HBM / L2 (reads 2 + outputs rows of d floats, writes the residual row and one row per plane).
#include <algorithm>

#include "bf16_ops.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// V consecutive floats (V = 4: 16-byte accesses).
template <int V> struct Vec { float v[V]; };
template <int V>
__device__ __forceinline__ Vec<V> ld(const float* p) {
    Vec<V> r;
    if constexpr (V == 4) { const float4 x = *(const float4*)p; r.v[0] = x.x; r.v[1] = x.y; r.v[2] = x.z; r.v[3] = x.w; }
    else r.v[0] = *p;
    return r;
}
template <int V>
__device__ __forceinline__ void st(float* p, const Vec<V>& x) {
    if constexpr (V == 4) *(float4*)p = make_float4(x.v[0], x.v[1], x.v[2], x.v[3]);
    else *p = x.v[0];
}
template <int V>
__device__ __forceinline__ void st(uint16_t* p, const Vec<V>& x) {
    if constexpr (V == 4) *(uint2*)p = make_uint2(tc::pack2(x.v[0], x.v[1]), tc::pack2(x.v[2], x.v[3]));
    else *p = __bfloat16_as_ushort(__float2bfloat16_rn(x.v[0]));
}
}  // namespace

template <class OT, int V>
__global__ void __launch_bounds__(512) mix_rows_kernel(const MixRows p, int rpc, int W) {
    extern __shared__ __align__(16) float sm[];            // h of rows r0 - 1 .. r0 + rpc - 1
    __shared__ float2 red[16];
    const int d = p.d, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, r0 = blockIdx.x * rpc, ahead = p.mu[0] ? 1 : 0;
    const int slot = warp / W, r = r0 + slot - ahead;      // this warp's row
    const int c0 = ((warp - slot * W) * 32 + lane) * V, step = W * 32 * V;
    const bool live = r >= 0 && r < p.M;
    const int src = live ? (p.row_idx ? p.row_idx[r] : r) : 0;
    float* h = sm + (size_t)slot * d;
    // the sums of the W warps of a row, in warp order
    auto row_sum2 = [&](float a, float b) -> float2 {
        a = warp_sum(a);
        b = warp_sum(b);
        __syncthreads();
        if (lane == 0) red[warp] = make_float2(a, b);
        __syncthreads();
        float2 s = red[slot * W];
        for (int i = 1; i < W; ++i) { s.x += red[slot * W + i].x; s.y += red[slot * W + i].y; }
        return s;
    };
    const bool keep = live && p.x_out && r >= r0;          // the residual is stored by the row's owner
    float ss = 0.0f;
    if (p.prev.outs) {
        const float* lo = p.prev.outs + (size_t)src * d;
        const float* ro = lo + p.prev.stride;
        float a = 0.0f, b = 0.0f;
        if (live)
#pragma unroll 4
            for (int c = c0; c < d; c += step) {
                const Vec<V> u = ld<V>(lo + c), v = ld<V>(ro + c);
#pragma unroll
                for (int e = 0; e < V; ++e) { a = fmaf(u.v[e], u.v[e], a); b = fmaf(v.v[e], v.v[e], b); }
            }
        const float2 s = row_sum2(a, b);
        const float il = 1.0f / sqrtf(s.x / (float)d + p.eps), ir = 1.0f / sqrtf(s.y / (float)d + p.eps);
        if (live)
#pragma unroll 2
            for (int c = c0; c < d; c += step) {
                const Vec<V> u = ld<V>(lo + c), v = ld<V>(ro + c), wl = ld<V>(p.prev.left_w + c), wr = ld<V>(p.prev.right_w + c);
                Vec<V> x = ld<V>(p.x_in + (size_t)src * d + c), y;
#pragma unroll
                for (int e = 0; e < V; ++e) y.v[e] = 0.5f * (u.v[e] * il * wl.v[e] + v.v[e] * ir * wr.v[e]);
                for (int f = 0; f < p.prev.n_ff; ++f) {
                    const Vec<V> z = ld<V>(lo + (size_t)(2 + f) * p.prev.stride + c);
#pragma unroll
                    for (int e = 0; e < V; ++e) y.v[e] += z.v[e];
                }
#pragma unroll
                for (int e = 0; e < V; ++e) { x.v[e] += y.v[e]; ss = fmaf(x.v[e], x.v[e], ss); }
                if (keep) st(p.x_out + (size_t)r * d + c, x);
                st(h + c, x);
            }
    } else if (live) {
        int id = p.ids[src];
        if (id < 0 || id >= p.embed.vocab) {
            if (lane == 0) atomicExch(p.error_flag, FC_E_DIM);
            id = 0;
        }
        const uint16_t* e16 = p.embed.table + (size_t)id * p.embed.ld;
        for (int c = c0; c < d; c += step) {
            Vec<V> x;
#pragma unroll
            for (int e = 0; e < V; ++e) {
                x.v[e] = __uint_as_float((uint32_t)e16[c + e] << 16) * p.embed.scale;
                ss = fmaf(x.v[e], x.v[e], ss);
            }
            if (keep) st(p.x_out + (size_t)r * d + c, x);
            st(h + c, x);
        }
    }
    if (p.norm_w) {
        const float inv = 1.0f / sqrtf(row_sum2(ss, 0.0f).x / (float)d + p.eps);
        if (live)
            for (int c = c0; c < d; c += step) {           // every lane reads back what it wrote
                Vec<V> x = ld<V>(h + c);
                const Vec<V> w = ld<V>(p.norm_w + c);
#pragma unroll
                for (int e = 0; e < V; ++e) x.v[e] = x.v[e] * inv * w.v[e];
                st(h + c, x);
            }
        else if (r < 0)
            for (int c = c0; c < d; c += step) st(h + c, ld<V>(p.h_first + c));
    }
    if (!p.norm_w) return;
    __syncthreads();
    OT* planes = (OT*)p.planes;
    const int rows = min(rpc, p.M - r0), units = d / V;
    for (int i = threadIdx.x; i < rows * units; i += blockDim.x) {
        const int rr = i / units, c = (i - rr * units) * V;
        const Vec<V> x = ld<V>(sm + (size_t)(rr + ahead) * d + c);
        OT* out = planes + (size_t)(r0 + rr) * p.ld + c;
        st(out, x);
        if (!ahead) continue;
        const Vec<V> before = ld<V>(sm + (size_t)rr * d + c);
#pragma unroll
        for (int s = 0; s < kMixes; ++s) {
            const Vec<V> mu = ld<V>(p.mu[s] + c);
            Vec<V> y;
#pragma unroll
            for (int e = 0; e < V; ++e) y.v[e] = fmaf(before.v[e] - x.v[e], mu.v[e], x.v[e]);
            st(out + (size_t)(1 + s) * p.plane_stride, y);
        }
        if (p.h_last && r0 + rr == p.M - 1) st(p.h_last + c, x);
    }
}

template <class OT, int V>
static int launch_mix(const MixRows& p, cudaStream_t st) {
    constexpr int kSmem = 200 * 1024;
    const size_t row = (size_t)p.d * sizeof(float);
    int rpc = p.M >= 512 ? 4 : (p.M >= 256 ? 2 : 1);
    while (rpc > 1 && (rpc + 1) * row > kSmem) rpc /= 2;
    const size_t smem = (rpc + 1) * row;
    if (smem > kSmem) return fail(FC_E_SHAPE, "rows of %d values exceed the row kernel's staging", p.d);
    // above 48 KB with the static part, shared memory has to be asked for
    if (smem > 47 * 1024) FC_CUDA(cudaFuncSetAttribute(mix_rows_kernel<OT, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, kSmem));
    const int slots = rpc + (p.mu[0] ? 1 : 0);
    int W = 16 / slots;
    while (W > 1 && (W - 1) * 32 * V >= p.d) --W;          // no warp without columns
    mix_rows_kernel<OT, V><<<(p.M + rpc - 1) / rpc, 32 * slots * W, smem, st>>>(p, rpc, W);
    FC_LAUNCHED();
    return FC_OK;
}
int launch_mix_rows(const MixRows& p, bool f32_planes, cudaStream_t st) {
    if (p.M <= 0) return FC_OK;
    const bool vec = p.d % 4 == 0;                          // every buffer is 16-byte aligned
    if (f32_planes) return vec ? launch_mix<float, 4>(p, st) : launch_mix<float, 1>(p, st);
    return vec ? launch_mix<uint16_t, 4>(p, st) : launch_mix<uint16_t, 1>(p, st);
}

}  // namespace fc
