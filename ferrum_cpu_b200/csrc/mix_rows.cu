// Row kernels of layers whose sublayers stand side by side on one norm: the residual update of the layer before,
// the norm, and the token-shift mixes of a recurrence, in one pass over the rows.
//
// x' = x + (rms(left) w_l + rms(right) w_r) / 2 + feed-forward;  h = rms(x') w;  m_s = h + (h_before - h) mu_s.
// The residual, every norm and every mix are f32; what the products read is written once as bf16 (or f32) planes.
// A CTA owns `rpc` consecutive rows and recomputes h of the row ahead of them, so no CTA waits for another.
//
// Bound: HBM / L2 (reads 2 + outputs rows of d floats, writes the residual row and one row per plane).
#include <algorithm>

#include "bf16_ops.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
constexpr int NT = 256;

// Sum over the block; `red` holds 2 * 8 floats per use, two values at once.
__device__ __forceinline__ float2 block_sum2(float a, float b, float2* red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        a += __shfl_xor_sync(0xffffffffu, a, o);
        b += __shfl_xor_sync(0xffffffffu, b, o);
    }
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = make_float2(a, b);
    __syncthreads();
    float2 t = red[0];
#pragma unroll
    for (int w = 1; w < NT / 32; ++w) { t.x += red[w].x; t.y += red[w].y; }
    return t;
}

template <class OT>
__device__ __forceinline__ void put(OT* p, float v) {
    if constexpr (sizeof(OT) == 2) *p = __bfloat16_as_ushort(__float2bfloat16_rn(v));
    else *p = v;
}
}  // namespace

template <class OT>
__global__ void __launch_bounds__(NT) mix_rows_kernel(const MixRows p, int rpc) {
    extern __shared__ float sm[];            // h of the row before | h of this row
    __shared__ float2 red[NT / 32];
    const int d = p.d, tid = threadIdx.x;
    float* hp = sm;
    float* hc = sm + d;
    // residual and norm of one row into dst; the row's owner also stores the residual
    auto row_h = [&](int r, float* dst, bool owner) {
        const int src = p.row_idx ? p.row_idx[r] : r;
        float ss = 0.0f;
        if (p.prev.outs) {
            const float* lo = p.prev.outs + (size_t)src * d;
            const float* ro = lo + p.prev.stride;
            float a = 0.0f, b = 0.0f;
            for (int c = tid; c < d; c += NT) { const float u = lo[c], v = ro[c]; a = fmaf(u, u, a); b = fmaf(v, v, b); }
            const float2 t = block_sum2(a, b, red);
            const float il = 1.0f / sqrtf(t.x / (float)d + p.eps), ir = 1.0f / sqrtf(t.y / (float)d + p.eps);
            for (int c = tid; c < d; c += NT) {
                float y = 0.5f * (lo[c] * il * p.prev.left_w[c] + ro[c] * ir * p.prev.right_w[c]);
                for (int f = 0; f < p.prev.n_ff; ++f) y += lo[(size_t)(2 + f) * p.prev.stride + c];
                const float x = p.x_in[(size_t)src * d + c] + y;
                if (owner && p.x_out) p.x_out[(size_t)r * d + c] = x;
                dst[c] = x;
                ss = fmaf(x, x, ss);
            }
        } else {
            int id = p.ids[src];
            if (id < 0 || id >= p.embed.vocab) {
                if (tid == 0) atomicExch(p.error_flag, FC_E_DIM);
                id = 0;
            }
            const uint16_t* e = p.embed.table + (size_t)id * p.embed.ld;
            for (int c = tid; c < d; c += NT) {
                const float x = __uint_as_float((uint32_t)e[c] << 16) * p.embed.scale;
                if (owner && p.x_out) p.x_out[(size_t)r * d + c] = x;
                dst[c] = x;
                ss = fmaf(x, x, ss);
            }
        }
        if (!p.norm_w) return;
        const float inv = 1.0f / sqrtf(block_sum2(ss, 0.0f, red).x / (float)d + p.eps);
        for (int c = tid; c < d; c += NT) dst[c] = dst[c] * inv * p.norm_w[c];
    };
    const int r0 = blockIdx.x * rpc, r1 = min(p.M, r0 + rpc);
    if (p.mu[0]) {
        if (r0 == 0) for (int c = tid; c < d; c += NT) hp[c] = p.h_first[c];
        else row_h(r0 - 1, hp, false);
    }
    OT* planes = (OT*)p.planes;
    for (int r = r0; r < r1; ++r) {
        row_h(r, hc, true);
        if (p.norm_w) {
            // every thread reads back only the columns it wrote
            OT* out = planes + (size_t)r * p.ld;
            for (int c = tid; c < d; c += NT) {
                const float h = hc[c];
                put(out + c, h);
                if (p.mu[0]) {
                    const float dh = hp[c] - h;
#pragma unroll
                    for (int s = 0; s < kMixes; ++s) put(out + (size_t)(1 + s) * p.plane_stride + c, fmaf(dh, p.mu[s][c], h));
                    if (p.h_last && r == p.M - 1) p.h_last[c] = h;
                }
            }
        }
        float* t = hp; hp = hc; hc = t;
    }
}

int launch_mix_rows(const MixRows& p, bool f32_planes, cudaStream_t st) {
    if (p.M <= 0) return FC_OK;
    const size_t smem = (size_t)2 * p.d * sizeof(float);
    if (smem > 200 * 1024) return fail(FC_E_SHAPE, "rows of %d values exceed the row kernel's staging", p.d);
    if (smem > 48 * 1024) {
        FC_CUDA(cudaFuncSetAttribute(mix_rows_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        FC_CUDA(cudaFuncSetAttribute(mix_rows_kernel<uint16_t>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    }
    const int rpc = !p.mu[0] ? 1 : (p.M >= 1024 ? 4 : (p.M >= 512 ? 2 : 1));
    const int grid = (p.M + rpc - 1) / rpc;
    if (f32_planes) mix_rows_kernel<float><<<grid, NT, smem, st>>>(p, rpc);
    else mix_rows_kernel<uint16_t><<<grid, NT, smem, st>>>(p, rpc);
    FC_LAUNCHED();
    return FC_OK;
}

}  // namespace fc
