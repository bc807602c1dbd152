// Row kernel of layers that norm what a sublayer adds to the residual: x <- x + rms(y) w with y the sum of a row's parts (K
// slices of one product, or the chosen experts' rows times their weights), and x written as the operand of the next products;
// or, at the start, x = rms(embedding) w; or, at the end, the final norm of some rows.
// The residual, sums and norms are f32; the operand is bf16 (or f32). One CTA a row.
//
// Bound: HBM / L2 (reads the parts and the residual row, writes the residual and the operand row).
#include <algorithm>

#include "bf16_ops.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
constexpr int NT = 256;
__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = red[0];
#pragma unroll
    for (int w = 1; w < NT / 32; ++w) t += red[w];
    return t;
}
template <class T, int V>
__device__ __forceinline__ void put(T* p, const float* x) {
    if constexpr (V == 1) {
        if constexpr (sizeof(T) == 2) *p = __bfloat16_as_ushort(__float2bfloat16_rn(x[0]));
        else *p = x[0];
    } else if constexpr (sizeof(T) == 2) {
        *(uint2*)p = make_uint2(tc::pack2(x[0], x[1]), tc::pack2(x[2], x[3]));
    } else {
        *(float4*)p = make_float4(x[0], x[1], x[2], x[3]);
    }
}
template <int V>
__device__ __forceinline__ void get(const float* p, float* x) {
    if constexpr (V == 4) { const float4 v = *(const float4*)p; x[0] = v.x; x[1] = v.y; x[2] = v.z; x[3] = v.w; }
    else x[0] = *p;
}
}  // namespace

template <class T, int V>
__global__ void __launch_bounds__(NT) post_norm_rows_kernel(const PostNormRows p) {
    extern __shared__ __align__(16) float row[];           // [d]: every thread reads back what it wrote
    __shared__ float red[NT / 32];
    const int d = p.d, r = blockIdx.x, tid = threadIdx.x;
    const size_t src = p.row_idx ? p.row_idx[r] : r;
    float* x = p.x + src * d;
    float ss = 0.0f;
    if (p.add.y) {
        const PostNorm& a = p.add;
        for (int c = tid * V; c < d; c += NT * V) {
            float y[V] = {};
#pragma unroll 4
            for (int s = 0; s < a.n_parts; ++s) {
                const size_t at = src * a.n_parts + s, yr = a.index ? (size_t)a.index[at] : (size_t)s * a.part_rows + src;
                const float w = a.weight ? a.weight[at] : 1.0f;
                float v[V];
                get<V>(a.y + yr * d + c, v);
#pragma unroll
                for (int e = 0; e < V; ++e) y[e] = fmaf(w, v[e], y[e]);
            }
#pragma unroll
            for (int e = 0; e < V; ++e) { row[c + e] = y[e]; ss = fmaf(y[e], y[e], ss); }
        }
    } else if (p.ids) {
        int id = p.ids[src];
        if (id < 0 || id >= p.embed.vocab) {
            if (tid == 0) atomicExch(p.error_flag, FC_E_DIM);
            id = 0;
        }
        const uint16_t* e16 = p.embed.table + (size_t)id * p.embed.ld;
        for (int c = tid * V; c < d; c += NT * V)
#pragma unroll
            for (int e = 0; e < V; ++e) {
                const float y = __uint_as_float((uint32_t)e16[c + e] << 16) * p.embed.scale;
                row[c + e] = y;
                ss = fmaf(y, y, ss);
            }
    } else {
        for (int c = tid * V; c < d; c += NT * V) {
            float y[V];
            get<V>(x + c, y);
#pragma unroll
            for (int e = 0; e < V; ++e) { row[c + e] = y[e]; ss = fmaf(y[e], y[e], ss); }
        }
    }
    T* out = (T*)p.plane + (size_t)r * p.ld;
    if (p.add.y || p.ids) {
        const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + p.eps);
        ss = 0.0f;
        for (int c = tid * V; c < d; c += NT * V) {
            float w[V], y[V] = {};
            get<V>(p.add.norm_w + c, w);
            if (p.add.y) get<V>(x + c, y);
#pragma unroll
            for (int e = 0; e < V; ++e) {
                y[e] = fmaf(row[c + e] * inv, w[e], y[e]);
                row[c + e] = y[e];
                ss = fmaf(y[e], y[e], ss);
            }
            put<float, V>(x + c, y);
            if (!p.out_norm_w) put<T, V>(out + c, y);
        }
    }
    if (!p.out_norm_w) return;
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + p.eps);
    for (int c = tid * V; c < d; c += NT * V) {
        float w[V], y[V];
        get<V>(p.out_norm_w + c, w);
#pragma unroll
        for (int e = 0; e < V; ++e) y[e] = row[c + e] * inv * w[e];
        put<T, V>(out + c, y);
    }
}

template <class T, int V>
static int launch(const PostNormRows& p, cudaStream_t st) {
    const size_t smem = (size_t)p.d * sizeof(float);
    if (smem > 200 * 1024) return fail(FC_E_SHAPE, "rows of %d values exceed the row kernel's staging", p.d);
    if (smem > 47 * 1024) FC_CUDA(cudaFuncSetAttribute(post_norm_rows_kernel<T, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    post_norm_rows_kernel<T, V><<<p.M, NT, smem, st>>>(p);
    FC_LAUNCHED();
    return FC_OK;
}
int launch_post_norm_rows(const PostNormRows& p, bool f32_plane, cudaStream_t st) {
    if (p.M <= 0) return FC_OK;
    const bool vec = p.d % 4 == 0;                          // every buffer is 16-byte aligned
    if (f32_plane) return vec ? launch<float, 4>(p, st) : launch<float, 1>(p, st);
    return vec ? launch<uint16_t, 4>(p, st) : launch<uint16_t, 1>(p, st);
}

}  // namespace fc
