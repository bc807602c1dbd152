// The residual of one token ahead of a decode kernel's own work, for layers that norm what a sublayer adds (PostNorm): every
// CTA computes the row for itself.
#pragma once
#include "bf16_ops.cuh"

namespace fc {

// NT threads; rows of up to 16 * NT * CH / 4 values whose length is a multiple of four take the 16-byte path, whose loads go out
// together: the norm's weights before the wait on the kernel ahead (load), the rest after it (run).
template <int NT, int CH>
struct PostRow {
    float4 w[CH];
    bool vec;
    __device__ __forceinline__ void load(const float* norm_w, int d) {
        vec = d % 4 == 0 && d <= 4 * NT * CH;
#pragma unroll
        for (int i = 0; i < CH; ++i) {
            const int c = (threadIdx.x + i * NT) * 4;
            w[i] = vec && c < d ? __ldg((const float4*)(norm_w + c)) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
    }
    // put(c, x'[c]) for this thread's columns; sum(v): the block's sum; row(c): a float per column between the passes (the
    // other path). Returns the thread's sum of squares of x'.
    template <class Put, class Sum, class Row>
    __device__ __forceinline__ float run(const PostNorm& p, const float* x_in, int d, float eps, Put put, Sum sum, Row row) {
        float ss = 0.0f, yy = 0.0f;
        if (!vec) {
            for (int c = threadIdx.x; c < d; c += NT) {
                const float y = post_norm_sum(p, 0, c, d);
                row(c) = y;
                yy = fmaf(y, y, yy);
            }
            const float inv = 1.0f / sqrtf(sum(yy) / (float)d + eps);
            for (int c = threadIdx.x; c < d; c += NT) {
                const float x = fmaf(row(c) * inv, p.norm_w[c], x_in[c]);
                put(c, x);
                ss = fmaf(x, x, ss);
            }
            return ss;
        }
        float4 x[CH], y[CH];
#pragma unroll
        for (int i = 0; i < CH; ++i) {
            const int c = (threadIdx.x + i * NT) * 4;
            x[i] = c < d ? *(const float4*)(x_in + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            y[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        }
        for (int s0 = 0; s0 < p.n_parts; s0 += 4) {
#pragma unroll
            for (int i = 0; i < CH; ++i) {
                const int c = (threadIdx.x + i * NT) * 4;
                if (i * NT * 4 >= d) continue;                           // uniform
                float4 v[4];
                float wt[4];
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const int s = s0 + k;
                    const bool on = s < p.n_parts && c < d;
                    v[k] = on ? *(const float4*)(p.y + (size_t)s * p.part_rows * d + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                    wt[k] = on && p.weight ? p.weight[s] : 1.0f;
                }
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    y[i].x = fmaf(wt[k], v[k].x, y[i].x); y[i].y = fmaf(wt[k], v[k].y, y[i].y);
                    y[i].z = fmaf(wt[k], v[k].z, y[i].z); y[i].w = fmaf(wt[k], v[k].w, y[i].w);
                }
            }
        }
#pragma unroll
        for (int i = 0; i < CH; ++i) yy += y[i].x * y[i].x + y[i].y * y[i].y + y[i].z * y[i].z + y[i].w * y[i].w;
        const float inv = 1.0f / sqrtf(sum(yy) / (float)d + eps);
#pragma unroll
        for (int i = 0; i < CH; ++i) {
            const int c = (threadIdx.x + i * NT) * 4;
            if (c >= d) continue;
            const float o[4] = {fmaf(y[i].x * inv, w[i].x, x[i].x), fmaf(y[i].y * inv, w[i].y, x[i].y), fmaf(y[i].z * inv, w[i].z, x[i].z),
                                fmaf(y[i].w * inv, w[i].w, x[i].w)};
#pragma unroll
            for (int e = 0; e < 4; ++e) { put(c + e, o[e]); ss = fmaf(o[e], o[e], ss); }
        }
        return ss;
    }
};

}  // namespace fc
