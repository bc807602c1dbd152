// What a portion's attention with rotated positions needs ahead of the softmax: queries (normed, rotated, scaled) as operands,
// and the cache rows of its tokens.
//
//   rot_prep_kernel      grouped-query attention: q and k normed over the whole projection, rotated; values as they are
//   latent_prep_kernel   latent attention: rotated part of every query head, normed latent and the rotated key part of a row
// One CTA per token; norms, angles and rotation are f32 (the angle's product in double).
// Bound: HBM / L2.
#include <algorithm>

#include "rot_rows.cuh"

namespace fc {

namespace {
constexpr int NT = 256;
}

template <class T>
__global__ void __launch_bounds__(NT) rot_prep_kernel(const RotAttn t, const float* __restrict__ proj, int ldp, int pos0, float factor,
                                                      T* __restrict__ q, T* __restrict__ kc, T* __restrict__ vc) {
    extern __shared__ float2 cs[];                 // [dims / 2]
    __shared__ float red[NT / 32];
    const int tid = threadIdx.x, row = blockIdx.x, pos = pos0 + row, dim = t.dim, qn = t.H * dim, kn = t.KV * dim;
    const float* src = proj + (size_t)row * ldp;
    for (int i = tid; i < t.rot.dims / 2; i += NT) cs[i] = rot_cs(pos, t.rot.freq[i]);
    float qi = 1.0f, ki = 1.0f;
    if (t.q_norm) {
        float s = 0.0f;
        for (int i = tid; i < qn; i += NT) s = fmaf(src[i], src[i], s);
        qi = 1.0f / sqrtf(block_sum_of<NT>(s, red) / (float)qn + t.eps);
    }
    if (t.own_kv && t.k_norm) {
        float s = 0.0f;
        for (int i = tid; i < kn; i += NT) s = fmaf(src[qn + i], src[qn + i], s);
        ki = 1.0f / sqrtf(block_sum_of<NT>(s, red) / (float)kn + t.eps);
    }
    __syncthreads();
    qi *= t.scale * factor;
    auto head = [&](const float* x, const float* w, float inv, int width, T* out) {      // two elements a thread
        for (int h = tid >> 5; h < width; h += NT / 32) {
            auto at = [&](int k) { return x[h * dim + k] * (w ? w[h * dim + k] : 1.0f); };
#pragma unroll 2
            for (int e = (tid & 31) * 2; e < t.kp; e += 64) {
                const float a = e < dim ? rotated(t.rot.neighbours, t.rot.dims, cs, e, at) * inv : 0.0f;
                const float b = e + 1 < dim ? rotated(t.rot.neighbours, t.rot.dims, cs, e + 1, at) * inv : 0.0f;
                put_pair(out + (size_t)h * t.kp + e, a, b);
            }
        }
    };
    head(src, t.q_norm, qi, t.H, q + (size_t)row * t.H * t.kp);
    if (!t.own_kv) return;
    head(src + qn, t.k_norm, ki, t.KV, kc + (size_t)pos * t.KV * t.kp);
    const float* v = src + qn + kn;
    for (int i = tid; i < t.KV * t.vp; i += NT) {
        const int c = i / t.vp, e = i - c * t.vp;
        put_row(vc + (size_t)pos * t.KV * t.vp + i, e < t.vdim ? v[c * t.vdim + e] : 0.0f);
    }
}
int launch_rot_prep(const RotAttn& t, const float* proj, int ldp, int M, int pos0, float factor, void* q, void* kc, void* vc, bool f32,
                    cudaStream_t st) {
    const size_t smem = (size_t)t.rot.dims / 2 * sizeof(float2);
    if (smem > 40 * 1024) return fail(FC_E_SHAPE, "%d rotated dimensions", t.rot.dims);
    if (f32) rot_prep_kernel<float><<<M, NT, smem, st>>>(t, proj, ldp, pos0, factor, (float*)q, (float*)kc, (float*)vc);
    else rot_prep_kernel<uint16_t><<<M, NT, smem, st>>>(t, proj, ldp, pos0, factor, (uint16_t*)q, (uint16_t*)kc, (uint16_t*)vc);
    FC_LAUNCHED();
    return FC_OK;
}
Flash rot_flash(const RotAttn& t, const void* kc, const void* vc, int ctx) {
    Flash f;
    f.H = t.H; f.KV = t.KV; f.vdim = t.vdim;
    f.k0.p = kc; f.k0.rows = ctx; f.k0.ld = t.KV * t.kp; f.k0.head_stride = t.kp; f.k0.width = t.kp;
    f.v.p = vc; f.v.rows = ctx; f.v.ld = t.KV * t.vp; f.v.head_stride = t.vp; f.v.width = t.vp;
    f.window = t.window; f.has_sink = t.has_sink;
    return f;
}

template <class T>
__global__ void __launch_bounds__(NT) latent_prep_kernel(const LatentAttn t, const float* __restrict__ proj, int ldp, int pos0, float factor,
                                                         T* __restrict__ q, T* __restrict__ cache) {
    extern __shared__ float2 cs[];
    __shared__ float red[NT / 32];
    const int tid = threadIdx.x, row = blockIdx.x, pos = pos0 + row, rot = t.rot.dims, hq = t.dim + rot, wq = t.dp + t.rot_p;
    const float* src = proj + (size_t)row * ldp;
    for (int i = tid; i < rot / 2; i += NT) cs[i] = rot_cs(pos, t.rot.freq[i]);
    const float* lat = src + (size_t)t.H * hq;
    float s = 0.0f;
    for (int i = tid; i < t.rank; i += NT) s = fmaf(lat[i], lat[i], s);
    const float inv = 1.0f / sqrtf(block_sum_of<NT>(s, red) / (float)t.rank + t.eps);      // also the barrier behind cs
    const float qs = t.scale * factor;
    T* out = q + (size_t)row * t.H * wq;
    for (int h = tid >> 5; h < t.H; h += NT / 32)
#pragma unroll 2
    for (int e0 = (tid & 31) * 2; e0 < wq; e0 += 64) {
        const float* x = src + (size_t)h * hq;
        float v[2];
#pragma unroll
        for (int y = 0; y < 2; ++y) {
            const int e = e0 + y, r = e - t.dp;
            if (r < 0) v[y] = e < t.dim ? x[e] * qs : 0.0f;
            else v[y] = r < rot ? rotated(t.rot.neighbours, rot, cs, r, [&](int k) { return x[t.dim + k]; }) * qs : 0.0f;
        }
        put_pair(out + (size_t)h * wq + e0, v[0], v[1]);
    }
    T* to = cache + (size_t)pos * (t.lat + t.rot_p);
    for (int i = tid; i < t.lat; i += NT) put_row(to + i, i < t.rank ? lat[i] * inv * t.c_norm[i] : 0.0f);
    for (int r = tid; r < t.rot_p; r += NT)
        put_row(to + t.lat + r, r < rot ? rotated(t.rot.neighbours, rot, cs, r, [&](int k) { return lat[t.rank + k]; }) : 0.0f);
}
int launch_latent_prep(const LatentAttn& t, const float* proj, int ldp, int M, int pos0, float factor, void* q, void* cache, bool f32,
                       cudaStream_t st) {
    const size_t smem = (size_t)t.rot.dims / 2 * sizeof(float2);
    if (smem > 40 * 1024) return fail(FC_E_SHAPE, "%d rotated dimensions", t.rot.dims);
    if (f32) latent_prep_kernel<float><<<M, NT, smem, st>>>(t, proj, ldp, pos0, factor, (float*)q, (float*)cache);
    else latent_prep_kernel<uint16_t><<<M, NT, smem, st>>>(t, proj, ldp, pos0, factor, (uint16_t*)q, (uint16_t*)cache);
    FC_LAUNCHED();
    return FC_OK;
}
Flash latent_flash(const LatentAttn& t, const void* k, const void* v, int rows, int base, const void* cache, int ctx) {
    Flash f;
    f.H = f.KV = t.H; f.vdim = t.vdim;
    f.k0.p = k; f.k0.rows = rows; f.k0.ld = t.H * t.dp; f.k0.head_stride = t.dp; f.k0.width = t.dp; f.k0.pos0 = base;
    f.k1.p = cache; f.k1.rows = ctx; f.k1.ld = t.row(); f.k1.col = t.lat; f.k1.width = t.rot_p;
    f.v.p = v; f.v.rows = rows; f.v.ld = t.H * t.vp; f.v.head_stride = t.vp; f.v.width = t.vp; f.v.pos0 = base;
    f.window = t.window;
    return f;
}

}  // namespace fc
