// Attention whose heads' scores are mixed before the softmax ("talking heads"), with a learned bias per distance,
// a sink in the denominator, a query temperature that grows with the position, and normed values.
//
// Mixing commutes with the product: the mixed score of head h is q'_h . (keys of all key/value heads side by side) with
// q'_h = [sum_{g in group 0} talk[h][g] q_g | sum_{g in group 1} ... ], plus a per-head table of the distance whose
// heads are mixed once at load. So after `talk_prep_kernel` this is ordinary attention with one wide shared key head.
//
//   talk_prep_kernel   one CTA per token: mixed queries out, key row and normed value row into the cache
// The attention itself: flash_tc.cu, flash_f32.cu. Bound: HBM / L2.
#include <algorithm>

#include "bf16_ops.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
template <class T>
__device__ __forceinline__ void put(T* p, float v) {
    if constexpr (sizeof(T) == 2) *p = __bfloat16_as_ushort(__float2bfloat16_rn(v));
    else *p = v;
}
}  // namespace

// PER: query heads per key/value head when it is one of the unrolled counts, 0: any.
template <class T, int PER>
__global__ void __launch_bounds__(256) talk_prep_kernel(const TalkAttn t, const float* __restrict__ proj, int ldp, int pos0, float factor,
                                                        T* __restrict__ qm, T* __restrict__ kc, T* __restrict__ vc) {
    extern __shared__ float sm[];              // talk [H][H] | q [H * dim]
    const int tid = threadIdx.x, row = blockIdx.x, pos = pos0 + row, H = t.H, dim = t.dim, per = H / t.KV;
    float* tk = sm;
    float* q = sm + H * H;
    const float* src = proj + (size_t)row * ldp;
    const float temp = 1.0f + t.temp_coef * logf((float)(floor((double)(pos + 1) / t.temp_every) + 1.0));
    for (int i = tid; i < H * H; i += 256) tk[i] = t.talk[i];
    const float qs = t.scale * temp * factor;
    for (int i = tid; i < H * dim; i += 256) q[i] = src[i] * qs;
    __syncthreads();
    const int width = t.KV * dim;
    T* out = qm + (size_t)row * H * t.kd;
    // two neighbouring columns a thread (kd is even); they may belong to different key/value heads
    for (int f = 2 * tid; f < t.kd; f += 512) {
        const int c0 = min(f, width - 1) / dim, c1 = min(f + 1, width - 1) / dim;
        const float z0 = f < width ? 1.0f : 0.0f, z1 = f + 1 < width ? 1.0f : 0.0f;
        const float* q0 = q + (size_t)c0 * per * dim + (min(f, width - 1) - c0 * dim);
        const float* q1 = q + (size_t)c1 * per * dim + (min(f + 1, width - 1) - c1 * dim);
        auto store = [&](int h, float a, float b) {
            T* to = out + (size_t)h * t.kd + f;
            if constexpr (sizeof(T) == 2) *(uint32_t*)to = tc::pack2(a, b);
            else *(float2*)to = make_float2(a, b);
        };
        if constexpr (PER > 0) {
            float a[PER], b[PER];
#pragma unroll
            for (int g = 0; g < PER; ++g) { a[g] = q0[g * dim] * z0; b[g] = q1[g * dim] * z1; }
            if (c0 == c1) {
#pragma unroll 4
                for (int h = 0; h < H; ++h) {
                    const float* w = tk + h * H + c0 * PER;
                    float x = 0.0f, y = 0.0f;
#pragma unroll
                    for (int g = 0; g < PER; ++g) { x = fmaf(w[g], a[g], x); y = fmaf(w[g], b[g], y); }
                    store(h, x, y);
                }
                continue;
            }
        }
        for (int h = 0; h < H; ++h) {
            float x = 0.0f, y = 0.0f;
            for (int g = 0; g < per; ++g) {
                x = fmaf(tk[h * H + c0 * per + g], q0[g * dim] * z0, x);
                y = fmaf(tk[h * H + c1 * per + g], q1[g * dim] * z1, y);
            }
            store(h, x, y);
        }
    }
    const float* ks = src + H * dim;
    for (int f = tid; f < t.kd; f += 256) put(kc + (size_t)pos * t.kd + f, f < width ? ks[f] : 0.0f);
    const float* vs = ks + width;
    for (int c = tid >> 5; c < t.KV; c += 8) {
        const int lane = tid & 31;
        float s = 0.0f;
        for (int e = lane; e < t.vdim; e += 32) { const float v = vs[c * t.vdim + e]; s = fmaf(v, v, s); }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        const float inv = 1.0f / sqrtf(s / (float)t.vdim + t.eps);
        for (int e = lane; e < t.vp; e += 32) put(vc + ((size_t)pos * t.KV + c) * t.vp + e, e < t.vdim ? vs[c * t.vdim + e] * inv : 0.0f);
    }
}

template <class T>
static int prep(const TalkAttn& t, const float* proj, int ldp, int M, int pos0, float factor, void* qm, void* kc, void* vc, cudaStream_t st) {
    const size_t smem = (size_t)(t.H * t.H + t.H * t.dim) * sizeof(float);
    if (smem > 200 * 1024) return fail(FC_E_SHAPE, "%d query heads of %d exceed the staging of the query mixing", t.H, t.dim);
#define FC_PREP(P)                                                                                                              \
    do {                                                                                                                        \
        if (smem > 47 * 1024) FC_CUDA(cudaFuncSetAttribute(talk_prep_kernel<T, P>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        talk_prep_kernel<T, P><<<M, 256, smem, st>>>(t, proj, ldp, pos0, factor, (T*)qm, (T*)kc, (T*)vc);                        \
    } while (0)
    switch (t.H / t.KV) {
        case 1: FC_PREP(1); break;
        case 2: FC_PREP(2); break;
        case 3: FC_PREP(3); break;
        case 4: FC_PREP(4); break;
        case 8: FC_PREP(8); break;
        default: FC_PREP(0);
    }
#undef FC_PREP
    FC_LAUNCHED();
    return FC_OK;
}
int launch_talk_prep(const TalkAttn& t, const float* proj, int ldp, int M, int pos0, float factor, void* qm, void* kc, void* vc, bool f32,
                     cudaStream_t st) {
    return f32 ? prep<float>(t, proj, ldp, M, pos0, factor, qm, kc, vc, st) : prep<uint16_t>(t, proj, ldp, M, pos0, factor, qm, kc, vc, st);
}

// What the attention of a portion reads: one wide key all heads share, values by key/value head, the bias, the sink.
Flash talk_flash(const TalkAttn& t, const void* kc, const void* vc, int ctx) {
    Flash f;
    f.H = t.H; f.KV = t.KV; f.vdim = t.vdim;
    f.k0.p = kc; f.k0.rows = ctx; f.k0.ld = t.kd; f.k0.width = t.kd;
    f.v.p = vc; f.v.rows = ctx; f.v.ld = t.KV * t.vp; f.v.head_stride = t.vp; f.v.width = t.vp;
    f.bias = t.bias; f.far = t.far; f.sink = t.sink; f.has_sink = true;
    return f;
}

}  // namespace fc
