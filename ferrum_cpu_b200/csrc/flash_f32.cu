// The attention of flash_tc.cu in true f32 on CUDA cores: 16 query rows of one head per CTA, online softmax over key tiles
// of 32 from the first key the window of its rows reaches.
// Bound: fp32 FMA.
#include <algorithm>

#include "bf16_ops.cuh"

namespace fc {

namespace {
constexpr int QR = 16, KT = 32, KC = 64, PNT = 128, VCOLS = 2;     // value columns per thread: heads of at most 256
}
__global__ void __launch_bounds__(PNT) flash_f32_kernel(const Flash t, const float* __restrict__ qm, int M, int pos0, float* __restrict__ out, int ldo) {
    __shared__ float Qs[QR][KC + 1], Ks[KT][KC + 1], P[QR][KT + 1];
    __shared__ float corr_s[QR], l_s[QR];
    const int tid = threadIdx.x, h = blockIdx.y, row0 = (gridDim.x - 1 - blockIdx.x) * QR, kv = h / (t.H / t.KV);
    const int rows = min(QR, M - row0), last = pos0 + row0 + rows - 1;
    const int qi = tid >> 3, k8 = tid & 7, qpos = pos0 + row0 + qi;
    const int w0 = t.k0.width, kq = w0 + (t.k1.p ? t.k1.width : 0), first = max(0, pos0 + row0 - t.window + 1);
    // rows of position 0 (the base is subtracted as an index: rows ahead of the buffer are never touched)
    const float* k0p = (const float*)t.k0.p + t.k0.col + kv * t.k0.head_stride;
    const float* k1p = (const float*)t.k1.p + t.k1.col;
    const float* vp = (const float*)t.v.p + t.v.col + kv * t.v.head_stride;
    const float* bias = t.bias ? t.bias + (size_t)h * (t.far + 1) : nullptr;
    // the sink: weight exp(sink - m) = 1 so far, no key, no value; without one the maximum starts below every score
    float m = t.has_sink ? (t.sink ? t.sink[h] : 0.0f) : -1e30f, l = t.has_sink ? 1.0f : 0.0f;
    float acc[VCOLS][QR];
#pragma unroll
    for (int c = 0; c < VCOLS; ++c)
#pragma unroll
        for (int r = 0; r < QR; ++r) acc[c][r] = 0.0f;
    for (int k0 = first; k0 <= last; k0 += KT) {
        float s[4] = {0.0f, 0.0f, 0.0f, 0.0f};
        for (int e0 = 0; e0 < kq; e0 += KC) {
            __syncthreads();
            for (int i = tid; i < QR * KC; i += PNT) {
                const int r = i / KC, e = i - r * KC;
                Qs[r][e] = r < rows && e0 + e < kq ? qm[((size_t)(row0 + r) * t.H + h) * kq + e0 + e] : 0.0f;
            }
            for (int i = tid; i < KT * KC; i += PNT) {
                const int r = i / KC, e = i - r * KC, c = e0 + e;
                float x = 0.0f;
                if (k0 + r <= last && c < kq)
                    x = c < w0 ? k0p[(size_t)(k0 + r - t.k0.pos0) * t.k0.ld + c] : k1p[(size_t)(k0 + r - t.k1.pos0) * t.k1.ld + c - w0];
                Ks[r][e] = x;
            }
            __syncthreads();
#pragma unroll 8
            for (int e = 0; e < KC; ++e) {
                const float q = Qs[qi][e];
#pragma unroll
                for (int x = 0; x < 4; ++x) s[x] = fmaf(q, Ks[k8 + 8 * x][e], s[x]);
            }
        }
        float mx = -INFINITY;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const int n = qpos - (k0 + k8 + 8 * x);
            s[x] = n >= 0 && n < t.window ? s[x] + (bias ? bias[min(n, t.far)] : 0.0f) : -INFINITY;
            mx = fmaxf(mx, s[x]);
        }
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float mn = fmaxf(m, mx), corr = expf(m - mn);
        float ps = 0.0f;
#pragma unroll
        for (int x = 0; x < 4; ++x) {
            const float p = expf(s[x] - mn);
            P[qi][k8 + 8 * x] = p;
            ps += p;
        }
#pragma unroll
        for (int o = 4; o > 0; o >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
        l = fmaf(l, corr, ps);
        m = mn;
        if (k8 == 0) { corr_s[qi] = corr; l_s[qi] = l; }
        __syncthreads();
        const int nk = min(KT, last - k0 + 1);
#pragma unroll
        for (int c = 0; c < VCOLS; ++c) {
            const int col = tid + c * PNT;
            if (col >= t.vdim) continue;
#pragma unroll
            for (int r = 0; r < QR; ++r) acc[c][r] *= corr_s[r];
            const float* v = vp + (size_t)(k0 - t.v.pos0) * t.v.ld + col;
            for (int j = 0; j < nk; ++j) {
                const float x = v[(size_t)j * t.v.ld];
#pragma unroll
                for (int r = 0; r < QR; ++r) acc[c][r] = fmaf(P[r][j], x, acc[c][r]);
            }
        }
    }
    __syncthreads();
#pragma unroll
    for (int c = 0; c < VCOLS; ++c) {
        const int col = tid + c * PNT;
        if (col >= t.vdim) continue;
#pragma unroll
        for (int r = 0; r < QR; ++r)
            if (r < rows) out[(size_t)(row0 + r) * ldo + (size_t)h * t.vdim + col] = acc[c][r] / l_s[r];
    }
}
int launch_flash_f32(const Flash& f, const float* q, int M, int pos0, float* out, int ldo, cudaStream_t st) {
    if (f.vdim > VCOLS * PNT) return fail(FC_E_SHAPE, "value heads of %d: at most %d", f.vdim, VCOLS * PNT);
    flash_f32_kernel<<<dim3((M + QR - 1) / QR, f.H), PNT, 0, st>>>(f, q, M, pos0, out, ldo);
    FC_LAUNCHED();
    return FC_OK;
}

}  // namespace fc
