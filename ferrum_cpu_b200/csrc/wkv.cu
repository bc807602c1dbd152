// Linear-attention state with per-channel decay (the RWKV form), over the tokens of a portion:
//     o_t = (S + diag(u) k_t v_t^T)^T r_t,     S <- diag(w_t) S + k_t v_t^T
// for every head, from the state an earlier portion left; everything is f32.
//
// A column j of S needs only v_t[j] and the row vectors r, k, w of the head, so columns are independent: a CTA takes 16
// columns of one head, eight lanes a column, each lane the rows 32 m + 4 l + e (m < M, e < 4) in registers. The tokens'
// vectors come in chunks of 16 through double-buffered shared memory (cp.async), so the only chain from token to token
// is the state's own multiply-add. The eight partial sums of o are exchanged for eight tokens at a time: seven shuffles
// leave lane l with token l's sum.
//
// Bound: issue (about 4 * dim * dim operations per token and head), latency when heads x columns do not fill the GPU.
#include <algorithm>

#include "bf16_ops.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
constexpr int COLS = 16, LANES = 8, NT = COLS * LANES, CHUNK = 16;

__device__ __forceinline__ void cp4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(tc::s32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(tc::s32(dst)), "l"(src) : "memory");
}
}  // namespace

template <int M>
__global__ void __launch_bounds__(NT) wkv_scan_kernel(const float* __restrict__ r, const float* __restrict__ k, const float* __restrict__ v,
                                                      int ld, const float* __restrict__ w, int ldw, const float* __restrict__ u,
                                                      float* __restrict__ state, float* __restrict__ o, int ldo, int T, int dim, int vec4) {
    constexpr int DP = 32 * M;
    extern __shared__ __align__(16) float sm[];     // [2][CHUNK][3][DP] r | k | w, then [2][CHUNK][COLS] v
    float* rows = sm;
    float* vs = sm + 2 * CHUNK * 3 * DP;
    const int tid = threadIdx.x, l = tid & 7, col = tid >> 3, head = blockIdx.y, j = blockIdx.x * COLS + col;
    const size_t h0 = (size_t)head * dim;
    for (int i = tid; i < 2 * CHUNK * (3 * DP + COLS); i += NT) sm[i] = 0.0f;    // rows and columns past dim stay zero
    __syncthreads();
    auto fetch = [&](int c) {                       // chunk c into buffer c & 1
        const int t0 = c * CHUNK, n = min(CHUNK, T - t0), b = c & 1;
        if (vec4) {
            const int q = dim >> 2;
            for (int i = tid; i < n * 3 * q; i += NT) {
                const int t = i / (3 * q), x = i - t * 3 * q, a = x / q, e = (x - a * q) * 4;
                const float* src = a == 2 ? w + (size_t)(t0 + t) * ldw : (a == 1 ? k : r) + (size_t)(t0 + t) * ld;
                cp16(rows + ((b * CHUNK + t) * 3 + a) * DP + e, src + h0 + e);
            }
        } else {
            for (int i = tid; i < n * 3 * dim; i += NT) {
                const int t = i / (3 * dim), x = i - t * 3 * dim, a = x / dim, e = x - a * dim;
                const float* src = a == 2 ? w + (size_t)(t0 + t) * ldw : (a == 1 ? k : r) + (size_t)(t0 + t) * ld;
                cp4(rows + ((b * CHUNK + t) * 3 + a) * DP + e, src + h0 + e);
            }
        }
        for (int i = tid; i < n * COLS; i += NT) {
            const int t = i / COLS, e = i - t * COLS;
            if (blockIdx.x * COLS + e < dim) cp4(vs + (b * CHUNK + t) * COLS + e, v + (size_t)(t0 + t) * ld + h0 + blockIdx.x * COLS + e);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float S[4 * M], ub[4 * M];
#pragma unroll
    for (int m = 0; m < M; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 32 * m + 4 * l + e;
            const bool in = i < dim;
            S[4 * m + e] = in && j < dim ? state[(h0 + i) * dim + j] : 0.0f;
            ub[4 * m + e] = in ? u[h0 + i] : 0.0f;
        }
    const int n_chunks = (T + CHUNK - 1) / CHUNK;
    fetch(0);
    for (int c = 0; c < n_chunks; ++c) {
        if (c + 1 < n_chunks) {
            fetch(c + 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const int n = min(CHUNK, T - c * CHUNK), b = c & 1;
#pragma unroll 1
        for (int g = 0; g < n; g += 8) {
            float acc[8];
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                acc[x] = 0.0f;
                if (g + x < n) {                     // uniform over the block
                    const float* p = rows + ((b * CHUNK + g + x) * 3) * DP + 4 * l;
                    const float vv = vs[(b * CHUNK + g + x) * COLS + col];
#pragma unroll
                    for (int m = 0; m < M; ++m) {
                        const float4 rr = *(const float4*)(p + 32 * m), kk = *(const float4*)(p + DP + 32 * m),
                                     ww = *(const float4*)(p + 2 * DP + 32 * m);
                        const float r4[4] = {rr.x, rr.y, rr.z, rr.w}, k4[4] = {kk.x, kk.y, kk.z, kk.w}, w4[4] = {ww.x, ww.y, ww.z, ww.w};
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const float kv = k4[e] * vv;
                            acc[x] = fmaf(r4[e], fmaf(ub[4 * m + e], kv, S[4 * m + e]), acc[x]);
                            S[4 * m + e] = fmaf(w4[e], S[4 * m + e], kv);
                        }
                    }
                }
            }
            // lane l ends with the sum over the eight lanes of acc[l]
#pragma unroll
            for (int x = 0; x < 4; ++x) {
                const bool up = l & 4;
                const float give = up ? acc[x] : acc[x + 4], keep = up ? acc[x + 4] : acc[x];
                acc[x] = keep + __shfl_xor_sync(0xffffffffu, give, 4);
            }
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const bool up = l & 2;
                const float give = up ? acc[x] : acc[x + 2], keep = up ? acc[x + 2] : acc[x];
                acc[x] = keep + __shfl_xor_sync(0xffffffffu, give, 2);
            }
            const bool up = l & 1;
            const float give = up ? acc[0] : acc[1], keep = up ? acc[1] : acc[0];
            const float s = keep + __shfl_xor_sync(0xffffffffu, give, 1);
            if (g + l < n && j < dim) o[(size_t)(c * CHUNK + g + l) * ldo + h0 + j] = s;
        }
        __syncthreads();                             // the buffer is filled again two chunks on
    }
#pragma unroll
    for (int m = 0; m < M; ++m)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int i = 32 * m + 4 * l + e;
            if (i < dim && j < dim) state[(h0 + i) * dim + j] = S[4 * m + e];
        }
}

int launch_wkv_scan(const float* r, const float* k, const float* v, int ld, const float* w, int ldw, const float* u, float* state, float* o,
                    int ldo, int M, int H, int dim, cudaStream_t st) {
    if (M <= 0 || H <= 0 || dim <= 0 || dim > 256) return fail(FC_E_SHAPE, "recurrence heads of %d channels (at most 256)", dim);
    const dim3 grid((dim + COLS - 1) / COLS, H);
    const int vec4 = dim % 4 == 0 && ld % 4 == 0 && ldw % 4 == 0 && aligned16(r) && aligned16(k) && aligned16(w);
    const int m = (dim + 31) / 32;
    const size_t smem = (size_t)2 * CHUNK * (3 * 32 * m + COLS) * sizeof(float);
#define FC_SCAN(MM)                                                                                                                  \
    case MM:                                                                                                                         \
        if (smem > 48 * 1024) FC_CUDA(cudaFuncSetAttribute(wkv_scan_kernel<MM>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        wkv_scan_kernel<MM><<<grid, NT, smem, st>>>(r, k, v, ld, w, ldw, u, state, o, ldo, M, dim, vec4);                             \
        break;
    switch (m) {
        FC_SCAN(1) FC_SCAN(2) FC_SCAN(3) FC_SCAN(4) FC_SCAN(5) FC_SCAN(6) FC_SCAN(7) FC_SCAN(8)
    }
#undef FC_SCAN
    FC_LAUNCHED();
    return FC_OK;
}

// One CTA per token, one warp per head: o / sqrt(mean(o^2) + eps) * norm * silu(gate).
template <class OT>
__global__ void __launch_bounds__(256) wkv_finish_kernel(const float* __restrict__ o, int ldo, const float* __restrict__ gate, int ldg,
                                                         const float* __restrict__ norm, float eps, int H, int dim, OT* __restrict__ y, int ldy) {
    const int lane = threadIdx.x & 31, row = blockIdx.x;
    for (int h = threadIdx.x >> 5; h < H; h += 8) {
        const float* x = o + (size_t)row * ldo + (size_t)h * dim;
        const float* g = gate + (size_t)row * ldg + (size_t)h * dim;
        float s = 0.0f;
        for (int c = lane; c < dim; c += 32) s = fmaf(x[c], x[c], s);
#pragma unroll
        for (int w = 16; w > 0; w >>= 1) s += __shfl_xor_sync(0xffffffffu, s, w);
        const float inv = 1.0f / sqrtf(s / (float)dim + eps);
        for (int c = lane; c < dim; c += 32) {
            const float z = g[c], v = x[c] * inv * norm[h * dim + c] * (z / (1.0f + expf(-z)));
            OT* d = y + (size_t)row * ldy + (size_t)h * dim + c;
            if constexpr (sizeof(OT) == 2) *d = __bfloat16_as_ushort(__float2bfloat16_rn(v));
            else *d = v;
        }
    }
}
int launch_wkv_finish(const float* o, int ldo, const float* gate, int ldg, const float* norm, float eps, int M, int H, int dim, void* y,
                      int ldy, bool f32, cudaStream_t st) {
    if (f32) wkv_finish_kernel<float><<<M, 256, 0, st>>>(o, ldo, gate, ldg, norm, eps, H, dim, (float*)y, ldy);
    else wkv_finish_kernel<uint16_t><<<M, 256, 0, st>>>(o, ldo, gate, ldg, norm, eps, H, dim, (uint16_t*)y, ldy);
    FC_LAUNCHED();
    return FC_OK;
}

}  // namespace fc
