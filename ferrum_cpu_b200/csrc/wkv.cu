// Linear-attention state with per-channel decay (the RWKV form), over the tokens of a portion:
//     o_t = (S + diag(u) k_t v_t^T)^T r_t,     S <- diag(w_t) S + k_t v_t^T
// for every head, from the state an earlier portion left; everything is f32.
//
// A column j of S needs only v_t[j] and the row vectors r, k, w of the head, so columns are independent: a warp takes four
// columns of one head, its lanes the rows R l .. R l + R - 1 of all four in registers (one vector load per row vector
// serves them), four warps a CTA. The tokens' vectors come in chunks of 16 through double-buffered shared memory
// (cp.async), so the only chain from token to token is the state's own multiply-add. The partial sums of o (32 lanes, four
// columns) are exchanged for eight tokens at a time: 31 shuffles leave every lane with one finished value. Tokens past the
// end of the portion are filled in as k = v = r = 0, w = 1, which change nothing.
//
// Bound: issue (about 4 dim^2 operations per token and head) when heads x columns fill the GPU.
#include <algorithm>

#include "bf16_ops.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
constexpr int WARPS = 4, NT = WARPS * 32, COLS = WARPS * 4, CHUNK = 16;

__device__ __forceinline__ void cp4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(tc::s32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(tc::s32(dst)), "l"(src) : "memory");
}
template <int R>
__device__ __forceinline__ void ld_rows(float (&x)[R], const float* p) {
    if constexpr (R == 1) x[0] = *p;
    else if constexpr (R == 2) { const float2 a = *(const float2*)p; x[0] = a.x; x[1] = a.y; }
    else {
#pragma unroll
        for (int i = 0; i < R; i += 4) {
            const float4 a = *(const float4*)(p + i);
            x[i] = a.x; x[i + 1] = a.y; x[i + 2] = a.z; x[i + 3] = a.w;
        }
    }
}
}  // namespace

// R rows a lane (1, 2, 4, 8: heads of up to 32 R channels); VEC: 16-byte copies.
template <int R, bool VEC>
__global__ void __launch_bounds__(NT) wkv_scan_kernel(const float* __restrict__ r, const float* __restrict__ k, const float* __restrict__ v,
                                                      int ld, const float* __restrict__ w, int ldw, const float* __restrict__ u,
                                                      float* __restrict__ state, float* __restrict__ o, int ldo, int T, int dim) {
    constexpr int DP = 32 * R;
    extern __shared__ __align__(16) float sm[];     // [2][CHUNK][3][DP] r | k | w, then [2][CHUNK][COLS] v
    float* rows = sm;
    float* vs = sm + 2 * CHUNK * 3 * DP;
    const int tid = threadIdx.x, lane = tid & 31, wc = (tid >> 5) * 4, head = blockIdx.y, j0 = blockIdx.x * COLS + wc;
    const size_t h0 = (size_t)head * dim;
    for (int i = tid; i < 2 * CHUNK * (3 * DP + COLS); i += NT) sm[i] = 0.0f;    // rows and columns past dim stay zero
    __syncthreads();
    auto fetch = [&](int c) {                       // chunk c into buffer c & 1
        const int t0 = c * CHUNK, n = min(CHUNK, T - t0), b = c & 1;
        float* dst = rows + b * CHUNK * 3 * DP;
        constexpr int E = VEC ? 4 : 1;
#pragma unroll 4
        for (int i = tid; i < CHUNK * 3 * DP / E; i += NT) {
            const int t = i / (3 * DP / E), a = i / (DP / E) % 3, e = i % (DP / E) * E;
            if (e < dim) {
                const float* src = (a == 2 ? w + (size_t)(t0 + t) * ldw : (a == 1 ? k : r) + (size_t)(t0 + t) * ld) + h0 + e;
                float* to = dst + (t * 3 + a) * DP + e;
                const float fill = a == 2 ? 1.0f : 0.0f;
                if (t >= n) {
#pragma unroll
                    for (int x = 0; x < E; ++x) to[x] = fill;
                } else if constexpr (VEC) cp16(to, src);
                else cp4(to, src);
            }
        }
#pragma unroll
        for (int x = 0; x < CHUNK * COLS / NT; ++x) {
            const int i = tid + x * NT, t = i / COLS, e = i % COLS;
            if (blockIdx.x * COLS + e < dim) {
                if (t < n) cp4(vs + (b * CHUNK + t) * COLS + e, v + (size_t)(t0 + t) * ld + h0 + blockIdx.x * COLS + e);
                else vs[(b * CHUNK + t) * COLS + e] = 0.0f;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float S[R][4], ub[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int row = R * lane + i;
        ub[i] = row < dim ? u[h0 + row] : 0.0f;
#pragma unroll
        for (int c = 0; c < 4; ++c) S[i][c] = row < dim && j0 + c < dim ? state[(h0 + row) * dim + j0 + c] : 0.0f;
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
            float acc[32];                           // [token][column]
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                const float* p = rows + ((b * CHUNK + g + x) * 3) * DP + R * lane;
                float rr[R], kk[R], ww[R];
                ld_rows<R>(rr, p);
                ld_rows<R>(kk, p + DP);
                ld_rows<R>(ww, p + 2 * DP);
                const float4 v4 = *(const float4*)(vs + (b * CHUNK + g + x) * COLS + wc);
                const float vv[4] = {v4.x, v4.y, v4.z, v4.w};
#pragma unroll
                for (int cc = 0; cc < 4; ++cc) {
                    float s = 0.0f;
#pragma unroll
                    for (int i = 0; i < R; ++i) {
                        const float kv = kk[i] * vv[cc];
                        s = fmaf(rr[i], fmaf(ub[i], kv, S[i][cc]), s);
                        S[i][cc] = fmaf(ww[i], S[i][cc], kv);
                    }
                    acc[x * 4 + cc] = s;
                }
            }
            // lane l ends with the sum over all lanes of acc[l]
#pragma unroll
            for (int m = 16; m > 0; m >>= 1) {
                const bool up = lane & m;
#pragma unroll
                for (int x = 0; x < m; ++x) {
                    const float give = up ? acc[x] : acc[x + m], mine = up ? acc[x + m] : acc[x];
                    acc[x] = mine + __shfl_xor_sync(0xffffffffu, give, m);
                }
            }
            const int t = g + (lane >> 2), j = j0 + (lane & 3);
            if (t < n && j < dim) o[(size_t)(c * CHUNK + t) * ldo + h0 + j] = acc[0];
        }
        __syncthreads();                             // the buffer is filled again two chunks on
    }
#pragma unroll
    for (int i = 0; i < R; ++i)
#pragma unroll
        for (int c = 0; c < 4; ++c) {
            const int row = R * lane + i;
            if (row < dim && j0 + c < dim) state[(h0 + row) * dim + j0 + c] = S[i][c];
        }
}

int launch_wkv_scan(const float* r, const float* k, const float* v, int ld, const float* w, int ldw, const float* u, float* state, float* o,
                    int ldo, int M, int H, int dim, cudaStream_t st) {
    if (M <= 0 || H <= 0 || dim <= 0 || dim > 256) return fail(FC_E_SHAPE, "recurrence heads of %d channels (at most 256)", dim);
    const dim3 grid((dim + COLS - 1) / COLS, H);
    const int vec4 = dim % 4 == 0 && ld % 4 == 0 && ldw % 4 == 0 && aligned16(r) && aligned16(k) && aligned16(w);
    const int R = dim <= 32 ? 1 : (dim <= 64 ? 2 : (dim <= 128 ? 4 : 8));
    const size_t smem = (size_t)2 * CHUNK * (3 * 32 * R + COLS) * sizeof(float);
#define FC_SCAN2(MM, VV)                                                                                                                   \
    do {                                                                                                                                  \
        if (smem > 48 * 1024) FC_CUDA(cudaFuncSetAttribute(wkv_scan_kernel<MM, VV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem)); \
        wkv_scan_kernel<MM, VV><<<grid, NT, smem, st>>>(r, k, v, ld, w, ldw, u, state, o, ldo, M, dim);                                    \
    } while (0)
#define FC_SCAN(MM)                                   \
    case MM:                                          \
        if (vec4) FC_SCAN2(MM, true);                 \
        else FC_SCAN2(MM, false);                     \
        break;
    switch (R) {
        FC_SCAN(1) FC_SCAN(2) FC_SCAN(4) FC_SCAN(8)
    }
#undef FC_SCAN
#undef FC_SCAN2
    FC_LAUNCHED();
    return FC_OK;
}

// One warp per token and head: o / sqrt(mean(o^2) + eps) * norm * silu(gate).
template <class OT>
__global__ void __launch_bounds__(256) wkv_finish_kernel(const float* __restrict__ o, int ldo, const float* __restrict__ gate, int ldg,
                                                         const float* __restrict__ norm, float eps, int H, int dim, OT* __restrict__ y, int ldy) {
    const int lane = threadIdx.x & 31, row = blockIdx.x, h = blockIdx.y * 8 + (threadIdx.x >> 5);
    if (h >= H) return;
    const float* x = o + (size_t)row * ldo + (size_t)h * dim;
    const float* g = gate + (size_t)row * ldg + (size_t)h * dim;
    float xv[8], gv[8], s = 0.0f;                    // heads of at most 256 channels
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c < dim) { xv[i] = x[c]; gv[i] = g[c]; s = fmaf(xv[i], xv[i], s); }
    }
#pragma unroll
    for (int w = 16; w > 0; w >>= 1) s += __shfl_xor_sync(0xffffffffu, s, w);
    const float inv = 1.0f / sqrtf(s / (float)dim + eps);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int c = lane + 32 * i;
        if (c < dim) {
            const float v = xv[i] * inv * norm[h * dim + c] * (gv[i] / (1.0f + expf(-gv[i])));
            OT* d = y + (size_t)row * ldy + (size_t)h * dim + c;
            if constexpr (sizeof(OT) == 2) *d = __bfloat16_as_ushort(__float2bfloat16_rn(v));
            else *d = v;
        }
    }
}
int launch_wkv_finish(const float* o, int ldo, const float* gate, int ldg, const float* norm, float eps, int M, int H, int dim, void* y,
                      int ldy, bool f32, cudaStream_t st) {
    const dim3 grid(M, (H + 7) / 8);
    if (f32) wkv_finish_kernel<float><<<grid, 256, 0, st>>>(o, ldo, gate, ldg, norm, eps, H, dim, (float*)y, ldy);
    else wkv_finish_kernel<uint16_t><<<grid, 256, 0, st>>>(o, ldo, gate, ldg, norm, eps, H, dim, (uint16_t*)y, ldy);
    FC_LAUNCHED();
    return FC_OK;
}

}  // namespace fc
