// Linear-attention state with per-channel decay (the RWKV form), over the tokens of a portion:
//     o_t = (S + diag(u) k_t v_t^T)^T r_t,     S <- diag(w_t) S + k_t v_t^T
// for every head, from the state an earlier portion left; everything is f32.
//
// A column j of S needs only v_t[j] and the row vectors r, k, w of the head, so columns are independent: 16 lanes take two
// columns of one head, each lane R rows of both in registers (one set of vector loads per row vector serves them), four warps
// a CTA. The tokens' vectors come in chunks of 16 through double-buffered shared memory (cp.async), so the only chain from
// token to token is the state's own multiply-add. The partial sums of o are exchanged for eight tokens at a time: 15
// shuffles leave every lane with one finished value. Tokens past the end are filled in as k = v = r = 0, w = 1, which change
// nothing.
//
// Long portions are cut into segments that run side by side: a first pass leaves each segment's state from zero and the
// product of its decays, a small kernel chains them (S <- P S + E), and the second pass starts every segment from its own
// state and writes o.
//
// Bound: issue (about 4 dim^2 operations per token and head, half of that again for the first pass).
#include <algorithm>

#include "bf16_ops.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
constexpr int WARPS = 4, NT = WARPS * 32, COLS = WARPS * 4, CHUNK = 16, SEG_MIN = 64;

__device__ __forceinline__ void cp4(void* dst, const void* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(tc::s32(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(tc::s32(dst)), "l"(src) : "memory");
}
// Row i of lane l: 2 l + i for two rows a lane, else 64 (i / 4) + 4 l + i % 4.
template <int R>
__device__ __forceinline__ int row_of(int l, int i) { return R == 2 ? 2 * l + i : 64 * (i >> 2) + 4 * l + (i & 3); }
template <int R>
__device__ __forceinline__ void ld_rows(float (&x)[R], const float* p, int l) {
    if constexpr (R == 2) { const float2 a = *(const float2*)(p + 2 * l); x[0] = a.x; x[1] = a.y; }
    else {
#pragma unroll
        for (int i = 0; i < R; i += 4) {
            const float4 a = *(const float4*)(p + 16 * i + 4 * l);
            x[i] = a.x; x[i + 1] = a.y; x[i + 2] = a.z; x[i + 3] = a.w;
        }
    }
}
struct ScanArgs {
    const float *r, *k, *v;
    int ld;
    const float* w;
    int ldw;
    const float* u;
    float* state;        // [H][dim][dim]
    float* o;
    int ldo, T, dim;
    int seg;             // tokens of a segment
    float *ein, *prod;   // more than one segment: [segments][H][dim][dim] states at their starts, [segments][H][dim] decays
};
}  // namespace

// R rows a lane (heads of up to 16 R channels); VEC: 16-byte copies; LOCAL: the first pass.
template <int R, bool VEC, bool LOCAL>
__global__ void __launch_bounds__(NT) wkv_scan_kernel(const ScanArgs a) {
    constexpr int DP = 16 * R;
    extern __shared__ __align__(16) float sm[];     // [2][CHUNK][3][DP] r | k | w, then [2][CHUNK][COLS] v
    float* rows = sm;
    float* vs = sm + 2 * CHUNK * 3 * DP;
    const int tid = threadIdx.x, lane = tid & 31, l = lane & 15, wc = (tid >> 4) * 2, head = blockIdx.y, H = gridDim.y, s = blockIdx.z;
    const int dim = a.dim, j0 = blockIdx.x * COLS + wc, first = s * a.seg, T = min(a.seg, a.T - first);
    const size_t h0 = (size_t)head * dim, sd = (size_t)H * dim * dim;
    for (int i = tid; i < 2 * CHUNK * (3 * DP + COLS); i += NT) sm[i] = 0.0f;    // rows and columns past dim stay zero
    __syncthreads();
    auto fetch = [&](int c) {                       // chunk c into buffer c & 1
        const int t0 = c * CHUNK, n = min(CHUNK, T - t0), b = c & 1;
        float* dst = rows + b * CHUNK * 3 * DP;
        constexpr int E = VEC ? 4 : 1, Q = DP / E;
#pragma unroll 4
        for (int i = tid; i < CHUNK * 3 * Q; i += NT) {
            const int t = i / (3 * Q), x = i / Q % 3, e = i % Q * E;
            if (LOCAL && x == 0) continue;
            if (e < dim) {
                const size_t at = (size_t)(first + t0 + t);
                const float* src = (x == 2 ? a.w + at * a.ldw : (x == 1 ? a.k : a.r) + at * a.ld) + h0 + e;
                float* to = dst + (t * 3 + x) * DP + e;
                if (t >= n) {
#pragma unroll
                    for (int y = 0; y < E; ++y) to[y] = x == 2 ? 1.0f : 0.0f;
                } else if constexpr (VEC) cp16(to, src);
                else cp4(to, src);
            }
        }
#pragma unroll
        for (int x = 0; x < CHUNK * COLS / NT; ++x) {
            const int i = tid + x * NT, t = i / COLS, e = i % COLS;
            if (blockIdx.x * COLS + e < dim) {
                if (t < n) cp4(vs + (b * CHUNK + t) * COLS + e, a.v + (size_t)(first + t0 + t) * a.ld + h0 + blockIdx.x * COLS + e);
                else vs[(b * CHUNK + t) * COLS + e] = 0.0f;
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    const float* from = a.ein ? a.ein + (size_t)s * sd : a.state;
    float S[R][2], ub[R], prod[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int row = row_of<R>(l, i);
        prod[i] = 1.0f;
        ub[i] = !LOCAL && row < dim ? a.u[h0 + row] : 0.0f;
#pragma unroll
        for (int c = 0; c < 2; ++c) S[i][c] = !LOCAL && row < dim && j0 + c < dim ? from[(h0 + row) * dim + j0 + c] : 0.0f;
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
            float acc[16];                           // [token][column]
#pragma unroll
            for (int x = 0; x < 8; ++x) {
                const float* p = rows + ((b * CHUNK + g + x) * 3) * DP;
                float rr[R], kk[R], ww[R];
                if (!LOCAL) ld_rows<R>(rr, p, l);
                ld_rows<R>(kk, p + DP, l);
                ld_rows<R>(ww, p + 2 * DP, l);
                const float2 v2 = *(const float2*)(vs + (b * CHUNK + g + x) * COLS + wc);
                const float vv[2] = {v2.x, v2.y};
#pragma unroll
                for (int cc = 0; cc < 2; ++cc) {
                    float y = 0.0f;
#pragma unroll
                    for (int i = 0; i < R; ++i) {
                        const float kv = kk[i] * vv[cc];
                        if (!LOCAL) y = fmaf(rr[i], fmaf(ub[i], kv, S[i][cc]), y);
                        S[i][cc] = fmaf(ww[i], S[i][cc], kv);
                    }
                    acc[x * 2 + cc] = y;
                }
                if (LOCAL)
#pragma unroll
                    for (int i = 0; i < R; ++i) prod[i] *= ww[i];
            }
            if (!LOCAL) {
                // lane l of 16 ends with the sum over them of acc[l]
#pragma unroll
                for (int m = 8; m > 0; m >>= 1) {
                    const bool up = lane & m;
#pragma unroll
                    for (int x = 0; x < m; ++x) {
                        const float give = up ? acc[x] : acc[x + m], mine = up ? acc[x + m] : acc[x];
                        acc[x] = mine + __shfl_xor_sync(0xffffffffu, give, m);
                    }
                }
                const int t = g + (l >> 1), j = j0 + (l & 1);
                if (t < n && j < dim) a.o[(size_t)(first + c * CHUNK + t) * a.ldo + h0 + j] = acc[0];
            }
        }
        __syncthreads();                             // the buffer is filled again two chunks on
    }
    if (!LOCAL && s + 1 < (int)gridDim.z) return;    // only the last segment leaves the portion's state
    float* to = LOCAL ? a.ein + (size_t)(s + 1) * sd : a.state;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int row = row_of<R>(l, i);
#pragma unroll
        for (int c = 0; c < 2; ++c)
            if (row < dim && j0 + c < dim) to[(h0 + row) * dim + j0 + c] = S[i][c];
        if (LOCAL && blockIdx.x == 0 && tid < 16 && row < dim) a.prod[(size_t)s * H * dim + h0 + row] = prod[i];
    }
}

// States at the starts of the segments: ein[0] = state, ein[s + 1] = prod[s] ein[s] + (what the first pass left there).
__global__ void __launch_bounds__(256) wkv_chain_kernel(const float* __restrict__ state, float* __restrict__ ein, const float* __restrict__ prod,
                                                        int n_seg, int rows, int dim) {
    const size_t i = (size_t)blockIdx.x * 256 + threadIdx.x, n = (size_t)rows * dim;
    if (i >= n) return;
    float S = state[i];
    ein[i] = S;
    for (int s = 0; s + 1 < n_seg; ++s) {
        S = fmaf(prod[(size_t)s * rows + i / dim], S, ein[(size_t)(s + 1) * n + i]);
        ein[(size_t)(s + 1) * n + i] = S;
    }
}

template <int R, bool VEC>
static int scan(ScanArgs a, int H, int n_seg, cudaStream_t st) {
    const size_t smem = (size_t)2 * CHUNK * (3 * 16 * R + COLS) * sizeof(float);
    if (smem > 47 * 1024) {
        FC_CUDA(cudaFuncSetAttribute(wkv_scan_kernel<R, VEC, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
        FC_CUDA(cudaFuncSetAttribute(wkv_scan_kernel<R, VEC, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    }
    const int cols = (a.dim + COLS - 1) / COLS;
    if (n_seg > 1) {
        wkv_scan_kernel<R, VEC, true><<<dim3(cols, H, n_seg - 1), NT, smem, st>>>(a);
        FC_LAUNCHED();
        const size_t n = (size_t)H * a.dim * a.dim;
        wkv_chain_kernel<<<(unsigned)((n + 255) / 256), 256, 0, st>>>(a.state, a.ein, a.prod, n_seg, H * a.dim, a.dim);
        FC_LAUNCHED();
    } else {
        a.ein = nullptr;
    }
    wkv_scan_kernel<R, VEC, false><<<dim3(cols, H, n_seg), NT, smem, st>>>(a);
    FC_LAUNCHED();
    return FC_OK;
}

size_t wkv_scratch_floats(int H, int dim) { return (size_t)kWkvSegments * H * dim * (dim + 1); }

int launch_wkv_scan(const float* r, const float* k, const float* v, int ld, const float* w, int ldw, const float* u, float* state, float* o,
                    int ldo, int M, int H, int dim, float* scratch, cudaStream_t st) {
    if (M <= 0 || H <= 0 || dim <= 0 || dim > 256) return fail(FC_E_SHAPE, "recurrence heads of %d channels (at most 256)", dim);
    // as many segments as give every scheduler of the GPU about four warps
    int n_seg = std::min({kWkvSegments, M / SEG_MIN, (148 * 16 + H * ((dim + 3) / 4) - 1) / (H * ((dim + 3) / 4))});
    n_seg = std::max(n_seg, 1);
    ScanArgs a = {r, k, v, ld, w, ldw, u, state, o, ldo, M, dim, 0, scratch, scratch + (size_t)kWkvSegments * H * dim * dim};
    a.seg = pad_to((M + n_seg - 1) / n_seg, CHUNK);
    n_seg = (M + a.seg - 1) / a.seg;
    const bool vec = dim % 4 == 0 && ld % 4 == 0 && ldw % 4 == 0 && aligned16(r) && aligned16(k) && aligned16(w);
    if (dim <= 32) return vec ? scan<2, true>(a, H, n_seg, st) : scan<2, false>(a, H, n_seg, st);
    if (dim <= 64) return vec ? scan<4, true>(a, H, n_seg, st) : scan<4, false>(a, H, n_seg, st);
    if (dim <= 128) return vec ? scan<8, true>(a, H, n_seg, st) : scan<8, false>(a, H, n_seg, st);
    return vec ? scan<16, true>(a, H, n_seg, st) : scan<16, false>(a, H, n_seg, st);
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
