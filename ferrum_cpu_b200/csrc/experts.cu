// Routing of feed-forwards that are cut into experts: which experts a token uses and with what weight, and the rows of a
// portion regrouped so that every expert's products read consecutive rows.
//
//   route_rows_kernel    8 tokens a CTA: logits in f32 (rows in shared memory, a warp holds four experts at a time,
//                        the block's halves every other 256 columns), softmax
//                        over all experts, the best groups (a group's score is its largest), the best experts in them; a slot's
//                        place within its expert from an atomic counter (the order of an expert's rows does not matter)
//   gather_rows_kernel   a CTA per token: places become rows (prefix sums of the counts), its operand row copied to each; the
//                        first CTA writes the table of row tiles
// The products themselves: launch_gemm_bf16_ragged. One token: launch_gemv_bf16_group, for the logits, the first matrices (whose
// launch chooses) and the second (whose rows run through all chosen experts).
//
// Bound: fp32 FMA (2 experts d FLOP per token) and L2; the gather HBM / L2.
#include <algorithm>

#include "route.cuh"

namespace fc {

namespace {
constexpr int NT = 256, RT = 512, TOK = 8, EPW = 4;      // tokens a CTA, experts a warp holds at once

// Place of column k in shared memory: within 256 values, lane l's eight are two float4 at 4 l and 128 + 4 l.
__device__ __forceinline__ int spot(int k) {
    const int e = k & 7;
    return (k & ~255) + ((k >> 3) & 31) * 4 + (e & 3) + (e & 4) * 32;
}
__device__ __forceinline__ void dot8(const uint4& w, const float4& u, const float4& v, float& s) {
    s = fmaf(__uint_as_float(w.x << 16), u.x, s); s = fmaf(__uint_as_float(w.x & 0xffff0000u), u.y, s);
    s = fmaf(__uint_as_float(w.y << 16), u.z, s); s = fmaf(__uint_as_float(w.y & 0xffff0000u), u.w, s);
    s = fmaf(__uint_as_float(w.z << 16), v.x, s); s = fmaf(__uint_as_float(w.z & 0xffff0000u), v.y, s);
    s = fmaf(__uint_as_float(w.w << 16), v.z, s); s = fmaf(__uint_as_float(w.w & 0xffff0000u), v.w, s);
}
// Sums over the warp of 32 values a lane holds: lane i receives value i's.
__device__ __forceinline__ float warp_sums32(float (&v)[32]) {
    const int lane = threadIdx.x & 31;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const bool up = lane & o;
#pragma unroll
        for (int i = 0; i < o; ++i) {
            const float mine = up ? v[i + o] : v[i], other = up ? v[i] : v[i + o];
            v[i] = mine + __shfl_xor_sync(0xffffffffu, other, o);
        }
    }
    return v[0];
}
}  // namespace

__global__ void __launch_bounds__(RT) route_rows_kernel(const RouteRows p, int kc) {
    extern __shared__ __align__(16) float sm[];              // x [TOK][kc] | z of either half [TOK][experts] | groups [TOK][groups]
    const int tid = threadIdx.x, lane = tid & 31, half = tid / (RT / 2), warp = (tid >> 5) % (RT / 64), E = p.r.experts, t0 = blockIdx.x * TOK, nt = min(TOK, p.M - t0);
    float* xs = sm;
    float* z = sm + TOK * kc;
    float* gs = z + 2 * TOK * E;
    for (int i = tid; i < 2 * TOK * E; i += RT) z[i] = 0.0f;
    const bool vec = p.d % 4 == 0;
    for (int k0 = 0; k0 < p.r.ld; k0 += kc) {                // all columns at once where they fit
        __syncthreads();
        for (int t = 0; t < TOK; ++t) {
            const float* x = p.x + (size_t)(t0 + t) * p.d;
            if (vec) {
#pragma unroll 4
                for (int k = tid * 4; k < kc; k += RT * 4)
                    *(float4*)(xs + t * kc + spot(k)) = t < nt && k0 + k < p.d ? *(const float4*)(x + k0 + k) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            } else {
                for (int k = tid; k < kc; k += RT) xs[t * kc + spot(k)] = t < nt && k0 + k < p.d ? x[k0 + k] : 0.0f;
            }
        }
        __syncthreads();
        for (int e0 = warp * EPW; e0 < E; e0 += RT / 64 * EPW) {
            float s[EPW * TOK] = {};
#pragma unroll 2
            for (int c = half * 256; c < kc; c += 512) {          // the halves of the block take turns
                const int k = k0 + c + lane * 8;
                uint4 w[EPW];
#pragma unroll
                for (int y = 0; y < EPW; ++y)
                    w[y] = e0 + y < E && k < p.r.ld ? __ldg((const uint4*)(p.r.w + (size_t)(e0 + y) * p.r.ld + k)) : make_uint4(0, 0, 0, 0);
#pragma unroll
                for (int t = 0; t < TOK; ++t) {
                    const float4 u = *(const float4*)(xs + t * kc + c + lane * 4), v = *(const float4*)(xs + t * kc + c + lane * 4 + 128);
#pragma unroll
                    for (int y = 0; y < EPW; ++y) dot8(w[y], u, v, s[y * TOK + t]);
                }
            }
            static_assert(EPW * TOK == 32, "a sum a lane");
            const float v = warp_sums32(s);
            if (e0 + lane / TOK < E) z[(half * TOK + lane % TOK) * E + e0 + lane / TOK] += v;
        }
    }
    __syncthreads();
    for (int i = tid; i < TOK * E; i += RT) z[i] += z[TOK * E + i];
    __syncthreads();
    const int t = warp;
    if (half == 0 && t < nt)
        choose(z + t * E, gs + t * p.r.groups, p.r, [&](int k, int e, float w) {
            const size_t at = (size_t)(t0 + t) * p.r.top + k;
            p.expert[at] = e;
            p.weight[at] = w;
            p.index[at] = atomicAdd(p.counts + e, 1);
        });
}

__global__ void __launch_bounds__(NT) gather_rows_kernel(const RouteRows p, const unsigned char* __restrict__ plane, int row16) {
    extern __shared__ int off[];                             // first row of every expert's run
    __shared__ int place[64];
    const int tid = threadIdx.x, lane = tid & 31, E = p.r.experts, m = blockIdx.x, top = p.r.top;
    const int per = (E + 31) / 32;
    if (tid < 32) {                                          // a lane sums `per` neighbouring experts
        int n = 0;
        for (int i = lane * per; i < min(E, (lane + 1) * per); ++i) n += p.counts[i];
        int at = n;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int x = __shfl_up_sync(0xffffffffu, at, o);
            if (lane >= o) at += x;
        }
        at -= n;
        for (int i = lane * per; i < min(E, (lane + 1) * per); ++i) { off[i] = at; at += p.counts[i]; }
    }
    __syncthreads();
    if (m == 0 && tid < 32) {
        int n = 0;
        for (int i = lane * per; i < min(E, (lane + 1) * per); ++i) n += (p.counts[i] + p.tile_rows - 1) / p.tile_rows;
        int at = n;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int x = __shfl_up_sync(0xffffffffu, at, o);
            if (lane >= o) at += x;
        }
        if (lane == 31) *p.n_table = at;
        at -= n;
        for (int i = lane * per; i < min(E, (lane + 1) * per); ++i)
            for (int r = 0; r < p.counts[i]; r += p.tile_rows) p.table[at++] = make_int4(off[i] + r, min(p.tile_rows, p.counts[i] - r), i, 0);
    }
    for (int s = tid; s < top; s += NT) {
        const size_t at = (size_t)m * top + s;
        const int row = off[p.expert[at]] + p.index[at];
        p.index[at] = row;
        place[s] = row;
    }
    __syncthreads();
    const uint4* src = (const uint4*)(plane + (size_t)m * row16 * 16);
    uint4* dst = (uint4*)p.rows;
    for (int i = tid; i < row16; i += NT) {
        const uint4 v = src[i];
        for (int s = 0; s < top; ++s) dst[(size_t)place[s] * row16 + i] = v;
    }
}

int max_row_tiles(const Router& r, int M, int tile_rows) {
    const long long rows = (long long)M * r.top;
    return (int)std::min<long long>(rows, rows / tile_rows + r.experts);
}
int launch_route_rows(const RouteRows& p, const void* plane, bool f32_rows, cudaStream_t st) {
    const Router& r = p.r;
    if (r.experts > kMaxExperts || r.groups > kMaxGroups || r.top > 64) return fail(FC_E_SHAPE, "%d experts in %d groups, %d chosen", r.experts, r.groups, r.top);
    const int rest = TOK * (2 * r.experts + r.groups) * 4, kc = std::min(pad_to(r.ld, 256), (200 * 1024 - rest) / (TOK * 4) / 256 * 256);
    const size_t smem = (size_t)TOK * kc * 4 + rest;
    if (smem > 47 * 1024) FC_CUDA(cudaFuncSetAttribute(route_rows_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    route_rows_kernel<<<(p.M + TOK - 1) / TOK, RT, smem, st>>>(p, kc);
    FC_LAUNCHED();
    gather_rows_kernel<<<p.M, NT, (size_t)r.experts * sizeof(int), st>>>(p, (const unsigned char*)plane, p.ld * (f32_rows ? 4 : 2) / 16);
    FC_LAUNCHED();
    return FC_OK;
}

}  // namespace fc
