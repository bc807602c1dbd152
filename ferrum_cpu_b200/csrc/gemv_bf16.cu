// Several products of one activation row in one launch, on bf16 weights: the decode counterpart of the grouped GEMM.
//
// The rows of all segments form one list that is cut into equal shares of bytes, one persistent CTA of 16 warps per SM.
// A warp takes pieces of 2048 weights, two in flight: a row (or a K slice given as a segment of its own) that is longer takes
// several, of rows of at most 1024, 512 or 256 weights a piece holds 2, 4 or 8. 16-byte loads, activations f32 in shared
// memory, f32 sums. A segment's rows may begin at an index read from the device (an expert chosen there).
// Launched as a programmatic dependent: the first two pieces of every warp are requested before the wait on the kernel
// ahead, since weights never change.
//
// Prologues: plain inputs; the residual of layers that norm what they add (and a norm of it); or the residual update of the
// layer before, the norm and the token-shift mixes of the row (every CTA computes them for itself, CTA 0 stores the residual and the token-shift row); or residual and norm alone
// (the head). The residual alternates between two buffers and the token-shift row between two slots (by the position's
// parity), so that no CTA overwrites what another still reads.
//
// Bound: HBM (2 bytes per weight).
#include <algorithm>

#include "bf16_ops.cuh"
#include "pdl.cuh"
#include "post_norm.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
constexpr int NW = 16, NT = NW * 32;
constexpr int PIECE = 2048;               // weights of a row per register piece: 8 loads of 16 bytes per lane

__device__ __forceinline__ uint4 ld_stream(const uint16_t* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];"
                 : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
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
    for (int w = 1; w < NW; ++w) { t.x += red[w].x; t.y += red[w].y; }
    return t;
}
// Place of activation k in shared memory: within 256 values, lane l's eight are two float4 at 4 l and 128 + 4 l.
__device__ __forceinline__ int spot(int k) {
    const int e = k & 7;
    return (k & ~255) + ((k >> 3) & 31) * 4 + (e & 3) + (e & 4) * 32;
}
struct Piece { uint4 w[8]; };
template <int V> struct Const { static constexpr int value = V; };

// This CTA's rows of segment s, repetitions one after the other: [first, last). Costs are counted in 64 weights.
__device__ __forceinline__ void share(const GemvGroup& g, int s, int lo, int hi, int* first, int* last) {
    const int cost = g.seg[s].cost, rows = g.seg[s].n * max(1, g.seg[s].reps), a = lo - g.seg[s].cost0, b = hi - g.seg[s].cost0;
    *first = *last = 0;
    if (b <= 0 || a >= rows * cost) return;
    *first = a <= 0 ? 0 : (a + cost - 1) / cost;
    *last = min((b + cost - 1) / cost, rows);
}
}  // namespace

__global__ void __launch_bounds__(NT, 1) gemv_bf16_group_kernel(const __grid_constant__ GemvGroup g, int x_cap) {
    extern __shared__ __align__(16) float sm[];    // staged input [x_cap] | h [d] | token-shift row [d]
    __shared__ float2 red[NW];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, d = g.d;
    float* xs = sm;
    float* hs = sm + x_cap;
    float* hp = hs + d;

    auto bound = [&](int b) { return g.share * b + g.rest * b / (int)gridDim.x; };
    const int lo = bound(blockIdx.x), hi = bound(blockIdx.x + 1);
    int cur = 0, lim = 0, seg = 0;                 // rows cur .. lim - 1 of segment seg are still to do
    int rep = 0, row = 0, end = 0;                 // of these, rows row + warp, + NW, ... < end of repetition rep now
    auto seek = [&]() {
        for (; seg < g.n_seg; ++seg) {
            share(g, seg, lo, hi, &cur, &lim);
            if (cur < lim) break;
        }
    };
    const uint16_t* base = nullptr;
    int ldw = 0, K_pad = 0, pieces = 1, lc = 3, items = 0;    // a piece holds 8 >> lc rows of 1 << lc loads of 256 weights
    bool ready = false;                            // past the wait: indices may be read
    auto open = [&]() {
        items = 0;
        if (seg >= g.n_seg) return;
        const GemvSeg& s = g.seg[seg];
        rep = cur / s.n;
        row = cur - rep * s.n;
        end = min(s.n, row + lim - cur);
        ldw = s.ldw;
        K_pad = s.K_pad;
        pieces = (K_pad + PIECE - 1) / PIECE;
        lc = K_pad > 1024 ? 3 : (K_pad > 512 ? 2 : (K_pad > 256 ? 1 : 0));
        const int rp = 8 >> lc, mine = end - row - warp * rp;
        if (s.index && !s.early && !ready) return;             // loaded after the wait
        base = s.w + (size_t)row * ldw;
        if (s.index) base += (size_t)s.index[rep] * s.w_step;
        items = mine > 0 ? (mine + NW * rp - 1) / (NW * rp) * pieces : 0;
    };
    // item i: piece i % pieces of the rows from (warp + (i / pieces) NW) rp on; LC is lc as a constant
    auto load = [&](auto LC, Piece& p, int i) {
        constexpr int L = decltype(LC)::value, RP = 8 >> L;
        if constexpr (RP == 1) {
            const int ri = i / pieces, k0 = (i - ri * pieces) * PIECE + lane * 8;
            const uint16_t* src = base + (size_t)(warp + ri * NW) * ldw;
#pragma unroll
            for (int c = 0; c < 8; ++c) p.w[c] = i < items && k0 + c * 256 < K_pad ? ld_stream(src + k0 + c * 256) : make_uint4(0, 0, 0, 0);
        } else {                                   // such rows are one piece long
            const int r0 = (warp + i * NW) * RP, rows = end - row - r0, k0 = lane * 8;
            const uint16_t* src = base + (size_t)r0 * ldw;
#pragma unroll
            for (int q = 0; q < RP; ++q, src += ldw)
#pragma unroll
                for (int c = 0; c < 8 / RP; ++c)
                    p.w[q * (8 / RP) + c] = i < items && q < rows && k0 + c * 256 < K_pad ? ld_stream(src + k0 + c * 256) : make_uint4(0, 0, 0, 0);
        }
    };
    auto by_length = [&](auto f) {
        if (lc == 3) f(Const<3>{});
        else if (lc == 2) f(Const<2>{});
        else if (lc == 1) f(Const<1>{});
        else f(Const<0>{});
    };
    Piece pa, pb;
    seek();
    open();
    auto load_first = [&]() { by_length([&](auto LC) { load(LC, pa, 0); load(LC, pb, 1); }); };
    load_first();
    PostRow<NT, 2> post_row;
    if (g.mode >= 3) post_row.load(g.post.norm_w, d);
    pdl_wait();
    pdl_trigger();
    if (g.state->done | g.state->error) return;
    ready = true;
    if (seg < g.n_seg && g.seg[seg].index && !g.seg[seg].early) { open(); load_first(); }

    if (g.mode != 0) {
        const int pos = g.state->pos;
        float ss = 0.0f;
        const bool post = g.mode >= 3;
        if (post && g.post.y) {
            ss = post_row.run(g.post, g.x_in, d, g.eps, [&](int c, float x) {
                if (blockIdx.x == 0 && g.x_out) g.x_out[c] = x;
                hs[c] = x;
            }, [&](float v) { return block_sum2(v, 0.0f, red).x; }, [&](int c) -> float& { return hs[c]; });
        } else
        if (g.prev.outs) {
            const float* lo = g.prev.outs;
            const float* ro = lo + g.prev.stride;
            float a = 0.0f, b = 0.0f;
            for (int c = tid; c < d; c += NT) { const float u = lo[c], v = ro[c]; a = fmaf(u, u, a); b = fmaf(v, v, b); }
            const float2 t = block_sum2(a, b, red);
            const float il = 1.0f / sqrtf(t.x / (float)d + g.eps), ir = 1.0f / sqrtf(t.y / (float)d + g.eps);
            for (int c = tid; c < d; c += NT) {
                float y = 0.5f * (lo[c] * il * g.prev.left_w[c] + ro[c] * ir * g.prev.right_w[c]);
                for (int f = 0; f < g.prev.n_ff; ++f) y += lo[(size_t)(2 + f) * g.prev.stride + c];
                const float x = g.x_in[c] + y;
                if (blockIdx.x == 0 && g.x_out) g.x_out[c] = x;
                hs[c] = x;
                ss = fmaf(x, x, ss);
            }
        } else if (g.queue) {
            const int id = g.queue[g.state->fed];
            if (id < 0 || id >= g.embed.vocab || pos >= g.ctx) {       // the same in every CTA; the step ends here
                __syncthreads();
                if (blockIdx.x == 0 && tid == 0) g.state->error = FC_E_DIM;
                return;
            }
            const uint16_t* e = g.embed.table + (size_t)id * g.embed.ld;
            for (int c = tid; c < d; c += NT) {
                const float x = __uint_as_float((uint32_t)e[c] << 16) * g.embed.scale;
                if (!post && blockIdx.x == 0 && g.x_out) g.x_out[c] = x;
                hs[c] = x;
                ss = fmaf(x, x, ss);
            }
            if (post) {                             // the normed embedding is the residual's first value
                const float ie = 1.0f / sqrtf(block_sum2(ss, 0.0f, red).x / (float)d + g.eps);
                ss = 0.0f;
                for (int c = tid; c < d; c += NT) {
                    const float x = hs[c] * ie * g.post.norm_w[c];
                    if (blockIdx.x == 0 && g.x_out) g.x_out[c] = x;
                    hs[c] = x;
                    ss = fmaf(x, x, ss);
                }
            }
        } else {
            for (int c = tid; c < d; c += NT) { const float x = g.x_in[c]; hs[c] = x; ss = fmaf(x, x, ss); }
        }
        const float inv = g.mode == 3 ? 1.0f : 1.0f / sqrtf(block_sum2(ss, 0.0f, red).x / (float)d + g.eps);
        const float* before = g.mode == 1 ? g.shift + (size_t)(pos & 1) * g.shift_slot : nullptr;
        float* after = g.mode == 1 ? g.shift + (size_t)((pos + 1) & 1) * g.shift_slot : nullptr;
        for (int c = tid; g.mode != 3 && c < d; c += NT) {
            const float h = hs[c] * inv * g.norm_w[c];
            hs[c] = h;
            if (before) {
                hp[c] = before[c];
                if (blockIdx.x == 0) after[c] = h;
            }
        }
    }

    while (seg < g.n_seg) {
        const GemvSeg& s = g.seg[seg];
        __syncthreads();                            // hs is complete / the last segment's input has been read
        const int kr = pieces > 1 ? pieces * PIECE : 256 << lc;
        if (g.mode == 0) {
            const float* x = g.x[s.src] + rep * s.x_step;
            if (s.K % 4 == 0 && ((uintptr_t)x & 15) == 0) {
#pragma unroll 2
                for (int k = tid * 4; k < kr; k += NT * 4) *(float4*)(xs + spot(k)) = k < s.K ? *(const float4*)(x + k) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            } else {
                for (int k = tid; k < kr; k += NT) xs[spot(k)] = k < s.K ? x[k] : 0.0f;
            }
        } else if (s.src == 0) {
            for (int k = tid; k < kr; k += NT) xs[spot(k)] = k < d ? hs[k] : 0.0f;
        } else {
            const float* mu = g.mu[s.src - 1];
            for (int k = tid; k < kr; k += NT) xs[spot(k)] = k < d ? fmaf(hp[k] - hs[k], mu[k], hs[k]) : 0.0f;
        }
        __syncthreads();
        auto dot = [&](const uint4& w, const float* x, float& a0, float& a1) {
            const float4 u = *(const float4*)x, v = *(const float4*)(x + 128);
            a0 = fmaf(__uint_as_float(w.x << 16), u.x, a0); a1 = fmaf(__uint_as_float(w.x & 0xffff0000u), u.y, a1);
            a0 = fmaf(__uint_as_float(w.y << 16), u.z, a0); a1 = fmaf(__uint_as_float(w.y & 0xffff0000u), u.w, a1);
            a0 = fmaf(__uint_as_float(w.z << 16), v.x, a0); a1 = fmaf(__uint_as_float(w.z & 0xffff0000u), v.y, a1);
            a0 = fmaf(__uint_as_float(w.w << 16), v.z, a0); a1 = fmaf(__uint_as_float(w.w & 0xffff0000u), v.w, a1);
        };
        auto store = [&](float v, int r) {         // row r of this repetition's share
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
            if (lane == 0 && r < end - row) {
                if (s.epi == ROW_XIELU) v = xielu_f(v, s.c0, s.c1);
                else if (s.epi == ROW_GELU) v = gelu_erf_f(v);
                s.y[rep * s.y_step + row + r] = v;
            }
        };
        by_length([&](auto LC) {
            constexpr int L = decltype(LC)::value, RP = 8 >> L;
            float acc = 0.0f;
            auto work = [&](const Piece& p, int i) {
                if constexpr (RP == 1) {
                    const int ri = i / pieces, pc = i - ri * pieces;
                    const float* x = xs + pc * PIECE + lane * 4;
                    float a0 = 0.0f, a1 = 0.0f;
#pragma unroll
                    for (int c = 0; c < 8; ++c)
                        if (pc * PIECE + c * 256 < K_pad) dot(p.w[c], x + c * 256, a0, a1);      // uniform
                    acc += a0 + a1;
                    if (pc + 1 == pieces) {
                        store(acc, warp + ri * NW);
                        acc = 0.0f;
                    }
                } else {
                    const float* x = xs + lane * 4;
#pragma unroll
                    for (int q = 0; q < RP; ++q) {
                        float a0 = 0.0f, a1 = 0.0f;
#pragma unroll
                        for (int c = 0; c < 8 / RP; ++c)
                            if (c * 256 < K_pad) dot(p.w[q * (8 / RP) + c], x + c * 256, a0, a1);
                        store(a0 + a1, (warp + i * NW) * RP + q);
                    }
                }
            };
            for (int i = 0; i < items; i += 2) {
                work(pa, i);
                load(LC, pa, i + 2);
                if (i + 1 < items) work(pb, i + 1);
                load(LC, pb, i + 3);
            }
        });
        cur += end - row;
        if (cur >= lim) { ++seg; seek(); }
        open();
        if (seg < g.n_seg) load_first();
    }
}

int launch_gemv_bf16_group(GemvGroup g, cudaStream_t st) {
    static int sms[64] = {};
    int dev = 0;
    FC_CUDA(cudaGetDevice(&dev));
    if (dev >= 64) return fail(FC_E_ARG, "device %d out of range", dev);
    if (!sms[dev]) {
        FC_CUDA(cudaFuncSetAttribute(gemv_bf16_group_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
        FC_CUDA(cudaDeviceGetAttribute(&sms[dev], cudaDevAttrMultiProcessorCount, dev));
    }
    if (g.n_seg <= 0 || g.n_seg > kGemvSegs) return fail(FC_E_SHAPE, "grouped GEMV: %d segments", g.n_seg);
    long long cost = 0, rows = 0;
    int x_cap = 0;
    for (int i = 0; i < g.n_seg; ++i) {
        const long long n = (long long)g.seg[i].n * std::max(1, g.seg[i].reps);
        g.seg[i].cost0 = (int)cost;
        g.seg[i].cost = g.seg[i].K_pad / 64;
        cost += n * g.seg[i].cost;
        rows += n;
        x_cap = std::max(x_cap, pad_to(g.seg[i].K_pad, PIECE));
    }
    if (cost >= 1LL << 30) return fail(FC_E_SHAPE, "grouped GEMV: %lld x 64 weights", cost);
    const size_t smem = (size_t)(x_cap + (g.mode ? 2 * g.d : 0)) * sizeof(float);
    if (smem > 220 * 1024) return fail(FC_E_SHAPE, "rows of %d values exceed the staging of the decode products", x_cap);
    const int grid = (int)std::min<long long>(sms[dev], std::max<long long>(1, rows / 4));
    g.share = (int)(cost / grid); g.rest = (int)(cost % grid);
    FC_CUDA(launch_pdl(gemv_bf16_group_kernel, dim3(grid), dim3(NT), smem, st, g, x_cap));
    ++g_launches;
    return FC_OK;
}

}  // namespace fc
