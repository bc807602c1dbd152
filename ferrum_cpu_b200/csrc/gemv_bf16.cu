// Several products of one activation row in one launch, on bf16 weights: the decode counterpart of the grouped GEMM.
//
// The rows of all segments form one list that is cut into equal shares of bytes, one persistent CTA of 16 warps per SM.
// A warp takes pieces of 2048 weights, two in flight: a row (or a K slice given as a segment of its own) that is longer takes
// several, of rows of at most 1024, 512 or 256 weights a piece holds 2, 4 or 8. 16-byte loads, activations f32 in shared
// memory, f32 sums. A segment's rows may begin at an index read from the device (an expert chosen there).
// Launched as a programmatic dependent: the first two pieces of every warp are requested before the wait on the kernel
// ahead, since weights never change.
//
// Prologues: plain inputs; the residual of layers that norm what they add (and a norm of it); or the residual update of the layer before, the norm and the token-shift mixes of the row
// (every CTA computes them for itself, CTA 0 stores the residual and the token-shift row); or residual and norm alone
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

// This CTA's rows of segment s: [first, last).
__device__ __forceinline__ void share(const GemvGroup& g, int s, int* first, int* last) {
    const long long cost = g.seg[s].K_pad;
    const long long lo = g.total_cost * blockIdx.x / gridDim.x, hi = g.total_cost * (blockIdx.x + 1) / gridDim.x;
    const long long a = lo - g.seg[s].cost0, b = hi - g.seg[s].cost0;
    *first = a <= 0 ? 0 : (int)min((a + cost - 1) / cost, (long long)g.seg[s].n);
    *last = b <= 0 ? 0 : (int)min((b + cost - 1) / cost, (long long)g.seg[s].n);
}
}  // namespace

__global__ void __launch_bounds__(NT, 1) gemv_bf16_group_kernel(const __grid_constant__ GemvGroup g, int x_cap) {
    extern __shared__ __align__(16) float sm[];    // staged input [x_cap] | h [d] | token-shift row [d]
    __shared__ float2 red[NW];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, d = g.d;
    float* xs = sm;
    float* hs = sm + x_cap;
    float* hp = hs + d;

    int row = 0, end = 0, seg = 0;                 // rows row + warp, + NW, ... < end of segment seg
    for (; seg < g.n_seg; ++seg) {
        share(g, seg, &row, &end);
        if (row < end) break;
    }
    const uint16_t* base = nullptr;
    int ldw = 0, K_pad = 0, pieces = 1, lc = 3, items = 0;    // a piece holds 8 >> lc rows of 1 << lc loads of 256 weights
    bool ready = false;                            // past the wait: indices may be read
    auto open = [&]() {
        items = 0;
        if (seg >= g.n_seg) return;
        const GemvSeg& s = g.seg[seg];
        ldw = s.ldw;
        K_pad = s.K_pad;
        pieces = (K_pad + PIECE - 1) / PIECE;
        lc = K_pad > 1024 ? 3 : (K_pad > 512 ? 2 : (K_pad > 256 ? 1 : 0));
        const int rp = 8 >> lc, mine = end - row - warp * rp;
        if (s.index && !s.early && !ready) return;             // loaded after the wait
        base = s.w + (size_t)row * ldw;
        if (s.index) base += (size_t)*s.index * s.w_step;
        items = mine > 0 ? (mine + NW * rp - 1) / (NW * rp) * pieces : 0;
    };
    auto load = [&](Piece& p, int i) {             // item i: piece i % pieces of the rows from (warp + (i / pieces) NW) rp on
        const int ri = i / pieces, k0 = (i - ri * pieces) * PIECE + lane * 8, rp = 8 >> lc, r0 = (warp + ri * NW) * rp;
#pragma unroll
        for (int c = 0; c < 8; ++c) {
            const int r = r0 + (c >> lc), k = k0 + (c & ((1 << lc) - 1)) * 256;
            p.w[c] = i < items && r < end - row && k < K_pad ? ld_stream(base + (size_t)r * ldw + k) : make_uint4(0, 0, 0, 0);
        }
    };
    Piece pa, pb;
    open();
    load(pa, 0);
    load(pb, 1);
    PostRow<NT, 2> post_row;
    if (g.mode >= 3) post_row.load(g.post.norm_w, d);
    pdl_wait();
    pdl_trigger();
    if (g.state->done | g.state->error) return;
    ready = true;
    if (seg < g.n_seg && g.seg[seg].index && !g.seg[seg].early) { open(); load(pa, 0); load(pb, 1); }

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
            const float* x = g.x[s.src];
            for (int k = tid; k < kr; k += NT) xs[spot(k)] = k < s.K ? x[k] : 0.0f;
        } else if (s.src == 0) {
            for (int k = tid; k < kr; k += NT) xs[spot(k)] = k < d ? hs[k] : 0.0f;
        } else {
            const float* mu = g.mu[s.src - 1];
            for (int k = tid; k < kr; k += NT) xs[spot(k)] = k < d ? fmaf(hp[k] - hs[k], mu[k], hs[k]) : 0.0f;
        }
        __syncthreads();
        float acc = 0.0f;
        auto work = [&](const Piece& p, int i) {
            const int ri = i / pieces, pc = i - ri * pieces, mask = (1 << lc) - 1, r0 = (warp + ri * NW) * (8 >> lc);
            const float* x = xs + pc * PIECE + lane * 4;
            float a0 = 0.0f, a1 = 0.0f;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                const int kc = (c & mask) * 256;
                if (pc * PIECE + kc < K_pad) {                          // uniform
                    const float4 u = *(const float4*)(x + kc), v = *(const float4*)(x + kc + 128);
                    const uint4 w = p.w[c];
                    a0 = fmaf(__uint_as_float(w.x << 16), u.x, a0); a1 = fmaf(__uint_as_float(w.x & 0xffff0000u), u.y, a1);
                    a0 = fmaf(__uint_as_float(w.y << 16), u.z, a0); a1 = fmaf(__uint_as_float(w.y & 0xffff0000u), u.w, a1);
                    a0 = fmaf(__uint_as_float(w.z << 16), v.x, a0); a1 = fmaf(__uint_as_float(w.z & 0xffff0000u), v.y, a1);
                    a0 = fmaf(__uint_as_float(w.w << 16), v.z, a0); a1 = fmaf(__uint_as_float(w.w & 0xffff0000u), v.w, a1);
                }
                if ((c & mask) == mask) {                               // uniform: the end of a row of this piece
                    acc += a0 + a1;
                    a0 = a1 = 0.0f;
                    if (pc + 1 == pieces) {
                        float v = acc;
                        acc = 0.0f;
#pragma unroll
                        for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
                        const int r = r0 + (c >> lc);
                        if (lane == 0 && r < end - row) {
                            if (s.epi == ROW_XIELU) v = xielu_f(v, s.c0, s.c1);
                            else if (s.epi == ROW_GELU) v = gelu_erf_f(v);
                            s.y[row + r] = v;
                        }
                    }
                }
            }
        };
        for (int i = 0; i < items; i += 2) {
            work(pa, i);
            load(pa, i + 2);
            if (i + 1 < items) work(pb, i + 1);
            load(pb, i + 3);
        }
        for (++seg; seg < g.n_seg; ++seg) {
            share(g, seg, &row, &end);
            if (row < end) break;
        }
        open();
        if (seg < g.n_seg) { load(pa, 0); load(pb, 1); }
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
        g.seg[i].cost0 = cost;
        cost += (long long)g.seg[i].n * g.seg[i].K_pad;
        rows += g.seg[i].n;
        x_cap = std::max(x_cap, pad_to(g.seg[i].K_pad, PIECE));
    }
    g.total_cost = cost;
    const size_t smem = (size_t)(x_cap + (g.mode ? 2 * g.d : 0)) * sizeof(float);
    if (smem > 220 * 1024) return fail(FC_E_SHAPE, "rows of %d values exceed the staging of the decode products", x_cap);
    const int grid = (int)std::min<long long>(sms[dev], std::max<long long>(1, rows / 4));
    FC_CUDA(launch_pdl(gemv_bf16_group_kernel, dim3(grid), dim3(NT), smem, st, g, x_cap));
    ++g_launches;
    return FC_OK;
}

}  // namespace fc
