// Several products of one activation row in one launch, on bf16 weights: the decode counterpart of the grouped GEMM.
//
// The rows of all segments form one list that is cut into equal shares of bytes, one persistent CTA of 16 warps per SM.
// A warp takes pieces of 2048 weights, two in flight: a row (or a K slice given as a segment of its own) that is longer takes
// several, of rows of at most 1024, 512 or 256 weights a piece holds 2, 4 or 8. 16-byte loads, activations f32 in shared
// memory, f32 sums. A segment may be repeated over experts, which every CTA chooses from the router's logits itself, its
// rows following one another; or over experts chosen by an earlier kernel, its rows running through all of them, summed with
// their weights.
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
#include "route.cuh"
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
// The layout of rows of K_pad weights: how many loads of 256 a row takes, as a power of two (3: eight or more).
__host__ __device__ inline int lay_of(int K_pad) { return K_pad > 1024 ? 3 : (K_pad > 512 ? 2 : (K_pad > 256 ? 1 : 0)); }
template <int V> struct Const { static constexpr int value = V; };

// This CTA's rows of segment s, repetitions one after the other: [first, last). Costs are counted in 64 weights.
__device__ __forceinline__ void share(const GemvGroup& g, int s, int lo, int hi, int* first, int* last) {
    const int cost = g.seg[s].cost, rows = g.seg[s].n * (g.seg[s].sum ? 1 : max(1, g.seg[s].reps)), a = lo - g.seg[s].cost0, b = hi - g.seg[s].cost0;
    *first = *last = 0;
    if (b <= 0 || a >= rows * cost) return;
    *first = a <= 0 ? 0 : (a + cost - 1) / cost;
    *last = min((b + cost - 1) / cost, rows);
}
}  // namespace

// MODE: what precedes the products (kPlain: inputs as they are; kSide: modes 1 and 2; kPost: modes 3 and 4; kChoose: plain inputs
// of experts chosen here). LAY: the piece layout all segments share (rows of more than 1024, 512, 256 weights, or fewer: 3 .. 0;
// kSum: rows that run through all chosen experts), or kAny. Small instances keep the instruction caches warm.
enum : int { kPlain = 0, kSide = 1, kPost = 2, kChoose = 3 };
enum : int { kSum = 4, kAny = 5 };
constexpr int kSumChunks = 1024, kMaxChosen = 64;

template <int MODE, int LAY>
__global__ void __launch_bounds__(NT, 1) gemv_bf16_group_kernel(const __grid_constant__ GemvGroup g, int x_cap) {
    extern __shared__ __align__(16) float sm[];    // staged input [x_cap] | h [d] | token-shift row [d]; or expert logits behind xs
    __shared__ float2 red[NW];
    __shared__ unsigned sum_at[LAY == kSum ? kSumChunks : 1];      // where 256 weights of a row begin, in 64s, times 8; plus how many 64s
    __shared__ int chosen[MODE == kChoose ? kMaxChosen : 1];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, d = g.d;
    float* xs = sm;
    float* hs = sm + x_cap;
    float* hp = hs + d;

    auto bound = [&](int b) { return g.share * b + g.rest * b / (int)gridDim.x; };
    const int lo = bound(blockIdx.x), hi = bound(blockIdx.x + 1);
    int cur = 0, lim = 0, seg = 0;                 // rows cur .. lim - 1 of segment seg are still to do
    int rep = 0, row = 0, end = 0;                 // of these, rows row + warp, + NW, ... < end of repetition rep now
    auto seek = [&]() {
#pragma unroll 1
        for (; seg < g.n_seg; ++seg) {
            share(g, seg, lo, hi, &cur, &lim);
            if (cur < lim) break;
        }
    };
    const uint16_t* base = nullptr;
    int ldw = 0, K_pad = 0, pieces = 1, lc = 3, items = 0;    // a piece holds 8 >> lc rows of 1 << lc loads of 256 weights
    int chunks = 0, per_rep = 0;                   // kSum: loads of 256 weights of a row, of one repetition of it
    bool ready = false;                            // past the wait: indices may be read
    auto open = [&]() {
        items = 0;
        const GemvSeg& s = g.seg[seg];
        rep = LAY == kSum ? 0 : cur / s.n;
        row = cur - rep * s.n;
        end = min(s.n, row + lim - cur);
        ldw = s.ldw;
        K_pad = s.K_pad;
        if ((MODE == kChoose || LAY == kSum) && !ready) return;      // loaded after the wait
        base = s.w + (size_t)row * ldw;
        if (LAY == kSum) {
            per_rep = (K_pad + 255) / 256;
            chunks = s.reps * per_rep;
            pieces = (chunks + 7) / 8;
        } else {
            lc = LAY != kAny ? LAY : lay_of(K_pad);
            pieces = lc == 3 ? (K_pad + PIECE - 1) / PIECE : 1;
            if (MODE == kChoose) base += (size_t)chosen[rep] * s.w_step;
        }
        const int rp = LAY == kSum ? 1 : 8 >> lc, mine = end - row - warp * rp;
        items = mine > 0 ? (mine + NW * rp - 1) / (NW * rp) * pieces : 0;
    };
    // item i: piece i % pieces of the rows from (warp + (i / pieces) NW) rp on; LC is lc as a constant
    auto load = [&](auto LC, Piece& p, int i) {
        constexpr int L = decltype(LC)::value;
        if constexpr (L == kSum) {
            const int ri = i / pieces, c0 = (i - ri * pieces) * 8;
            const uint16_t* src = base + (size_t)(warp + ri * NW) * ldw + lane * 8;
#pragma unroll
            for (int c = 0; c < 8; ++c) {
                const unsigned at = c0 + c < chunks ? sum_at[c0 + c] : 0;
                p.w[c] = i < items && lane < (int)(at & 7) * 8 ? ld_stream(src + (size_t)(at >> 3) * 64) : make_uint4(0, 0, 0, 0);
            }
        } else if constexpr (L == 3) {
            const int ri = i / pieces, k0 = (i - ri * pieces) * PIECE + lane * 8;
            const uint16_t* src = base + (size_t)(warp + ri * NW) * ldw;
#pragma unroll
            for (int c = 0; c < 8; ++c) p.w[c] = i < items && k0 + c * 256 < K_pad ? ld_stream(src + k0 + c * 256) : make_uint4(0, 0, 0, 0);
        } else {                                   // such rows are one piece long
            constexpr int RP = 8 >> L;
            const int r0 = (warp + i * NW) * RP, rows = end - row - r0, k0 = lane * 8;
            const uint16_t* src = base + (size_t)r0 * ldw;
#pragma unroll
            for (int q = 0; q < RP; ++q, src += ldw)
#pragma unroll
                for (int c = 0; c < 8 / RP; ++c)
                    p.w[q * (8 / RP) + c] = i < items && q < rows && k0 + c * 256 < K_pad ? ld_stream(src + k0 + c * 256) : make_uint4(0, 0, 0, 0);
        }
    };
    auto by_layout = [&](auto f) {
        if constexpr (LAY != kAny) f(Const<LAY>{});
        else if (lc == 3) f(Const<3>{});
        else if (lc == 2) f(Const<2>{});
        else if (lc == 1) f(Const<1>{});
        else f(Const<0>{});
    };
    Piece pa, pb;
    PostRow<NT, 2> post_row;
    seek();
    while (true) {
        if (seg < g.n_seg) {
            open();
            by_layout([&](auto LC) { load(LC, pa, 0); load(LC, pb, 1); });
        }
        if (!ready) {
            if constexpr (MODE == kPost) post_row.load(g.post.norm_w, d);
            pdl_wait();
            pdl_trigger();
            if (g.state->done | g.state->error) return;
            ready = true;
            if constexpr (MODE == kChoose) {
                if (warp == 0) {                   // every CTA for itself; the first tells the kernels behind
                    float* z = sm + x_cap;
                    for (int i = lane; i < g.router.experts; i += 32) z[i] = __ldcg(g.z + i);
                    __syncwarp();
                    choose(z, z + g.router.experts, g.router, [&](int k, int e, float w) {
                        chosen[k] = e;
                        if (blockIdx.x == 0) { g.expert[k] = e; g.weight[k] = w; }
                    });
                }
                __syncthreads();
                continue;
            }
            if constexpr (LAY == kSum) {
                const GemvSeg& s = g.seg[0];
                const int n = (s.K_pad + 255) / 256;
                for (int i = tid; i < s.reps * n; i += NT) {
                    const int r = i / n, c = i - r * n;
                    sum_at[i] = ((unsigned)((size_t)__ldcg(g.expert + r) * (s.w_step / 64)) + c * 4) * 8 + min(4, s.K_pad / 64 - c * 4);
                }
                __syncthreads();
                continue;
            }
            if constexpr (MODE == kSide || MODE == kPost) {
                const int pos = g.state->pos;
                float ss = 0.0f;
                if (MODE == kPost && g.post.y) {
                    if constexpr (MODE == kPost)
                        ss = post_row.run(g.post, g.x_in, d, g.eps, [&](int c, float x) {
                            if (blockIdx.x == 0 && g.x_out) g.x_out[c] = x;
                            hs[c] = x;
                        }, [&](float v) { return block_sum2(v, 0.0f, red).x; }, [&](int c) -> float& { return hs[c]; });
                } else if (MODE == kSide && g.prev.outs) {
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
                        if (MODE == kSide && blockIdx.x == 0 && g.x_out) g.x_out[c] = x;
                        hs[c] = x;
                        ss = fmaf(x, x, ss);
                    }
                    if (MODE == kPost) {            // the normed embedding is the residual's first value
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
                if (g.mode != 3) {
                    const float inv = 1.0f / sqrtf(block_sum2(ss, 0.0f, red).x / (float)d + g.eps);
                    const float* before = g.mode == 1 ? g.shift + (size_t)(pos & 1) * g.shift_slot : nullptr;
                    float* after = g.mode == 1 ? g.shift + (size_t)((pos + 1) & 1) * g.shift_slot : nullptr;
                    for (int c = tid; c < d; c += NT) {
                        const float h = hs[c] * inv * g.norm_w[c];
                        hs[c] = h;
                        if (before) {
                            hp[c] = before[c];
                            if (blockIdx.x == 0) after[c] = h;
                        }
                    }
                }
            }
        }
        if (seg >= g.n_seg) break;
        const GemvSeg& s = g.seg[seg];
        __syncthreads();                            // hs is complete / the last segment's input has been read
        const int kr = LAY == kSum ? chunks * 256 : (pieces > 1 ? pieces * PIECE : 256 << lc);
        if constexpr (LAY == kSum) {
#pragma unroll 2
            for (int ci = warp; ci < chunks; ci += NW) {          // 256 values of one expert's input
                const int r = ci / per_rep, e = (ci - r * per_rep) * 256 + lane * 8;
                const float* x = g.x[s.src] + (size_t)r * s.x_step + e;
                const float w = __ldcg(g.weight + r);
                float v[8];
                if (s.K % 8 == 0 && s.x_step % 4 == 0) {
                    const float4 a = e < s.K ? *(const float4*)x : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                    const float4 b = e < s.K ? *(const float4*)(x + 4) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
                    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
                } else {
#pragma unroll
                    for (int k = 0; k < 8; ++k) v[k] = e + k < s.K ? x[k] : 0.0f;
                }
                *(float4*)(xs + ci * 256 + lane * 4) = make_float4(v[0] * w, v[1] * w, v[2] * w, v[3] * w);
                *(float4*)(xs + ci * 256 + lane * 4 + 128) = make_float4(v[4] * w, v[5] * w, v[6] * w, v[7] * w);
            }
            for (int k = chunks * 256 + tid; k < pieces * PIECE; k += NT) xs[k] = 0.0f;
        } else if constexpr (MODE == kPlain || MODE == kChoose) {
            const float* x = g.x[s.src] + rep * s.x_step;
            if (s.K % 4 == 0 && ((uintptr_t)x & 15) == 0) {
#pragma unroll 2
                for (int k = tid * 4; k < kr; k += NT * 4) *(float4*)(xs + spot(k)) = k < s.K ? *(const float4*)(x + k) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            } else {
                for (int k = tid; k < kr; k += NT) xs[spot(k)] = k < s.K ? x[k] : 0.0f;
            }
        } else if (MODE == kPost || s.src == 0) {
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
        by_layout([&](auto LC) {
            constexpr int L = decltype(LC)::value;
            float acc = 0.0f;
            auto work = [&](const Piece& p, int i) {
                if constexpr (L >= 3) {
                    const int ri = i / pieces, pc = i - ri * pieces, k_end = L == kSum ? kr : K_pad;
                    const float* x = xs + pc * PIECE + lane * 4;
                    float a0 = 0.0f, a1 = 0.0f;
#pragma unroll
                    for (int c = 0; c < 8; ++c)
                        if (pc * PIECE + c * 256 < k_end) dot(p.w[c], x + c * 256, a0, a1);      // uniform
                    acc += a0 + a1;
                    if (pc + 1 == pieces) {
                        store(acc, warp + ri * NW);
                        acc = 0.0f;
                    }
                } else {
                    constexpr int RP = 8 >> L;
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
        if (seg >= g.n_seg) break;
    }
}

template <int MODE, int LAY>
static int launch(const GemvGroup& g, int x_cap, int grid, size_t smem, cudaStream_t st) {
    static bool set[64] = {};
    int dev = 0;
    FC_CUDA(cudaGetDevice(&dev));
    if (!set[dev]) {
        FC_CUDA(cudaFuncSetAttribute(gemv_bf16_group_kernel<MODE, LAY>, cudaFuncAttributeMaxDynamicSharedMemorySize, 216 * 1024));
        set[dev] = true;
    }
    FC_CUDA(launch_pdl(gemv_bf16_group_kernel<MODE, LAY>, dim3(grid), dim3(NT), smem, st, g, x_cap));
    ++g_launches;
    return FC_OK;
}
template <int MODE>
static int launch_layout(int lay, const GemvGroup& g, int x_cap, int grid, size_t smem, cudaStream_t st) {
    switch (lay) {
        case 3: return launch<MODE, 3>(g, x_cap, grid, smem, st);
        case 2: return launch<MODE, 2>(g, x_cap, grid, smem, st);
        case 1: return launch<MODE, 1>(g, x_cap, grid, smem, st);
        case 0: return launch<MODE, 0>(g, x_cap, grid, smem, st);
        default: return launch<MODE, kAny>(g, x_cap, grid, smem, st);
    }
}

int launch_gemv_bf16_group(GemvGroup g, cudaStream_t st) {
    static int sms[64] = {};
    int dev = 0;
    FC_CUDA(cudaGetDevice(&dev));
    if (dev >= 64) return fail(FC_E_ARG, "device %d out of range", dev);
    if (!sms[dev]) FC_CUDA(cudaDeviceGetAttribute(&sms[dev], cudaDevAttrMultiProcessorCount, dev));
    if (g.n_seg <= 0 || g.n_seg > kGemvSegs) return fail(FC_E_SHAPE, "grouped GEMV: %d segments", g.n_seg);
    long long cost = 0, rows = 0;
    int x_cap = 0, lay = lay_of(g.seg[0].K_pad);
    const bool sum = g.seg[0].sum, choosing = !sum && g.router.experts > 0;
    for (int i = 0; i < g.n_seg; ++i) {
        GemvSeg& s = g.seg[i];
        const int reps = std::max(1, s.reps), chunks = (s.K_pad + 255) / 256 * reps;
        const long long n = (long long)s.n * (sum ? 1 : reps);
        if (sum && (chunks > kSumChunks || s.w_step % 64)) return fail(FC_E_SHAPE, "product summed over %d experts of %d inputs", reps, s.K);
        s.cost0 = (int)cost;
        s.cost = sum ? chunks * 4 : s.K_pad / 64;
        cost += n * s.cost;
        rows += n;
        x_cap = std::max(x_cap, sum ? pad_to(chunks * 256, PIECE) : pad_to(s.K_pad, PIECE));
        if (lay_of(s.K_pad) != lay) lay = kAny;
    }
    if (cost >= 1LL << 30) return fail(FC_E_SHAPE, "grouped GEMV: %lld x 64 weights", cost);
    if (choosing && (g.router.top > kMaxChosen || g.router.experts > kMaxExperts || g.router.groups > kMaxGroups || g.mode != 0))
        return fail(FC_E_SHAPE, "%d of %d experts in %d groups", g.router.top, g.router.experts, g.router.groups);
    if (sum && (g.n_seg != 1 || g.mode != 0)) return fail(FC_E_SHAPE, "a product summed over experts stands alone");
    const size_t smem = (size_t)(x_cap + (g.mode ? 2 * g.d : 0) + (choosing ? g.router.experts + g.router.groups : 0)) * sizeof(float);
    if (smem > 216 * 1024) return fail(FC_E_SHAPE, "rows of %d values exceed the staging of the decode products", x_cap);
    const int grid = (int)std::min<long long>(sms[dev], std::max<long long>(1, rows / 4));
    g.share = (int)(cost / grid); g.rest = (int)(cost % grid);
    if (sum) return launch<kPlain, kSum>(g, x_cap, grid, smem, st);
    if (choosing) return launch_layout<kChoose>(lay, g, x_cap, grid, smem, st);
    if (g.mode == 0) return launch_layout<kPlain>(lay, g, x_cap, grid, smem, st);
    if (g.mode >= 3) return launch_layout<kPost>(lay, g, x_cap, grid, smem, st);
    return launch_layout<kSide>(lay, g, x_cap, grid, smem, st);
}

}  // namespace fc
