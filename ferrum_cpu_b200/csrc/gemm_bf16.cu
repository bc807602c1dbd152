// Several products of a layer in one launch on bf16 weights: Y_s = A_s W_s^T for the segments s of a group
// (for instance q | k | v, the feed-forward's first matrix and the inputs of a recurrence, each reading its own
// plane of activations), bf16 operands, fp32 accumulation in TMEM.
//
// Persistent kernel, one CTA per SM, 256 x 128 output tiles (two 128-row MMA tiles sharing one weight tile),
// k-blocks of 64, four stages of 48 KB; two accumulator buffers, so a tile's epilogue overlaps the next tile's MMAs.
//   warp 8      TMA producer of the activation and weight tiles (128-byte swizzle, K-major)
//   warp 9      TMEM allocation, tcgen05.mma issue by one thread, tcgen05.commit
//   warps 0-7   epilogue: tcgen05.ld, activation function, f32 or bf16 rows out
// Every mbarrier wait is bounded by a cycle budget; when it runs out the status word is raised and the CTA leaves.
//
// Bound: tensor pipe (2 M N K FLOP) for long portions, HBM (the weights once) for short ones.
#include <algorithm>

#include "bf16_ops.cuh"
#include "tc_common.cuh"

namespace fc {

using namespace tc;

namespace {
constexpr int BM = 256, BN = 128, BK = 64, STAGES = 4;
constexpr int TILE_BYTES = 128 * BK * 2;             // 16 KiB
constexpr int STAGE_BYTES = 3 * TILE_BYTES;          // two activation tiles, one weight tile
constexpr int EPI_WARPS = 8, TMA_WARP = 8, MMA_WARP = 9, THREADS = 320, TMEM_COLS = 512;
constexpr uint32_t IDESC = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(BN >> 3) << 17) | ((uint32_t)(128 >> 4) << 24);

struct Bars {
    unsigned long long full[STAGES], empty[STAGES], acc_full[2], acc_empty[2];
    uint32_t tmem_base;
    volatile int abort;
};
constexpr int SMEM_BYTES = STAGES * STAGE_BYTES + 1024 + (int)sizeof(Bars);

// Rows [m0, m_end) of the operand plane (and of the output), columns from n0 on, weight rows from b0 on.
struct Tile { int seg, m0, m_end, n0, b0; };
template <bool RAGGED>
__device__ __forceinline__ Tile locate(const GemmGroup& g, int tile) {
    if constexpr (RAGGED) {
        const int e = tile / g.seg[0].tiles_n;
        const int4 t = __ldg(g.ragged.table + e);
        return {0, t.x, t.x + t.y, (tile - e * g.seg[0].tiles_n) * BN, g.seg[0].b_row0 + t.z * g.ragged.b_step};
    }
    int s = 0;
    while (s + 1 < g.n_seg && tile >= g.seg[s + 1].tile0) ++s;
    const int local = tile - g.seg[s].tile0;
    return {s, (local / g.seg[s].tiles_n) * BM, g.M, (local % g.seg[s].tiles_n) * BN, g.seg[s].b_row0};
}
}  // namespace

template <bool RAGGED>
__global__ void __launch_bounds__(THREADS, 1)
gemm_bf16_group_kernel(const __grid_constant__ GemmMaps maps, const __grid_constant__ GemmGroup g) {
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    Bars* bars = (Bars*)(smem + STAGES * STAGE_BYTES);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    const int n_tiles = RAGGED ? *g.ragged.n * g.seg[0].tiles_n : g.n_tiles;
    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; ++s) { mbar_init(&bars->full[s], 1); mbar_init(&bars->empty[s], 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(&bars->acc_full[b], 1); mbar_init(&bars->acc_empty[b], EPI_WARPS); }
        bars->abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == MMA_WARP) tmem_alloc(&bars->tmem_base, TMEM_COLS);
    fence_before();
    __syncthreads();
    fence_after();
    const uint32_t tmem = bars->tmem_base;

    if (warp == TMA_WARP) {
        if (lane == 0 && !g.withhold) {
            int it = 0;
            for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x) {
                const Tile t = locate<RAGGED>(g, tile);
                const GemmSeg& s = g.seg[t.seg];
                const bool two = t.m0 + 128 < t.m_end;
                const CUtensorMap* ma = &maps.a[s.a_map];
                const CUtensorMap* mb = &maps.b[s.b_map];
                for (int kb = 0; kb < s.kb; ++kb, ++it) {
                    const int st = it % STAGES;
                    if (!wait_bar(&bars->abort, &bars->empty[st], ((it / STAGES) & 1) ^ 1, g.status, g.wait_cycles)) { tile = n_tiles; break; }
                    unsigned char* p = smem + st * STAGE_BYTES;
                    mbar_expect_tx(&bars->full[st], (two ? 3 : 2) * TILE_BYTES);
                    const int x = (s.kb0 + kb) * BK;
                    tma_load_2d(p, ma, x, s.a_row0 + t.m0, &bars->full[st]);
                    if (two) tma_load_2d(p + TILE_BYTES, ma, x, s.a_row0 + t.m0 + 128, &bars->full[st]);
                    tma_load_2d(p + 2 * TILE_BYTES, mb, x, t.b0 + t.n0, &bars->full[st]);
                }
            }
            if (bars->abort)                              // leaving early: no copy may still be on its way into this CTA
                for (int i = max(0, it - STAGES); i < it; ++i) {
                    const long long t0 = clock64();
                    while (!mbar_try_wait(&bars->full[i % STAGES], (i / STAGES) & 1) && clock64() - t0 < g.wait_cycles) {}
                }
        }
    } else if (warp == MMA_WARP) {
        if (lane == 0) {
            int it = 0, ti = 0;
            bool ok = true;
            for (int tile = blockIdx.x; tile < n_tiles && ok; tile += gridDim.x, ++ti) {
                const Tile t = locate<RAGGED>(g, tile);
                const int nkb = g.seg[t.seg].kb, halves = t.m0 + 128 < t.m_end ? 2 : 1, buf = ti & 1;
                ok = wait_bar(&bars->abort, &bars->acc_empty[buf], ((ti >> 1) & 1) ^ 1, g.status, g.wait_cycles);
                if (!ok) break;
                fence_after();
                const uint32_t acc = tmem + (uint32_t)(buf * 2 * BN);
                for (int kb = 0; kb < nkb; ++kb, ++it) {
                    const int st = it % STAGES;
                    ok = wait_bar(&bars->abort, &bars->full[st], (it / STAGES) & 1, g.status, g.wait_cycles);
                    if (!ok) break;
                    fence_after();
                    const uint32_t base = s32(smem + st * STAGE_BYTES);
                    const uint64_t b = smem_desc(base + 2 * TILE_BYTES);
                    for (int hm = 0; hm < halves; ++hm) {
                        const uint64_t a = smem_desc(base + hm * TILE_BYTES);
#pragma unroll
                        for (int ks = 0; ks < BK / 16; ++ks) umma(acc + hm * BN, a + (uint64_t)(ks * 2), b + (uint64_t)(ks * 2), IDESC, (kb | ks) != 0);
                    }
                    umma_commit(&bars->empty[st]);
                }
                if (ok) umma_commit(&bars->acc_full[buf]);
            }
        }
    } else {
        int ti = 0;
        const int hm = warp >> 2, quarter = warp & 3;
        for (int tile = blockIdx.x; tile < n_tiles; tile += gridDim.x, ++ti) {
            const Tile t = locate<RAGGED>(g, tile);
            const GemmSeg& s = g.seg[t.seg];
            const int buf = ti & 1;
            if (!wait_bar(&bars->abort, &bars->acc_full[buf], (ti >> 1) & 1, g.status, g.wait_cycles)) break;
            fence_after();
            const int m = t.m0 + hm * 128 + quarter * 32 + lane;
            const bool f32_vec = s.y && (s.ldy & 7) == 0 && ((uintptr_t)s.y & 31) == 0;
            const bool b16_vec = s.yb && (s.ldy & 15) == 0 && ((uintptr_t)s.yb & 31) == 0;
#pragma unroll 1
            for (int c = 0; c < BN / 32; ++c) {
                uint32_t r[32];
                tmem_ld32(tmem + ((uint32_t)(quarter * 32) << 16) + (uint32_t)((buf * 2 + hm) * BN + c * 32), r);
                if (c == BN / 32 - 1) {
                    fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(&bars->acc_empty[buf]);
                }
                const int nb = t.n0 + c * 32;
                if (m < t.m_end && nb < s.n) {
                    if (s.epi == ROW_XIELU) {
#pragma unroll
                        for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(xielu_f(__uint_as_float(r[i]), s.c0, s.c1));
                    } else if (s.epi == ROW_GELU) {
#pragma unroll
                        for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(gelu_erf_f(__uint_as_float(r[i])));
                    }
                    const bool full = nb + 32 <= s.n;
                    const size_t off = (size_t)m * s.ldy + nb;
                    if (s.y) {
                        if (full && f32_vec) {
#pragma unroll
                            for (int i = 0; i < 4; ++i) st256(s.y + off + 8 * i, r + 8 * i);
                        } else {
#pragma unroll
                            for (int i = 0; i < 32; ++i)
                                if (nb + i < s.n) s.y[off + i] = __uint_as_float(r[i]);
                        }
                    } else if (full && b16_vec) {
                        uint32_t p[16];
#pragma unroll
                        for (int i = 0; i < 16; ++i) p[i] = pack2(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1]));
                        st256(s.yb + off, p);
                        st256(s.yb + off + 16, p + 8);
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                            if (nb + i < s.n) s.yb[off + i] = __bfloat16_as_ushort(__float2bfloat16_rn(__uint_as_float(r[i])));
                    }
                }
                __syncwarp();
            }
        }
    }
    fence_before();
    __syncthreads();
    if (warp == MMA_WARP) {
        fence_after();
        tmem_dealloc(tmem, TMEM_COLS);
    }
}

static int prepare(int* sms_out) {
    static int sms[64] = {};
    int dev = 0;
    FC_CUDA(cudaGetDevice(&dev));
    if (dev >= 64) return fail(FC_E_ARG, "device %d out of range", dev);
    if (!sms[dev]) {
        FC_CUDA(cudaFuncSetAttribute(gemm_bf16_group_kernel<false>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_BYTES));
        FC_CUDA(cudaFuncSetAttribute(gemm_bf16_group_kernel<true>, cudaFuncAttributeMaxDynamicSharedMemorySize, SMEM_BYTES));
        FC_CUDA(cudaDeviceGetAttribute(&sms[dev], cudaDevAttrMultiProcessorCount, dev));
    }
    *sms_out = sms[dev];
    return FC_OK;
}
int launch_gemm_bf16_group(const GemmMaps& maps, GemmGroup g, int M, int* status, cudaStream_t st) {
    int sms = 0;
    FC_TRY(prepare(&sms));
    if (M <= 0 || g.n_seg <= 0 || g.n_seg > kGemmSegs) return fail(FC_E_SHAPE, "grouped GEMM: M = %d, %d segments", M, g.n_seg);
    const int tiles_m = (M + BM - 1) / BM;
    int tiles = 0;
    for (int i = 0; i < g.n_seg; ++i) {
        g.seg[i].tile0 = tiles;
        g.seg[i].tiles_n = (g.seg[i].n + BN - 1) / BN;
        tiles += g.seg[i].tiles_n * tiles_m;
    }
    g.M = M; g.n_tiles = tiles; g.status = status;
    g.wait_cycles = g_debug.wait_cycles; g.withhold = g_debug.withhold;
    gemm_bf16_group_kernel<false><<<std::min(tiles, sms), THREADS, SMEM_BYTES, st>>>(maps, g);
    FC_LAUNCHED();
    return FC_OK;
}
int launch_gemm_bf16_ragged(const GemmMaps& maps, const GemmSeg& seg, const Ragged& r, int max_entries, int* status, cudaStream_t st) {
    static_assert(kRaggedRows == BM, "a table entry is a tile's rows");
    int sms = 0;
    FC_TRY(prepare(&sms));
    GemmGroup g = {};
    g.seg[0] = seg; g.n_seg = 1; g.ragged = r; g.status = status;
    g.seg[0].tiles_n = (seg.n + BN - 1) / BN;
    g.wait_cycles = g_debug.wait_cycles; g.withhold = g_debug.withhold;
    if (max_entries <= 0 || seg.n <= 0) return fail(FC_E_SHAPE, "product over runs: %d entries, n = %d", max_entries, seg.n);
    gemm_bf16_group_kernel<true><<<(int)std::min<long long>((long long)max_entries * g.seg[0].tiles_n, sms), THREADS, SMEM_BYTES, st>>>(maps, g);
    FC_LAUNCHED();
    return FC_OK;
}

// ------------------------------------------------------------------------------ true f32 on CUDA cores
// 64 x 64 tiles, k-steps of 32, 4 x 4 outputs per thread; the bf16 weights are exact in f32, every product and sum is f32.
namespace {
constexpr int FM = 64, FN = 64, FK = 32;
}
__global__ void __launch_bounds__(256) gemm_bf16w_f32_kernel(const uint16_t* __restrict__ w, int K_pad, int n, const GemmF32 p, int M,
                                                             const Ragged runs) {
    __shared__ __align__(16) float As[FK][FM + 4], Bs[FK][FN + 4];
    const int t = threadIdx.x, n0 = blockIdx.x * FN;
    int m0 = blockIdx.y * FM;
    if (runs.table) {                                     // rows m0 .. M - 1 of one run, with its weights
        if ((int)blockIdx.y >= *runs.n) return;
        const int4 e = __ldg(runs.table + blockIdx.y);
        m0 = e.x; M = e.x + e.y;
        w += (size_t)e.z * runs.b_step * K_pad;
    }
    const int row = t >> 2, k8 = (t & 3) * 8;             // this thread loads 8 consecutive k of one row
    const bool va = m0 + row < M, vb = n0 + row < n;
    const float* ap = p.a + (size_t)(va ? m0 + row : 0) * p.lda + k8;
    const uint16_t* bp = w + (size_t)(vb ? n0 + row : 0) * K_pad + k8;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) acc[i][j] = 0.0f;
    const int ty = t >> 4, tx = t & 15;
    float4 av[2] = {};
    uint4 bv = make_uint4(0, 0, 0, 0);
    auto load = [&](int k0) {
        if (va) { av[0] = *(const float4*)(ap + k0); av[1] = *(const float4*)(ap + k0 + 4); }
        if (vb) bv = *(const uint4*)(bp + k0);
    };
    load(0);
    for (int k0 = 0; k0 < K_pad; k0 += FK) {
        float x[8] = {av[0].x, av[0].y, av[0].z, av[0].w, av[1].x, av[1].y, av[1].z, av[1].w};
        const uint32_t y[4] = {bv.x, bv.y, bv.z, bv.w};
        if (p.tanh_in)
#pragma unroll
            for (int i = 0; i < 8; ++i) x[i] = tanhf(x[i]);
        __syncthreads();
#pragma unroll
        for (int i = 0; i < 8; ++i) As[k8 + i][row] = x[i];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            Bs[k8 + 2 * i][row] = __uint_as_float(y[i] << 16);
            Bs[k8 + 2 * i + 1][row] = __uint_as_float(y[i] & 0xffff0000u);
        }
        __syncthreads();
        if (k0 + FK < K_pad) load(k0 + FK);
#pragma unroll
        for (int k = 0; k < FK; ++k) {
            const float4 a = *(const float4*)&As[k][ty * 4], b = *(const float4*)&Bs[k][tx * 4];
            const float aa[4] = {a.x, a.y, a.z, a.w}, bb[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(aa[i], bb[j], acc[i][j]);
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int m = m0 + ty * 4 + i;
        if (m >= M) continue;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int c = n0 + tx * 4 + j;
            if (c >= n) continue;
            float v = acc[i][j];
            if (p.epi == ROW_XIELU) v = xielu_f(v, p.c0, p.c1);
            else if (p.epi == ROW_GELU) v = gelu_erf_f(v);
            else if (p.epi == ROW_DECAY) v = expf(-expf(v + p.vec[c]));
            if (p.y) p.y[(size_t)m * p.ldy + c] = v;
            else p.yb[(size_t)m * p.ldy + c] = __bfloat16_as_ushort(__float2bfloat16_rn(v));
        }
    }
}
int launch_gemm_bf16w_f32(const BMat& w, int row0, int n, const GemmF32& p, int M, cudaStream_t st) {
    if (M <= 0 || n <= 0 || p.lda % 4 || ((uintptr_t)p.a & 15)) return fail(FC_E_SHAPE, "f32 product: M = %d, n = %d, lda = %d", M, n, p.lda);
    gemm_bf16w_f32_kernel<<<dim3((n + FN - 1) / FN, (M + FM - 1) / FM), 256, 0, st>>>(w.w + (size_t)row0 * w.K_pad, w.K_pad, n, p, M, Ragged{});
    FC_LAUNCHED();
    return FC_OK;
}
int launch_gemm_bf16w_f32_ragged(const BMat& w, int n, const GemmF32& p, const Ragged& r, int max_entries, cudaStream_t st) {
    static_assert(kRaggedRowsF32 == FM, "a table entry is a tile's rows");
    if (max_entries <= 0 || n <= 0 || p.lda % 4 || ((uintptr_t)p.a & 15)) return fail(FC_E_SHAPE, "f32 product over runs: %d entries, n = %d, lda = %d", max_entries, n, p.lda);
    gemm_bf16w_f32_kernel<<<dim3((n + FN - 1) / FN, max_entries), 256, 0, st>>>(w.w, w.K_pad, n, p, 0, r);
    FC_LAUNCHED();
    return FC_OK;
}

}  // namespace fc
