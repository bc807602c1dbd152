// Attention of a portion's rows over cached keys on the tcgen05 tensor cores: bf16 queries (scale and log2(e) inside), keys
// and values, fp32 scores, softmax and sums.
//
// One CTA owns 128 query rows of one head; key tiles of 64, from the first the window of its rows reaches.
//   warp 8      TMA: the query tile once (k-chunks of 64 columns; a tile too wide to stay travels again with every key
//               tile), then per key tile the chunks of the key row (the head's own part, then the part all heads share)
//               through a ring, and the value tile of the head's key/value head (two buffers)
//   warp 9      tcgen05.mma: S = q K^T into one of two score buffers, one tile ahead; O += P V (V consumed MN-major),
//               P as bf16 hi + lo so that the weights keep 16 bits
//   warps 0-7   two threads per query row, 32 keys each: score + a 191-entry slice per tile of the distance's bias (0 without
//               one), -inf for keys ahead of the query or behind its window; online softmax in base 2 that starts from the
//               sink (max = sink, sum = 1) or from nothing, P to shared memory. O stays in TMEM; it is rescaled only when a
//               row's maximum has grown by more than 8. Tiles that no edge crosses skip the slice when there is no bias.
// Every mbarrier wait is bounded; on a timeout the status word is raised and the CTA leaves.
//
// Bound: tensor pipe / special-function unit. Per (query, key) pair and head w0 + w1 + 2 vdim multiply-adds executed.
#include <algorithm>

#include "bf16_ops.cuh"
#include "tc_common.cuh"

namespace fc {

using namespace tc;

namespace {
constexpr int QT = 128, KT = 64, CH = 64;
constexpr int Q_CHUNK = QT * CH * 2;       // 16 KiB
constexpr int K_CHUNK = KT * CH * 2;       // 8 KiB
constexpr int P_BYTES = QT * KT * 2;       // 16 KiB
constexpr int MAX_KS = 8;
constexpr int SM_WARPS = 8, TMA_WARP = 8, MMA_WARP = 9, THREADS = 10 * 32;
constexpr uint32_t IDESC_S = (1u << 4) | (1u << 7) | (1u << 10) | ((uint32_t)(KT >> 3) << 17) | ((uint32_t)(QT >> 4) << 24);
constexpr uint32_t IDESC_O = (1u << 4) | (1u << 7) | (1u << 10) | (1u << 16) | ((uint32_t)(CH >> 3) << 17) | ((uint32_t)(QT >> 4) << 24);
constexpr float GROW = 8.0f;               // log2: how far a row's maximum may run ahead of the one its sums are relative to

struct Bars {
    unsigned long long q_full, k_full[MAX_KS], k_empty[MAX_KS], v_full[2], v_empty[2], s_full[2], s_empty[2], p_full, o_done;
    uint32_t tmem_base;
    volatile int abort;
    float bias[2][192];
    float half[2][2][QT];            // per buffer, half of the tile's keys: a row's largest score; at the end its sums
};
struct Args {
    int M, pos0, kq, nkc, ks, nv, H, KV, vdim, far, ldo, window;
    int nc0, w0, last0, last1;       // chunks and columns of the head's own key part; MMA steps of either part's last chunk
    int k0_col, k0_head, k0_base, k1_col, k1_base, v_col, v_head, v_base;
    int has_sink;
    int q_stream;        // the query tile is too wide to stay in shared memory: its chunks travel with the key chunks
    const float *bias, *sink;        // bias null: none; has_sink with sink null: a score of 0
    uint16_t* out;
    int* status;
    long long wait_cycles;
    int withhold;
    uint32_t tmem_cols;
};
size_t smem_bytes(int nkc, int ks, int nv, bool q_stream) {
    return (q_stream ? (size_t)ks * Q_CHUNK : (size_t)nkc * Q_CHUNK) + (size_t)ks * K_CHUNK + (size_t)2 * nv * K_CHUNK + 2 * P_BYTES + 1024 +
           sizeof(Bars);
}
// Key-ring stages: as many as keep two CTAs on an SM, else as many as fit one. 0: does not fit.
int plan_stages(int nkc, int nv, bool q_stream) {
    if (!q_stream)
        for (int ks = MAX_KS; ks >= 3; --ks)
            if (smem_bytes(nkc, ks, nv, false) <= 113 * 1024) return ks;
    for (int ks = MAX_KS; ks >= 2; --ks)
        if (smem_bytes(nkc, ks, nv, q_stream) <= 226 * 1024) return ks;
    return 0;
}
}  // namespace

__global__ void __launch_bounds__(THREADS, 1)
flash_tc_kernel(const __grid_constant__ CUtensorMap mq, const __grid_constant__ CUtensorMap mk0, const __grid_constant__ CUtensorMap mk1,
                const __grid_constant__ CUtensorMap mv, const Args a) {
    extern __shared__ unsigned char smem_raw[];
    unsigned char* smem = (unsigned char*)(((uintptr_t)smem_raw + 1023) & ~(uintptr_t)1023);
    unsigned char* sk = smem + (a.q_stream ? a.ks : a.nkc) * Q_CHUNK;
    unsigned char* sv_ = sk + a.ks * K_CHUNK;
    unsigned char* sp = sv_ + 2 * a.nv * K_CHUNK;
    Bars* bars = (Bars*)(sp + 2 * P_BYTES);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int q0 = ((int)gridDim.y - 1 - (int)blockIdx.y) * QT, h = blockIdx.x, kv = h / (a.H / a.KV);
    const int last = a.pos0 + min(a.M, q0 + QT) - 1;       // the last key any row of the tile sees
    const int kt0 = max(0, a.pos0 + q0 - a.window + 1) / KT;    // the first tile any of them sees
    const int n_kt = last / KT + 1 - kt0;                  // tiles are counted from there

    if (threadIdx.x == 0) {
        mbar_init(&bars->q_full, 1);
        for (int i = 0; i < a.ks; ++i) { mbar_init(&bars->k_full[i], 1); mbar_init(&bars->k_empty[i], 1); }
        for (int i = 0; i < 2; ++i) {
            mbar_init(&bars->v_full[i], 1); mbar_init(&bars->v_empty[i], 1);
            mbar_init(&bars->s_full[i], 1); mbar_init(&bars->s_empty[i], SM_WARPS);
        }
        mbar_init(&bars->p_full, SM_WARPS);
        mbar_init(&bars->o_done, 1);
        bars->abort = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == MMA_WARP) tmem_alloc(&bars->tmem_base, a.tmem_cols);
    fence_before();
    __syncthreads();
    fence_after();
    const uint32_t tmem = bars->tmem_base, tmem_o = tmem + 2 * KT;
    auto wait = [&](unsigned long long* b, uint32_t par) { return wait_bar(&bars->abort, b, par, a.status, a.wait_cycles); };

    if (warp == TMA_WARP) {
        if (lane == 0 && !a.withhold) {
            if (!a.q_stream) mbar_expect_tx(&bars->q_full, a.nkc * Q_CHUNK);
            auto q_x = [&](int c) { return h * a.kq + (c < a.nc0 ? c * CH : a.w0 + (c - a.nc0) * CH); };
            for (int c = 0; !a.q_stream && c < a.nkc; ++c) tma_load_2d(smem + c * Q_CHUNK, &mq, q_x(c), q0, &bars->q_full);
            int s = 0, issued = 0, nvt = 0;               // ring stage, key chunks and value tiles asked for
            uint32_t ph = 1;                              // parity of k_empty: a fresh ring is empty
            bool ok = true;
            for (int kt = 0; kt < n_kt && ok; ++kt) {
                for (int c = 0; c < a.nkc && ok; ++c) {
                    ok = wait(&bars->k_empty[s], ph);
                    if (!ok) break;
                    mbar_expect_tx(&bars->k_full[s], a.q_stream ? K_CHUNK + Q_CHUNK : K_CHUNK);
                    if (a.q_stream) tma_load_2d(smem + s * Q_CHUNK, &mq, q_x(c), q0, &bars->k_full[s]);
                    if (c < a.nc0) tma_load_2d(sk + s * K_CHUNK, &mk0, a.k0_col + kv * a.k0_head + c * CH, (kt0 + kt) * KT - a.k0_base, &bars->k_full[s]);
                    else tma_load_2d(sk + s * K_CHUNK, &mk1, a.k1_col + (c - a.nc0) * CH, (kt0 + kt) * KT - a.k1_base, &bars->k_full[s]);
                    ++issued;
                    if (++s == a.ks) { s = 0; ph ^= 1; }
                }
                const int b = kt & 1;
                ok = ok && wait(&bars->v_empty[b], ((kt >> 1) & 1) ^ 1);
                if (!ok) break;
                mbar_expect_tx(&bars->v_full[b], a.nv * K_CHUNK);
                for (int c = 0; c < a.nv; ++c) tma_load_2d(sv_ + (b * a.nv + c) * K_CHUNK, &mv, a.v_col + kv * a.v_head + c * CH, (kt0 + kt) * KT - a.v_base, &bars->v_full[b]);
                ++nvt;
            }
            if (bars->abort) {                            // leaving early: no copy may still be on its way into this CTA
                auto drain = [&](unsigned long long* b, uint32_t par) {
                    const long long t0 = clock64();
                    while (!mbar_try_wait(b, par) && clock64() - t0 < a.wait_cycles) {}
                };
                if (!a.q_stream) drain(&bars->q_full, 0);
                for (int i = max(0, issued - a.ks); i < issued; ++i) drain(&bars->k_full[i % a.ks], (i / a.ks) & 1);
                for (int i = max(0, nvt - 2); i < nvt; ++i) drain(&bars->v_full[i & 1], (i >> 1) & 1);
            }
        }
    } else if (warp == MMA_WARP) {
        if (lane == 0) {
            const uint32_t sb = s32(smem), kb = s32(sk), vb = s32(sv_);
            const uint64_t ph = smem_desc(s32(sp)), pl = smem_desc(s32(sp) + P_BYTES);
            int s = 0;                                    // ring stage (no divisions here: this thread's pace is the kernel's)
            uint32_t kph = 0;
            const uint64_t q_desc = smem_desc(sb), k_desc = smem_desc(kb), v_desc = smem_desc(vb);
            auto scores = [&](int kt) -> bool {
                const int b = kt & 1;
                if (!wait(&bars->s_empty[b], ((kt >> 1) & 1) ^ 1)) return false;
                fence_after();
                for (int c = 0; c < a.nkc; ++c) {
                    if (!wait(&bars->k_full[s], kph)) return false;
                    fence_after();
                    const int steps = c + 1 == a.nc0 ? a.last0 : (c + 1 == a.nkc ? a.last1 : CH / 16);
                    const uint64_t qd = q_desc + (uint64_t)((a.q_stream ? s : c) * (Q_CHUNK >> 4)), kd = k_desc + (uint64_t)(s * (K_CHUNK >> 4));
#pragma unroll
                    for (int ks = 0; ks < CH / 16; ++ks)
                        if (ks < steps) umma(tmem + b * KT, qd + (uint64_t)(ks * 2), kd + (uint64_t)(ks * 2), IDESC_S, (c | ks) != 0);
                    umma_commit(&bars->k_empty[s]);
                    if (++s == a.ks) { s = 0; kph ^= 1; }
                }
                umma_commit(&bars->s_full[b]);
                return true;
            };
            bool ok = (a.q_stream || wait(&bars->q_full, 0)) && scores(0);
            for (int kt = 0; kt < n_kt && ok; ++kt) {
                if (kt + 1 < n_kt && !(ok = scores(kt + 1))) break;
                const int b = kt & 1;
                ok = wait(&bars->v_full[b], (kt >> 1) & 1) && wait(&bars->p_full, kt & 1);
                if (!ok) break;
                fence_after();
                for (int c = 0; c < a.nv; ++c) {
                    const uint64_t vd = v_desc + (uint64_t)((b * a.nv + c) * (K_CHUNK >> 4));
#pragma unroll
                    for (int ks = 0; ks < KT / 16; ++ks) {
                        umma(tmem_o + c * CH, ph + (uint64_t)(ks * 2), vd + (uint64_t)(ks * 128), IDESC_O, (kt | ks) != 0);
                        umma(tmem_o + c * CH, pl + (uint64_t)(ks * 2), vd + (uint64_t)(ks * 128), IDESC_O, 1);
                    }
                }
                umma_commit(&bars->v_empty[b]);
                umma_commit(&bars->o_done);
            }
        }
    } else {
        // two threads a query row, each with half of the tile's keys (and of the output's columns)
        const int hf = warp >> 2, r = (warp & 3) * 32 + lane, tid = threadIdx.x;
        const float* bias = a.bias ? a.bias + (size_t)h * (a.far + 1) : nullptr;
        // without a sink the maximum starts below every score, and what precedes the first visible key is scaled away
        float m = a.has_sink ? (a.sink ? a.sink[h] * kLog2e : 0.0f) : -1e30f, l = a.has_sink && hf == 0 ? 1.0f : 0.0f;
        unsigned char* ph = sp + r * 128;
        unsigned char* pl = ph + P_BYTES;
        const uint32_t lane_addr = (uint32_t)((warp & 3) * 32) << 16;
        constexpr int HK = KT / 2;
        auto bias_at = [&](int kt) -> float {              // entry tid of tile kt's slice of the table
            const int n = a.pos0 + q0 - (kt0 + kt) * KT - (KT - 1) + tid;
            if (n < 0 || n >= a.window) return -INFINITY;
            return bias ? __ldg(bias + min(n, a.far)) * kLog2e : 0.0f;
        };
        auto edges = [&](int kt) -> bool {                 // does any pair of tile kt need the slice?
            const int n = a.pos0 + q0 - (kt0 + kt) * KT;   // distance of the first row to the first key
            return bias || n < KT - 1 || n + QT - 1 >= a.window;
        };
        float next_bias = bias_at(0);
        bool ok = true;
        for (int kt = 0; kt < n_kt; ++kt) {
            const int b = kt & 1;
            float* bt = bars->bias[b];
            const bool slice = edges(kt);
            if (slice && tid < QT + KT - 1) bt[tid] = next_bias;
            if (kt + 1 < n_kt) next_bias = bias_at(kt + 1);
            ok = __all_sync(0xffffffffu, wait(&bars->s_full[b], (kt >> 1) & 1));
            uint32_t sr[HK];
            float mx = -INFINITY;
            if (ok) {
                fence_after();
                tmem_ld32(tmem + b * KT + hf * HK + lane_addr, sr);
                fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(&bars->s_empty[b]);
            }
            // one warp's timeout must not leave the others at a named barrier: everybody goes on to them, tile by tile, with
            // waits that the abort flag ends at once
            // (a slice's buffer is written again two tiles on, after o_done of this tile, which every warp's P precedes)
            if (slice) asm volatile("bar.sync 1, 256;" ::: "memory");
            if (ok) {
                if (slice) {
#pragma unroll
                    for (int j = 0; j < HK; ++j) sr[j] = __float_as_uint(__uint_as_float(sr[j]) + bt[r + (KT - 1) - hf * HK - j]);
                }
#pragma unroll
                for (int j = 0; j < HK; ++j) mx = fmaxf(mx, __uint_as_float(sr[j]));
                bars->half[b][hf][r] = mx;
            }
            // the two warps of these 32 rows
            asm volatile("bar.sync %0, 64;" ::"r"(2 + (warp & 3)) : "memory");
            if (ok) mx = fmaxf(mx, bars->half[b][hf ^ 1][r]);
            if (ok && kt > 0) ok = wait(&bars->o_done, (kt - 1) & 1);     // P may be overwritten, O holds tiles 0 .. kt - 1
            ok = __all_sync(0xffffffffu, ok);
            if (ok) {
                fence_after();
                const bool grow = mx > m + GROW;
                if (__any_sync(0xffffffffu, grow)) {
                    const float mn = grow ? mx : m, corr = ex2_approx(m - mn);
                    l *= corr;
                    m = mn;
                    if (kt > 0)
                        for (int c = hf; c < 2 * a.nv; c += 2) {
                            uint32_t o[32];
                            tmem_ld32(tmem_o + c * 32 + lane_addr, o);
#pragma unroll
                            for (int i = 0; i < 32; ++i) o[i] = __float_as_uint(__uint_as_float(o[i]) * corr);
                            tmem_st32(tmem_o + c * 32 + lane_addr, o);
                        }
                }
                float ps = 0.0f;
#pragma unroll
                for (int c = 0; c < HK / 8; ++c) {
                    float p[8];
#pragma unroll
                    for (int e = 0; e < 8; ++e) { p[e] = ex2_approx(__uint_as_float(sr[8 * c + e]) - m); ps += p[e]; }
                    uint4 hi, lo;
                    split2(p[0], p[1], &hi.x, &lo.x);
                    split2(p[2], p[3], &hi.y, &lo.y);
                    split2(p[4], p[5], &hi.z, &lo.z);
                    split2(p[6], p[7], &hi.w, &lo.w);
                    const int chunk = ((hf * (HK / 8) + c) ^ (r & 7)) * 16;
                    *(uint4*)(ph + chunk) = hi;
                    *(uint4*)(pl + chunk) = lo;
                }
                l += ps;
                asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
                fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(&bars->p_full);
            }
        }
        ok = __all_sync(0xffffffffu, wait(&bars->o_done, (n_kt - 1) & 1) && ok && !bars->abort);
        bars->half[n_kt & 1][hf][r] = l;                   // not the buffer of the last tile's maxima
        asm volatile("bar.sync %0, 64;" ::"r"(2 + (warp & 3)) : "memory");
        if (ok) {
            fence_after();
            const float inv = 1.0f / (bars->half[n_kt & 1][0][r] + bars->half[n_kt & 1][1][r]);
            const bool store = q0 + r < a.M, vec = (a.vdim & 7) == 0 && (a.ldo & 7) == 0;
            uint16_t* dst = a.out + (size_t)(q0 + r) * a.ldo + (size_t)h * a.vdim;
            for (int c = hf; c < 2 * a.nv; c += 2) {
                if (c * 32 >= a.vdim) break;
                uint32_t o[32];
                tmem_ld32(tmem_o + c * 32 + lane_addr, o);
                if (store) {
                    if (vec) {
#pragma unroll
                        for (int i = 0; i < 4; ++i)
                            if (c * 32 + 8 * i < a.vdim) {
                                uint4 w;
                                w.x = pack2(__uint_as_float(o[8 * i]) * inv, __uint_as_float(o[8 * i + 1]) * inv);
                                w.y = pack2(__uint_as_float(o[8 * i + 2]) * inv, __uint_as_float(o[8 * i + 3]) * inv);
                                w.z = pack2(__uint_as_float(o[8 * i + 4]) * inv, __uint_as_float(o[8 * i + 5]) * inv);
                                w.w = pack2(__uint_as_float(o[8 * i + 6]) * inv, __uint_as_float(o[8 * i + 7]) * inv);
                                *(uint4*)(dst + c * 32 + 8 * i) = w;
                            }
                    } else {
#pragma unroll
                        for (int i = 0; i < 32; ++i)
                            if (c * 32 + i < a.vdim) dst[c * 32 + i] = __bfloat16_as_ushort(__float2bfloat16_rn(__uint_as_float(o[i]) * inv));
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
        tmem_dealloc(tmem, a.tmem_cols);
    }
}

int launch_flash_tc(const Flash& f, const void* q, int M, int pos0, void* out, int ldo, int* status, cudaStream_t st) {
    const int w0 = f.k0.width, w1 = f.k1.p ? f.k1.width : 0;
    if (f.vdim > 256) return fail(FC_E_SHAPE, "value heads of %d do not fit the tensor-core attention", f.vdim);
    if (w0 <= 0 || w0 % 16 || w1 % 16 || f.k0.col % 16 || f.k0.head_stride % 16 || f.k1.col % 16 || f.v.head_stride % 16 || f.v.width % 16)
        return fail(FC_E_SHAPE, "tensor-core attention: key parts of %d and %d columns", w0, w1);
    Args a = {};
    a.nc0 = (w0 + CH - 1) / CH;
    const int nc1 = (w1 + CH - 1) / CH;
    a.nkc = a.nc0 + nc1;
    a.last0 = (w0 - (a.nc0 - 1) * CH) / 16;
    a.last1 = nc1 ? (w1 - (nc1 - 1) * CH) / 16 : a.last0;
    a.nv = (f.v.width + CH - 1) / CH;
    a.ks = plan_stages(a.nkc, a.nv, false);
    if (!a.ks) { a.q_stream = 1; a.ks = plan_stages(a.nkc, a.nv, true); }
    static bool attr_set[64] = {};
    int dev = 0;
    FC_CUDA(cudaGetDevice(&dev));
    if (dev < 64 && !attr_set[dev]) {
        FC_CUDA(cudaFuncSetAttribute(flash_tc_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        attr_set[dev] = true;
    }
    CUtensorMap mq, mk0, mk1, mv;
    a.kq = w0 + w1;
    FC_TRY(encode_bf16(&mq, q, M, (size_t)f.H * a.kq, (size_t)f.H * a.kq, QT));
    FC_TRY(encode_bf16(&mk0, f.k0.p, f.k0.rows, f.k0.ld, f.k0.ld, KT));
    mk1 = mk0;
    if (w1) FC_TRY(encode_bf16(&mk1, f.k1.p, f.k1.rows, f.k1.ld, f.k1.ld, KT));
    FC_TRY(encode_bf16(&mv, f.v.p, f.v.rows, f.v.ld, f.v.ld, KT));
    a.M = M; a.pos0 = pos0; a.H = f.H; a.KV = f.KV; a.vdim = f.vdim; a.far = f.far; a.ldo = ldo; a.window = f.window; a.w0 = w0;
    a.k0_col = f.k0.col; a.k0_head = f.k0.head_stride; a.k0_base = f.k0.pos0; a.k1_col = f.k1.col; a.k1_base = f.k1.pos0;
    a.v_col = f.v.col; a.v_head = f.v.head_stride; a.v_base = f.v.pos0;
    a.bias = f.bias; a.has_sink = f.has_sink; a.sink = f.sink; a.out = (uint16_t*)out; a.status = status;
    a.wait_cycles = g_debug.wait_cycles; a.withhold = g_debug.withhold;
    a.tmem_cols = a.nv <= 2 ? 256 : 512;
    flash_tc_kernel<<<dim3(f.H, (M + QT - 1) / QT), THREADS, smem_bytes(a.nkc, a.ks, a.nv, a.q_stream), st>>>(mq, mk0, mk1, mv, a);
    FC_LAUNCHED();
    return FC_OK;
}

}  // namespace fc
