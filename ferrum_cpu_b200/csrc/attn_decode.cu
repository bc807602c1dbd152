// Attention of one decoded token over the cached rows its window reaches.
//
//   attn_decode_kernel     the rows are cut into splits, one CTA each per block of at most 16 heads that read the same key/value
//                          head: a tile of rows goes to shared memory (cp.async), a thread takes a row (or a piece of it) and
//                          four heads for the scores, two columns and four heads for the values. Grouped-query layers prepare
//                          their queries and the token's own row here (norm, rotation), and the last split of a block to
//                          finish (an atomic counter, no waiting) merges in split order. Scores, softmax, sums are f32.
//   latent_absorb_kernel   latent layers ahead of it: a head's query through W_uk^T, so that all heads meet the cached latents
//                          themselves (one key row shared by all, its first part the value row too); the token's cache row
//   latent_expand_kernel   and behind it: splits merged, the head's sum of latents through W_uv
//
// Launched as programmatic dependents. Every kernel of the step lets its successor start only after its own wait, so cached rows
// of earlier tokens and weights are asked for before the wait.
//
// Bound: HBM / latency (cached rows once per block of heads, W_uk and W_uv once).
#include <cooperative_groups.h>

#include <algorithm>

#include "pdl.cuh"
#include "rot_rows.cuh"

namespace fc {

namespace {
constexpr int NT = 256, HB = 16, PER = 4;

// What a launch derives from the sizes: rows of a tile, heads of a block (and up to fours), parts a key row and a tile's rows are
// cut into so that all threads have work, bytes of a staged row.
struct Plan {
    int kt, hb, hb4, nb, np, nkp, krow, vrow, vw4;
    int q, k, v, raw, p, acc, ml, cs, bytes;     // offsets into shared memory
};
bool plan_of(const AttnDecode& a, int kt, Plan* o) {
    const int e = a.f32 ? 4 : 2, per = a.H / a.KV;
    Plan& l = *o;
    l.kt = kt;
    l.hb = std::min(per, HB);
    l.nb = (per + HB - 1) / HB;
    const int ng = (l.hb + PER - 1) / PER;
    l.hb4 = ng * PER;
    l.np = std::max(1, std::min(8, NT / (kt * ng)));
    l.vw4 = (a.vw + 3) / 4 * 4;
    l.nkp = std::max(1, std::min(8, NT / (ng * ((a.vw + 1) / 2))));
    l.krow = a.kw * e + 16;
    l.vrow = a.vc ? (a.vw + 7) / 8 * 8 * e + 16 : l.krow;
    int at = 0;
    auto take = [&](int bytes) { const int x = at; at += (bytes + 15) / 16 * 16; return x; };
    l.q = take(l.hb4 * a.kw * 4);
    l.k = take(kt * l.krow);
    l.v = a.vc ? take(kt * l.vrow) : l.k;
    l.raw = take(std::max(l.np * l.hb4 * (kt + 1), l.hb4 * kMaxSplitsRow) * 4);
    l.p = take(kt * (l.hb4 + 4) * 4);
    l.acc = take(l.nkp * l.hb4 * l.vw4 * 4);
    l.ml = take(l.hb4 * 3 * 4);
    l.cs = take(a.prep.rot.dims / 2 * 8);
    l.bytes = at;
    return at <= 200 * 1024;
}
int make_plan(const AttnDecode& a, Plan* l) {
    // the smallest tile with which the splits reach every visible row; several tiles a split where that is too large
    int want = 16;
    while (want < 64 && want * a.max_splits < a.reach) want *= 2;
    for (int kt = want; kt >= 16; kt /= 2)
        if (plan_of(a, kt, l)) return FC_OK;
    return fail(FC_E_SHAPE, "decode attention: rows of %d values do not fit shared memory", a.kw);
}
// Rows [begin, end) of split sp; splits: how many there are.
struct Range { int splits, begin, end; };
__device__ __forceinline__ Range range_of(int len, int window, int kt, int max_splits, int sp) {
    const int visible = min(len, window), splits = min(max_splits, (visible + kt - 1) / kt), per = (visible + splits - 1) / splits;
    const int b = len - visible + sp * per;
    return {splits, b, min(len, b + per)};
}

template <class T> constexpr int kVec = 16 / sizeof(T);
template <class T>
__device__ __forceinline__ void unpack(const uint4& w, float* x) {
    const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        if constexpr (sizeof(T) == 2) { x[2 * i] = __uint_as_float(u[i] << 16); x[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u); }
        else x[i] = __uint_as_float(u[i]);
    }
}
__device__ __forceinline__ void copy16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ float warp_max(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v = fmaxf(v, __shfl_xor_sync(0xffffffffu, v, o));
    return v;
}
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Weights of at most kMaxSplitsRow splits of head h, normalised: lane's two into w.
__device__ __forceinline__ void split_weights(const float* part_ml, int H, int h, int splits, bool has_sink, float* w) {
    const int lane = threadIdx.x & 31;
    float mv[2], lv[2];
#pragma unroll
    for (int y = 0; y < 2; ++y) {
        const int s = lane + 32 * y;
        mv[y] = s < splits ? __ldcg(part_ml + ((size_t)s * H + h) * 2) : -INFINITY;
        lv[y] = s < splits ? __ldcg(part_ml + ((size_t)s * H + h) * 2 + 1) : 0.0f;
    }
    float m = warp_max(fmaxf(mv[0], mv[1]));
    if (has_sink) m = fmaxf(m, 0.0f);
    const float w0 = expf(mv[0] - m), w1 = expf(mv[1] - m);
    const float l = warp_sum(w0 * lv[0] + w1 * lv[1]) + (has_sink ? expf(-m) : 0.0f);
    w[0] = w0 / l;
    w[1] = w1 / l;
}
}  // namespace

template <class T>
__global__ void __launch_bounds__(NT) attn_decode_kernel(const __grid_constant__ AttnDecode a, const Plan l) {
    extern __shared__ __align__(16) unsigned char sm[];
    __shared__ float red[NT / 32];
    __shared__ bool is_last;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, kw = a.kw, vw = a.vw, per = a.H / a.KV;
    const int c = blockIdx.y / l.nb, hk = blockIdx.y - c * l.nb, h0 = c * per + hk * HB, nh = min(HB, per - hk * HB);
    float* q = (float*)(sm + l.q);                 // [hb4][kw]
    float* raw = (float*)(sm + l.raw);             // [np][hb4][kt + 1]
    float* p = (float*)(sm + l.p);                 // [kt][hb4 + 4]
    float* acc = (float*)(sm + l.acc);             // [nkp][hb4][vw4]
    float* ml = (float*)(sm + l.ml);               // [hb4][3]: max, sum, correction
    float2* cs = (float2*)(sm + l.cs);
    const RotAttn& t = a.prep;
    const int pos = a.state->pos, len = pos + 1;   // as the kernels of the step before left it
    const Range r = range_of(len, a.window, l.kt, a.max_splits, blockIdx.x);
    const bool live = (int)blockIdx.x < r.splits && r.begin < r.end;
    const char* kbase = (const char*)((const T*)a.kc + (size_t)c * a.k_head);
    const char* vbase = a.vc ? (const char*)((const T*)a.vc + (size_t)c * a.v_head) : nullptr;
    const int kv16 = kw * (int)sizeof(T) / 16, vv16 = a.vc ? (l.vrow - 16) / 16 : 0;
    auto stage = [&](int k0, int from, int to) {   // rows from .. to - 1 of the tile that begins at k0
        const int n = to - from;
        for (int i = tid; i < n * kv16; i += NT) {
            const int j = i / kv16, e = i - j * kv16;
            copy16(sm + l.k + (from + j - k0) * l.krow + e * 16, kbase + (size_t)(from + j) * a.k_ld * sizeof(T) + e * 16);
        }
        for (int i = tid; i < n * vv16; i += NT) {
            const int j = i / vv16, e = i - j * vv16;
            copy16(sm + l.v + (from + j - k0) * l.vrow + e * 16, vbase + (size_t)(from + j) * a.v_ld * sizeof(T) + e * 16);
        }
    };
    if (live) stage(r.begin, r.begin, min(min(r.end, r.begin + l.kt), pos));
    for (int i = tid; i < l.hb4; i += NT) { ml[3 * i] = -1e30f; ml[3 * i + 1] = 0.0f; ml[3 * i + 2] = 0.0f; }
    for (int i = tid; i < t.rot.dims / 2; i += NT) cs[i] = rot_cs(pos, t.rot.freq[i]);
    pdl_wait();
    pdl_trigger();
    if (a.state->done | a.state->error) return;
    if ((int)blockIdx.x >= r.splits) return;
    const bool own = live && r.end == len;         // the split that holds the token's own row
    if (t.H) {
        const int qn = t.H * t.dim, kn = t.KV * t.dim;
        float inv = t.scale;
        if (t.q_norm) {
            float s = 0.0f;
#pragma unroll 8
            for (int i = tid; i < qn; i += NT) s = fmaf(a.q[i], a.q[i], s);
            inv = t.scale / sqrtf(block_sum_of<NT>(s, red) / (float)qn + t.eps);
        }
        __syncthreads();                           // cs
        for (int h = warp; h < l.hb4; h += NT / 32) {
            const float* x = a.q + (size_t)(h0 + h) * t.dim;
            const float* w = t.q_norm + (size_t)(h0 + h) * t.dim;
#pragma unroll 4
            for (int e = lane; e < kw; e += 32)
                q[h * kw + e] = h < nh && e < t.dim ? rotated(t.rot.neighbours, t.rot.dims, cs, e, [&](int k) { return x[k] * (t.q_norm ? w[k] : 1.0f); }) * inv : 0.0f;
        }
        if (own && t.own_kv) {
            float ki = 1.0f;
            if (t.k_norm) {
                float s = 0.0f;
                for (int i = tid; i < kn; i += NT) s = fmaf(a.q[qn + i], a.q[qn + i], s);
                ki = 1.0f / sqrtf(block_sum_of<NT>(s, red) / (float)kn + t.eps);
            }
            const float* x = a.q + qn + (size_t)c * t.dim;
            const float* w = t.k_norm + (size_t)c * t.dim;
            T* kr = (T*)a.kc + (size_t)pos * a.k_ld + (size_t)c * a.k_head;
            for (int e = tid; e < kw; e += NT) {
                const float v = e < t.dim ? rotated(t.rot.neighbours, t.rot.dims, cs, e, [&](int k) { return x[k] * (t.k_norm ? w[k] : 1.0f); }) * ki : 0.0f;
                if (hk == 0) put_row(kr + e, v);
                if (r.end - r.begin <= l.kt) put_row((T*)(sm + l.k + (pos - r.begin) * l.krow) + e, v);
            }
            T* vr = (T*)a.vc + (size_t)pos * a.v_ld + (size_t)c * a.v_head;
            for (int e = tid; e < t.vp; e += NT) {
                const float v = e < t.vdim ? a.q[qn + kn + (size_t)c * t.vdim + e] : 0.0f;
                if (hk == 0) put_row(vr + e, v);
                if (r.end - r.begin <= l.kt && e < (l.vrow - 16) / (int)sizeof(T)) put_row((T*)(sm + l.v + (pos - r.begin) * l.vrow) + e, v);
            }
        }
    } else {
        const float4* src = (const float4*)(a.q + (size_t)h0 * kw);      // kw is a multiple of 8
#pragma unroll 4
        for (int i = tid; i < l.hb4 * kw / 4; i += NT) ((float4*)q)[i] = i < nh * kw / 4 ? src[i] : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    }
    const bool self = own && t.H && t.own_kv;      // the own row does not come from the cache when one tile holds the split
    const int ng = l.hb4 / PER, pst = l.hb4 + 4;
    // one tile, one piece of its rows, and splits to be merged: the values go from the registers to where they are merged
    const bool straight = r.end - r.begin <= l.kt && l.nkp == 1 && !(a.counter && r.splits == 1);
    for (int k0 = r.begin; k0 < r.end; k0 += l.kt) {
        const int nk = min(l.kt, r.end - k0);
        if (k0 > r.begin) {
            __syncthreads();
            const int to = k0 + nk;
            stage(k0, k0, to == len ? pos : to);
        }
        if (k0 + nk == len) {
            if (!self) stage(k0, pos, len);
            else if (r.end - r.begin > l.kt) {     // a later tile: the row again
                const int qn = t.H * t.dim, kn = t.KV * t.dim;
                float s = 0.0f, ki = 1.0f;
                if (t.k_norm) {
                    for (int i = tid; i < kn; i += NT) s = fmaf(a.q[qn + i], a.q[qn + i], s);
                    ki = 1.0f / sqrtf(block_sum_of<NT>(s, red) / (float)kn + t.eps);
                }
                const float* x = a.q + qn + (size_t)c * t.dim;
                const float* w = t.k_norm + (size_t)c * t.dim;
                for (int e = tid; e < kw; e += NT)
                    put_row((T*)(sm + l.k + (pos - k0) * l.krow) + e,
                            e < t.dim ? rotated(t.rot.neighbours, t.rot.dims, cs, e, [&](int k) { return x[k] * (t.k_norm ? w[k] : 1.0f); }) * ki : 0.0f);
                for (int e = tid; e < (l.vrow - 16) / (int)sizeof(T); e += NT)
                    put_row((T*)(sm + l.v + (pos - k0) * l.vrow) + e, e < t.vdim ? a.q[qn + kn + (size_t)c * t.vdim + e] : 0.0f);
            }
        }
        asm volatile("cp.async.wait_all;" ::: "memory");
        __syncthreads();
        // scores: row j, heads 4 g .. 4 g + 3, piece s of the row
        for (int i = tid; i < l.kt * ng * l.np; i += NT) {
            const int j = i % l.kt, gs = i / l.kt, g = gs % ng, s = gs / ng;
            if (j >= nk) continue;
            constexpr int V = kVec<T>;
            const int nv = kw / V, v0 = nv * s / l.np, v1 = nv * (s + 1) / l.np;
            const unsigned char* kr = sm + l.k + j * l.krow;
            const float* qg = q + g * PER * kw;
            float d[PER] = {};
#pragma unroll 2
            for (int v = v0; v < v1; ++v) {
                float x[V];
                unpack<T>(*(const uint4*)(kr + v * 16), x);
#pragma unroll
                for (int y = 0; y < PER; ++y)
#pragma unroll
                    for (int e = 0; e < V; e += 4) {
                        const float4 qq = *(const float4*)(qg + y * kw + v * V + e);
                        d[y] = fmaf(qq.x, x[e], d[y]); d[y] = fmaf(qq.y, x[e + 1], d[y]);
                        d[y] = fmaf(qq.z, x[e + 2], d[y]); d[y] = fmaf(qq.w, x[e + 3], d[y]);
                    }
            }
#pragma unroll
            for (int y = 0; y < PER; ++y) raw[(s * l.hb4 + g * PER + y) * (l.kt + 1) + j] = d[y];
        }
        __syncthreads();
        for (int h = warp; h < l.hb4; h += NT / 32) {
            float b[2];
#pragma unroll
            for (int y = 0; y < 2; ++y) {
                const int j = lane + 32 * y;
                b[y] = j < nk ? 0.0f : -INFINITY;
                if (j < nk)
                    for (int s = 0; s < l.np; ++s) b[y] += raw[(s * l.hb4 + h) * (l.kt + 1) + j];
            }
            const float m0 = ml[3 * h], mn = fmaxf(m0, warp_max(fmaxf(b[0], b[1])));
            const float p0 = expf(b[0] - mn), p1 = expf(b[1] - mn);
            if (lane < l.kt) p[lane * pst + h] = p0;
            if (lane + 32 < l.kt) p[(lane + 32) * pst + h] = p1;
            const float ps = warp_sum(p0 + p1);
            __syncwarp();
            if (lane == 0) {
                const float corr = expf(m0 - mn);
                ml[3 * h] = mn;
                ml[3 * h + 1] = fmaf(ml[3 * h + 1], corr, ps);
                ml[3 * h + 2] = corr;
            }
        }
        __syncthreads();
        // values: columns 2 u and 2 u + 1, heads 4 g .., rows of piece s
        const int up = (vw + 1) / 2;
        for (int i = tid; i < up * ng * l.nkp; i += NT) {
            const int u = i % up, gs = i / up, g = gs % ng, s = gs / ng, j1 = nk * (s + 1) / l.nkp;
            const T* v = (const T*)(sm + l.v) + 2 * u;
            float o[PER][2] = {};
#pragma unroll 4
            for (int j = nk * s / l.nkp; j < j1; ++j) {
                const T* vr = (const T*)((const unsigned char*)v + j * l.vrow);
                float x, y;
                if constexpr (sizeof(T) == 2) {
                    const uint32_t w = *(const uint32_t*)vr;
                    x = __uint_as_float(w << 16); y = __uint_as_float(w & 0xffff0000u);
                } else {
                    const float2 w = *(const float2*)vr;
                    x = w.x; y = w.y;
                }
                const float4 pp = *(const float4*)(p + j * pst + g * PER);
                o[0][0] = fmaf(pp.x, x, o[0][0]); o[0][1] = fmaf(pp.x, y, o[0][1]);
                o[1][0] = fmaf(pp.y, x, o[1][0]); o[1][1] = fmaf(pp.y, y, o[1][1]);
                o[2][0] = fmaf(pp.z, x, o[2][0]); o[2][1] = fmaf(pp.z, y, o[2][1]);
                o[3][0] = fmaf(pp.w, x, o[3][0]); o[3][1] = fmaf(pp.w, y, o[3][1]);
            }
#pragma unroll
            for (int y = 0; y < PER; ++y) {
                const int h = g * PER + y;
                if (straight) {
                    if (h < nh) *(float2*)(a.part + ((size_t)blockIdx.x * a.H + h0 + h) * l.vw4 + 2 * u) = make_float2(o[y][0], o[y][1]);
                    continue;
                }
                float2* to = (float2*)(acc + ((size_t)s * l.hb4 + h) * l.vw4 + 2 * u);
                if (k0 == r.begin) {
                    *to = make_float2(o[y][0], o[y][1]);
                } else {
                    const float corr = ml[3 * h + 2];
                    *to = make_float2(fmaf(to->x, corr, o[y][0]), fmaf(to->y, corr, o[y][1]));
                }
            }
        }
    }
    __syncthreads();
    auto total = [&](int h, int e) {
        float o = 0.0f;
        for (int s = 0; s < l.nkp; ++s) o += acc[((size_t)s * l.hb4 + h) * l.vw4 + e];
        return o;
    };
    if (a.counter && r.splits == 1) {
        for (int i = tid; i < nh * vw; i += NT) {
            const int h = i / vw;
            const float m0 = ml[3 * h], m = a.has_sink ? fmaxf(m0, 0.0f) : m0, w = expf(m0 - m);
            a.out[(size_t)h0 * vw + i] = total(h, i - h * vw) * w / fmaf(ml[3 * h + 1], w, a.has_sink ? expf(-m) : 0.0f);
        }
        return;
    }
    const size_t sp = blockIdx.x;
    if (!straight || !live)
        for (int i = tid; i < nh * l.vw4; i += NT) {
            const int h = i / l.vw4, e = i - h * l.vw4;
            a.part[(sp * a.H + h0 + h) * l.vw4 + e] = live && e < vw ? total(h, e) : 0.0f;
        }
    for (int h = tid; h < nh; h += NT) {
        a.part_ml[(sp * a.H + h0 + h) * 2] = ml[3 * h];
        a.part_ml[(sp * a.H + h0 + h) * 2 + 1] = ml[3 * h + 1];
    }
    if (!a.counter) return;
    __threadfence();
    __syncthreads();
    if (tid == 0) is_last = atomicAdd(a.counter + blockIdx.y, 1u) == (unsigned)(r.splits - 1);
    __syncthreads();
    if (!is_last) return;
    __threadfence();
    if (tid == 0) a.counter[blockIdx.y] = 0;
    for (int h = warp; h < nh; h += NT / 32) {
        float w[2];
        split_weights(a.part_ml, a.H, h0 + h, r.splits, a.has_sink, w);
        raw[h * kMaxSplitsRow + lane] = w[0];
        raw[h * kMaxSplitsRow + lane + 32] = w[1];
    }
    __syncthreads();
    for (int i = tid; i < nh * vw; i += NT) {
        const int h = i / vw, e = i - h * vw;
        float o = 0.0f;
#pragma unroll 8
        for (int s = 0; s < r.splits; ++s) o = fmaf(raw[h * kMaxSplitsRow + s], __ldcg(a.part + ((size_t)s * a.H + h0 + h) * l.vw4 + e), o);
        a.out[(size_t)h0 * vw + i] = o;
    }
}

int attn_decode_blocks(const AttnDecode& a) { return a.KV * ((a.H / a.KV + HB - 1) / HB); }

int launch_attn_decode_rows(const AttnDecode& a, cudaStream_t st) {
    Plan l;
    if (a.max_splits > kMaxSplitsRow) return fail(FC_E_SHAPE, "%d attention splits (at most %d)", a.max_splits, kMaxSplitsRow);
    if (a.kw % 8 || (!a.vc && a.vw > a.kw)) return fail(FC_E_SHAPE, "decode attention: key rows of %d values", a.kw);
    FC_TRY(make_plan(a, &l));
    if (l.bytes > 47 * 1024) {
        FC_CUDA(cudaFuncSetAttribute(attn_decode_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        FC_CUDA(cudaFuncSetAttribute(attn_decode_kernel<uint16_t>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    }
    const dim3 grid(a.max_splits, attn_decode_blocks(a));
    if (a.f32) FC_CUDA(launch_pdl(attn_decode_kernel<float>, grid, dim3(NT), (size_t)l.bytes, st, a, l));
    else FC_CUDA(launch_pdl(attn_decode_kernel<uint16_t>, grid, dim3(NT), (size_t)l.bytes, st, a, l));
    ++g_launches;
    return FC_OK;
}

// ------------------------------------------------------------------------------------------ latent layers
namespace {
constexpr int RC = 128, SL = NT / (RC / 8), DPRE = 8;   // latents of a CTA, slices of the head's dimensions, rows loaded ahead of the wait
}
template <class T>
__global__ void __launch_bounds__(NT) latent_absorb_kernel(const LatentAttn t, const float* __restrict__ proj, float* __restrict__ q, T* cache,
                                                           const StepState* state) {
    extern __shared__ __align__(16) float smf[];        // query [dim], partial sums [SL][RC]; or cos / sin pairs
    __shared__ float red[NT / 32];
    const int tid = threadIdx.x, h = blockIdx.y, chunk = blockIdx.x, rot = t.rot.dims, hq = t.dim + rot, kw = t.lat + t.rot_p;
    const float* qh = proj + (size_t)h * hq;
    if (chunk * RC < t.lat) {
        const int r8 = chunk * RC + (tid % (RC / 8)) * 8, sl = tid / (RC / 8);
        const bool mine = r8 < t.lat;
        const uint16_t* w = t.uk + (size_t)h * t.dp * t.lat + r8;
        uint4 pre[DPRE];
#pragma unroll
        for (int i = 0; i < DPRE; ++i) pre[i] = mine && sl + i * SL < t.dim ? *(const uint4*)(w + (size_t)(sl + i * SL) * t.lat) : make_uint4(0, 0, 0, 0);
        pdl_wait();
        pdl_trigger();
        if (state->done | state->error) return;
        float* part = smf + (t.dim + 3) / 4 * 4;
        for (int i = tid; i < t.dim; i += NT) smf[i] = qh[i];
        __syncthreads();
        float s[8] = {};
        auto add = [&](const uint4& v, float x) {
            float k[8];
            unpack<uint16_t>(v, k);
#pragma unroll
            for (int e = 0; e < 8; ++e) s[e] = fmaf(x, k[e], s[e]);
        };
#pragma unroll
        for (int i = 0; i < DPRE; ++i)
            if (sl + i * SL < t.dim) add(pre[i], smf[sl + i * SL]);
        if (mine)
            for (int d = sl + DPRE * SL; d < t.dim; d += SL) add(*(const uint4*)(w + (size_t)d * t.lat), smf[d]);
#pragma unroll
        for (int e = 0; e < 8; ++e) part[sl * RC + (tid % (RC / 8)) * 8 + e] = s[e];
        __syncthreads();
        if (tid < RC && chunk * RC + tid < t.lat) {
            float o = 0.0f;
#pragma unroll
            for (int i = 0; i < SL; ++i) o += part[i * RC + tid];
            q[(size_t)h * kw + chunk * RC + tid] = o * t.scale;
        }
        return;
    }
    const int pos = state->pos;
    float2* cs = (float2*)smf;
    for (int i = tid; i < rot / 2; i += NT) cs[i] = rot_cs(pos, t.rot.freq[i]);
    pdl_wait();
    pdl_trigger();
    if (state->done | state->error) return;
    __syncthreads();
    for (int r = tid; r < t.rot_p; r += NT)
        q[(size_t)h * kw + t.lat + r] = r < rot ? rotated(t.rot.neighbours, rot, cs, r, [&](int k) { return qh[t.dim + k]; }) * t.scale : 0.0f;
    if (h) return;
    const float* lat = proj + (size_t)t.H * hq;
    float s = 0.0f;
    for (int i = tid; i < t.rank; i += NT) s = fmaf(lat[i], lat[i], s);
    const float inv = 1.0f / sqrtf(block_sum_of<NT>(s, red) / (float)t.rank + t.eps);
    T* to = cache + (size_t)pos * kw;
    for (int i = tid; i < t.lat; i += NT) put_row(to + i, i < t.rank ? lat[i] * inv * t.c_norm[i] : 0.0f);
    for (int r = tid; r < t.rot_p; r += NT)
        put_row(to + t.lat + r, r < rot ? rotated(t.rot.neighbours, rot, cs, r, [&](int k) { return lat[t.rank + k]; }) : 0.0f);
}
int launch_latent_absorb(const LatentAttn& t, const float* proj, float* q, void* cache, bool f32, const StepState* state, cudaStream_t st) {
    const size_t smem = std::max<size_t>(((size_t)(t.dim + 3) / 4 * 4 + SL * RC) * 4, (size_t)t.rot.dims / 2 * 8);
    if (smem > 47 * 1024) return fail(FC_E_SHAPE, "latent attention: heads of %d dimensions", t.dim);
    const dim3 grid((t.lat + RC - 1) / RC + 1, t.H);
    if (f32) FC_CUDA(launch_pdl(latent_absorb_kernel<float>, grid, dim3(NT), smem, st, t, proj, q, (float*)cache, state));
    else FC_CUDA(launch_pdl(latent_absorb_kernel<uint16_t>, grid, dim3(NT), smem, st, t, proj, q, (uint16_t*)cache, state));
    ++g_launches;
    return FC_OK;
}

namespace {
constexpr int VC = 32, kMaxCluster = 8;                 // value rows of a CTA; CTAs of a head
}
// The CTAs of a head form a cluster: each merges a share of the latents and hands it to the others' shared memory, then
// multiplies its own value rows.
__global__ void __launch_bounds__(NT) latent_expand_kernel(const LatentAttn t, const __grid_constant__ AttnDecode a, int kt, float* __restrict__ out) {
    extern __shared__ __align__(16) float smf[];        // sum of latents [lat], partial sums [4 NT]
    __shared__ float wgt[kMaxSplitsRow];
    namespace cg = cooperative_groups;
    cg::cluster_group cluster = cg::this_cluster();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, n = gridDim.x, v0 = blockIdx.x * VC, nv = min(VC, t.vdim - v0);
    const uint16_t* w = t.uv + ((size_t)h * t.vp + v0) * t.lat;
    for (int i = tid * 64; i < nv * t.lat; i += NT * 64) asm volatile("prefetch.global.L2 [%0];" ::"l"(w + i));
    for (int i = t.rank + tid; i < t.lat; i += NT) smf[i] = 0.0f;
    const Range r = range_of(a.state->pos + 1, a.window, kt, a.max_splits, 0);
    pdl_wait();
    pdl_trigger();
    if (a.state->done | a.state->error) return;         // the same in every CTA
    if (warp == 0) {
        float x[2];
        split_weights(a.part_ml, a.H, h, r.splits, a.has_sink, x);
        wgt[lane] = x[0];
        wgt[lane + 32] = x[1];
    }
    cluster.sync();                                     // weights; every CTA of the cluster runs
    // four latents a thread, the splits dealt out over what is left of the block
    const int vw4 = (a.vw + 3) / 4 * 4, n4 = vw4 / 4, u0 = n4 * (int)blockIdx.x / n, u1 = n4 * ((int)blockIdx.x + 1) / n;
    float* part = smf + t.lat;
    for (int ub = u0; ub < u1; ub += NT) {
        const int nu = min(NT, u1 - ub), lanes = NT / nu, sg = tid / nu, u = tid - sg * nu;
        if (sg < lanes) {
            float4 o = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 8
            for (int s = sg; s < r.splits; s += lanes) {
                const float4 x = __ldcg((const float4*)(a.part + ((size_t)s * a.H + h) * vw4 + (ub + u) * 4));
                o.x = fmaf(wgt[s], x.x, o.x); o.y = fmaf(wgt[s], x.y, o.y); o.z = fmaf(wgt[s], x.z, o.z); o.w = fmaf(wgt[s], x.w, o.w);
            }
            *(float4*)(part + (sg * nu + u) * 4) = o;
        }
        __syncthreads();
        for (int i = tid; i < nu * 4; i += NT) {
            float o = 0.0f;
            for (int s = 0; s < lanes; ++s) o += part[s * nu * 4 + i];
            const int at = ub * 4 + i;
            if (at < t.rank)
                for (int c = 0; c < n; ++c) cluster.map_shared_rank(smf, c)[at] = o;
        }
        __syncthreads();
    }
    cluster.sync();
#pragma unroll 4
    for (int v = warp; v < nv; v += NT / 32) {
        float s = 0.0f;
        for (int k = lane * 8; k < t.lat; k += 256) {
            float x[8];
            unpack<uint16_t>(*(const uint4*)(w + (size_t)v * t.lat + k), x);
            const float4 y = *(const float4*)(smf + k), z = *(const float4*)(smf + k + 4);
            s = fmaf(x[0], y.x, s); s = fmaf(x[1], y.y, s); s = fmaf(x[2], y.z, s); s = fmaf(x[3], y.w, s);
            s = fmaf(x[4], z.x, s); s = fmaf(x[5], z.y, s); s = fmaf(x[6], z.z, s); s = fmaf(x[7], z.w, s);
        }
        s = warp_sum(s);
        if (lane == 0) out[(size_t)h * t.vdim + v0 + v] = s;
    }
}
int launch_latent_expand(const LatentAttn& t, const AttnDecode& a, float* out, cudaStream_t st) {
    Plan l;
    FC_TRY(make_plan(a, &l));
    const int n = (t.vdim + VC - 1) / VC;
    const size_t smem = (size_t)(t.lat + 4 * NT) * 4;
    if (n > kMaxCluster || smem > 200 * 1024) return fail(FC_E_SHAPE, "latents of %d values, value heads of %d", t.rank, t.vdim);
    if (smem > 47 * 1024) FC_CUDA(cudaFuncSetAttribute(latent_expand_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    FC_CUDA(launch_pdl_cluster(latent_expand_kernel, dim3(n, t.H), dim3(NT), n, smem, st, t, a, l.kt, out));
    ++g_launches;
    return FC_OK;
}

}  // namespace fc
