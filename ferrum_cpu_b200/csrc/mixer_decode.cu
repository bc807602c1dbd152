// The two mixers of one decoded token in one launch.
//
// Attention (blocks rH ..): the cached keys are cut into splits, one CTA each, that compute the scores of ALL heads for
// their keys (the heads are mixed before the softmax), in tiles of 64 keys:
//   raw[g][j] = q_g . k_j   a thread takes one key and one key/value head: its part of the key row straight from the cache
//                           with 16-byte loads, against the queries of that head's group in shared memory
//   mixed[h][j] = sum_g talk[h][g] raw[g][j] + bias[h][i - j]     a warp takes four heads, a lane two keys
//   values: a thread takes two columns and half of the keys, with the weights of the group's heads
// The last split to finish (an atomic counter, no waiting) merges the partial results in split order and adds the sink.
// The split that holds the token's own position writes its key row and normed value row to the cache first.
//
// Recurrence (blocks 0 .. rH - 1): one head each: decay from the low-rank projection, o = (S + diag(u) k v^T)^T r,
// S <- diag(w) S + k v^T, head norm and gate. State and arithmetic are f32.
//
// Launched as a programmatic dependent. Every kernel of the step lets its successor start only after its own wait, so what
// kernels before the one ahead wrote (cached rows of earlier tokens, the state, the position) may be asked for before the
// wait: the splits prefetch their cache rows into L2, the recurrences load their state.
//
// Bound: HBM / latency (cache rows once, the recurrence states once in and out).
#include <algorithm>

#include "bf16_ops.cuh"
#include "pdl.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
constexpr int NT = 512, KT = 64, RST = KT + 1;
constexpr int PER = 4;                    // heads of a group served by one pass over a key part / value column
constexpr int SPRE = 16;                  // state values of a thread loaded ahead of the wait

template <class T>
__device__ __forceinline__ float get(const T* p) {
    if constexpr (sizeof(T) == 2) return __uint_as_float((uint32_t)*p << 16);
    else return *p;
}
template <class T>
__device__ __forceinline__ void put(T* p, float v) {
    if constexpr (sizeof(T) == 2) *p = __bfloat16_as_ushort(__float2bfloat16_rn(v));
    else *p = v;
}
// Values in 16 bytes of a cached row.
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
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ float block_sum(float v, float* red) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = red[0];
#pragma unroll
    for (int w = 1; w < NT / 32; ++w) t += red[w];
    return t;
}

__device__ void recurrence(const MixerDecode& a, float* sm) {
    __shared__ float red[NT / 32];
    const int head = blockIdx.x, D = a.rdim, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const size_t h0 = (size_t)head * D;
    float *r = sm, *k = r + D, *w = k + D, *v = w + D, *low = v + D, *part = low + a.rank;     // part [slices][D]
    // column j of the state, rows sl, sl + slices, ...
    const int slices = max(1, NT / D), j = tid % D, sl = tid / D;
    const bool mine = sl < slices;
    float* S = a.wkv_state + h0 * D + j;
    float pre[SPRE];
#pragma unroll
    for (int x = 0; x < SPRE; ++x) pre[x] = mine && sl + x * slices < D ? S[(size_t)(sl + x * slices) * D] : 0.0f;
    pdl_wait();
    pdl_trigger();
    if (a.state->done | a.state->error) return;
    for (int i = tid; i < a.rank; i += NT) low[i] = tanhf(a.w1[i]);
    float bonus = 0.0f;
    for (int i = tid; i < D; i += NT) {
        const float x = a.r[h0 + i], y = a.k[h0 + i];
        r[i] = x; k[i] = y; v[i] = a.v[h0 + i];
        bonus = fmaf(x * a.u[h0 + i], y, bonus);
    }
    bonus = block_sum(bonus, red);              // also the barrier in front of low
#pragma unroll 4
    for (int i = warp; i < D; i += NT / 32) {   // a warp per channel
        const uint16_t* row = a.w2 + (h0 + i) * a.w2_ld;
        float s = 0.0f;
        for (int c = lane; c < a.rank; c += 32) s = fmaf(get(row + c), low[c], s);
        s = warp_sum(s);
        if (lane == 0) w[i] = expf(-expf(s + a.w0[h0 + i]));
    }
    __syncthreads();
    if (mine) {
        const float vj = v[j];
        float o = 0.0f;
#pragma unroll
        for (int x = 0; x < SPRE; ++x) {
            const int i = sl + x * slices;
            if (i < D) {
                o = fmaf(pre[x], r[i], o);
                S[(size_t)i * D] = fmaf(w[i], pre[x], k[i] * vj);
            }
        }
#pragma unroll 4
        for (int i = sl + SPRE * slices; i < D; i += slices) {
            const float s = S[(size_t)i * D];
            o = fmaf(s, r[i], o);
            S[(size_t)i * D] = fmaf(w[i], s, k[i] * vj);
        }
        part[sl * D + j] = o;
    }
    __syncthreads();
    float o = 0.0f;
    if (tid < D) {
        for (int x = 0; x < slices; ++x) o += part[x * D + tid];
        o = fmaf(bonus, v[tid], o);
    }
    const float inv = 1.0f / sqrtf(block_sum(o * o, red) / (float)D + a.eps);
    if (tid < D) {
        const float z = a.g[h0 + tid];
        a.ro[h0 + tid] = o * inv * a.rnorm[h0 + tid] * (z / (1.0f + expf(-z)));
    }
}

// Dot products of the key part at kr (dim values) with PER queries: vectors of 16 bytes when `vec`.
template <class T>
__device__ __forceinline__ void scores_of(const T* kr, const float* q, int qst, int dim, bool vec, float (&s)[PER]) {
    constexpr int V = kVec<T>;
    if (vec) {
        constexpr int F = 8;                             // loads in flight
        for (int e0 = 0; e0 < dim; e0 += F * V) {
            uint4 w[F];
#pragma unroll
            for (int x = 0; x < F; ++x) w[x] = e0 + x * V < dim ? *(const uint4*)(kr + e0 + x * V) : make_uint4(0, 0, 0, 0);
#pragma unroll
            for (int x = 0; x < F; ++x)
                if (e0 + x * V < dim) {
                    float kv[V];
                    unpack<T>(w[x], kv);
#pragma unroll
                    for (int y = 0; y < PER; ++y)
#pragma unroll
                        for (int e = 0; e < V; e += 4) {
                            const float4 qq = *(const float4*)(q + y * qst + e0 + x * V + e);
                            s[y] = fmaf(qq.x, kv[e], s[y]); s[y] = fmaf(qq.y, kv[e + 1], s[y]);
                            s[y] = fmaf(qq.z, kv[e + 2], s[y]); s[y] = fmaf(qq.w, kv[e + 3], s[y]);
                        }
                }
        }
    } else {
        for (int e = 0; e < dim; ++e) {
            const float k = get(kr + e);
#pragma unroll
            for (int y = 0; y < PER; ++y) s[y] = fmaf(q[y * qst + e], k, s[y]);
        }
    }
}

template <class T>
__device__ void attention(const MixerDecode& a, float* sm) {
    __shared__ bool is_last;
    const TalkAttn& t = a.t;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, H = t.H, dim = t.dim, per = H / t.KV, width = t.KV * dim, vd = t.vdim;
    const int pos = a.state->pos, len = pos + 1;         // as the kernels of the step before left it
    const int splits = min(a.max_splits, (len + KT - 1) / KT), sp = blockIdx.x - a.rH;
    const int per_split = ((len + splits - 1) / splits + 15) & ~15;
    const int k_begin = sp * per_split, k_end = min(len, k_begin + per_split);
    T* kc = (T*)a.kc;
    T* vc = (T*)a.vc;
    const size_t vst = (size_t)t.KV * t.vp;
    if (sp < splits) {                                   // rows of earlier tokens, one request per 128 bytes
        const char* kb = (const char*)(kc + (size_t)k_begin * t.kd);
        const char* vb = (const char*)(vc + (size_t)k_begin * vst);
        const long long rows = max(0, min(k_end, pos) - k_begin);
        const long long kn = min(rows * t.kd * (long long)sizeof(T), 1LL << 18), vn = min(rows * (long long)vst * (long long)sizeof(T), 1LL << 18);
        for (long long i = tid * 128LL; i < kn; i += NT * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(kb + i));
        for (long long i = tid * 128LL; i < vn; i += NT * 128) asm volatile("prefetch.global.L2 [%0];" ::"l"(vb + i));
    }
    const int Hp = (H + 3) & ~3, qd = (dim + 3) & ~3, qg = per * qd + 4;     // groups of queries a few banks apart
    float* q = sm;                               // [KV][qg]: the queries of a group, then the next group's
    float* talk = q + t.KV * qg + PER * qd;      // [H][Hp], transposed: talk[g][h] (the gap: reads past a group's last query)
    float* raw = talk + H * Hp;                  // [H + PER][RST]
    float* mix = raw + (H + PER) * RST;          // [KT][Hp + 4]: weights of a key for all heads
    const int mst = Hp + 4;
    float* acc = mix + KT * mst;                 // [2][H][vd]: halves of the keys
    float* ml = acc + 2 * H * vd;                // [H][3]: max, sum, correction
    float* bsm = ml + 3 * H;                     // [H][RST]: bias of the tile's distances
    auto load_bias = [&](int k0) {
        for (int i = tid; i < H * KT; i += NT) {
            const int h = i / KT, j = i - h * KT;
            bsm[h * RST + j] = __ldg(t.bias + (size_t)h * (t.far + 1) + min(max(pos - (k0 + j), 0), t.far));
        }
    };
    if (sp < splits) load_bias(k_begin);
    for (int i = tid; i < H * H; i += NT) { const int h = i / H, g = i - h * H; talk[g * Hp + h] = t.talk[i]; }
    for (int i = tid; i < 2 * H * vd; i += NT) acc[i] = 0.0f;
    for (int h = tid; h < H; h += NT) { ml[3 * h] = -INFINITY; ml[3 * h + 1] = 0.0f; ml[3 * h + 2] = 0.0f; }
    for (int i = tid; i < PER * qd; i += NT) q[t.KV * qg + i] = 0.0f;
    const float temp = 1.0f + t.temp_coef * logf((float)(floor((double)len / t.temp_every) + 1.0));
    pdl_wait();
    pdl_trigger();
    if (a.state->done | a.state->error) return;
    if (sp >= splits) return;
    for (int i = tid; i < H * qd; i += NT) {
        const int g = i / qd, e = i - g * qd, c = g / per;
        q[c * qg + (g - c * per) * qd + e] = e < dim ? a.q[g * dim + e] * (t.scale * temp) : 0.0f;
    }
    if (k_end == len && k_begin < len) {         // this split owns the token's own row
        const float* src = a.q + H * dim;
        for (int f = tid; f < t.kd; f += NT) put(kc + (size_t)pos * t.kd + f, f < width ? src[f] : 0.0f);
        for (int c = warp; c < t.KV; c += NT / 32) {
            const float* v = src + width + c * vd;
            float s = 0.0f;
            for (int e = lane; e < vd; e += 32) s = fmaf(v[e], v[e], s);
            const float inv = 1.0f / sqrtf(warp_sum(s) / (float)vd + t.eps);
            for (int e = lane; e < t.vp; e += 32) put(vc + (size_t)pos * vst + c * t.vp + e, e < vd ? v[e] * inv : 0.0f);
        }
    }
    __syncthreads();
    const bool vec = dim % kVec<T> == 0;         // every key part starts on 16 bytes then
    for (int k0 = k_begin; k0 < k_end; k0 += KT) {
        const int nk = min(KT, k_end - k0);
        if (k0 > k_begin) load_bias(k0);
        for (int i = tid; i < nk * t.KV; i += NT) {
            const int j = i / t.KV, c = i - j * t.KV;
            const T* kr = kc + (size_t)(k0 + j) * t.kd + c * dim;
            for (int g0 = 0; g0 < per; g0 += PER) {
                float s[PER] = {};
                scores_of<T>(kr, q + c * qg + g0 * qd, qd, dim, vec, s);
#pragma unroll
                for (int y = 0; y < PER; ++y)
                    if (g0 + y < per) raw[(c * per + g0 + y) * RST + j] = s[y];
            }
        }
        __syncthreads();
        for (int h0 = warp * 4; h0 < H; h0 += NT / 32 * 4) {
            float s[4][2] = {};
            for (int g = 0; g < H; ++g) {
                const float4 tk = *(const float4*)(talk + g * Hp + h0);
                const float x = raw[g * RST + lane], y = raw[g * RST + lane + 32];
                s[0][0] = fmaf(tk.x, x, s[0][0]); s[0][1] = fmaf(tk.x, y, s[0][1]);
                s[1][0] = fmaf(tk.y, x, s[1][0]); s[1][1] = fmaf(tk.y, y, s[1][1]);
                s[2][0] = fmaf(tk.z, x, s[2][0]); s[2][1] = fmaf(tk.z, y, s[2][1]);
                s[3][0] = fmaf(tk.w, x, s[3][0]); s[3][1] = fmaf(tk.w, y, s[3][1]);
            }
#pragma unroll
            for (int z = 0; z < 4; ++z) {
                const int h = h0 + z;
                if (h >= H) break;
                float b[2];
#pragma unroll
                for (int y = 0; y < 2; ++y) {
                    const int j = lane + 32 * y;
                    b[y] = j < nk ? s[z][y] + bsm[h * RST + j] : -INFINITY;
                }
                float mx = fmaxf(b[0], b[1]);
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
                const float m0 = ml[3 * h], mn = fmaxf(m0, mx);
                const float p0 = expf(b[0] - mn), p1 = expf(b[1] - mn);
                mix[lane * mst + h] = p0;
                mix[(lane + 32) * mst + h] = p1;
                const float ps = warp_sum(p0 + p1);
                if (lane == 0) {
                    const float corr = expf(m0 - mn);
                    ml[3 * h] = mn;
                    ml[3 * h + 1] = fmaf(ml[3 * h + 1], corr, ps);
                    ml[3 * h + 2] = corr;
                }
            }
        }
        __syncthreads();
        // values: columns 2 u, 2 u + 1 of a value head (the last may stand alone) and half of the tile's keys
        const int up = (vd + 1) / 2, units = t.KV * up, half = (nk + 1) / 2;
        for (int i = tid; i < 2 * units; i += NT) {
            const int kh = i / units, u = i - kh * units, c = u / up, e = 2 * (u - c * up), j_end = kh ? nk : half;
            const bool two = e + 1 < vd;
            const T* v = vc + (size_t)k0 * vst + c * t.vp + e;         // vp is even: pairs are aligned
            for (int g0 = 0; g0 < per; g0 += PER) {
                float s[PER][2] = {};
                const float* mp = mix + c * per + g0;
                for (int j0 = kh ? half : 0; j0 < j_end; j0 += 16) {
                    float vv[16][2];
#pragma unroll
                    for (int x = 0; x < 16; ++x) {
                        vv[x][0] = vv[x][1] = 0.0f;
                        if (j0 + x < j_end) {
                            const T* p = v + (size_t)(j0 + x) * vst;
                            if constexpr (sizeof(T) == 2) {
                                const uint32_t w = *(const uint32_t*)p;
                                vv[x][0] = __uint_as_float(w << 16); vv[x][1] = __uint_as_float(w & 0xffff0000u);
                            } else {
                                const float2 w = *(const float2*)p;
                                vv[x][0] = w.x; vv[x][1] = w.y;
                            }
                        }
                    }
#pragma unroll
                    for (int x = 0; x < 16; ++x) {
                        const float* mr = mp + min(j0 + x, KT - 1) * mst;
#pragma unroll
                        for (int y = 0; y < PER; ++y) {
                            const float p = mr[y];                      // past the group's last head: the next one's, not stored
                            s[y][0] = fmaf(p, vv[x][0], s[y][0]);
                            s[y][1] = fmaf(p, vv[x][1], s[y][1]);
                        }
                    }
                }
#pragma unroll
                for (int y = 0; y < PER; ++y)
                    if (g0 + y < per) {
                        const int h = c * per + g0 + y;
                        float* to = acc + ((size_t)kh * H + h) * vd + e;
                        const float corr = ml[3 * h + 2];
                        to[0] = fmaf(to[0], corr, s[y][0]);
                        if (two) to[1] = fmaf(to[1], corr, s[y][1]);
                    }
            }
        }
        __syncthreads();
    }
    const float* acc1 = acc + H * vd;
    if (splits > 1) {
        for (int i = tid; i < H * vd; i += NT) a.part[(size_t)sp * H * vd + i] = acc[i] + acc1[i];
        for (int h = tid; h < H; h += NT) {
            a.part_ml[((size_t)sp * H + h) * 2] = ml[3 * h];
            a.part_ml[((size_t)sp * H + h) * 2 + 1] = ml[3 * h + 1];
        }
        __threadfence();
        __syncthreads();
        if (tid == 0) is_last = atomicAdd(a.counter, 1u) == (unsigned)(splits - 1);
        __syncthreads();
        if (!is_last) return;
        __threadfence();
        if (tid == 0) *a.counter = 0;
        float* wgt = raw;                        // [H][splits]: at most KT splits
        for (int h = warp; h < H; h += NT / 32) {
            const float sink = t.sink[h];
            float mv[2], lv[2];
#pragma unroll
            for (int y = 0; y < 2; ++y) {
                const int s = lane + 32 * y;
                mv[y] = s < splits ? __ldcg(a.part_ml + ((size_t)s * H + h) * 2) : -INFINITY;
                lv[y] = s < splits ? __ldcg(a.part_ml + ((size_t)s * H + h) * 2 + 1) : 0.0f;
            }
            float m = fmaxf(fmaxf(mv[0], mv[1]), sink);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) m = fmaxf(m, __shfl_xor_sync(0xffffffffu, m, o));
            const float w0 = expf(mv[0] - m), w1 = expf(mv[1] - m);
            const float l = warp_sum(w0 * lv[0] + w1 * lv[1]) + expf(sink - m);
            if (lane < splits) wgt[h * RST + lane] = w0 / l;
            if (lane + 32 < splits) wgt[h * RST + lane + 32] = w1 / l;
        }
        __syncthreads();
        for (int i = tid; i < H * vd; i += NT) {
            const float* w = wgt + i / vd * RST;
            float o = 0.0f;
#pragma unroll 8
            for (int s = 0; s < splits; ++s) o = fmaf(w[s], __ldcg(a.part + (size_t)s * H * vd + i), o);
            a.att[i] = o;
        }
    } else {
        for (int i = tid; i < H * vd; i += NT) {
            const int h = i / vd;
            const float m0 = ml[3 * h], sink = t.sink[h], m = fmaxf(m0, sink), w = expf(m0 - m);
            a.att[i] = (acc[i] + acc1[i]) * w / fmaf(ml[3 * h + 1], w, expf(sink - m));
        }
    }
}
}  // namespace

template <class T>
__global__ void __launch_bounds__(NT) mixer_decode_kernel(const __grid_constant__ MixerDecode a) {
    extern __shared__ __align__(16) float sm[];
    if ((int)blockIdx.x < a.rH) recurrence(a, sm);
    else attention<T>(a, sm);
}

int launch_mixer_decode(const MixerDecode& a, cudaStream_t st) {
    const TalkAttn& t = a.t;
    const int qd = (t.dim + 3) & ~3, Hp = (t.H + 3) & ~3;
    if (a.max_splits > KT) return fail(FC_E_SHAPE, "%d attention splits (at most %d)", a.max_splits, KT);
    const size_t att = (size_t)(t.KV * (t.H / t.KV * qd + 4) + PER * qd + t.H * Hp + (t.H + PER) * RST + KT * (Hp + 4) + 2 * t.H * t.vdim + 3 * t.H + t.H * RST) * 4;
    const size_t rec = (size_t)(4 * a.rdim + a.rank + std::max(1, NT / a.rdim) * a.rdim) * 4;
    const size_t smem = std::max(att, rec);
    if (smem > 220 * 1024) return fail(FC_E_SHAPE, "the decode mixers need %zu bytes of shared memory", smem);
    if (smem > 47 * 1024) {
        FC_CUDA(cudaFuncSetAttribute(mixer_decode_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
        FC_CUDA(cudaFuncSetAttribute(mixer_decode_kernel<uint16_t>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
    }
    const dim3 grid(a.rH + a.max_splits);
    if (a.f32_cache) FC_CUDA(launch_pdl(mixer_decode_kernel<float>, grid, dim3(NT), smem, st, a));
    else FC_CUDA(launch_pdl(mixer_decode_kernel<uint16_t>, grid, dim3(NT), smem, st, a));
    ++g_launches;
    return FC_OK;
}

}  // namespace fc
