// The two mixers of one decoded token in one launch.
//
// Attention (blocks rH ..): the cached keys are cut into splits, one CTA each, that compute the scores of ALL heads for
// their keys (the heads are mixed before the softmax), in tiles of 32 keys:
//   raw[g][j] = q_g . k_j   thread per (head, group of keys), query in registers, key tile in shared memory
//   mixed[h][j] = sum_g talk[h][g] raw[g][j] + bias[h][i - j]
//   running max / sum per head, values accumulated by the threads that own their columns.
// The last split to finish (an atomic counter, no waiting) merges the partial results in split order and adds the sink.
// The split that holds the token's own position writes its key row and normed value row to the cache first.
//
// Recurrence (blocks 0 .. rH - 1): one head each: decay from the low-rank projection, o = (S + diag(u) k v^T)^T r,
// S <- diag(w) S + k v^T, head norm and gate. State and arithmetic are f32.
//
// Bound: HBM / latency (cache rows once, the recurrence states once in and out).
#include <algorithm>

#include "bf16_ops.cuh"
#include "pdl.cuh"
#include "tc_common.cuh"

namespace fc {

namespace {
constexpr int NT = 256, KT = 32, SPLIT_KEYS = 64;
constexpr int KPT = 8;                    // keys of a tile a thread scores at once
constexpr int QREG = 16;                  // query values in registers at once

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
// Four consecutive values from shared memory (16-byte aligned rows for f32, 8-byte for bf16).
template <class T>
__device__ __forceinline__ float4 get4(const T* p) {
    if constexpr (sizeof(T) == 2) {
        const uint2 w = *(const uint2*)p;
        return make_float4(__uint_as_float(w.x << 16), __uint_as_float(w.x & 0xffff0000u), __uint_as_float(w.y << 16), __uint_as_float(w.y & 0xffff0000u));
    } else {
        return *(const float4*)p;
    }
}
__device__ __forceinline__ float block_sum(float v, float* red) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
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
    const int head = blockIdx.x, D = a.rdim, tid = threadIdx.x;
    const size_t h0 = (size_t)head * D;
    float *r = sm, *k = r + D, *w = k + D, *v = w + D, *low = v + D, *part = low + a.rank;     // part [slices][D]
    for (int i = tid; i < a.rank; i += NT) low[i] = tanhf(a.w1[i]);
    for (int i = tid; i < D; i += NT) { r[i] = a.r[h0 + i]; k[i] = a.k[h0 + i]; v[i] = a.v[h0 + i]; }
    __syncthreads();
    float bonus = 0.0f;
    for (int i = tid; i < D; i += NT) {
        const uint16_t* row = a.w2 + (h0 + i) * a.w2_ld;
        float s = 0.0f;
        for (int c = 0; c < a.rank; ++c) s = fmaf(get(row + c), low[c], s);
        w[i] = expf(-expf(s + a.w0[h0 + i]));
        bonus = fmaf(r[i] * a.u[h0 + i], k[i], bonus);
    }
    bonus = block_sum(bonus, red);              // also the barrier in front of w
    // column j of the state, rows sl, sl + slices, ...
    const int slices = max(1, NT / D), j0 = tid % D, sl = tid / D;
    float* S = a.wkv_state + h0 * D;
    if (sl < slices) {
        for (int j = j0; j < D; j += NT) {      // one pass unless D > NT
            const float vj = v[j];
            float o = 0.0f;
            int i = sl;
            for (; i + 3 * slices < D; i += 4 * slices) {
                float s4[4];
#pragma unroll
                for (int x = 0; x < 4; ++x) s4[x] = S[(size_t)(i + x * slices) * D + j];
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const int ii = i + x * slices;
                    o = fmaf(s4[x], r[ii], o);
                    S[(size_t)ii * D + j] = fmaf(w[ii], s4[x], k[ii] * vj);
                }
            }
            for (; i < D; i += slices) {
                const float s = S[(size_t)i * D + j];
                o = fmaf(s, r[i], o);
                S[(size_t)i * D + j] = fmaf(w[i], s, k[i] * vj);
            }
            part[sl * D + j] = o;
        }
    }
    __syncthreads();
    float ss = 0.0f;
    for (int j = tid; j < D; j += NT) {
        float o = 0.0f;
        for (int x = 0; x < slices; ++x) o += part[x * D + j];
        o = fmaf(bonus, v[j], o);
        part[j] = o;
        ss = fmaf(o, o, ss);
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)D + a.eps);
    for (int j = tid; j < D; j += NT) {
        const float z = a.g[h0 + j];
        a.ro[h0 + j] = part[j] * inv * a.rnorm[h0 + j] * (z / (1.0f + expf(-z)));
    }
}

template <class T>
__device__ void attention(const MixerDecode& a, float* sm) {
    __shared__ bool is_last;
    const TalkAttn& t = a.t;
    const int tid = threadIdx.x, lane = tid & 31, H = t.H, dim = t.dim, per = H / t.KV, width = t.KV * dim, vd = t.vdim;
    const int pos = a.state->pos, len = pos + 1;
    const int splits = min(a.max_splits, (len + SPLIT_KEYS - 1) / SPLIT_KEYS), sp = blockIdx.x - a.rH;
    if (sp >= splits) return;
    const int per_split = ((len + splits - 1) / splits + KT - 1) / KT * KT;
    const int k_begin = sp * per_split, k_end = min(len, k_begin + per_split);
    // rows of queries and cached keys are a few banks apart
    const int dq = (dim + 3) & ~3, qst = dq + 4, hk = H * (KT + 1), khs = dq + (sizeof(T) == 2 ? 8 : 4), kst = a.kv_block * khs;
    T* ks = (T*)sm;                              // [KT][kst]
    float* q = sm + KT * kst * sizeof(T) / 4;    // [H][qst]
    float* talk = q + H * qst;                   // [H][H], transposed: talk[g][h]
    float* raw = talk + H * H;                   // [H][KT + 1]
    float* mix = raw + hk;                       // [H][KT + 1]
    float* acc = mix + hk;                       // [H][vd]
    float* ml = acc + H * vd;                    // [H][3]: max, sum, correction
    T* kc = (T*)a.kc;
    T* vc = (T*)a.vc;
    const float temp = 1.0f + t.temp_coef * logf((float)(floor((double)len / t.temp_every) + 1.0));
    for (int i = tid; i < H * dq; i += NT) {
        const int g = i / dq, e = i - g * dq;
        q[g * qst + e] = e < dim ? a.q[g * dim + e] * (t.scale * temp) : 0.0f;
    }
    for (int i = tid; i < H * H; i += NT) { const int h = i / H, g = i - h * H; talk[g * H + h] = t.talk[i]; }
    for (int i = tid; i < H * vd; i += NT) acc[i] = 0.0f;
    for (int h = tid; h < H; h += NT) { ml[3 * h] = -INFINITY; ml[3 * h + 1] = 0.0f; ml[3 * h + 2] = 0.0f; }
    for (int i = tid; i < KT * kst; i += NT) put(ks + i, 0.0f);
    if (k_end == len && k_begin < len) {         // this split owns the token's own row
        const float* src = a.q + H * dim;
        for (int f = tid; f < t.kd; f += NT) put(kc + (size_t)pos * t.kd + f, f < width ? src[f] : 0.0f);
        for (int c = tid >> 5; c < t.KV; c += NT / 32) {
            const float* v = src + width + c * vd;
            float s = 0.0f;
            for (int e = lane; e < vd; e += 32) s = fmaf(v[e], v[e], s);
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
            const float inv = 1.0f / sqrtf(s / (float)vd + t.eps);
            for (int e = lane; e < t.vp; e += 32) put(vc + ((size_t)pos * t.KV + c) * t.vp + e, e < vd ? v[e] * inv : 0.0f);
        }
    }
    __syncthreads();
    for (int k0 = k_begin; k0 < k_end; k0 += KT) {
        const int nk = min(KT, k_end - k0);
        for (int c0 = 0; c0 < t.KV; c0 += a.kv_block) {              // as many key heads at a time as shared memory holds
            const int nc = min(a.kv_block, t.KV - c0), wb = nc * dim, Hb = nc * per, groups = max(1, NT / Hb);
            if (c0) __syncthreads();
            for (int i = tid; i < nk * wb; i += NT) {
                const int j = i / wb, f = i - j * wb, c = f / dim;
                ks[j * kst + c * khs + (f - c * dim)] = kc[(size_t)(k0 + j) * t.kd + c0 * dim + f];
            }
            __syncthreads();
            for (int w = tid; w < Hb * groups; w += NT) {
                const int gl = w % Hb, kg = w / Hb, g = c0 * per + gl;
                const float* qg = q + g * qst;
                const T* kb = ks + (gl / per) * khs;
                for (int jb = kg; jb < KT; jb += groups * KPT) {
                    float s[KPT];
#pragma unroll
                    for (int x = 0; x < KPT; ++x) s[x] = 0.0f;
                    for (int e0 = 0; e0 < dq; e0 += QREG) {
                        float4 qr[QREG / 4];
#pragma unroll
                        for (int e = 0; e < QREG / 4; ++e) qr[e] = e0 + 4 * e < dq ? *(const float4*)(qg + e0 + 4 * e) : make_float4(0, 0, 0, 0);
#pragma unroll
                        for (int x = 0; x < KPT; ++x) {
                            const int j = jb + x * groups;
                            if (j < KT) {
                                const T* kr = kb + j * kst + e0;
#pragma unroll
                                for (int e = 0; e < QREG / 4; ++e)
                                    if (e0 + 4 * e < dq) {
                                        const float4 k4 = get4(kr + 4 * e);
                                        s[x] = fmaf(qr[e].x, k4.x, s[x]); s[x] = fmaf(qr[e].y, k4.y, s[x]);
                                        s[x] = fmaf(qr[e].z, k4.z, s[x]); s[x] = fmaf(qr[e].w, k4.w, s[x]);
                                    }
                            }
                        }
                    }
#pragma unroll
                    for (int x = 0; x < KPT; ++x)
                        if (jb + x * groups < KT) raw[g * (KT + 1) + jb + x * groups] = s[x];
                }
            }
        }
        __syncthreads();
        // mixed scores: a warp takes a head, a lane a key
        for (int h = tid >> 5; h < H; h += NT / 32) {
            float s = -INFINITY;
            if (lane < nk) {
                s = 0.0f;
                for (int g = 0; g < H; ++g) s = fmaf(talk[g * H + h], raw[g * (KT + 1) + lane], s);
                s += t.bias[(size_t)h * (t.far + 1) + min(pos - (k0 + lane), t.far)];
            }
            float mx = s;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float m0 = ml[3 * h], mn = fmaxf(m0, mx);
            const float p = lane < nk ? expf(s - mn) : 0.0f;
            mix[h * (KT + 1) + lane] = p;
            float ps = p;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) ps += __shfl_xor_sync(0xffffffffu, ps, o);
            __syncwarp();
            if (lane == 0) {
                const float corr = expf(m0 - mn);
                ml[3 * h] = mn;
                ml[3 * h + 1] = fmaf(ml[3 * h + 1], corr, ps);
                ml[3 * h + 2] = corr;
            }
        }
        __syncthreads();
        for (int col = tid; col < t.KV * vd; col += NT) {
            const int c = col / vd, e = col - c * vd;
            const T* v = vc + ((size_t)k0 * t.KV + c) * t.vp + e;
            const size_t vs = (size_t)t.KV * t.vp;
            for (int g0 = 0; g0 < per; g0 += 4) {
                float s[4];
#pragma unroll
                for (int x = 0; x < 4; ++x) {
                    const int h = c * per + g0 + x;
                    s[x] = g0 + x < per ? acc[h * vd + e] * ml[3 * h + 2] : 0.0f;
                }
                const float* mp = mix + (c * per + g0) * (KT + 1);
                for (int j0 = 0; j0 < nk; j0 += 8) {
                    float vv[8];
#pragma unroll
                    for (int x = 0; x < 8; ++x) vv[x] = j0 + x < nk ? get(v + (size_t)(j0 + x) * vs) : 0.0f;
#pragma unroll
                    for (int x = 0; x < 8; ++x)
#pragma unroll
                        for (int y = 0; y < 4; ++y)
                            if (g0 + y < per) s[y] = fmaf(mp[y * (KT + 1) + j0 + x], vv[x], s[y]);
                }
#pragma unroll
                for (int x = 0; x < 4; ++x)
                    if (g0 + x < per) acc[(c * per + g0 + x) * vd + e] = s[x];
            }
        }
        __syncthreads();
    }
    if (splits > 1) {
        for (int i = tid; i < H * vd; i += NT) a.part[(size_t)sp * H * vd + i] = acc[i];
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
        float* wgt = raw;                        // [splits] weights of one head at a time would serialise: [H][splits] in `raw` | `mix`
        const bool fits = H * splits <= 2 * hk;
        for (int h = tid; h < H; h += NT) {
            float m = t.sink[h];
            for (int s = 0; s < splits; ++s) m = fmaxf(m, __ldcg(a.part_ml + ((size_t)s * H + h) * 2));
            float l = expf(t.sink[h] - m);
            for (int s = 0; s < splits; ++s) {
                const float w = expf(__ldcg(a.part_ml + ((size_t)s * H + h) * 2) - m);
                l = fmaf(w, __ldcg(a.part_ml + ((size_t)s * H + h) * 2 + 1), l);
                if (fits) wgt[h * splits + s] = w;
            }
            ml[3 * h] = m;
            ml[3 * h + 1] = 1.0f / l;
        }
        __syncthreads();
        for (int i = tid; i < H * vd; i += NT) {
            const int h = i / vd;
            float o = 0.0f;
#pragma unroll 8
            for (int s = 0; s < splits; ++s) {
                const float w = fits ? wgt[h * splits + s] : expf(__ldcg(a.part_ml + ((size_t)s * H + h) * 2) - ml[3 * h]);
                o = fmaf(w, __ldcg(a.part + (size_t)s * H * vd + i), o);
            }
            a.att[i] = o * ml[3 * h + 1];
        }
    } else {
        for (int i = tid; i < H * vd; i += NT) {
            const int h = i / vd;
            const float m0 = ml[3 * h], sink = t.sink[h], m = fmaxf(m0, sink), w = expf(m0 - m);
            a.att[i] = acc[i] * w / fmaf(ml[3 * h + 1], w, expf(sink - m));
        }
    }
}
}  // namespace

template <class T>
__global__ void __launch_bounds__(NT) mixer_decode_kernel(const MixerDecode a) {
    extern __shared__ __align__(16) float sm[];
    pdl_wait();
    pdl_trigger();
    if (a.state->done | a.state->error) return;
    if ((int)blockIdx.x < a.rH) recurrence(a, sm);
    else attention<T>(a, sm);
}

int launch_mixer_decode(MixerDecode a, cudaStream_t st) {
    const TalkAttn& t = a.t;
    const int dq = (t.dim + 3) & ~3, el = a.f32_cache ? 4 : 2, khs = dq + (a.f32_cache ? 4 : 8);
    const size_t fixed = (size_t)(t.H * (dq + 4) + t.H * t.H + 2 * t.H * (KT + 1) + t.H * t.vdim + 3 * t.H) * 4, head = (size_t)KT * khs * el;
    a.kv_block = t.KV;
    while (a.kv_block > 1 && fixed + a.kv_block * head > 220 * 1024) a.kv_block = (a.kv_block + 1) / 2;
    const size_t att = fixed + a.kv_block * head;
    const size_t rec = (size_t)(4 * a.rdim + a.rank + std::max(1, NT / a.rdim) * a.rdim) * 4;
    const size_t smem = std::max(att, rec);
    if (smem > 220 * 1024) return fail(FC_E_SHAPE, "the decode mixers need %zu bytes of shared memory", smem);
    if (smem > 48 * 1024) {
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
