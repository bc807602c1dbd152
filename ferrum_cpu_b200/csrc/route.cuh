// Choice of a token's experts by one warp.
#pragma once
#include "bf16_ops.cuh"

namespace fc {

constexpr int kMaxExperts = 1024, kMaxGroups = 256;

// The place and value of the largest entry (the first of equals), in every lane. n may exceed what a lane sees.
static __device__ __forceinline__ int warp_argmax(const float* z, int n, float* best) {
    const int lane = threadIdx.x & 31;
    float b = -INFINITY;
    int at = 1 << 30;
    for (int i = lane; i < n; i += 32)
        if (z[i] > b) { b = z[i]; at = i; }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ob = __shfl_xor_sync(0xffffffffu, b, o);
        const int oa = __shfl_xor_sync(0xffffffffu, at, o);
        if (ob > b || (ob == b && oa < at)) { b = ob; at = oa; }
    }
    *best = b;
    return at;
}
// One warp chooses from logits z (overwritten) of a token; gs: room for the groups' scores. emit(slot, expert, weight) runs in
// one lane per slot. Softmax keeps the logits' order, so they are compared in its place; of equals the first counts as larger.
// Few entries are ranked by counting those ahead of each, more are taken one by one.
constexpr int kRankBy = 128;
static __device__ __forceinline__ int rank_of(const float* z, int n, int i) {
    const float v = z[i];
    int ahead = 0;
#pragma unroll 8
    for (int k = 0; k < n; ++k) ahead += z[k] > v || (z[k] == v && k < i);
    return ahead;
}
template <class F>
__device__ __forceinline__ void choose(float* z, float* gs, const Router& r, F emit) {
    const int lane = threadIdx.x & 31, E = r.experts;
    if (E <= 32) {                                                   // an expert a lane, in few instructions (they are run once)
        float v = lane < E ? z[lane] : -INFINITY;
        if (v != v) v = -INFINITY;
        float top = v;
#pragma unroll 1
        for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
        float sum = expf(v - top);
        const float e = sum;
#pragma unroll 1
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        if (r.keep < r.groups) {
            const int size = E / r.groups, g = lane / size;
            float mine = -INFINITY;
#pragma unroll 1
            for (int k = 0; k < size; ++k) mine = fmaxf(mine, __shfl_sync(0xffffffffu, v, min(g * size + k, 31)));
            int ahead = 0;
#pragma unroll 1
            for (int k = 0; k < r.groups; ++k) {
                const float o = __shfl_sync(0xffffffffu, mine, k * size);
                ahead += o > mine || (o == mine && k < g);
            }
            if (ahead >= r.keep) v = -INFINITY;
        }
        int ahead = 0;
#pragma unroll 4
        for (int k = 0; k < E; ++k) {
            const float o = __shfl_sync(0xffffffffu, v, k);
            ahead += o > v || (o == v && k < lane);
        }
        if (lane < E && ahead < r.top) emit(ahead, lane, e / sum);
        return;
    }
    for (int i = lane; i < E; i += 32)
        if (z[i] != z[i]) z[i] = -INFINITY;                          // what is not a number comes last: every slot gets an expert
    __syncwarp();
    float top;
    warp_argmax(z, E, &top);
    float sum = 0.0f;
    for (int i = lane; i < E; i += 32) sum += expf(z[i] - top);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
    if (r.keep < r.groups) {
        const int size = E / r.groups;
        for (int g = lane; g < r.groups; g += 32) {
            float m = -INFINITY;
            for (int i = 0; i < size; ++i) m = fmaxf(m, z[g * size + i]);
            gs[g] = m;
        }
        __syncwarp();
        for (int i = lane; i < E; i += 32)
            if (rank_of(gs, r.groups, i / size) >= r.keep) z[i] = -INFINITY;
        __syncwarp();
    }
    if (E <= kRankBy) {
        for (int i = lane; i < E; i += 32) {
            const int k = rank_of(z, E, i);
            if (k < r.top) emit(k, i, expf(z[i] - top) / sum);
        }
        return;
    }
    for (int k = 0; k < r.top; ++k) {
        float v;
        int e = warp_argmax(z, E, &v);
        if (e >= E) e = 0;                                           // only where logits are not numbers
        __syncwarp();
        if (lane == 0) { z[e] = -INFINITY; emit(k, e, expf(v - top) / sum); }
        __syncwarp();
    }
}

}  // namespace fc
