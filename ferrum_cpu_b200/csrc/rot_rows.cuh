// Device helpers of attention with rotated positions, shared by its prefill and decode kernels.
#pragma once
#include "bf16_ops.cuh"

namespace fc {

// Cosine and sine of position * freq: the product and its reduction to one turn in double, so that the f32 functions see a
// small argument whatever the position.
__device__ __forceinline__ float2 rot_cs(int pos, double freq) {
    constexpr double kTurn = 6.283185307179586476925286766559, kInv = 0.15915494309189533576888376337251;
    const double a = (double)pos * freq;
    float s, c;
    sincosf((float)(a - kTurn * rint(a * kInv)), &s, &c);
    return make_float2(c, s);
}
// Element e of a head whose first r.dims elements are rotated; x(i) gives the unrotated element i, cs[i] pair i's turn.
template <class F>
__device__ __forceinline__ float rotated(bool neighbours, int dims, const float2* cs, int e, F x) {
    if (e >= dims) return x(e);
    if (neighbours) {
        const float2 t = cs[e >> 1];
        return e & 1 ? x(e) * t.x + x(e - 1) * t.y : x(e) * t.x - x(e + 1) * t.y;
    }
    const int n = dims / 2;
    if (e < n) return x(e) * cs[e].x - x(e + n) * cs[e].y;
    return x(e) * cs[e - n].x + x(e - n) * cs[e - n].y;
}
template <class T>
__device__ __forceinline__ void put_row(T* p, float v) {
    if constexpr (sizeof(T) == 2) *p = __bfloat16_as_ushort(__float2bfloat16_rn(v));
    else *p = v;
}
// Two neighbouring elements (p on an even element).
template <class T>
__device__ __forceinline__ void put_pair(T* p, float a, float b) {
    if constexpr (sizeof(T) == 2) {
        const __nv_bfloat162 h = __float22bfloat162_rn(make_float2(a, b));
        *(uint32_t*)p = *(const uint32_t*)&h;
    } else *(float2*)p = make_float2(a, b);
}
// Sum over the NT threads of a block; red: one float a warp.
template <int NT>
__device__ __forceinline__ float block_sum_of(float v, float* red) {
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

}  // namespace fc
