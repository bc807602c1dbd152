// Products and mixers on weights stored as bf16: device layout, grouped GEMM / GEMV, and the row kernels
// of layers that put several sublayers side by side. Everything is parameterised by sizes and constants;
// nothing here belongs to one model.
#pragma once
#include <cuda.h>

#include "fc_common.cuh"

namespace fc {

// A bf16 matrix [N][K] on the device, rows padded to K_pad (a multiple of 64) and N_pad (of 128) with zeros.
struct BMat {
    const uint16_t* w = nullptr;
    int N = 0, K = 0, N_pad = 0, K_pad = 0;
};
inline int pad_to(int v, int m) { return (v + m - 1) / m * m; }

// What happens to a product before it is stored. XIELU: z > 0: c0 z^2 + z / 2, else c1 (e^z - 1 - z) + z / 2.
// DECAY: exp(-exp(v + vec[n])).
enum RowEpi : int { ROW_NONE = 0, ROW_XIELU = 1, ROW_DECAY = 2 };
__device__ __forceinline__ float xielu_f(float z, float c0, float c1) {
    return z > 0.0f ? fmaf(c0 * z, z, 0.5f * z) : fmaf(c1, expm1f(z) - z, 0.5f * z);
}

// ---- gemm_bf16.cu: several products in one launch ---------------------------------------------------
// Segment: columns [0, n) of Y = A W^T with A rows taken from a plane of one of the operand maps and W rows
// b_row0.. of one of the weight maps, over k-blocks [kb0, kb0 + kb) of 64.
struct GemmSeg {
    int a_map, a_row0, b_map, b_row0, kb0, kb, n;
    float* y;         // f32 rows, or
    uint16_t* yb;     // bf16 rows
    int ldy, epi;
    float c0, c1;
    int tile0, tiles_n;   // filled by the launcher
};
constexpr int kGemmSegs = 16;
struct GemmMaps { CUtensorMap a[3], b[3]; };
struct GemmGroup {
    GemmSeg seg[kGemmSegs];
    int n_seg, M, n_tiles;
    int* status;
    long long wait_cycles;
    int withhold;
};
constexpr int kGemmBoxRows = 128;     // rows of every box of the operand and weight maps
int launch_gemm_bf16_group(const GemmMaps& maps, GemmGroup g, int M, int* status, cudaStream_t st);
// One product in true f32 on CUDA cores: Y[M][n] = f(A)[M][K] W^T, A f32 rows lda apart (K = w.K_pad columns are
// read), W rows row0.. of the matrix; tanh_in applies tanh to A on the way in. y or yb.
struct GemmF32 {
    const float* a; int lda, tanh_in;
    float* y; uint16_t* yb; int ldy;
    int epi; float c0, c1; const float* vec;
};
int launch_gemm_bf16w_f32(const BMat& w, int row0, int n, const GemmF32& p, int M, cudaStream_t st);

// ---- rows of side-by-side layers (mix_rows.cu) ------------------------------------------------------
// Residual update of the layer before (x + (half the sum of two normed outputs + feed-forward partials)), the norm of
// the layer that follows, and the token-shift mixes h + (h' - h) mu_s of every row.
constexpr int kMixes = 5;
struct SideOutputs {              // outputs of the layer before; outs == null: x comes from the embedding
    const float* outs = nullptr;  // [2 + n_ff][stride]: left, right, feed-forward partial sums
    size_t stride = 0;
    int n_ff = 0;
    const float *left_w = nullptr, *right_w = nullptr;
};
struct EmbedSrc {
    const uint16_t* table = nullptr;   // bf16 [vocab][ld]
    int vocab = 0, ld = 0;
    float scale = 1.0f;
};
struct MixRows {
    EmbedSrc embed; const int* ids;    // used when prev.outs is null
    SideOutputs prev;
    const float* x_in; float* x_out;   // [M][d]; x_out may be null
    const float* norm_w; float eps;    // norm_w null: only x_out is written
    const float* mu[kMixes];           // null: only the plane of h
    const float* h_first;              // h of the token before row 0 (token shift)
    float* h_last;                     // receives h of row M - 1
    const int* row_idx;                // rows of x_in / prev to take (null: 0..M-1); no token shift then
    int M, d, ld;                      // planes have rows of ld elements
    void* planes; size_t plane_stride; // plane 0: h, 1..: mixes; bf16 or f32
    int* error_flag;
};
int launch_mix_rows(const MixRows& p, bool f32_planes, cudaStream_t st);

// ---- talk_attn.cu / talk_attn_tc.cu: attention with mixed heads ------------------------------------
// score[h](i, j) = sum_g talk[h][g] (scale temp(i) q_g(i) . k_kv(g)(j) + rel[bucket(i - j)][g]), softmax with one extra
// exp(sink[h]) in the denominator, values divided by their root mean square. Mixing is linear, so it is applied to the
// queries: with q'_h = the concatenation over key/value heads c of sum_{g in c} talk[h][g] q_g, the mixed score is
// q'_h . (all keys of j side by side) plus a per-head table of the distance.
struct TalkAttn {
    int H = 0, KV = 0, dim = 0, vdim = 0;
    int kd = 0;         // elements of a cached key row: KV * dim rounded up to 16
    int vp = 0;         // elements of one cached value head: vdim rounded up to 16
    int far = 0;        // the last distance with an entry of its own in `bias`
    float scale = 1.0f, temp_coef = 0.0f, eps = 0.0f;
    double temp_every = 1.0;
    const float* talk = nullptr;   // [H][H]
    const float* bias = nullptr;   // [H][far + 1], heads already mixed
    const float* sink = nullptr;   // [H]
};
// Positions pos0 .. pos0 + M - 1: mixed queries (times scale, temperature and `factor`), cache rows of keys and values.
// proj rows: q | k | v. qm [M][H * kd], bf16 or f32; caches in the same type.
int launch_talk_prep(const TalkAttn& t, const float* proj, int ldp, int M, int pos0, float factor, void* qm, void* kc, void* vc, bool f32,
                     cudaStream_t st);
// Rows of a portion against an f32 cache (positions 0 .. pos0 + i) on CUDA cores; out rows ldo apart. Queries prepared
// with factor 1; value heads of at most 256.
int launch_talk_prefill_f32(const TalkAttn& t, const float* qm, const float* kc, const float* vc, int M, int pos0, float* out, int ldo,
                            cudaStream_t st);
// The same on tcgen05 with bf16 queries, cache and output; queries prepared with factor log2(e).
int launch_talk_prefill_tc(const TalkAttn& t, const void* qm, const void* kc, const void* vc, int M, int pos0, int ctx, void* out, int ldo,
                           int* status, cudaStream_t st);
constexpr float kLog2e = 1.4426950408889634f;

// ---- wkv.cu: linear-attention state with per-channel decay and a bonus for the current token --------
// o_t = (S + diag(u) k_t v_t^T)^T r_t, S <- diag(w_t) S + k_t v_t^T; state [H][dim][dim] f32 in and out. scratch:
// wkv_scratch_floats(H, dim), for portions long enough to be cut into segments.
constexpr int kWkvSegments = 8;
size_t wkv_scratch_floats(int H, int dim);
int launch_wkv_scan(const float* r, const float* k, const float* v, int ld, const float* w, int ldw, const float* u, float* state, float* o,
                    int ldo, int M, int H, int dim, float* scratch, cudaStream_t st);
// o / rms(o) per head, times norm, times silu(gate): rows of ldy elements, bf16 or f32.
int launch_wkv_finish(const float* o, int ldo, const float* gate, int ldg, const float* norm, float eps, int M, int H, int dim, void* y,
                      int ldy, bool f32, cudaStream_t st);

// ---- one decode step --------------------------------------------------------------------------------
// gemv_bf16.cu: several products of one activation row in one launch. src: index of the input (plane of the mix
// prologue, or x[src]).
struct GemvSeg {
    const uint16_t* w;    // first row; rows ldw apart, K_pad weights of each (a multiple of 64), K inputs
    int n, ldw, K_pad, src, K;
    float* y;
    int epi;
    float c0, c1;
    long long cost0;      // filled by the launcher
};
constexpr int kGemvSegs = 16;
struct GemvGroup {
    GemvSeg seg[kGemvSegs];
    int n_seg;
    const float* x[8];                 // plain inputs (mode 0)
    int mode;                          // 0: plain inputs; 1: residual + norm + mixes of the row; 2: residual + norm
    EmbedSrc embed; const int* queue; int ctx;
    SideOutputs prev;
    const float* x_in; float* x_out;
    const float* norm_w; float eps;
    const float* mu[kMixes];
    float* shift; size_t shift_slot;   // two slots of h, read at position parity, written at the other
    int d;
    StepState* state;
    long long total_cost;
};
int launch_gemv_bf16_group(GemvGroup g, cudaStream_t st);

// mixer_decode.cu: attention splits and recurrence heads of one token in one launch.
struct MixerDecode {
    TalkAttn t;
    const float* q;                    // proj row: q | k | v
    void *kc, *vc; bool f32_cache; int ctx;
    float* att;                        // [H * vdim]
    float *part, *part_ml;             // [splits][H][vdim], [splits][H][2]
    int max_splits; unsigned int* counter;
    // recurrence
    int rH, rdim, rank;
    const float *r, *k, *v, *g, *w1;   // projections of the row (w1: [rank])
    const uint16_t* w2; int w2_ld; const float* w0;
    const float *u, *rnorm; float eps;
    float* wkv_state; float* ro;
    StepState* state;
};
int launch_mixer_decode(const MixerDecode& a, cudaStream_t st);

}  // namespace fc
