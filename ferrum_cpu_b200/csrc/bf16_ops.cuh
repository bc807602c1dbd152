// Products and mixers on weights stored as bf16: device layout, grouped GEMM / GEMV, and the row kernels
// of layers that put several sublayers side by side. Everything is parameterised by sizes and constants;
// nothing here belongs to one model.
#pragma once
#include <cuda.h>
#include <cuda_bf16.h>

#include "fc_common.cuh"

namespace fc {

// A bf16 matrix [N][K] on the device, rows padded to K_pad (a multiple of 64) and N_pad (of 128) with zeros.
struct BMat {
    const uint16_t* w = nullptr;
    int N = 0, K = 0, N_pad = 0, K_pad = 0;
};
inline int pad_to(int v, int m) { return (v + m - 1) / m * m; }

// What happens to a product before it is stored. XIELU: z > 0: c0 z^2 + z / 2, else c1 (e^z - 1 - z) + z / 2.
// DECAY: exp(-exp(v + vec[n])). GELU: the exact form, z / 2 (1 + erf(z / sqrt 2)).
enum RowEpi : int { ROW_NONE = 0, ROW_XIELU = 1, ROW_DECAY = 2, ROW_GELU = 3 };
__device__ __forceinline__ float xielu_f(float z, float c0, float c1) {
    return z > 0.0f ? fmaf(c0 * z, z, 0.5f * z) : fmaf(c1, expm1f(z) - z, 0.5f * z);
}

__device__ __forceinline__ float gelu_erf_f(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752f)); }

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
// Row tiles of a product with runs of rows: {first row, rows, index of the run's weights, 0}, and how many there are.
struct Ragged {
    const int4* table;
    const int* n;
    int b_step;       // weight rows from one index to the next
};
struct GemmGroup {
    GemmSeg seg[kGemmSegs];
    int n_seg, M, n_tiles;
    int* status;
    long long wait_cycles;
    int withhold;
    Ragged ragged;
};
constexpr int kGemmBoxRows = 128;     // rows of every box of the operand and weight maps
int launch_gemm_bf16_group(const GemmMaps& maps, GemmGroup g, int M, int* status, cudaStream_t st);
// One product whose rows fall into runs, each with weights of its own (rows of one expert after the other): the segment's
// b_row0 and b_step give the first weight row of a run's index. Tiles are counted on the device; at most max_tiles entries.
constexpr int kRaggedRows = 256, kRaggedRowsF32 = 64;   // most rows of a table entry
int launch_gemm_bf16_ragged(const GemmMaps& maps, const GemmSeg& seg, const Ragged& r, int max_entries, int* status, cudaStream_t st);
// One product in true f32 on CUDA cores: Y[M][n] = f(A)[M][K] W^T, A f32 rows lda apart (K = w.K_pad columns are
// read), W rows row0.. of the matrix; tanh_in applies tanh to A on the way in. y or yb.
struct GemmF32 {
    const float* a; int lda, tanh_in;
    float* y; uint16_t* yb; int ldy;
    int epi; float c0, c1; const float* vec;
};
int launch_gemm_bf16w_f32(const BMat& w, int row0, int n, const GemmF32& p, int M, cudaStream_t st);
// The same over runs of rows (table entries of at most kRaggedRowsF32 rows): weight rows index * b_step ..
int launch_gemm_bf16w_f32_ragged(const BMat& w, int n, const GemmF32& p, const Ragged& r, int max_entries, cudaStream_t st);

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

// ---- rows of layers that norm what a sublayer adds (post_norm_rows.cu) --------------------------------------
// x' = x + rms(y) w, y = sum of parts, part s of a row being weight[row * n_parts + s] y[index[row * n_parts + s]] (index null:
// row s * part_rows + row of y; weight null: 1). Without y: x' = rms(embed[id]) w.
struct PostNorm {
    const float* y = nullptr;
    int n_parts = 0, part_rows = 0;
    const int* index = nullptr;
    const float* weight = nullptr;
    const float* norm_w = nullptr;
};
// Value c of the sum of a row's parts.
__device__ __forceinline__ float post_norm_sum(const PostNorm& p, size_t row, int c, int d) {
    float y = 0.0f;
    for (int s = 0; s < p.n_parts; ++s) {
        const size_t at = row * p.n_parts + s, r = p.index ? (size_t)p.index[at] : (size_t)s * p.part_rows + row;
        const float v = p.y[r * d + c];
        y = p.weight ? fmaf(p.weight[at], v, y) : y + v;
    }
    return y;
}
struct PostNormRows {
    PostNorm add;
    EmbedSrc embed; const int* ids;    // used when add.y is null and ids is set
    float* x;                          // [M][d] residual, updated in place (rows row_idx[r] of it when that is set)
    const int* row_idx;
    const float* out_norm_w;           // not null: the plane receives rms(x') out_norm_w, and x stays as it is when add.y is null
    float eps;
    int M, d, ld;
    void* plane;                       // [M][ld], bf16 or f32: x', or its norm
    int* error_flag;
};
int launch_post_norm_rows(const PostNormRows& p, bool f32_plane, cudaStream_t st);

// ---- flash_tc.cu / flash_f32.cu: attention of a portion's rows over cached keys ---------------------------
// score[h](i, j) = q_h(i) . k_h(j) (+ bias[h][min(i - j, far)]) for 0 <= i - j < window; softmax, with one extra exp(sink) in
// the denominator when there is a sink. A key row is a part of the head's own (head h reads key/value head h / (H / KV);
// head_stride 0: all read the same) and, when k1.p is set, a part all heads share. Columns col + head * head_stride +
// 0 .. width - 1 of rows ld elements apart; row r holds position pos0 + r. Widths, strides and first columns are multiples of 16.
constexpr float kLog2e = 1.4426950408889634f;
constexpr int kNoWindow = 1 << 30;
struct FlashPart {
    const void* p = nullptr;
    int rows = 0, ld = 0, col = 0, head_stride = 0, width = 0, pos0 = 0;
};
struct Flash {
    int H = 0, KV = 0, vdim = 0;
    FlashPart k0, k1, v;
    int window = kNoWindow;
    const float* bias = nullptr; int far = 0;       // [H][far + 1]
    bool has_sink = false; const float* sink = nullptr;   // [H]; null: a score of 0 for every head
};
// Rows at positions pos0 .. pos0 + M - 1. q [M][H * (k0.width + k1.width)]; out rows ldo apart, head by head; value heads of at
// most 256. tcgen05 form: bf16 everywhere, queries times log2(e).
int launch_flash_tc(const Flash& f, const void* q, int M, int pos0, void* out, int ldo, int* status, cudaStream_t st);
int launch_flash_f32(const Flash& f, const float* q, int M, int pos0, float* out, int ldo, cudaStream_t st);

// ---- talk_attn.cu: attention with mixed heads --------------------------------------------------------
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
Flash talk_flash(const TalkAttn& t, const void* kc, const void* vc, int ctx);

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
    // the product again with the weights of every chosen expert (GemvGroup): rep r reads the rows expert * w_step weights
    // further on and the input x_step * r values further on, and writes y_step * r values further on. sum: one row of results
    // instead, the sum over the repetitions with the experts' weights (w_step a multiple of 64).
    int reps;             // 0 or 1: once
    int sum;
    size_t w_step;
    int x_step, y_step;
    int cost0, cost;      // filled by the launcher
};
constexpr int kGemvSegs = 16;
struct Router {
    int experts = 0, top = 0, groups = 1, keep = 1;
    const uint16_t* w = nullptr; int ld = 0;         // [experts][ld]
};
struct GemvGroup {
    GemvSeg seg[kGemvSegs];
    int n_seg;
    const float* x[8];                 // plain inputs (mode 0)
    int mode;                          // 0: plain inputs; 1: residual + norm + mixes of the row; 2: residual + norm;
                                       // 3: residual of PostNorm; 4: the same and a norm (norm_w)
    PostNorm post;                     // modes 3 and 4 (x_in, x_out, queue and embed as in the others)
    EmbedSrc embed; const int* queue; int ctx;
    SideOutputs prev;
    const float* x_in; float* x_out;
    const float* norm_w; float eps;
    const float* mu[kMixes];
    float* shift; size_t shift_slot;   // two slots of h, read at position parity, written at the other
    int d;
    // experts > 0 (mode 0): the segments' experts are chosen from the logits z and left in expert / weight [top]; a segment that
    // is a sum reads these instead
    Router router; const float* z; int* expert; float* weight;
    StepState* state;
    int share, rest;      // filled by the launcher: cost of a CTA, and what the division leaves
};
int launch_gemv_bf16_group(GemvGroup g, cudaStream_t st);

// ---- rot_attn.cu: what attention with rotated positions needs around the softmax ----------------------------
// Pair i of `dims` elements turns by position * base^(-2i/dims); freq[i] is that power in double. neighbours: elements 2i and
// 2i + 1 form a pair, else i and i + dims / 2.
struct Rot {
    int dims = 0;
    bool neighbours = false;
    const double* freq = nullptr;
};
// Grouped-query attention: q and k normed over their whole projection (q_norm / k_norm null: not), rotated on the first
// rot.dims elements of every head; scores times scale. Cached rows: KV heads of kp (keys) and vp (values) elements.
struct RotAttn {
    int H = 0, KV = 0, dim = 0, vdim = 0, kp = 0, vp = 0;
    float scale = 1.0f, eps = 0.0f;
    Rot rot;
    const float *q_norm = nullptr, *k_norm = nullptr;
    int window = kNoWindow;
    bool has_sink = false;             // one more exp(0) in the denominator
    bool own_kv = true;                // false: the keys and values of another layer's cache
};
// Rows at pos0 ..: q [M][H * kp] (times scale and factor) and, with own_kv, cache rows. proj rows: q | k | v.
int launch_rot_prep(const RotAttn& t, const float* proj, int ldp, int M, int pos0, float factor, void* q, void* kc, void* vc, bool f32, cudaStream_t st);
Flash rot_flash(const RotAttn& t, const void* kc, const void* vc, int ctx);

// Latent attention: a cached row is one normed latent of `rank` values, then one rotated key part of `rot.dims`, both shared by
// all heads; a head's own key part and its values are products of the latent. Row: [lat | rot_p], lat = rank up to 64s.
struct LatentAttn {
    int H = 0, dim = 0, vdim = 0, rank = 0;
    int dp = 0, vp = 0, lat = 0, rot_p = 0;     // elements of a head's expanded key / value row, of either part of a cached row
    float scale = 1.0f, eps = 0.0f;
    Rot rot;
    const float* c_norm = nullptr;
    int window = kNoWindow;
    const uint16_t *uk = nullptr, *uv = nullptr;     // [H * dp][lat], [H * vp][lat]: rows of a head padded with zeros
    int row() const { return lat + rot_p; }
};
// Rows at pos0 ..: q [M][H * (dp + rot_p)] (times scale and factor), cache rows. proj rows: q | latent | shared key part.
int launch_latent_prep(const LatentAttn& t, const float* proj, int ldp, int M, int pos0, float factor, void* q, void* cache, bool f32,
                       cudaStream_t st);
// Keys and values of positions base .. as expanded by products of the cached latents (rows of H * dp and H * vp).
Flash latent_flash(const LatentAttn& t, const void* k, const void* v, int rows, int base, const void* cache, int ctx);

// One token (attn_decode.cu). Latent: q' = [W_uk^T q | rotated part] per head, f32 [H][lat + rot_p], and the token's cache row.
int launch_latent_absorb(const LatentAttn& t, const float* proj, float* q, void* cache, bool f32, const StepState* state, cudaStream_t st);
// Splits of the visible cached rows against all heads. Grouped-query: prepares q itself, writes the token's cache row (own_kv),
// and the last split of a block of heads merges into out [H * vdim].
struct AttnDecode {
    int H = 0, KV = 0, kw = 0, vw = 0;               // values of a key / value row of one head (kw a multiple of 8)
    int k_ld = 0, k_head = 0, v_ld = 0, v_head = 0;  // row stride and head stride of the caches
    void *kc = nullptr, *vc = nullptr;               // vc null: the values are the first vw of a key row
    bool f32 = false;
    int window = kNoWindow;
    bool has_sink = false;
    RotAttn prep;                                    // H 0: q is ready (f32 [H][kw], scaled), the cache row written
    const float* q = nullptr;                        // the projection row q | k | v, or the ready queries
    float *part = nullptr, *part_ml = nullptr;       // [splits][H][vw up to 4s], [splits][H][2]
    int max_splits = 1, reach = 0;                   // reach: most rows a token can see
    unsigned int* counter = nullptr;                 // one a block of heads; null: the splits stay as they are
    float* out = nullptr;
    const StepState* state = nullptr;
};
constexpr int kMaxSplitsRow = 64;                     // most splits of a token
int launch_attn_decode_rows(const AttnDecode& a, cudaStream_t st);
int attn_decode_blocks(const AttnDecode& a);         // blocks of heads: counters needed
// Merges the splits of latent decoding and expands the values: out [H * vdim].
int launch_latent_expand(const LatentAttn& t, const AttnDecode& a, float* out, cudaStream_t st);

// ---- experts.cu: routed feed-forwards -----------------------------------------------------------------
// Routes M rows of x (f32, d apart; the same as operand rows in `plane`, ld apart): chosen expert and weight (softmax over all
// experts, not renormalised) of every slot, the places of the slots' rows once they are grouped by expert, those rows (bf16 or
// f32, ld apart) and the row tiles of the products. counts starts as zeros.
struct RouteRows {
    Router r;
    const float* x; int M, d;
    int *expert, *index, *counts; float* weight;     // [M][top], [M][top], [experts], [M][top]
    void* rows; int ld;
    int4* table; int* n_table; int tile_rows;
};
int max_row_tiles(const Router& r, int M, int tile_rows);
int launch_route_rows(const RouteRows& p, const void* plane, bool f32_rows, cudaStream_t st);
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
