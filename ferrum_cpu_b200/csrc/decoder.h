// Decoders whose model is a folder (config.json + model.safetensors): what every design of that kind shares. A design
// brings its configuration, tensors, cache contents and the kernels of a portion and of a decode step; loading, portions,
// the captured decode step, scoring, generation and the C ABI are here, once.
#pragma once
#include <cuda.h>

#include <initializer_list>
#include <string>
#include <utility>
#include <vector>

#include "bf16_ops.cuh"
#include "model_dir.h"

struct fc_decoder_cache;

// A model of some design on one GPU.
struct fc_decoder {
    // set by parse()
    int vocab = 0, width = 0, n_layers = 0, n_own_layers = 0;
    // set by the loader
    int device = 0, ctx = 0;
    bool f32 = false;
    cudaStream_t st = nullptr;
    cudaEvent_t ev0 = nullptr, ev1 = nullptr;
    fc::Arena arena, ws_arena;
    fc::BMat embed, head;
    float* final_norm = nullptr;
    CUtensorMap m_head, a_head;
    int64_t weight_bytes = 0;           // matrices a decode step reads: the head here, the layers' in tensors()
    // workspace of a portion of ws_rows tokens
    int ws_rows = 0, head_chunk = 0;
    void* planes = nullptr;             // n_planes() operands [ws_rows][head.K_pad]; the head reads plane 0
    float* logits = nullptr;
    int *ids_d = nullptr, *rows_d = nullptr, *targets_d = nullptr, *status = nullptr;     // status: [0] timeout, [1] bad id
    double* lp_d = nullptr;
    uint8_t* gr_d = nullptr;
    float last_forward_ms = 0.0f;

    virtual ~fc_decoder() {}
    virtual int parse(const fc::Json& config) = 0;
    // Looks up and checks every tensor of the layers; with `upload` puts them on the device.
    virtual int tensors(const fc::ModelDir& md, bool upload) = 0;
    virtual int n_planes() const { return 1; }
    virtual int workspace(int rows) = 0;                             // the design's own buffers, from ws_arena
    virtual fc_decoder_cache* make_cache() = 0;
    // M tokens whose ids are in ids_d through all layers, from the cache's position on. layers_out (host, may be null):
    // the residual stream after every layer.
    virtual int portion(fc_decoder_cache* s, int M, float* layers_out) = 0;
    // Final norm of n rows of the portion (indices on the device at `rows`) into plane 0.
    virtual int final_rows(const int* rows, int n) = 0;
    // The kernels of one decode step (without the bookkeeping at its end); logits to the cache's.
    virtual int step(fc_decoder_cache* s, bool with_head) = 0;

    size_t el() const { return f32 ? 4 : 2; }
    int zeroed(fc::Arena& a, void** p, size_t bytes);                // device memory that starts as zero
    template <class T>
    int zeroed_n(fc::Arena& a, T** p, size_t n) { return zeroed(a, (void**)p, n * sizeof(T)); }
};

// What one sequence holds. A design derives its own from it.
struct fc_decoder_cache {
    fc_decoder* m = nullptr;
    int device = 0;
    fc::Arena arena;
    float* logits = nullptr;
    int* queue = nullptr;
    int queue_cap = 0;
    fc::StepState* state = nullptr;
    unsigned long long* rng_d = nullptr;
    int host_pos = 0;
    cudaGraphExec_t graph[2] = {nullptr, nullptr};
    int graph_nodes[2] = {0, 0};
    cudaEvent_t ev0 = nullptr, ev1 = nullptr;
    float last_decode_ms = 0.0f;

    virtual ~fc_decoder_cache() {}
    virtual int create() = 0;                       // the design's buffers, from `arena`
    virtual int clear() { return FC_OK; }           // back to an empty sequence
};

namespace fc {

constexpr int kMaxPortion = 2048;       // tokens of one forward pass; longer portions are cut
constexpr int kMaxSplits = 64;          // attention splits of a decode step

// A design announces itself under the name config.json has in "architecture".
struct DecoderDesign {
    const char* architecture;
    fc_decoder* (*make)();
    const DecoderDesign* next;
    DecoderDesign(const char* name, fc_decoder* (*make)());
};

// Entries of a configuration; `where` names the object in messages.
int want_int(const Json* o, const char* key, const std::string& where, int* out);
int want_num(const Json* o, const char* key, const std::string& where, double* out);

// A tensor of the file with the shape it must have.
int find_tensor(const ModelDir& md, const std::string& name, std::initializer_list<int64_t> shape, const TensorView** out);
void to_f32(const TensorView& t, std::vector<float>* out);
// `rows` rows of a tensor from row `from` on.
struct Part { const TensorView* t; int rows; int from = 0; };
// Rows of several matrices with the same row length into one padded device matrix; every part starts at its row.
int upload_rows(Arena& ar, const std::vector<std::pair<int, Part>>& parts, int rows_total, int K, const char* what, BMat* out, cudaStream_t st);
int upload_vec(Arena& ar, const TensorView& t, float** out, cudaStream_t st);
int map_of(const BMat& w, CUtensorMap* m);

}  // namespace fc
