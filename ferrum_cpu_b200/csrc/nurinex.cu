// C ABI of the Nurinex decoder: a stack of layers in which attention (mixed heads, distance bias, sink) and a
// linear-attention recurrence stand side by side on one norm, next to a feed-forward on the same norm. Everything that
// differs between models of the design is read from the folder's config.json; a layer may use another layer's tensors
// with a cache and state of its own.
//
// Loading, the forward of a portion of tokens (prefill kernels), the decode step (captured in a CUDA graph), generation
// and scoring. Kernels: bf16_ops.cuh.
#include <algorithm>
#include <cmath>
#include <cstring>
#include <memory>
#include <string>
#include <vector>

#include "bf16_ops.cuh"
#include "decode_loop.cuh"
#include "llama_ops.cuh"
#include "model_dir.h"
#include "tc_common.cuh"

using namespace fc;

namespace {

constexpr int kMaxPortion = 2048;       // tokens of one forward pass; longer portions are cut
constexpr int kFfSplits = 4;            // most partial sums of the feed-forward's second product
constexpr int kMaxSplits = 64;          // attention splits of a decode step

// The entries of config.json for one layer.
struct LayerCfg {
    int owner = 0;                      // layer whose tensors it uses
    int H = 0, KV = 0, dim = 0, vdim = 0;
    double bias_max = 0, scale = 0, temp_coef = 0, temp_every = 1;
    int rH = 0, rdim = 0;
    int ff = 0;                         // 0: no feed-forward
};
struct Config {
    int vocab = 0, width = 0;
    double eps = 0, emb_scale = 1;
    std::vector<LayerCfg> layers;
};

int want_int(const Json* o, const char* key, const std::string& where, int* out) {
    const Json* v = o ? o->find(key) : nullptr;
    if (!v || v->kind != Json::Number || v->num != std::floor(v->num) || v->num < 1 || v->num > 1e9)
        return fail(FC_E_FORMAT, "config.json: %s.%s must be a positive whole number", where.c_str(), key);
    *out = (int)v->num;
    return FC_OK;
}
int want_num(const Json* o, const char* key, const std::string& where, double* out) {
    const Json* v = o ? o->find(key) : nullptr;
    if (!v || v->kind != Json::Number || !std::isfinite(v->num)) return fail(FC_E_FORMAT, "config.json: %s.%s must be a number", where.c_str(), key);
    *out = v->num;
    return FC_OK;
}

int parse_config(const Json& j, Config* c) {
    const Json* arch = j.find("architecture");
    if (!arch || arch->str != "Nurinex") return fail(FC_E_FORMAT, "config.json: architecture is not Nurinex");
    FC_TRY(want_int(&j, "vocab", "config", &c->vocab));
    FC_TRY(want_int(&j, "width", "config", &c->width));
    FC_TRY(want_num(j.find("norm"), "eps", "norm", &c->eps));
    if (j.has("embedding") && j.find("embedding")->has("scale")) FC_TRY(want_num(j.find("embedding"), "scale", "embedding", &c->emb_scale));
    const Json* layers = j.find("layers");
    if (!layers || layers->kind != Json::Array || layers->items.empty()) return fail(FC_E_FORMAT, "config.json: layers must be a list");
    const int n = (int)layers->items.size();
    c->layers.resize(n);
    for (int i = 0; i < n; ++i) {
        const Json& e = layers->items[i];
        LayerCfg& L = c->layers[i];
        const std::string at = "layers[" + std::to_string(i) + "]";
        const Json* type = e.find("type");
        if (!type || type->str != "parallel") return fail(FC_E_FORMAT, "config.json: %s: layer type '%s' is not known", at.c_str(), type ? type->str.c_str() : "");
        L.owner = i;
        if (e.has("weights_of")) {
            const double w = e.find("weights_of")->num;
            if (e.find("weights_of")->kind != Json::Number || w < 0 || w >= n || w != std::floor(w))
                return fail(FC_E_FORMAT, "config.json: %s.weights_of names no layer", at.c_str());
            L.owner = (int)w;
        }
        const Json* mix = e.find("mixer");
        const Json *l = mix ? mix->find("left") : nullptr, *r = mix ? mix->find("right") : nullptr;
        FC_TRY(want_int(l, "heads", at + ".mixer.left", &L.H));
        FC_TRY(want_int(l, "kv_heads", at + ".mixer.left", &L.KV));
        FC_TRY(want_int(l, "dim", at + ".mixer.left", &L.dim));
        FC_TRY(want_int(l, "vdim", at + ".mixer.left", &L.vdim));
        FC_TRY(want_num(l, "scale", at + ".mixer.left", &L.scale));
        FC_TRY(want_num(l, "bias_max", at + ".mixer.left", &L.bias_max));
        if (l->has("q_temp")) {
            FC_TRY(want_num(l->find("q_temp"), "coef", at + ".mixer.left.q_temp", &L.temp_coef));
            FC_TRY(want_num(l->find("q_temp"), "every", at + ".mixer.left.q_temp", &L.temp_every));
        }
        FC_TRY(want_int(r, "heads", at + ".mixer.right", &L.rH));
        FC_TRY(want_int(r, "dim", at + ".mixer.right", &L.rdim));
        if (L.H % L.KV) return fail(FC_E_DIM, "%s: %d query heads cannot share %d key/value heads", at.c_str(), L.H, L.KV);
        if (!(L.temp_every > 0)) return fail(FC_E_DIM, "%s: q_temp.every must be positive", at.c_str());
        if (L.vdim > 256 || L.rdim > 256) return fail(FC_E_SHAPE, "%s: value heads and recurrence heads of at most 256", at.c_str());
        if (e.has("mlp")) {
            const Json* kind = e.find("mlp")->find("kind");
            if (!kind || kind->str != "dense") return fail(FC_E_FORMAT, "config.json: %s: feed-forward kind '%s' is not known", at.c_str(), kind ? kind->str.c_str() : "");
            FC_TRY(want_int(e.find("mlp"), "ff", at + ".mlp", &L.ff));
        }
    }
    for (int i = 0; i < n; ++i) {           // follow references to the layer that has tensors
        int o = i, hops = 0;
        while (c->layers[o].owner != o && hops++ < n) o = c->layers[o].owner;
        if (c->layers[o].owner != o) return fail(FC_E_FORMAT, "config.json: layers[%d].weights_of runs in a circle", i);
        const LayerCfg &a = c->layers[i], &b = c->layers[o];
        if (a.H != b.H || a.KV != b.KV || a.dim != b.dim || a.vdim != b.vdim || a.rH != b.rH || a.rdim != b.rdim || a.ff != b.ff)
            return fail(FC_E_DIM, "config.json: layers[%d] does not have the sizes of the layer whose tensors it uses", i);
        c->layers[i].owner = o;
    }
    return FC_OK;
}

// The bias row of distance n: half the rows one by one, then equal steps of ln n up to bias_max. A quotient that is a
// whole number in exact arithmetic may come out a rounding below it; 1e-10 puts it back.
int distance_bucket(int n, int rows, double bias_max) {
    const int half = rows / 2;
    if (n < half) return n;
    const double f = std::log((double)n / half) / std::log(bias_max / half) * (rows - half);
    return (int)std::min<double>(rows - 1, half + std::floor(f + 1e-10));
}

// A tensor of the file with the shape it must have.
int find_tensor(const ModelDir& md, const std::string& name, std::initializer_list<int64_t> shape, const TensorView** out) {
    const TensorView* t = md.tensor(name);
    if (!t) return fail(FC_E_FORMAT, "tensor %s is missing", name.c_str());
    if (t->shape.size() != shape.size() || !std::equal(shape.begin(), shape.end(), t->shape.begin()))
        return fail(FC_E_DIM, "tensor %s does not have the shape the configuration asks for", name.c_str());
    if (t->dtype != "BF16" && t->dtype != "F32") return fail(FC_E_FORMAT, "tensor %s: type %s is not read here", name.c_str(), t->dtype.c_str());
    *out = t;
    return FC_OK;
}
float bf16_value(uint16_t b) {
    const uint32_t u = (uint32_t)b << 16;
    float f;
    std::memcpy(&f, &u, 4);
    return f;
}
void to_f32(const TensorView& t, std::vector<float>* out) {
    const size_t n = t.dtype == "F32" ? t.nbytes / 4 : t.nbytes / 2;
    out->resize(n);
    if (t.dtype == "F32") { std::memcpy(out->data(), t.data, t.nbytes); return; }
    for (size_t i = 0; i < n; ++i) {
        uint16_t b;
        std::memcpy(&b, t.data + 2 * i, 2);
        (*out)[i] = bf16_value(b);
    }
}

}  // namespace

// The tensors of one layer on the device.
struct NxWeights {
    TalkAttn t;
    int rH = 0, rdim = 0, rank = 0, ff = 0;
    BMat in, lo, ro, w2, down;          // `in`: rows of every product of the norm and its mixes, one after the other
    int row_up = 0, row_r = 0, row_k = 0, row_v = 0, row_g = 0, row_w1 = 0;      // first rows inside `in` (q | k | v at 0)
    int off_r = 0, off_k = 0, off_v = 0, off_g = 0, off_w1 = 0, proj = 0;        // columns of a projection row (q | k | v at 0)
    int n_qkv = 0;
    float *norm1 = nullptr, *mu[kMixes] = {}, *w0 = nullptr, *u = nullptr, *rnorm = nullptr, *left_out = nullptr, *right_out = nullptr;
    float c0 = 0, c1 = 0;               // the feed-forward's activation
    CUtensorMap m_in, m_lo, m_ro, m_down;              // weight maps
    CUtensorMap a_planes, a_att, a_ro, a_hid;          // operand maps into the workspace
};

struct fc_nurinex {
    Config cfg;
    int device = 0, mode = 0, ctx = 0;
    bool f32 = false;
    cudaStream_t st = nullptr, side = nullptr;
    cudaEvent_t fork = nullptr, join = nullptr, ev0 = nullptr, ev1 = nullptr;
    Arena arena, ws_arena;
    BMat embed, head;
    float* final_norm = nullptr;
    std::vector<std::unique_ptr<NxWeights>> own;       // by layer index; null where another layer's are used
    std::vector<const NxWeights*> run;                 // by layer
    int max_proj = 0, max_att = 0, max_ro = 0, max_hid = 0, max_qm = 0, max_rd = 0, max_qo = 0;
    int64_t weight_bytes = 0;                          // matrices a decode step reads
    CUtensorMap m_head, a_head;
    // workspace of a portion of ws_rows tokens
    int ws_rows = 0, head_chunk = 0;
    float *x[2] = {}, *proj = nullptr, *outs = nullptr, *decay = nullptr, *wkv_o = nullptr, *logits = nullptr, *h_last = nullptr, *wkv_scratch = nullptr;
    void *planes = nullptr, *att = nullptr, *ro = nullptr, *hid = nullptr, *qm = nullptr;
    int *ids_d = nullptr, *rows_d = nullptr, *targets_d = nullptr, *status = nullptr;     // status: [0] timeout, [1] bad id
    double* lp_d = nullptr;
    uint8_t* gr_d = nullptr;
    float last_forward_ms = 0.0f;
};

struct fc_nurinex_cache {
    fc_nurinex* m = nullptr;
    int device = 0;
    Arena arena;
    std::vector<void*> kc, vc;                 // per layer: [ctx][kd], [ctx][KV][vp]
    std::vector<float*> wkv;                   // per layer: [rH][rdim][rdim]
    float* shift = nullptr;                    // [2][layers][width]: h of the token before, by the parity of the position
    float* state_block = nullptr;              // recurrence states and `shift`, one block
    size_t state_floats = 0;
    float *x[2] = {}, *proj = nullptr, *outs = nullptr, *hid = nullptr, *att = nullptr, *ro = nullptr, *logits = nullptr;
    float *part = nullptr, *part_ml = nullptr;
    unsigned int* counter = nullptr;
    int max_splits = 1;
    int* queue = nullptr;
    int queue_cap = 0;
    StepState* state = nullptr;
    unsigned long long* rng_d = nullptr;
    int host_pos = 0;
    cudaGraphExec_t graph[2] = {nullptr, nullptr};
    int graph_nodes[2] = {0, 0};
    cudaEvent_t ev0 = nullptr, ev1 = nullptr;
    float last_decode_ms = 0.0f;
};

namespace {

// ------------------------------------------------------------------------------------ loading
struct Part { const TensorView* t; int rows; };
// Rows of several matrices with the same row length into one padded device matrix; every part starts at its row0.
int upload_rows(Arena& ar, const std::vector<std::pair<int, Part>>& parts, int rows_total, int K, const char* what, BMat* out, cudaStream_t st) {
    const int K_pad = pad_to(K, 64), N_pad = pad_to(rows_total, 128);
    std::vector<uint16_t> buf((size_t)N_pad * K_pad, 0);
    for (auto& p : parts) {
        if (p.second.t->dtype != "BF16") return fail(FC_E_FORMAT, "%s: matrices must be stored as BF16", what);
        for (int r = 0; r < p.second.rows; ++r)
            std::memcpy(buf.data() + (size_t)(p.first + r) * K_pad, p.second.t->data + (size_t)r * K * 2, (size_t)K * 2);
    }
    uint16_t* d = nullptr;
    FC_TRY(ar.alloc_n(&d, buf.size()));
    FC_CUDA(cudaMemcpyAsync(d, buf.data(), buf.size() * 2, cudaMemcpyHostToDevice, st));
    FC_CUDA(cudaStreamSynchronize(st));
    out->w = d; out->N = rows_total; out->K = K; out->N_pad = N_pad; out->K_pad = K_pad;
    return FC_OK;
}
int upload_vec(Arena& ar, const TensorView& t, float** out, cudaStream_t st) {
    std::vector<float> v;
    to_f32(t, &v);
    FC_TRY(upload_f32(ar, v.data(), v.size(), out, st));
    FC_CUDA(cudaStreamSynchronize(st));
    return FC_OK;
}
int map_of(const BMat& w, CUtensorMap* m) { return tc::encode_bf16(m, w.w, w.N_pad, w.K_pad, w.K_pad, kGemmBoxRows); }

// Looks up and checks every tensor of a layer; with `w` uploads them.
int load_layer(const ModelDir& md, const Config& c, int i, fc_nurinex* m, NxWeights* w) {
    const LayerCfg& L = c.layers[i];
    const int d = c.width, rd = L.rH * L.rdim;
    const std::string p = "l" + std::to_string(i) + ".";
    const TensorView *q, *k, *v, *rel, *talk, *sink, *lo, *mu[kMixes], *r, *rk, *rv, *rg, *w1, *w2, *w0, *u, *rn, *ro, *lout, *rout, *n1;
    const TensorView *up = nullptr, *down = nullptr, *act = nullptr;
    auto get = [&](const char* name, std::initializer_list<int64_t> shape, const TensorView** out) { return find_tensor(md, p + name, shape, out); };
    FC_TRY(get("norm1", {d}, &n1));
    FC_TRY(get("mix.left.q", {(int64_t)L.H * L.dim, d}, &q));
    FC_TRY(get("mix.left.k", {(int64_t)L.KV * L.dim, d}, &k));
    FC_TRY(get("mix.left.v", {(int64_t)L.KV * L.vdim, d}, &v));
    const TensorView* any = md.tensor(p + "mix.left.rel");
    const int rows = any && any->shape.size() == 2 ? (int)any->shape[0] : 0;
    FC_TRY(get("mix.left.rel", {rows, L.H}, &rel));
    FC_TRY(get("mix.left.talk", {L.H, L.H}, &talk));
    FC_TRY(get("mix.left.sink", {L.H}, &sink));
    FC_TRY(get("mix.left.o", {d, (int64_t)L.H * L.vdim}, &lo));
    const char* names[kMixes] = {"mix.right.mu.r", "mix.right.mu.k", "mix.right.mu.v", "mix.right.mu.g", "mix.right.mu.w"};
    for (int s = 0; s < kMixes; ++s) FC_TRY(get(names[s], {d}, &mu[s]));
    FC_TRY(get("mix.right.r", {rd, d}, &r));
    FC_TRY(get("mix.right.k", {rd, d}, &rk));
    FC_TRY(get("mix.right.v", {rd, d}, &rv));
    FC_TRY(get("mix.right.g", {rd, d}, &rg));
    any = md.tensor(p + "mix.right.w1");
    const int rank = any && any->shape.size() == 2 ? (int)any->shape[0] : 0;
    FC_TRY(get("mix.right.w1", {rank, d}, &w1));
    FC_TRY(get("mix.right.w2", {rd, rank}, &w2));
    FC_TRY(get("mix.right.w0", {rd}, &w0));
    FC_TRY(get("mix.right.u", {L.rH, L.rdim}, &u));
    FC_TRY(get("mix.right.norm", {rd}, &rn));
    FC_TRY(get("mix.right.o", {d, rd}, &ro));
    FC_TRY(get("mix.left.out", {d}, &lout));
    FC_TRY(get("mix.right.out", {d}, &rout));
    if (L.ff) {
        FC_TRY(get("mlp.up", {L.ff, d}, &up));
        FC_TRY(get("mlp.down", {d, L.ff}, &down));
        FC_TRY(get("mlp.act", {2}, &act));
    }
    if (rows < 2 || rank < 1) return fail(FC_E_SHAPE, "layer %d: the bias table and the decay projection need rows", i);
    if (!(L.bias_max > rows / 2) || L.bias_max > (1 << 20)) return fail(FC_E_DIM, "layer %d: bias_max must lie above half the table's rows", i);
    if (!w) return FC_OK;

    cudaStream_t st = m->st;
    Arena& ar = m->arena;
    TalkAttn& t = w->t;
    t.H = L.H; t.KV = L.KV; t.dim = L.dim; t.vdim = L.vdim;
    t.kd = pad_to(L.KV * L.dim, 16); t.vp = pad_to(L.vdim, 16);
    t.far = (int)std::ceil(L.bias_max);
    t.scale = (float)L.scale; t.temp_coef = (float)L.temp_coef; t.temp_every = L.temp_every; t.eps = (float)c.eps;
    w->rH = L.rH; w->rdim = L.rdim; w->rank = rank; w->ff = L.ff;
    // one matrix for every product of the norm's output and its mixes
    w->n_qkv = L.H * L.dim + L.KV * (L.dim + L.vdim);
    std::vector<std::pair<int, Part>> parts;
    int row = 0;
    auto add = [&](const TensorView* x, int n) { parts.push_back({row, {x, n}}); row += n; };
    auto align = [&] { row = pad_to(row, 128); };
    add(q, L.H * L.dim); add(k, L.KV * L.dim); add(v, L.KV * L.vdim); align();
    w->row_up = row; if (L.ff) { add(up, L.ff); align(); }
    w->row_r = row; add(r, rd); align();
    w->row_k = row; add(rk, rd); align();
    w->row_v = row; add(rv, rd); align();
    w->row_g = row; add(rg, rd); align();
    w->row_w1 = row; add(w1, rank); align();
    FC_TRY(upload_rows(ar, parts, row, d, "layer projections", &w->in, st));
    FC_TRY(upload_rows(ar, {{0, {lo, d}}}, d, L.H * L.vdim, "mix.left.o", &w->lo, st));
    FC_TRY(upload_rows(ar, {{0, {ro, d}}}, d, rd, "mix.right.o", &w->ro, st));
    FC_TRY(upload_rows(ar, {{0, {w2, rd}}}, rd, rank, "mix.right.w2", &w->w2, st));
    if (L.ff) FC_TRY(upload_rows(ar, {{0, {down, d}}}, d, L.ff, "mlp.down", &w->down, st));
    FC_TRY(map_of(w->in, &w->m_in));
    FC_TRY(map_of(w->lo, &w->m_lo));
    FC_TRY(map_of(w->ro, &w->m_ro));
    w->m_down = w->m_ro;
    if (L.ff) FC_TRY(map_of(w->down, &w->m_down));
    int off = pad_to(w->n_qkv, 8);
    w->off_r = off; off += pad_to(rd, 8);
    w->off_k = off; off += pad_to(rd, 8);
    w->off_v = off; off += pad_to(rd, 8);
    w->off_g = off; off += pad_to(rd, 8);
    w->off_w1 = off; off += w->w2.K_pad;
    w->proj = pad_to(off, 8);
    FC_TRY(upload_vec(ar, *n1, &w->norm1, st));
    for (int s = 0; s < kMixes; ++s) FC_TRY(upload_vec(ar, *mu[s], &w->mu[s], st));
    FC_TRY(upload_vec(ar, *w0, &w->w0, st));
    FC_TRY(upload_vec(ar, *u, &w->u, st));
    FC_TRY(upload_vec(ar, *rn, &w->rnorm, st));
    FC_TRY(upload_vec(ar, *lout, &w->left_out, st));
    FC_TRY(upload_vec(ar, *rout, &w->right_out, st));
    float* dev = nullptr;
    FC_TRY(upload_vec(ar, *talk, &dev, st)); t.talk = dev;
    FC_TRY(upload_vec(ar, *sink, &dev, st)); t.sink = dev;
    // the bias of every distance, heads already mixed: row h of talk times the table's row
    std::vector<float> tk, rl;
    to_f32(*talk, &tk);
    to_f32(*rel, &rl);
    std::vector<float> bias((size_t)L.H * (t.far + 1));
    for (int n = 0; n <= t.far; ++n) {
        const int b = distance_bucket(n, rows, L.bias_max);
        for (int h = 0; h < L.H; ++h) {
            double s = 0.0;
            for (int g = 0; g < L.H; ++g) s += (double)tk[(size_t)h * L.H + g] * rl[(size_t)b * L.H + g];
            bias[(size_t)h * (t.far + 1) + n] = (float)s;
        }
    }
    FC_TRY(upload_f32(ar, bias.data(), bias.size(), &dev, st)); t.bias = dev;
    FC_CUDA(cudaStreamSynchronize(st));
    if (L.ff) {
        std::vector<float> a;
        to_f32(*act, &a);
        auto softplus = [](double z) { return z > 30 ? z : std::log1p(std::exp(z)); };
        w->c0 = (float)softplus(a[0]);
        w->c1 = (float)(0.5 + softplus(a[1]));
    }
    return FC_OK;
}

size_t el(const fc_nurinex* m) { return m->f32 ? 4 : 2; }

int ensure_workspace(fc_nurinex* m, int rows) {
    if (rows <= m->ws_rows) return FC_OK;
    int R = 128;
    while (R < rows) R *= 2;
    FC_CUDA(cudaStreamSynchronize(m->st));
    m->ws_arena.release();
    m->ws_rows = 0;
    const int d = m->cfg.width, dp = m->head.K_pad;
    const size_t RR = R, e = el(m);
    Arena& a = m->ws_arena;
    // padding columns must hold finite values (they meet zero weights): everything starts as zero
    auto get = [&](void** p, size_t bytes) -> int {
        FC_TRY(a.alloc(p, bytes));
        FC_CUDA(cudaMemsetAsync(*p, 0, bytes ? bytes : 16, m->st));
        return FC_OK;
    };
    FC_TRY(get((void**)&m->x[0], RR * d * 4));
    FC_TRY(get((void**)&m->x[1], RR * d * 4));
    FC_TRY(get((void**)&m->proj, RR * m->max_proj * 4));
    FC_TRY(get((void**)&m->outs, (2 + kFfSplits) * RR * d * 4));
    FC_TRY(get((void**)&m->decay, RR * m->max_rd * 4));
    FC_TRY(get((void**)&m->wkv_o, RR * m->max_rd * 4));
    size_t scratch = 0;
    for (const NxWeights* w : m->run) scratch = std::max(scratch, wkv_scratch_floats(w->rH, w->rdim));
    FC_TRY(get((void**)&m->wkv_scratch, scratch * 4));
    FC_TRY(get((void**)&m->h_last, (size_t)m->cfg.layers.size() * d * 4));
    FC_TRY(get(&m->planes, (1 + kMixes) * RR * dp * e));
    FC_TRY(get(&m->att, RR * m->max_att * e));
    FC_TRY(get(&m->ro, RR * m->max_ro * e));
    FC_TRY(get(&m->hid, RR * m->max_hid * e));
    FC_TRY(get(&m->qm, RR * m->max_qm * e));
    m->head_chunk = (int)std::max<size_t>(1, std::min<size_t>(RR, ((size_t)1 << 27) / m->head.N_pad));
    FC_TRY(get((void**)&m->logits, (size_t)m->head_chunk * m->head.N_pad * 4));
    FC_TRY(get((void**)&m->ids_d, RR * 4));
    FC_TRY(get((void**)&m->rows_d, RR * 4));
    FC_TRY(get((void**)&m->targets_d, RR * 4));
    FC_TRY(get((void**)&m->lp_d, RR * 8));
    FC_TRY(get((void**)&m->gr_d, RR));
    FC_TRY(get((void**)&m->status, 8));
    if (!m->f32) {
        for (auto& w : m->own) {
            if (!w) continue;
            FC_TRY(tc::encode_bf16(&w->a_planes, m->planes, (1 + kMixes) * RR, dp, dp, kGemmBoxRows));
            FC_TRY(tc::encode_bf16(&w->a_att, m->att, RR, w->lo.K_pad, w->lo.K_pad, kGemmBoxRows));
            FC_TRY(tc::encode_bf16(&w->a_ro, m->ro, RR, w->ro.K_pad, w->ro.K_pad, kGemmBoxRows));
            w->a_hid = w->a_ro;
            if (w->ff) FC_TRY(tc::encode_bf16(&w->a_hid, m->hid, RR, w->down.K_pad, w->down.K_pad, kGemmBoxRows));
        }
        FC_TRY(tc::encode_bf16(&m->a_head, m->planes, RR, dp, dp, kGemmBoxRows));
    }
    m->ws_rows = R;
    return FC_OK;
}

int check_ids(const fc_nurinex* m, const int32_t* ids, size_t n) {
    for (size_t i = 0; i < n; ++i)
        if (ids[i] < 0 || ids[i] >= m->cfg.vocab) return fail(FC_E_DIM, "token %d ≥ vocab_size %d", ids[i], m->cfg.vocab);
    return FC_OK;
}
int check_status(fc_nurinex* m) {
    int s[2] = {0, 0};
    FC_CUDA(cudaMemcpyAsync(s, m->status, 8, cudaMemcpyDeviceToHost, m->st));
    FC_CUDA(cudaStreamSynchronize(m->st));
    if (s[0] || s[1]) cudaMemsetAsync(m->status, 0, 8, m->st);
    if (s[0]) return fail(FC_E_TIMEOUT, "a bounded wait inside a tensor-core kernel ran out (status %d)", s[0]);
    if (s[1]) return fail(s[1], "a token id was rejected on the device");
    return FC_OK;
}

// ---------------------------------------------------------------------- a portion of tokens
// How many partial sums the feed-forward's second product is cut into. The tiles of the three output products go round
// robin over the SMs, the longest first; with few tiles the feed-forward's long K decides, so the number is the one whose
// busiest SM has the least to do (each further partial sum counts as a little extra traffic).
int ff_splits(const NxWeights& w, int M) {
    if (!w.ff) return 0;
    const int tiles = ((w.down.N + 127) / 128) * ((M + 255) / 256), kb = w.down.K_pad / 64, lo = w.lo.K_pad / 64, ro = w.ro.K_pad / 64;
    int best = 1;
    double least = 1e30;
    for (int f = 1; f <= std::min(kFfSplits, kb); ++f) {
        std::vector<int> load(148, 0);
        int at = 0;
        auto add = [&](int n, int cost) { for (int i = 0; i < n; ++i) load[at++ % 148] += cost + 4; };
        add(tiles * f, (kb + f - 1) / f);
        add(tiles, lo);
        add(tiles, ro);
        const double cost = *std::max_element(load.begin(), load.end()) * (1.0 + 0.03 * (f - 1));
        if (cost < least) { least = cost; best = f; }
    }
    return best;
}

SideOutputs outputs_of(const NxWeights& w, const float* outs, size_t stride, int n_ff) {
    SideOutputs o;
    o.outs = outs; o.stride = stride; o.n_ff = n_ff; o.left_w = w.left_out; o.right_w = w.right_out;
    return o;
}

// One layer's products and mixers for M rows whose norm and mixes are in the planes; positions pos0...
int layer_forward(fc_nurinex* m, fc_nurinex_cache* s, int l, int M, int pos0, int* n_ff) {
    const NxWeights& w = *m->run[l];
    cudaStream_t st = m->st;
    const int R = m->ws_rows, dp = m->head.K_pad, d = m->cfg.width, rd = w.rH * w.rdim;
    const int ldp = w.proj;
    struct In { int plane, row, n, off; };
    const In in[6] = {{0, 0, w.n_qkv, 0}, {1, w.row_r, rd, w.off_r}, {2, w.row_k, rd, w.off_k}, {3, w.row_v, rd, w.off_v},
                      {4, w.row_g, rd, w.off_g}, {5, w.row_w1, w.rank, w.off_w1}};
    if (m->f32) {
        for (const In& x : in) {
            GemmF32 p = {};
            p.a = (const float*)m->planes + (size_t)x.plane * R * dp; p.lda = dp; p.y = m->proj + x.off; p.ldy = ldp;
            FC_TRY(launch_gemm_bf16w_f32(w.in, x.row, x.n, p, M, st));
        }
        if (w.ff) {
            GemmF32 p = {};
            p.a = (const float*)m->planes; p.lda = dp; p.y = (float*)m->hid; p.ldy = w.down.K_pad;
            p.epi = ROW_XIELU; p.c0 = w.c0; p.c1 = w.c1;
            FC_TRY(launch_gemm_bf16w_f32(w.in, w.row_up, w.ff, p, M, st));
        }
    } else {
        GemmMaps maps;
        for (int i = 0; i < 3; ++i) { maps.a[i] = w.a_planes; maps.b[i] = w.m_in; }
        GemmGroup g = {};
        for (const In& x : in) {
            GemmSeg& q = g.seg[g.n_seg++];
            q.a_row0 = x.plane * R; q.b_row0 = x.row; q.kb = dp / 64; q.n = x.n; q.y = m->proj + x.off; q.ldy = ldp;
        }
        if (w.ff) {
            GemmSeg& q = g.seg[g.n_seg++];
            q.b_row0 = w.row_up; q.kb = dp / 64; q.n = w.ff; q.yb = (uint16_t*)m->hid; q.ldy = w.down.K_pad;
            q.epi = ROW_XIELU; q.c0 = w.c0; q.c1 = w.c1;
        }
        FC_TRY(launch_gemm_bf16_group(maps, g, M, m->status, st));
    }
    // the recurrence runs beside the attention
    FC_CUDA(cudaEventRecord(m->fork, st));
    FC_CUDA(cudaStreamWaitEvent(m->side, m->fork, 0));
    {
        GemmF32 p = {};
        p.a = m->proj + w.off_w1; p.lda = ldp; p.tanh_in = 1; p.y = m->decay; p.ldy = rd; p.epi = ROW_DECAY; p.vec = w.w0;
        FC_TRY(launch_gemm_bf16w_f32(w.w2, 0, rd, p, M, m->side));
        FC_TRY(launch_wkv_scan(m->proj + w.off_r, m->proj + w.off_k, m->proj + w.off_v, ldp, m->decay, rd, w.u, s->wkv[l], m->wkv_o, rd, M, w.rH,
                               w.rdim, m->wkv_scratch, m->side));
        FC_TRY(launch_wkv_finish(m->wkv_o, rd, m->proj + w.off_g, ldp, w.rnorm, (float)m->cfg.eps, M, w.rH, w.rdim, m->ro, w.ro.K_pad, m->f32, m->side));
    }
    FC_CUDA(cudaEventRecord(m->join, m->side));
    FC_TRY(launch_talk_prep(w.t, m->proj, ldp, M, pos0, m->f32 ? 1.0f : kLog2e, m->qm, s->kc[l], s->vc[l], m->f32, st));
    if (m->f32) FC_TRY(launch_talk_prefill_f32(w.t, (const float*)m->qm, (const float*)s->kc[l], (const float*)s->vc[l], M, pos0, (float*)m->att, w.lo.K_pad, st));
    else FC_TRY(launch_talk_prefill_tc(w.t, m->qm, s->kc[l], s->vc[l], M, pos0, m->ctx, m->att, w.lo.K_pad, m->status, st));
    FC_CUDA(cudaStreamWaitEvent(st, m->join, 0));
    const size_t stride = (size_t)R * d;
    if (m->f32) {
        *n_ff = w.ff ? 1 : 0;
        GemmF32 p = {};
        p.ldy = d;
        p.a = (const float*)m->att; p.lda = w.lo.K_pad; p.y = m->outs;
        FC_TRY(launch_gemm_bf16w_f32(w.lo, 0, d, p, M, st));
        p.a = (const float*)m->ro; p.lda = w.ro.K_pad; p.y = m->outs + stride;
        FC_TRY(launch_gemm_bf16w_f32(w.ro, 0, d, p, M, st));
        if (w.ff) {
            p.a = (const float*)m->hid; p.lda = w.down.K_pad; p.y = m->outs + 2 * stride;
            FC_TRY(launch_gemm_bf16w_f32(w.down, 0, d, p, M, st));
        }
        return FC_OK;
    }
    GemmMaps maps;
    maps.a[0] = w.a_att; maps.a[1] = w.a_ro; maps.a[2] = w.a_hid;
    maps.b[0] = w.m_lo; maps.b[1] = w.m_ro; maps.b[2] = w.m_down;
    GemmGroup g = {};
    auto seg = [&](int which, int kb0, int kb, int out) {
        GemmSeg& q = g.seg[g.n_seg++];
        q.a_map = q.b_map = which; q.kb0 = kb0; q.kb = kb; q.n = d; q.y = m->outs + (size_t)out * stride; q.ldy = d;
    };
    *n_ff = ff_splits(w, M);
    const int kb = w.ff ? w.down.K_pad / 64 : 0;
    for (int f = 0; f < *n_ff; ++f) seg(2, kb * f / *n_ff, kb * (f + 1) / *n_ff - kb * f / *n_ff, 2 + f);
    seg(0, 0, w.lo.K_pad / 64, 0);
    seg(1, 0, w.ro.K_pad / 64, 1);
    return launch_gemm_bf16_group(maps, g, M, m->status, st);
}

// M tokens whose ids are in m->ids_d through all layers, from the cache's position on. Afterwards `tail` runs the rows
// it wants through the final norm (finish_rows). layers_out (host, may be null): residual stream after every layer.
struct Tail { MixRows rows; };
int portion_forward(fc_nurinex* m, fc_nurinex_cache* s, int M, float* layers_out, Tail* tail) {
    const Config& c = m->cfg;
    const int d = c.width, L = (int)c.layers.size(), R = m->ws_rows, dp = m->head.K_pad, pos0 = s->host_pos;
    cudaStream_t st = m->st;
    MixRows p = {};
    p.embed.table = m->embed.w; p.embed.vocab = c.vocab; p.embed.ld = m->embed.K_pad; p.embed.scale = (float)c.emb_scale;
    p.ids = m->ids_d; p.eps = (float)c.eps; p.M = M; p.d = d; p.ld = dp; p.planes = m->planes; p.plane_stride = (size_t)R * dp;
    p.error_flag = m->status + 1;
    int n_ff = 0;
    for (int l = 0; l < L; ++l) {
        const NxWeights& w = *m->run[l];
        if (l) p.prev = outputs_of(*m->run[l - 1], m->outs, (size_t)R * d, n_ff);
        p.x_in = m->x[l & 1]; p.x_out = m->x[(l + 1) & 1];
        p.norm_w = w.norm1;
        for (int i = 0; i < kMixes; ++i) p.mu[i] = w.mu[i];
        p.h_first = s->shift + ((size_t)(pos0 & 1) * L + l) * d;
        p.h_last = m->h_last + (size_t)l * d;
        FC_TRY(launch_mix_rows(p, m->f32, st));
        if (layers_out && l)
            FC_CUDA(cudaMemcpyAsync(layers_out + (size_t)(l - 1) * M * d, p.x_out, (size_t)M * d * 4, cudaMemcpyDeviceToHost, st));
        FC_TRY(layer_forward(m, s, l, M, pos0, &n_ff));
    }
    FC_CUDA(cudaMemcpyAsync(s->shift + (size_t)((pos0 + M) & 1) * L * d, m->h_last, (size_t)L * d * 4, cudaMemcpyDeviceToDevice, st));
    p.prev = outputs_of(*m->run[L - 1], m->outs, (size_t)R * d, n_ff);
    p.x_in = m->x[L & 1];
    p.x_out = nullptr;
    for (auto& x : p.mu) x = nullptr;
    p.h_first = nullptr; p.h_last = nullptr;
    if (layers_out) {
        p.x_out = m->x[(L + 1) & 1];
        p.norm_w = nullptr;
        FC_TRY(launch_mix_rows(p, m->f32, st));
        FC_CUDA(cudaMemcpyAsync(layers_out + (size_t)(L - 1) * M * d, p.x_out, (size_t)M * d * 4, cudaMemcpyDeviceToHost, st));
        p.x_out = nullptr;
    }
    p.norm_w = m->final_norm;
    tail->rows = p;
    s->host_pos += M;
    return launch_step_set(s->state, s->host_pos, s->host_pos, s->host_pos, st);
}

// Final norm and head for n rows of the portion (their indices on the device in m->rows_d + at); logits [n][ldl].
int head_rows(fc_nurinex* m, const Tail& tail, int at, int n, float* logits, int ldl) {
    MixRows p = tail.rows;
    p.row_idx = m->rows_d + at;
    p.M = n;
    FC_TRY(launch_mix_rows(p, m->f32, m->st));
    if (m->f32) {
        GemmF32 q = {};
        q.a = (const float*)m->planes; q.lda = m->head.K_pad; q.y = logits; q.ldy = ldl;
        return launch_gemm_bf16w_f32(m->head, 0, m->cfg.vocab, q, n, m->st);
    }
    GemmMaps maps;
    for (int i = 0; i < 3; ++i) { maps.a[i] = m->a_head; maps.b[i] = m->m_head; }
    GemmGroup g = {};
    GemmSeg& q = g.seg[g.n_seg++];
    q.kb = m->head.K_pad / 64; q.n = m->cfg.vocab; q.y = logits; q.ldy = ldl;
    return launch_gemm_bf16_group(maps, g, n, m->status, m->st);
}

// ------------------------------------------------------------------------------ decode step
int launch_step(fc_nurinex_cache* s, int with_head) {
    fc_nurinex* m = s->m;
    const Config& c = m->cfg;
    const int d = c.width, L = (int)c.layers.size();
    cudaStream_t st = m->st;
    GemvGroup base = {};
    base.eps = (float)c.eps; base.d = d; base.state = s->state; base.ctx = m->ctx;
    base.shift_slot = (size_t)L * d;
    SideOutputs prev;
    for (int l = 0; l < L; ++l) {
        const NxWeights& w = *m->run[l];
        const int rd = w.rH * w.rdim;
        GemvGroup g = base;
        g.mode = 1;
        g.prev = prev;
        if (!l) {
            g.embed.table = m->embed.w; g.embed.vocab = c.vocab; g.embed.ld = m->embed.K_pad; g.embed.scale = (float)c.emb_scale;
            g.queue = s->queue;
        }
        g.x_in = s->x[l & 1]; g.x_out = s->x[(l + 1) & 1];
        g.norm_w = w.norm1;
        for (int i = 0; i < kMixes; ++i) g.mu[i] = w.mu[i];
        g.shift = s->shift + (size_t)l * d;
        auto add = [&](int src, int row, int n, float* y) -> GemvSeg& {
            GemvSeg& q = g.seg[g.n_seg++];
            q.w = w.in.w + (size_t)row * w.in.K_pad; q.n = n; q.ldw = q.K_pad = w.in.K_pad; q.K = d; q.src = src; q.y = y;
            return q;
        };
        add(0, 0, w.n_qkv, s->proj);
        if (w.ff) {
            GemvSeg& q = add(0, w.row_up, w.ff, s->hid);
            q.epi = ROW_XIELU; q.c0 = w.c0; q.c1 = w.c1;
        }
        add(1, w.row_r, rd, s->proj + w.off_r);
        add(2, w.row_k, rd, s->proj + w.off_k);
        add(3, w.row_v, rd, s->proj + w.off_v);
        add(4, w.row_g, rd, s->proj + w.off_g);
        add(5, w.row_w1, w.rank, s->proj + w.off_w1);
        FC_TRY(launch_gemv_bf16_group(g, st));

        MixerDecode a = {};
        a.t = w.t;
        a.q = s->proj; a.kc = s->kc[l]; a.vc = s->vc[l]; a.f32_cache = m->f32; a.ctx = m->ctx;
        a.att = s->att; a.part = s->part; a.part_ml = s->part_ml; a.max_splits = s->max_splits; a.counter = s->counter;
        a.rH = w.rH; a.rdim = w.rdim; a.rank = w.rank;
        a.r = s->proj + w.off_r; a.k = s->proj + w.off_k; a.v = s->proj + w.off_v; a.g = s->proj + w.off_g; a.w1 = s->proj + w.off_w1;
        a.w2 = w.w2.w; a.w2_ld = w.w2.K_pad; a.w0 = w.w0; a.u = w.u; a.rnorm = w.rnorm; a.eps = (float)c.eps;
        a.wkv_state = s->wkv[l]; a.ro = s->ro; a.state = s->state;
        FC_TRY(launch_mixer_decode(a, st));

        GemvGroup o = base;
        o.x[0] = s->att; o.x[1] = s->ro;
        auto out = [&](const BMat& mat, int k0, int K, int src, int slot) {
            GemvSeg& q = o.seg[o.n_seg++];
            q.w = mat.w + k0; q.n = d; q.ldw = mat.K_pad; q.K_pad = pad_to(K, 64); q.K = K; q.src = src; q.y = s->outs + (size_t)slot * d;
        };
        out(w.lo, 0, w.lo.K, 0, 0);
        out(w.ro, 0, w.ro.K, 1, 1);
        int n_ff = 0;
        if (w.ff) {                                // K slices of about 2048, each a row list of its own
            const int kb = w.down.K_pad / 64;
            n_ff = std::max(1, std::min(kFfSplits, (kb + 31) / 32));
            for (int f = 0; f < n_ff; ++f) {
                const int k0 = kb * f / n_ff * 64, k1 = std::min(w.down.K, kb * (f + 1) / n_ff * 64);
                o.x[2 + f] = s->hid + k0;
                out(w.down, k0, k1 - k0, 2 + f, 2 + f);
            }
        }
        FC_TRY(launch_gemv_bf16_group(o, st));
        prev = outputs_of(w, s->outs, (size_t)d, n_ff);
    }
    if (with_head) {
        GemvGroup g = base;
        g.mode = 2;
        g.prev = prev;
        g.x_in = s->x[L & 1];
        g.norm_w = m->final_norm;
        GemvSeg& q = g.seg[g.n_seg++];
        q.w = m->head.w; q.n = c.vocab; q.ldw = q.K_pad = m->head.K_pad; q.K = d; q.y = s->logits;
        FC_TRY(launch_gemv_bf16_group(g, st));
    }
    return launch_step_advance_pdl(s->state, st);
}

int run_step(fc_nurinex_cache* s, int with_head) {
    if (!s->graph[with_head]) {
        cudaStream_t st = s->m->st;
        cudaGraph_t g = nullptr;
        const int64_t before = g_launches;
        FC_CUDA(cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal));
        const int rc = launch_step(s, with_head);
        const cudaError_t e = cudaStreamEndCapture(st, &g);
        s->graph_nodes[with_head] = (int)(g_launches - before);
        g_launches = before;
        if (rc != FC_OK) { if (g) cudaGraphDestroy(g); return rc; }
        FC_CUDA(e);
        const cudaError_t ei = cudaGraphInstantiate(&s->graph[with_head], g, 0);
        cudaGraphDestroy(g);
        FC_CUDA(ei);
    }
    FC_CUDA(cudaGraphLaunch(s->graph[with_head], s->m->st));
    g_launches += s->graph_nodes[with_head];
    return FC_OK;
}

int read_state(fc_nurinex_cache* s, StepState* out) {
    FC_CUDA(cudaMemcpyAsync(out, s->state, sizeof(StepState), cudaMemcpyDeviceToHost, s->m->st));
    FC_CUDA(cudaStreamSynchronize(s->m->st));
    return FC_OK;
}

int check_room(const fc_nurinex_cache* s, int n) {
    if (n > s->m->ctx - s->host_pos)
        return fail(FC_E_DIM, "%d more tokens do not fit the %d-token context (position %d)", n, s->m->ctx, s->host_pos);
    return FC_OK;
}

// Puts the next `n` ids on the device for a portion (and into the queue, the ids so far).
int stage_ids(fc_nurinex_cache* s, const int32_t* ids, int n) {
    FC_CUDA(cudaMemcpyAsync(s->m->ids_d, ids, (size_t)n * 4, cudaMemcpyHostToDevice, s->m->st));
    FC_CUDA(cudaMemcpyAsync(s->queue + s->host_pos, ids, (size_t)n * 4, cudaMemcpyHostToDevice, s->m->st));
    return FC_OK;
}

// One token through the decode step; logits stay in s->logits.
int feed_one(fc_nurinex_cache* s, int32_t id, int with_head) {
    FC_CUDA(cudaMemcpyAsync(s->queue + s->host_pos, &id, 4, cudaMemcpyHostToDevice, s->m->st));
    FC_TRY(launch_step_set(s->state, s->host_pos, s->host_pos, s->host_pos + 1, s->m->st));
    FC_TRY(run_step(s, with_head));
    s->host_pos += 1;
    StepState hs;
    FC_TRY(read_state(s, &hs));
    if (hs.error) { s->host_pos -= 1; return fail(hs.error, "the decode step rejected a token or position on the device"); }
    return FC_OK;
}

// A prompt of n ids; the logits of its last token in s->logits.
int feed_prompt(fc_nurinex_cache* s, const int32_t* ids, int n) {
    fc_nurinex* m = s->m;
    for (int at = 0; at < n;) {
        const int M = std::min(kMaxPortion, n - at);
        if (M == 1) {
            FC_TRY(feed_one(s, ids[at], at + 1 == n));
        } else {
            FC_TRY(ensure_workspace(m, M));
            FC_TRY(stage_ids(s, ids + at, M));
            Tail tail;
            FC_TRY(portion_forward(m, s, M, nullptr, &tail));
            if (at + M == n) {
                const int32_t last = M - 1;
                FC_CUDA(cudaMemcpyAsync(m->rows_d, &last, 4, cudaMemcpyHostToDevice, m->st));
                FC_TRY(head_rows(m, tail, 0, 1, s->logits, m->head.N_pad));
            }
            FC_TRY(check_status(m));
        }
        at += M;
    }
    return FC_OK;
}

}  // namespace

extern "C" {

static int probe_dir(const char* dir, ModelDir* md, Config* c) {
    FC_TRY(md->open(dir));
    FC_TRY(parse_config(md->config, c));
    const TensorView* t;
    FC_TRY(find_tensor(*md, "embed", {c->vocab, c->width}, &t));
    FC_TRY(find_tensor(*md, "head", {c->vocab, c->width}, &t));
    FC_TRY(find_tensor(*md, "final.norm", {c->width}, &t));
    for (size_t i = 0; i < c->layers.size(); ++i)
        if (c->layers[i].owner == (int)i) FC_TRY(load_layer(*md, *c, (int)i, nullptr, nullptr));
    return FC_OK;
}
static void fill_info(const Config& c, int ctx, int64_t weight_bytes, fc_nurinex_info* out) {
    out->vocab = c.vocab; out->width = c.width; out->n_layers = (int)c.layers.size(); out->ctx = ctx;
    out->n_own_layers = 0;
    for (size_t i = 0; i < c.layers.size(); ++i) out->n_own_layers += c.layers[i].owner == (int)i;
    out->weight_bytes = weight_bytes;
}

int fc_nurinex_probe(const char* dir, fc_nurinex_info* out) {
    if (!dir || !out) return fail(FC_E_ARG, "fc_nurinex_probe: null argument");
    ModelDir md;
    Config c;
    FC_TRY(probe_dir(dir, &md, &c));
    fill_info(c, 0, 0, out);
    return FC_OK;
}

int fc_nurinex_load(const char* dir, int device, int math_mode, int ctx, fc_nurinex** out) {
    if (!dir || !out) return fail(FC_E_ARG, "fc_nurinex_load: null argument");
    *out = nullptr;
    if (math_mode != FC_MATH_FP32 && math_mode != FC_MATH_BF16) return fail(FC_E_ARG, "math_mode %d: this decoder runs in f32 or bf16", math_mode);
    if (ctx <= 0) return fail(FC_E_SHAPE, "fc_nurinex_load: ctx = %d", ctx);
    ModelDir md;
    auto* m = new fc_nurinex();
    auto build = [&]() -> int {
        FC_TRY(probe_dir(dir, &md, &m->cfg));
        FC_TRY(select_device(device));
        m->device = device; m->mode = math_mode; m->f32 = math_mode == FC_MATH_FP32; m->ctx = ctx;
        FC_CUDA(cudaStreamCreateWithFlags(&m->st, cudaStreamNonBlocking));
        FC_CUDA(cudaStreamCreateWithFlags(&m->side, cudaStreamNonBlocking));
        FC_CUDA(cudaEventCreateWithFlags(&m->fork, cudaEventDisableTiming));
        FC_CUDA(cudaEventCreateWithFlags(&m->join, cudaEventDisableTiming));
        FC_CUDA(cudaEventCreate(&m->ev0));
        FC_CUDA(cudaEventCreate(&m->ev1));
        const Config& c = m->cfg;
        const TensorView* t;
        FC_TRY(find_tensor(md, "embed", {c.vocab, c.width}, &t));
        FC_TRY(upload_rows(m->arena, {{0, {t, c.vocab}}}, c.vocab, c.width, "embed", &m->embed, m->st));
        FC_TRY(find_tensor(md, "head", {c.vocab, c.width}, &t));
        FC_TRY(upload_rows(m->arena, {{0, {t, c.vocab}}}, c.vocab, c.width, "head", &m->head, m->st));
        FC_TRY(map_of(m->head, &m->m_head));
        FC_TRY(find_tensor(md, "final.norm", {c.width}, &t));
        FC_TRY(upload_vec(m->arena, *t, &m->final_norm, m->st));
        m->own.resize(c.layers.size());
        for (size_t i = 0; i < c.layers.size(); ++i) {
            if (c.layers[i].owner != (int)i) continue;
            m->own[i] = std::make_unique<NxWeights>();
            FC_TRY(load_layer(md, c, (int)i, m, m->own[i].get()));
        }
        for (size_t i = 0; i < c.layers.size(); ++i) m->run.push_back(m->own[c.layers[i].owner].get());
        m->weight_bytes = (int64_t)m->head.N * m->head.K * 2;
        for (const NxWeights* w : m->run) {
            const int rd = w->rH * w->rdim;
            m->max_proj = std::max(m->max_proj, w->proj);
            m->max_att = std::max(m->max_att, w->lo.K_pad);
            m->max_ro = std::max(m->max_ro, w->ro.K_pad);
            m->max_hid = std::max(m->max_hid, w->ff ? w->down.K_pad : 64);
            m->max_qm = std::max(m->max_qm, w->t.H * w->t.kd);
            m->max_qo = std::max(m->max_qo, w->t.H * w->t.vdim);
            m->max_rd = std::max(m->max_rd, rd);
            m->weight_bytes += 2LL * c.width * (w->n_qkv + 2 * w->ff + 5 * rd + w->rank + w->t.H * w->t.vdim) + 2LL * rd * w->rank;
        }
        return FC_OK;
    };
    const int rc = build();
    if (rc != FC_OK) { fc_nurinex_free(m); return rc; }
    *out = m;
    return FC_OK;
}

void fc_nurinex_free(fc_nurinex* m) {
    if (!m) return;
    if (m->st) {
        cudaSetDevice(m->device);
        cudaStreamSynchronize(m->st);
    }
    m->ws_arena.release();
    m->arena.release();
    for (cudaEvent_t e : {m->fork, m->join, m->ev0, m->ev1}) if (e) cudaEventDestroy(e);
    if (m->side) cudaStreamDestroy(m->side);
    if (m->st) cudaStreamDestroy(m->st);
    delete m;
}

int fc_nurinex_get_info(const fc_nurinex* m, fc_nurinex_info* out) {
    if (!m || !out) return fail(FC_E_ARG, "fc_nurinex_get_info: null argument");
    fill_info(m->cfg, m->ctx, m->weight_bytes, out);
    return FC_OK;
}
float fc_nurinex_last_forward_ms(const fc_nurinex* m) { return m ? m->last_forward_ms : 0.0f; }

int fc_nurinex_cache_create(fc_nurinex* m, fc_nurinex_cache** out) {
    if (!m || !out) return fail(FC_E_ARG, "fc_nurinex_cache_create: null argument");
    *out = nullptr;
    FC_CUDA(cudaSetDevice(m->device));
    const Config& c = m->cfg;
    const int L = (int)c.layers.size(), d = c.width;
    auto* s = new fc_nurinex_cache();
    s->m = m;
    s->device = m->device;
    auto build = [&]() -> int {
        Arena& a = s->arena;
        // rows a kernel may touch before they are written must hold finite values: the caches start as zero
        auto zero = [&](void** p, size_t bytes) -> int {
            FC_TRY(a.alloc(p, bytes));
            FC_CUDA(cudaMemsetAsync(*p, 0, bytes, m->st));
            return FC_OK;
        };
        s->state_floats = (size_t)2 * L * d;
        for (const NxWeights* w : m->run) {
            void *k = nullptr, *v = nullptr;
            FC_TRY(zero(&k, (size_t)m->ctx * w->t.kd * el(m)));
            s->kc.push_back(k);
            FC_TRY(zero(&v, (size_t)m->ctx * w->t.KV * w->t.vp * el(m)));
            s->vc.push_back(v);
            s->state_floats += (size_t)w->rH * w->rdim * w->rdim;
        }
        FC_TRY(a.alloc_n(&s->state_block, s->state_floats));
        s->shift = s->state_block;
        float* at = s->state_block + (size_t)2 * L * d;
        for (const NxWeights* w : m->run) { s->wkv.push_back(at); at += (size_t)w->rH * w->rdim * w->rdim; }
        s->max_splits = std::max(1, std::min(kMaxSplits, (m->ctx + 63) / 64));
        FC_TRY(a.alloc_n(&s->x[0], (size_t)d));
        FC_TRY(a.alloc_n(&s->x[1], (size_t)d));
        FC_TRY(a.alloc_n(&s->proj, (size_t)m->max_proj));
        FC_TRY(a.alloc_n(&s->outs, (size_t)(2 + kFfSplits) * d));
        FC_TRY(a.alloc_n(&s->hid, (size_t)m->max_hid));
        FC_TRY(a.alloc_n(&s->att, (size_t)m->max_qo));
        FC_TRY(a.alloc_n(&s->ro, (size_t)m->max_rd));
        FC_TRY(a.alloc_n(&s->logits, (size_t)m->head.N_pad));
        FC_TRY(a.alloc_n(&s->part, (size_t)s->max_splits * m->max_qo));
        int heads = 1;
        for (const NxWeights* w : m->run) heads = std::max(heads, w->t.H);
        FC_TRY(a.alloc_n(&s->part_ml, (size_t)s->max_splits * heads * 2));
        FC_TRY(zero((void**)&s->counter, 4));
        s->queue_cap = m->ctx + 1;
        FC_TRY(a.alloc_n(&s->queue, (size_t)s->queue_cap));
        FC_TRY(a.alloc_n(&s->state, 1));
        FC_TRY(a.alloc_n(&s->rng_d, 1));
        FC_CUDA(cudaEventCreate(&s->ev0));
        FC_CUDA(cudaEventCreate(&s->ev1));
        return fc_nurinex_cache_clear(s);
    };
    const int rc = build();
    if (rc != FC_OK) { fc_nurinex_cache_free(s); return rc; }
    *out = s;
    return FC_OK;
}

void fc_nurinex_cache_free(fc_nurinex_cache* s) {
    if (!s) return;
    cudaSetDevice(s->device);
    cudaDeviceSynchronize();              // the model (and its streams) may already be gone
    for (auto& g : s->graph) if (g) cudaGraphExecDestroy(g);
    if (s->ev0) cudaEventDestroy(s->ev0);
    if (s->ev1) cudaEventDestroy(s->ev1);
    s->arena.release();
    delete s;
}

int fc_nurinex_cache_clear(fc_nurinex_cache* s) {
    if (!s) return fail(FC_E_ARG, "fc_nurinex_cache_clear: null cache");
    FC_CUDA(cudaSetDevice(s->device));
    FC_CUDA(cudaMemsetAsync(s->state_block, 0, s->state_floats * 4, s->m->st));
    FC_TRY(launch_step_set(s->state, 0, 0, 0, s->m->st));
    s->host_pos = 0;
    return FC_OK;
}
int fc_nurinex_cache_pos(const fc_nurinex_cache* s) { return s ? s->host_pos : 0; }

int fc_nurinex_feed(fc_nurinex_cache* s, const int32_t* ids, int n, const int32_t* want, int n_want, float* logits) {
    if (!s || !ids || (n_want > 0 && (!want || !logits))) return fail(FC_E_ARG, "fc_nurinex_feed: null argument");
    if (n <= 0 || n_want < 0) return fail(FC_E_SHAPE, "fc_nurinex_feed: n = %d, n_want = %d", n, n_want);
    fc_nurinex* m = s->m;
    FC_CUDA(cudaSetDevice(m->device));
    FC_TRY(check_ids(m, ids, (size_t)n));
    FC_TRY(check_room(s, n));
    for (int k = 0; k < n_want; ++k)
        if (want[k] < 0 || want[k] >= n) return fail(FC_E_DIM, "wanted place %d is not among the %d tokens", want[k], n);
    const int V = m->cfg.vocab, ldl = m->head.N_pad;
    m->last_forward_ms = 0.0f;
    std::vector<int32_t> rows, dst;
    for (int at = 0; at < n;) {
        const int M = std::min(kMaxPortion, n - at);
        rows.clear(); dst.clear();
        for (int k = 0; k < n_want; ++k)
            if (want[k] >= at && want[k] < at + M) { rows.push_back(want[k] - at); dst.push_back(k); }
        if (M == 1) {
            FC_TRY(feed_one(s, ids[at], !rows.empty()));
            for (int32_t k : dst) FC_CUDA(cudaMemcpyAsync(logits + (size_t)k * V, s->logits, (size_t)V * 4, cudaMemcpyDeviceToHost, m->st));
            FC_CUDA(cudaStreamSynchronize(m->st));
        } else {
            FC_TRY(ensure_workspace(m, M));
            FC_TRY(stage_ids(s, ids + at, M));
            FC_CUDA(cudaEventRecord(m->ev0, m->st));
            Tail tail;
            FC_TRY(portion_forward(m, s, M, nullptr, &tail));
            for (size_t k = 0; k < rows.size();) {
                const int c = (int)std::min<size_t>(std::min(m->head_chunk, m->ws_rows), rows.size() - k);
                FC_CUDA(cudaMemcpyAsync(m->rows_d, rows.data() + k, (size_t)c * 4, cudaMemcpyHostToDevice, m->st));
                FC_TRY(head_rows(m, tail, 0, c, m->logits, ldl));
                for (int i = 0; i < c;) {                  // runs of neighbouring places in one copy
                    int e = i + 1;
                    while (e < c && dst[k + e] == dst[k + e - 1] + 1) ++e;
                    FC_CUDA(cudaMemcpy2DAsync(logits + (size_t)dst[k + i] * V, (size_t)V * 4, m->logits + (size_t)i * ldl, (size_t)ldl * 4, (size_t)V * 4,
                                              e - i, cudaMemcpyDeviceToHost, m->st));
                    i = e;
                }
                k += c;
            }
            FC_CUDA(cudaEventRecord(m->ev1, m->st));
            FC_TRY(check_status(m));
            float ms = 0.0f;
            FC_CUDA(cudaEventElapsedTime(&ms, m->ev0, m->ev1));
            m->last_forward_ms += ms;
        }
        at += M;
    }
    return FC_OK;
}

int fc_nurinex_feed_layers(fc_nurinex_cache* s, const int32_t* ids, int n, float* layers) {
    if (!s || !ids || !layers) return fail(FC_E_ARG, "fc_nurinex_feed_layers: null argument");
    if (n <= 0 || n > kMaxPortion) return fail(FC_E_SHAPE, "fc_nurinex_feed_layers: n = %d, at most %d", n, kMaxPortion);
    fc_nurinex* m = s->m;
    FC_CUDA(cudaSetDevice(m->device));
    FC_TRY(check_ids(m, ids, (size_t)n));
    FC_TRY(check_room(s, n));
    FC_TRY(ensure_workspace(m, n));
    FC_TRY(stage_ids(s, ids, n));
    Tail tail;
    FC_TRY(portion_forward(m, s, n, layers, &tail));
    return check_status(m);
}

int fc_nurinex_score(fc_nurinex_cache* s, const int32_t* ids, int n, int from, fc_score* score, float* lp, uint8_t* is_greedy) {
    if (!s || !ids || !score) return fail(FC_E_ARG, "fc_nurinex_score: null argument");
    if (n < 0 || from < 0) return fail(FC_E_SHAPE, "fc_nurinex_score: n = %d, from = %d", n, from);
    fc_nurinex* m = s->m;
    FC_CUDA(cudaSetDevice(m->device));
    FC_TRY(check_ids(m, ids, (size_t)n));
    score->logprob = 0.0; score->n_tokens = 0; score->greedy = 1;
    if (lp) std::fill(lp, lp + std::max(n - 1, 0), 0.0f);
    if (is_greedy) std::fill(is_greedy, is_greedy + std::max(n - 1, 0), (uint8_t)0);
    const int first = std::max(from, 1) - 1, feed = n - 1;       // row t predicts id t + 1
    if (first >= feed) return FC_OK;
    FC_TRY(fc_nurinex_cache_clear(s));
    FC_TRY(check_room(s, feed));
    m->last_forward_ms = 0.0f;
    std::vector<int32_t> rows, targets;
    std::vector<double> lps;
    std::vector<uint8_t> grs;
    for (int at = 0; at < feed;) {
        const int M = std::min(kMaxPortion, feed - at);
        FC_TRY(ensure_workspace(m, M));
        FC_TRY(stage_ids(s, ids + at, M));
        FC_CUDA(cudaEventRecord(m->ev0, m->st));
        Tail tail;
        FC_TRY(portion_forward(m, s, M, nullptr, &tail));
        rows.clear(); targets.clear();
        for (int t = std::max(first, at); t < at + M; ++t) { rows.push_back(t - at); targets.push_back(ids[t + 1]); }
        const int R = (int)rows.size();
        if (R) {
            FC_CUDA(cudaMemcpyAsync(m->rows_d, rows.data(), (size_t)R * 4, cudaMemcpyHostToDevice, m->st));
            FC_CUDA(cudaMemcpyAsync(m->targets_d, targets.data(), (size_t)R * 4, cudaMemcpyHostToDevice, m->st));
            for (int k = 0; k < R; k += m->head_chunk) {
                const int c = std::min(m->head_chunk, R - k);
                FC_TRY(head_rows(m, tail, k, c, m->logits, m->head.N_pad));
                FC_TRY(launch_llama_score_rows(m->logits, m->head.N_pad, m->cfg.vocab, m->targets_d + k, c, m->lp_d + k, m->gr_d + k, m->st));
            }
        }
        FC_CUDA(cudaEventRecord(m->ev1, m->st));
        lps.resize(R); grs.resize(R);
        if (R) {
            FC_CUDA(cudaMemcpyAsync(lps.data(), m->lp_d, (size_t)R * 8, cudaMemcpyDeviceToHost, m->st));
            FC_CUDA(cudaMemcpyAsync(grs.data(), m->gr_d, (size_t)R, cudaMemcpyDeviceToHost, m->st));
        }
        FC_TRY(check_status(m));
        float ms = 0.0f;
        FC_CUDA(cudaEventElapsedTime(&ms, m->ev0, m->ev1));
        m->last_forward_ms += ms;
        for (int i = 0; i < R; ++i) {
            const int t = at + rows[i];
            score->logprob += lps[i];
            score->n_tokens += 1;
            if (!grs[i]) score->greedy = 0;
            if (lp) lp[t] = (float)lps[i];
            if (is_greedy) is_greedy[t] = grs[i];
        }
        at += M;
    }
    return FC_OK;
}

int fc_nurinex_generate(fc_nurinex_cache* s, const int32_t* prompt, int n, int max_new, const fc_sampling* params, const int32_t* stops,
                        int n_stops, uint64_t* rng_state, const volatile int32_t* cancel, int32_t* out, int* n_out) {
    if (!s || !prompt || !params || !rng_state || !n_out || (max_new > 0 && !out) || (n_stops > 0 && !stops))
        return fail(FC_E_ARG, "fc_nurinex_generate: null argument");
    *n_out = 0;
    if (n <= 0) return fail(FC_E_DIM, "prompt must be non-empty");
    if (max_new < 0 || n_stops < 0) return fail(FC_E_SHAPE, "fc_nurinex_generate: max_new = %d, n_stops = %d", max_new, n_stops);
    fc_nurinex* m = s->m;
    FC_CUDA(cudaSetDevice(m->device));
    FC_TRY(check_ids(m, prompt, (size_t)n));
    if (n >= m->ctx) return fail(FC_E_DIM, "prompt of %d tokens does not fit the %d-token context", n, m->ctx);
    max_new = std::min(max_new, m->ctx - n);
    if (cancel && *cancel) return FC_OK;
    FC_TRY(fc_nurinex_cache_clear(s));
    FC_CUDA(cudaMemcpyAsync(s->rng_d, rng_state, 8, cudaMemcpyHostToDevice, m->st));
    FC_TRY(feed_prompt(s, prompt, n));
    const GenCtx g = {m->st, s->logits, m->cfg.vocab, s->queue, s->queue_cap, s->state, s->rng_d, s->ev0, s->ev1, &s->host_pos, &s->last_decode_ms};
    return generate_tokens(g, n, max_new, params, stops, n_stops, rng_state, cancel, out, n_out, [&] { return run_step(s, 1); },
                           [&](StepState* hs) { return read_state(s, hs); });
}
float fc_nurinex_last_decode_ms(const fc_nurinex_cache* s) { return s ? s->last_decode_ms : 0.0f; }

}  // extern "C"
