// The Nurinex decoder: a stack of layers in which attention (mixed heads, distance bias, sink) and a
// linear-attention recurrence stand side by side on one norm, next to a feed-forward on the same norm. Everything that
// differs between models of the design is read from the folder's config.json; a layer may use another layer's tensors
// with a cache and state of its own.
//
// Configuration, tensors, cache contents, the forward of a portion of tokens (prefill kernels) and the decode step; the
// rest is decoder.cu's. Kernels: bf16_ops.cuh.
#include <algorithm>
#include <cmath>
#include <memory>

#include "decoder.h"
#include "tc_common.cuh"

using namespace fc;

namespace {

constexpr int kFfSplits = 4;            // most partial sums of the feed-forward's second product

// The entries of config.json for one layer.
struct LayerCfg {
    int owner = 0;                      // layer whose tensors it uses
    int H = 0, KV = 0, dim = 0, vdim = 0;
    double bias_max = 0, scale = 0, temp_coef = 0, temp_every = 1;
    int rH = 0, rdim = 0;
    int ff = 0;                         // 0: no feed-forward
};
struct Config {
    double eps = 0, emb_scale = 1;
    std::vector<LayerCfg> layers;
};

int parse_config(const Json& j, Config* c) {
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

namespace {
struct Nurinex : fc_decoder {
    Config cfg;
    cudaStream_t side = nullptr;
    cudaEvent_t fork = nullptr, join = nullptr;
    std::vector<std::unique_ptr<NxWeights>> own;       // by layer index; null where another layer's are used
    std::vector<const NxWeights*> run;                 // by layer
    int max_proj = 0, max_att = 0, max_ro = 0, max_hid = 0, max_qm = 0, max_rd = 0, max_qo = 0;
    // workspace of a portion of ws_rows tokens
    float *x[2] = {}, *proj = nullptr, *outs = nullptr, *decay = nullptr, *wkv_o = nullptr, *h_last = nullptr, *wkv_scratch = nullptr;
    void *att = nullptr, *ro = nullptr, *hid = nullptr, *qm = nullptr;
    MixRows tail;                                      // final norm of the last portion, but for the rows

    ~Nurinex() override {
        for (cudaEvent_t e : {fork, join}) if (e) cudaEventDestroy(e);
        if (side) cudaStreamDestroy(side);
    }
    int parse(const Json& config) override;
    int tensors(const ModelDir& md, bool upload) override;
    int n_planes() const override { return 1 + kMixes; }
    int workspace(int rows) override;
    fc_decoder_cache* make_cache() override;
    int portion(fc_decoder_cache* s, int M, float* layers_out) override;
    int final_rows(const int* rows, int n) override;
    int step(fc_decoder_cache* s, bool with_head) override;
};
const DecoderDesign design("Nurinex", []() -> fc_decoder* { return new Nurinex(); });

struct NurinexCache : fc_decoder_cache {
    std::vector<void*> kc, vc;                 // per layer: [ctx][kd], [ctx][KV][vp]
    std::vector<float*> wkv;                   // per layer: [rH][rdim][rdim]
    float* shift = nullptr;                    // [2][layers][width]: h of the token before, by the parity of the position
    float* state_block = nullptr;              // recurrence states and `shift`, one block
    size_t state_floats = 0;
    float *x[2] = {}, *proj = nullptr, *outs = nullptr, *hid = nullptr, *att = nullptr, *ro = nullptr;
    float *part = nullptr, *part_ml = nullptr;
    unsigned int* counter = nullptr;
    int max_splits = 1;
    int create() override;
    int clear() override {
        FC_CUDA(cudaMemsetAsync(state_block, 0, state_floats * 4, m->st));
        return FC_OK;
    }
};

// ------------------------------------------------------------------------------------ loading
// Looks up and checks every tensor of a layer; with `w` uploads them.
int load_layer(const ModelDir& md, int i, Nurinex* m, NxWeights* w) {
    const Config& c = m->cfg;
    const LayerCfg& L = c.layers[i];
    const int d = m->width, rd = L.rH * L.rdim;
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
int layer_forward(Nurinex* m, NurinexCache* s, int l, int M, int pos0, int* n_ff) {
    const NxWeights& w = *m->run[l];
    cudaStream_t st = m->st;
    const int R = m->ws_rows, dp = m->head.K_pad, d = m->width, rd = w.rH * w.rdim;
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
    const Flash f = talk_flash(w.t, s->kc[l], s->vc[l], m->ctx);
    if (m->f32) FC_TRY(launch_flash_f32(f, (const float*)m->qm, M, pos0, (float*)m->att, w.lo.K_pad, st));
    else FC_TRY(launch_flash_tc(f, m->qm, M, pos0, m->att, w.lo.K_pad, m->status, st));
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

}  // namespace

int Nurinex::portion(fc_decoder_cache* sc, int M, float* layers_out) {
    Nurinex* m = this;
    auto* s = static_cast<NurinexCache*>(sc);
    const Config& c = m->cfg;
    const int d = width, L = (int)c.layers.size(), R = m->ws_rows, dp = m->head.K_pad, pos0 = s->host_pos;
    MixRows p = {};
    p.embed.table = m->embed.w; p.embed.vocab = vocab; p.embed.ld = m->embed.K_pad; p.embed.scale = (float)c.emb_scale;
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
    tail = p;
    return FC_OK;
}

int Nurinex::final_rows(const int* rows, int n) {
    MixRows p = tail;
    p.row_idx = rows;
    p.M = n;
    return launch_mix_rows(p, f32, st);
}

// ------------------------------------------------------------------------------ decode step
int Nurinex::step(fc_decoder_cache* sc, bool with_head) {
    Nurinex* m = this;
    auto* s = static_cast<NurinexCache*>(sc);
    const Config& c = cfg;
    const int d = width, L = (int)c.layers.size();
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
            g.embed.table = m->embed.w; g.embed.vocab = vocab; g.embed.ld = m->embed.K_pad; g.embed.scale = (float)c.emb_scale;
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
        q.w = m->head.w; q.n = vocab; q.ldw = q.K_pad = m->head.K_pad; q.K = d; q.y = s->logits;
        FC_TRY(launch_gemv_bf16_group(g, st));
    }
    return FC_OK;
}


int Nurinex::parse(const Json& j) {
    FC_TRY(parse_config(j, &cfg));
    n_layers = (int)cfg.layers.size();
    for (int i = 0; i < n_layers; ++i) n_own_layers += cfg.layers[i].owner == i;
    return FC_OK;
}

int Nurinex::tensors(const ModelDir& md, bool upload) {
    if (!upload) {
        for (int i = 0; i < n_layers; ++i)
            if (cfg.layers[i].owner == i) FC_TRY(load_layer(md, i, this, nullptr));
        return FC_OK;
    }
    FC_CUDA(cudaStreamCreateWithFlags(&side, cudaStreamNonBlocking));
    FC_CUDA(cudaEventCreateWithFlags(&fork, cudaEventDisableTiming));
    FC_CUDA(cudaEventCreateWithFlags(&join, cudaEventDisableTiming));
    own.resize(n_layers);
    for (int i = 0; i < n_layers; ++i) {
        if (cfg.layers[i].owner != i) continue;
        own[i] = std::make_unique<NxWeights>();
        FC_TRY(load_layer(md, i, this, own[i].get()));
    }
    for (int i = 0; i < n_layers; ++i) run.push_back(own[cfg.layers[i].owner].get());
    for (const NxWeights* w : run) {
        const int rd = w->rH * w->rdim;
        max_proj = std::max(max_proj, w->proj);
        max_att = std::max(max_att, w->lo.K_pad);
        max_ro = std::max(max_ro, w->ro.K_pad);
        max_hid = std::max(max_hid, w->ff ? w->down.K_pad : 64);
        max_qm = std::max(max_qm, w->t.H * w->t.kd);
        max_qo = std::max(max_qo, w->t.H * w->t.vdim);
        max_rd = std::max(max_rd, rd);
        weight_bytes += 2LL * width * (w->n_qkv + 2 * w->ff + 5 * rd + w->rank + w->t.H * w->t.vdim) + 2LL * rd * w->rank;
    }
    return FC_OK;
}

int Nurinex::workspace(int rows) {
    const int d = width, dp = head.K_pad;
    const size_t RR = rows, e = el();
    Arena& a = ws_arena;
    FC_TRY(zeroed_n(a, &x[0], RR * d));
    FC_TRY(zeroed_n(a, &x[1], RR * d));
    FC_TRY(zeroed_n(a, &proj, RR * max_proj));
    FC_TRY(zeroed_n(a, &outs, (2 + kFfSplits) * RR * d));
    FC_TRY(zeroed_n(a, &decay, RR * max_rd));
    FC_TRY(zeroed_n(a, &wkv_o, RR * max_rd));
    size_t scratch = 0;
    for (const NxWeights* w : run) scratch = std::max(scratch, wkv_scratch_floats(w->rH, w->rdim));
    FC_TRY(zeroed_n(a, &wkv_scratch, scratch));
    FC_TRY(zeroed_n(a, &h_last, (size_t)n_layers * d));
    FC_TRY(zeroed(a, &att, RR * max_att * e));
    FC_TRY(zeroed(a, &ro, RR * max_ro * e));
    FC_TRY(zeroed(a, &hid, RR * max_hid * e));
    FC_TRY(zeroed(a, &qm, RR * max_qm * e));
    if (f32) return FC_OK;
    for (auto& w : own) {
        if (!w) continue;
        FC_TRY(tc::encode_bf16(&w->a_planes, planes, (1 + kMixes) * RR, dp, dp, kGemmBoxRows));
        FC_TRY(tc::encode_bf16(&w->a_att, att, RR, w->lo.K_pad, w->lo.K_pad, kGemmBoxRows));
        FC_TRY(tc::encode_bf16(&w->a_ro, ro, RR, w->ro.K_pad, w->ro.K_pad, kGemmBoxRows));
        w->a_hid = w->a_ro;
        if (w->ff) FC_TRY(tc::encode_bf16(&w->a_hid, hid, RR, w->down.K_pad, w->down.K_pad, kGemmBoxRows));
    }
    return FC_OK;
}

fc_decoder_cache* Nurinex::make_cache() { return new NurinexCache(); }

int NurinexCache::create() {
    auto* n = static_cast<Nurinex*>(m);
    Arena& a = arena;
    const int L = n->n_layers, d = n->width;
    // rows a kernel may touch before they are written must hold finite values: the caches start as zero
    state_floats = (size_t)2 * L * d;
    for (const NxWeights* w : n->run) {
        void *k = nullptr, *v = nullptr;
        FC_TRY(n->zeroed(a, &k, (size_t)n->ctx * w->t.kd * n->el()));
        kc.push_back(k);
        FC_TRY(n->zeroed(a, &v, (size_t)n->ctx * w->t.KV * w->t.vp * n->el()));
        vc.push_back(v);
        state_floats += (size_t)w->rH * w->rdim * w->rdim;
    }
    FC_TRY(a.alloc_n(&state_block, state_floats));
    shift = state_block;
    float* at = state_block + (size_t)2 * L * d;
    for (const NxWeights* w : n->run) { wkv.push_back(at); at += (size_t)w->rH * w->rdim * w->rdim; }
    max_splits = std::max(1, std::min(kMaxSplits, (n->ctx + 63) / 64));
    FC_TRY(a.alloc_n(&x[0], (size_t)d));
    FC_TRY(a.alloc_n(&x[1], (size_t)d));
    FC_TRY(a.alloc_n(&proj, (size_t)n->max_proj));
    FC_TRY(a.alloc_n(&outs, (size_t)(2 + kFfSplits) * d));
    FC_TRY(a.alloc_n(&hid, (size_t)n->max_hid));
    FC_TRY(a.alloc_n(&att, (size_t)n->max_qo));
    FC_TRY(a.alloc_n(&ro, (size_t)n->max_rd));
    FC_TRY(a.alloc_n(&part, (size_t)max_splits * n->max_qo));
    int heads = 1;
    for (const NxWeights* w : n->run) heads = std::max(heads, w->t.H);
    FC_TRY(a.alloc_n(&part_ml, (size_t)max_splits * heads * 2));
    return n->zeroed_n(a, &counter, 1);
}
