// Decoders whose model is a folder: loading, portions of a sequence, the captured decode step, scoring, generation, and the
// C ABI (fc_decoder*). What a design computes is behind the virtual calls of decoder.h.
#include "decoder.h"

#include <algorithm>
#include <cmath>
#include <cstring>
#include <memory>

#include "decode_loop.cuh"
#include "llama_ops.cuh"
#include "tc_common.cuh"

using namespace fc;

namespace fc {

namespace {
const DecoderDesign* g_designs = nullptr;
}
DecoderDesign::DecoderDesign(const char* name, fc_decoder* (*mk)()) : architecture(name), make(mk), next(g_designs) { g_designs = this; }

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


int upload_rows(Arena& ar, const std::vector<std::pair<int, Part>>& parts, int rows_total, int K, const char* what, BMat* out, cudaStream_t st) {
    const int K_pad = pad_to(K, 64), N_pad = pad_to(rows_total, 128);
    std::vector<uint16_t> buf((size_t)N_pad * K_pad, 0);
    for (auto& p : parts) {
        if (p.second.t->dtype != "BF16") return fail(FC_E_FORMAT, "%s: matrices must be stored as BF16", what);
        for (int r = 0; r < p.second.rows; ++r)
            std::memcpy(buf.data() + (size_t)(p.first + r) * K_pad, p.second.t->data + (size_t)(p.second.from + r) * K * 2, (size_t)K * 2);
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


}  // namespace fc

int fc_decoder::zeroed(Arena& a, void** p, size_t bytes) {
    FC_TRY(a.alloc(p, bytes));
    FC_CUDA(cudaMemsetAsync(*p, 0, bytes ? bytes : 16, st));
    return FC_OK;
}

namespace {

int ensure_workspace(fc_decoder* m, int rows) {
    if (rows <= m->ws_rows) return FC_OK;
    int R = 128;
    while (R < rows) R *= 2;
    FC_CUDA(cudaStreamSynchronize(m->st));
    m->ws_arena.release();
    m->ws_rows = 0;
    const int dp = m->head.K_pad;
    const size_t RR = R;
    Arena& a = m->ws_arena;
    // padding columns must hold finite values (they meet zero weights): everything starts as zero
    FC_TRY(m->zeroed(a, &m->planes, m->n_planes() * RR * dp * m->el()));
    m->head_chunk = (int)std::max<size_t>(1, std::min<size_t>(RR, ((size_t)1 << 27) / m->head.N_pad));
    FC_TRY(m->zeroed_n(a, &m->logits, (size_t)m->head_chunk * m->head.N_pad));
    FC_TRY(m->zeroed_n(a, &m->ids_d, RR));
    FC_TRY(m->zeroed_n(a, &m->rows_d, RR));
    FC_TRY(m->zeroed_n(a, &m->targets_d, RR));
    FC_TRY(m->zeroed_n(a, &m->lp_d, RR));
    FC_TRY(m->zeroed_n(a, &m->gr_d, RR));
    FC_TRY(m->zeroed_n(a, &m->status, 2));
    if (!m->f32) FC_TRY(tc::encode_bf16(&m->a_head, m->planes, RR, dp, dp, kGemmBoxRows));
    m->ws_rows = R;                     // workspace() reads it
    const int rc = m->workspace(R);
    if (rc != FC_OK) m->ws_rows = 0;
    return rc;
}

int check_ids(const fc_decoder* m, const int32_t* ids, size_t n) {
    for (size_t i = 0; i < n; ++i)
        if (ids[i] < 0 || ids[i] >= m->vocab) return fail(FC_E_DIM, "token %d ≥ vocab_size %d", ids[i], m->vocab);
    return FC_OK;
}
int check_status(fc_decoder* m) {
    int s[2] = {0, 0};
    FC_CUDA(cudaMemcpyAsync(s, m->status, 8, cudaMemcpyDeviceToHost, m->st));
    FC_CUDA(cudaStreamSynchronize(m->st));
    if (s[0] || s[1]) cudaMemsetAsync(m->status, 0, 8, m->st);
    if (s[0]) return fail(FC_E_TIMEOUT, "a bounded wait inside a tensor-core kernel ran out (status %d)", s[0]);
    if (s[1]) return fail(s[1], "a token id was rejected on the device");
    return FC_OK;
}

// Final norm and head for n rows of the portion (their indices on the device in m->rows_d + at); logits [n][ldl].
int head_rows(fc_decoder* m, int at, int n, float* logits, int ldl) {
    FC_TRY(m->final_rows(m->rows_d + at, n));
    if (m->f32) {
        GemmF32 q = {};
        q.a = (const float*)m->planes; q.lda = m->head.K_pad; q.y = logits; q.ldy = ldl;
        return launch_gemm_bf16w_f32(m->head, 0, m->vocab, q, n, m->st);
    }
    GemmMaps maps;
    for (int i = 0; i < 3; ++i) { maps.a[i] = m->a_head; maps.b[i] = m->m_head; }
    GemmGroup g = {};
    GemmSeg& q = g.seg[g.n_seg++];
    q.kb = m->head.K_pad / 64; q.n = m->vocab; q.y = logits; q.ldy = ldl;
    return launch_gemm_bf16_group(maps, g, n, m->status, m->st);
}
// A portion and the position after it.
int run_portion(fc_decoder* m, fc_decoder_cache* s, int M, float* layers_out) {
    FC_TRY(m->portion(s, M, layers_out));
    s->host_pos += M;
    return launch_step_set(s->state, s->host_pos, s->host_pos, s->host_pos, m->st);
}

int run_step(fc_decoder_cache* s, int with_head) {
    if (!s->graph[with_head]) {
        cudaStream_t st = s->m->st;
        cudaGraph_t g = nullptr;
        const int64_t before = g_launches;
        FC_CUDA(cudaStreamBeginCapture(st, cudaStreamCaptureModeThreadLocal));
        int rc = s->m->step(s, with_head != 0);
        if (rc == FC_OK) rc = launch_step_advance_pdl(s->state, st);
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

int read_state(fc_decoder_cache* s, StepState* out) {
    FC_CUDA(cudaMemcpyAsync(out, s->state, sizeof(StepState), cudaMemcpyDeviceToHost, s->m->st));
    FC_CUDA(cudaStreamSynchronize(s->m->st));
    return FC_OK;
}

int check_room(const fc_decoder_cache* s, int n) {
    if (n > s->m->ctx - s->host_pos)
        return fail(FC_E_DIM, "%d more tokens do not fit the %d-token context (position %d)", n, s->m->ctx, s->host_pos);
    return FC_OK;
}

// Puts the next `n` ids on the device for a portion (and into the queue, the ids so far).
int stage_ids(fc_decoder_cache* s, const int32_t* ids, int n) {
    FC_CUDA(cudaMemcpyAsync(s->m->ids_d, ids, (size_t)n * 4, cudaMemcpyHostToDevice, s->m->st));
    FC_CUDA(cudaMemcpyAsync(s->queue + s->host_pos, ids, (size_t)n * 4, cudaMemcpyHostToDevice, s->m->st));
    return FC_OK;
}

// One token through the decode step; logits stay in s->logits.
int feed_one(fc_decoder_cache* s, int32_t id, int with_head) {
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
int feed_prompt(fc_decoder_cache* s, const int32_t* ids, int n) {
    fc_decoder* m = s->m;
    for (int at = 0; at < n;) {
        const int M = std::min(kMaxPortion, n - at);
        if (M == 1) {
            FC_TRY(feed_one(s, ids[at], at + 1 == n));
        } else {
            FC_TRY(ensure_workspace(m, M));
            FC_TRY(stage_ids(s, ids + at, M));
            FC_TRY(run_portion(m, s, M, nullptr));
            if (at + M == n) {
                const int32_t last = M - 1;
                FC_CUDA(cudaMemcpyAsync(m->rows_d, &last, 4, cudaMemcpyHostToDevice, m->st));
                FC_TRY(head_rows(m, 0, 1, s->logits, m->head.N_pad));
            }
            FC_TRY(check_status(m));
        }
        at += M;
    }
    return FC_OK;
}

// Sizes, tensors and constants of a folder, checked without a GPU.
int probe_dir(const char* dir, ModelDir* md, std::unique_ptr<fc_decoder>* out) {
    FC_TRY(md->open(dir));
    const Json* arch = md->config.find("architecture");
    const DecoderDesign* d = g_designs;
    while (d && !(arch && arch->str == d->architecture)) d = d->next;
    if (!d) return fail(FC_E_FORMAT, "config.json: the architecture '%s' is not known here", arch ? arch->str.c_str() : "");
    out->reset(d->make());
    fc_decoder* m = out->get();
    FC_TRY(want_int(&md->config, "vocab", "config", &m->vocab));
    FC_TRY(want_int(&md->config, "width", "config", &m->width));
    FC_TRY(m->parse(md->config));
    const TensorView* t;
    FC_TRY(find_tensor(*md, "embed", {m->vocab, m->width}, &t));
    FC_TRY(find_tensor(*md, "head", {m->vocab, m->width}, &t));
    FC_TRY(find_tensor(*md, "final.norm", {m->width}, &t));
    return m->tensors(*md, false);
}
void fill_info(const fc_decoder* m, fc_decoder_info* out) {
    std::memset(out, 0, sizeof *out);
    out->vocab = m->vocab; out->width = m->width; out->n_layers = m->n_layers; out->n_own_layers = m->n_own_layers;
    out->ctx = m->ctx; out->weight_bytes = m->weight_bytes;
}

}  // namespace

extern "C" {

int fc_decoder_probe(const char* dir, fc_decoder_info* out) {
    if (!dir || !out) return fail(FC_E_ARG, "fc_decoder_probe: null argument");
    ModelDir md;
    std::unique_ptr<fc_decoder> m;
    FC_TRY(probe_dir(dir, &md, &m));
    fill_info(m.get(), out);
    return FC_OK;
}

int fc_decoder_load(const char* dir, int device, int math_mode, int ctx, fc_decoder** out) {
    if (!dir || !out) return fail(FC_E_ARG, "fc_decoder_load: null argument");
    *out = nullptr;
    if (math_mode != FC_MATH_FP32 && math_mode != FC_MATH_BF16) return fail(FC_E_ARG, "math_mode %d: this decoder runs in f32 or bf16", math_mode);
    if (ctx <= 0) return fail(FC_E_SHAPE, "fc_decoder_load: ctx = %d", ctx);
    ModelDir md;
    std::unique_ptr<fc_decoder> made;
    FC_TRY(probe_dir(dir, &md, &made));
    FC_TRY(select_device(device));
    fc_decoder* m = made.release();
    auto build = [&]() -> int {
        m->device = device; m->f32 = math_mode == FC_MATH_FP32; m->ctx = ctx;
        FC_CUDA(cudaStreamCreateWithFlags(&m->st, cudaStreamNonBlocking));
        FC_CUDA(cudaEventCreate(&m->ev0));
        FC_CUDA(cudaEventCreate(&m->ev1));
        const TensorView* t;
        FC_TRY(find_tensor(md, "embed", {m->vocab, m->width}, &t));
        FC_TRY(upload_rows(m->arena, {{0, {t, m->vocab}}}, m->vocab, m->width, "embed", &m->embed, m->st));
        FC_TRY(find_tensor(md, "head", {m->vocab, m->width}, &t));
        FC_TRY(upload_rows(m->arena, {{0, {t, m->vocab}}}, m->vocab, m->width, "head", &m->head, m->st));
        FC_TRY(map_of(m->head, &m->m_head));
        FC_TRY(find_tensor(md, "final.norm", {m->width}, &t));
        FC_TRY(upload_vec(m->arena, *t, &m->final_norm, m->st));
        m->weight_bytes = (int64_t)m->head.N * m->head.K * 2;
        return m->tensors(md, true);
    };
    const int rc = build();
    if (rc != FC_OK) { fc_decoder_free(m); return rc; }
    *out = m;
    return FC_OK;
}

void fc_decoder_free(fc_decoder* m) {
    if (!m) return;
    if (m->st) {
        cudaSetDevice(m->device);
        cudaStreamSynchronize(m->st);
    }
    m->ws_arena.release();
    m->arena.release();
    for (cudaEvent_t e : {m->ev0, m->ev1}) if (e) cudaEventDestroy(e);
    if (m->st) cudaStreamDestroy(m->st);
    delete m;
}

int fc_decoder_get_info(const fc_decoder* m, fc_decoder_info* out) {
    if (!m || !out) return fail(FC_E_ARG, "fc_decoder_get_info: null argument");
    fill_info(m, out);
    return FC_OK;
}
float fc_decoder_last_forward_ms(const fc_decoder* m) { return m ? m->last_forward_ms : 0.0f; }

int fc_decoder_cache_create(fc_decoder* m, fc_decoder_cache** out) {
    if (!m || !out) return fail(FC_E_ARG, "fc_decoder_cache_create: null argument");
    *out = nullptr;
    FC_CUDA(cudaSetDevice(m->device));
    fc_decoder_cache* s = m->make_cache();
    s->m = m;
    s->device = m->device;
    auto build = [&]() -> int {
        Arena& a = s->arena;
        FC_TRY(s->create());
        FC_TRY(a.alloc_n(&s->logits, (size_t)m->head.N_pad));
        s->queue_cap = m->ctx + 1;
        FC_TRY(a.alloc_n(&s->queue, (size_t)s->queue_cap));
        FC_TRY(a.alloc_n(&s->state, 1));
        FC_TRY(a.alloc_n(&s->rng_d, 1));
        FC_CUDA(cudaEventCreate(&s->ev0));
        FC_CUDA(cudaEventCreate(&s->ev1));
        return fc_decoder_cache_clear(s);
    };
    const int rc = build();
    if (rc != FC_OK) { fc_decoder_cache_free(s); return rc; }
    *out = s;
    return FC_OK;
}

void fc_decoder_cache_free(fc_decoder_cache* s) {
    if (!s) return;
    cudaSetDevice(s->device);
    cudaDeviceSynchronize();              // the model (and its streams) may already be gone
    for (auto& g : s->graph) if (g) cudaGraphExecDestroy(g);
    if (s->ev0) cudaEventDestroy(s->ev0);
    if (s->ev1) cudaEventDestroy(s->ev1);
    s->arena.release();
    delete s;
}

int fc_decoder_cache_clear(fc_decoder_cache* s) {
    if (!s) return fail(FC_E_ARG, "fc_decoder_cache_clear: null cache");
    FC_CUDA(cudaSetDevice(s->device));
    FC_TRY(s->clear());
    FC_TRY(launch_step_set(s->state, 0, 0, 0, s->m->st));
    s->host_pos = 0;
    return FC_OK;
}
int fc_decoder_cache_pos(const fc_decoder_cache* s) { return s ? s->host_pos : 0; }

int fc_decoder_feed(fc_decoder_cache* s, const int32_t* ids, int n, const int32_t* want, int n_want, float* logits) {
    if (!s || !ids || (n_want > 0 && (!want || !logits))) return fail(FC_E_ARG, "fc_decoder_feed: null argument");
    if (n <= 0 || n_want < 0) return fail(FC_E_SHAPE, "fc_decoder_feed: n = %d, n_want = %d", n, n_want);
    fc_decoder* m = s->m;
    FC_CUDA(cudaSetDevice(m->device));
    FC_TRY(check_ids(m, ids, (size_t)n));
    FC_TRY(check_room(s, n));
    for (int k = 0; k < n_want; ++k)
        if (want[k] < 0 || want[k] >= n) return fail(FC_E_DIM, "wanted place %d is not among the %d tokens", want[k], n);
    const int V = m->vocab, ldl = m->head.N_pad;
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
            FC_TRY(run_portion(m, s, M, nullptr));
            for (size_t k = 0; k < rows.size();) {
                const int c = (int)std::min<size_t>(std::min(m->head_chunk, m->ws_rows), rows.size() - k);
                FC_CUDA(cudaMemcpyAsync(m->rows_d, rows.data() + k, (size_t)c * 4, cudaMemcpyHostToDevice, m->st));
                FC_TRY(head_rows(m, 0, c, m->logits, ldl));
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

int fc_decoder_feed_layers(fc_decoder_cache* s, const int32_t* ids, int n, float* layers) {
    if (!s || !ids || !layers) return fail(FC_E_ARG, "fc_decoder_feed_layers: null argument");
    if (n <= 0 || n > kMaxPortion) return fail(FC_E_SHAPE, "fc_decoder_feed_layers: n = %d, at most %d", n, kMaxPortion);
    fc_decoder* m = s->m;
    FC_CUDA(cudaSetDevice(m->device));
    FC_TRY(check_ids(m, ids, (size_t)n));
    FC_TRY(check_room(s, n));
    FC_TRY(ensure_workspace(m, n));
    FC_TRY(stage_ids(s, ids, n));
    FC_TRY(run_portion(m, s, n, layers));
    return check_status(m);
}

int fc_decoder_score(fc_decoder_cache* s, const int32_t* ids, int n, int from, fc_score* score, float* lp, uint8_t* is_greedy) {
    if (!s || !ids || !score) return fail(FC_E_ARG, "fc_decoder_score: null argument");
    if (n < 0 || from < 0) return fail(FC_E_SHAPE, "fc_decoder_score: n = %d, from = %d", n, from);
    fc_decoder* m = s->m;
    FC_CUDA(cudaSetDevice(m->device));
    FC_TRY(check_ids(m, ids, (size_t)n));
    score->logprob = 0.0; score->n_tokens = 0; score->greedy = 1;
    if (lp) std::fill(lp, lp + std::max(n - 1, 0), 0.0f);
    if (is_greedy) std::fill(is_greedy, is_greedy + std::max(n - 1, 0), (uint8_t)0);
    const int first = std::max(from, 1) - 1, feed = n - 1;       // row t predicts id t + 1
    if (first >= feed) return FC_OK;
    FC_TRY(fc_decoder_cache_clear(s));
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
        FC_TRY(run_portion(m, s, M, nullptr));
        rows.clear(); targets.clear();
        for (int t = std::max(first, at); t < at + M; ++t) { rows.push_back(t - at); targets.push_back(ids[t + 1]); }
        const int R = (int)rows.size();
        if (R) {
            FC_CUDA(cudaMemcpyAsync(m->rows_d, rows.data(), (size_t)R * 4, cudaMemcpyHostToDevice, m->st));
            FC_CUDA(cudaMemcpyAsync(m->targets_d, targets.data(), (size_t)R * 4, cudaMemcpyHostToDevice, m->st));
            for (int k = 0; k < R; k += m->head_chunk) {
                const int c = std::min(m->head_chunk, R - k);
                FC_TRY(head_rows(m, k, c, m->logits, m->head.N_pad));
                FC_TRY(launch_llama_score_rows(m->logits, m->head.N_pad, m->vocab, m->targets_d + k, c, m->lp_d + k, m->gr_d + k, m->st));
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

int fc_decoder_generate(fc_decoder_cache* s, const int32_t* prompt, int n, int max_new, const fc_sampling* params, const int32_t* stops,
                        int n_stops, uint64_t* rng_state, const volatile int32_t* cancel, int32_t* out, int* n_out) {
    if (!s || !prompt || !params || !rng_state || !n_out || (max_new > 0 && !out) || (n_stops > 0 && !stops))
        return fail(FC_E_ARG, "fc_decoder_generate: null argument");
    *n_out = 0;
    if (n <= 0) return fail(FC_E_DIM, "prompt must be non-empty");
    if (max_new < 0 || n_stops < 0) return fail(FC_E_SHAPE, "fc_decoder_generate: max_new = %d, n_stops = %d", max_new, n_stops);
    fc_decoder* m = s->m;
    FC_CUDA(cudaSetDevice(m->device));
    FC_TRY(check_ids(m, prompt, (size_t)n));
    if (n >= m->ctx) return fail(FC_E_DIM, "prompt of %d tokens does not fit the %d-token context", n, m->ctx);
    max_new = std::min(max_new, m->ctx - n);
    if (cancel && *cancel) return FC_OK;
    FC_TRY(fc_decoder_cache_clear(s));
    FC_CUDA(cudaMemcpyAsync(s->rng_d, rng_state, 8, cudaMemcpyHostToDevice, m->st));
    FC_TRY(feed_prompt(s, prompt, n));
    const GenCtx g = {m->st, s->logits, m->vocab, s->queue, s->queue_cap, s->state, s->rng_d, s->ev0, s->ev1, &s->host_pos, &s->last_decode_ms};
    return generate_tokens(g, n, max_new, params, stops, n_stops, rng_state, cancel, out, n_out, [&] { return run_step(s, 1); },
                           [&](StepState* hs) { return read_state(s, hs); });
}
float fc_decoder_last_decode_ms(const fc_decoder_cache* s) { return s ? s->last_decode_ms : 0.0f; }

}  // extern "C"
