// The Zogevik decoder: windowed attention, latent or grouped-query (whose cached keys and values another layer may use), and
// feed-forwards of routed experts; what a sublayer adds is normed on its way into the residual, which the sublayers read as it
// is. Everything that differs between models of the design is read from the folder's config.json.
//
// Configuration, tensors, cache contents, the forward of a portion of tokens and the decode step; the rest is decoder.cu's.
// Kernels: bf16_ops.cuh.
#include <algorithm>
#include <cmath>
#include <memory>

#include "decoder.h"
#include "tc_common.cuh"

using namespace fc;

namespace {

constexpr int kOutSplits = 4;           // most partial sums of the mixer's output product
constexpr int kMaxTop = 64;             // most experts a token uses

// The entries of config.json for one layer.
struct LayerCfg {
    bool latent = false;
    int H = 0, KV = 0, dim = 0, vdim = 0, rank = 0, rot = 0, window = kNoWindow, kv_from = -1;
    double scale = 0, base = 0;
    int ff = 0, experts = 0, top = 0, groups = 1, keep = 1;      // ff 0: no feed-forward
};

// The tensors of one layer on the device.
struct Layer {
    bool latent = false;
    LatentAttn lat;
    RotAttn att;
    int kv_from = -1, proj = 0, n_in = 0, row = 0, vrow = 0, attw = 0;     // row / vrow: elements of a cached (key) row / value row
    BMat in, uk, uv, o, up, down;
    Router router;
    int ff = 0;
    float *norm1 = nullptr, *norm2 = nullptr;
    CUtensorMap m_in, m_uk, m_uv, m_o, m_up, m_down;       // weight maps
    CUtensorMap a_att, a_rows, a_hid;                      // operand maps into the workspace
    int H() const { return latent ? lat.H : att.H; }
    int vdim() const { return latent ? lat.vdim : att.vdim; }
    int window() const { return latent ? lat.window : att.window; }
    int q_row() const { return latent ? lat.H * (lat.dp + lat.rot_p) : att.H * att.kp; }
};

struct Zogevik : fc_decoder {
    double eps = 0;
    std::vector<LayerCfg> cfg;
    std::vector<std::unique_ptr<Layer>> layers;
    float* embed_norm = nullptr;
    int max_proj = 0, max_att = 0, max_q = 0, max_hid = 0, max_ff_top = 0, max_top = 0, max_experts = 0, max_k = 0, max_v = 0, max_span = 0;
    // workspace of a portion of ws_rows tokens
    float *x = nullptr, *proj = nullptr, *outs = nullptr, *y = nullptr, *weight = nullptr;
    void *q = nullptr, *att = nullptr, *rows = nullptr, *hid = nullptr, *kx = nullptr, *vx = nullptr;
    int *expert = nullptr, *index = nullptr, *counts = nullptr, *n_table = nullptr;
    int4* table = nullptr;

    int parse(const Json& config) override;
    int tensors(const ModelDir& md, bool upload) override;
    int workspace(int rows) override;
    fc_decoder_cache* make_cache() override;
    int portion(fc_decoder_cache* s, int M, float* layers_out) override;
    int final_rows(const int* rows, int n) override;
    int step(fc_decoder_cache* s, bool with_head) override;

    int load_layer(const ModelDir& md, int i, Layer* w);
    int mixer(fc_decoder_cache* s, int l, int M, PostNorm* add);
    int experts(int l, int M, PostNorm* add);
};
const DecoderDesign design("Zogevik", []() -> fc_decoder* { return new Zogevik(); });

struct ZogevikCache : fc_decoder_cache {
    std::vector<void*> kc, vc;          // per layer: [ctx][row], [ctx][vrow]; a layer that uses another's has none, a latent one no vc
    float *x[2] = {}, *proj = nullptr, *q = nullptr, *att = nullptr, *outs = nullptr, *hid = nullptr, *y = nullptr, *z = nullptr, *weight = nullptr;
    float *part = nullptr, *part_ml = nullptr;
    int* expert = nullptr;
    unsigned int* counter = nullptr;    // one a block of heads
    int max_splits = 1;
    int create() override;
    Layer& layer(int l) const { return *static_cast<Zogevik*>(m)->layers[l]; }
    AttnDecode attend(int l) const;
};

}  // namespace

// --------------------------------------------------------------------------------------- configuration
int Zogevik::parse(const Json& j) {
    FC_TRY(want_num(j.find("norm"), "eps", "norm", &eps));
    const Json* list = j.find("layers");
    if (!list || list->kind != Json::Array || list->items.empty()) return fail(FC_E_FORMAT, "config.json: layers must be a list");
    n_layers = n_own_layers = (int)list->items.size();
    cfg.resize(n_layers);
    for (int i = 0; i < n_layers; ++i) {
        const Json& e = list->items[i];
        LayerCfg& c = cfg[i];
        const std::string at = "layers[" + std::to_string(i) + "]", mx = at + ".mixer";
        const Json *type = e.find("type"), *mix = e.find("mixer");
        const std::string name = type ? type->str : "";
        if (name != "attention" && name != "latent_attention") return fail(FC_E_FORMAT, "config.json: %s: layer type '%s' is not known", at.c_str(), name.c_str());
        c.latent = name == "latent_attention";
        FC_TRY(want_int(mix, "heads", mx, &c.H));
        FC_TRY(want_int(mix, "dim", mx, &c.dim));
        FC_TRY(want_int(mix, "vdim", mx, &c.vdim));
        FC_TRY(want_num(mix, "scale", mx, &c.scale));
        FC_TRY(want_int(mix->find("rot"), "dims", mx + ".rot", &c.rot));
        FC_TRY(want_num(mix->find("rot"), "base", mx + ".rot", &c.base));
        if (mix->has("mask")) FC_TRY(want_int(mix->find("mask"), "size", mx + ".mask", &c.window));
        c.window = std::min(c.window, kNoWindow);
        if (c.rot % 2 || !(c.base > 0)) return fail(FC_E_DIM, "config.json: %s.rot: an even number of dimensions and a positive base", mx.c_str());
        if (c.vdim > 256) return fail(FC_E_SHAPE, "%s: value heads of at most 256", at.c_str());
        if (c.latent) {
            int rot_dim = 0;
            FC_TRY(want_int(mix, "kv_rank", mx, &c.rank));
            FC_TRY(want_int(mix, "rot_dim", mx, &rot_dim));
            if (rot_dim != c.rot) return fail(FC_E_DIM, "config.json: %s: rot_dim and rot.dims differ", mx.c_str());
            c.KV = c.H;
        } else {
            FC_TRY(want_int(mix, "kv_heads", mx, &c.KV));
            if (c.H % c.KV) return fail(FC_E_DIM, "%s: %d query heads cannot share %d key/value heads", at.c_str(), c.H, c.KV);
            if (c.rot > c.dim) return fail(FC_E_DIM, "config.json: %s: more rotated than query/key dimensions", mx.c_str());
            if (mix->has("kv_from")) {
                const Json* f = mix->find("kv_from");
                const int n = f->kind == Json::Number && f->num == std::floor(f->num) && f->num >= 0 && f->num < i ? (int)f->num : -1;
                if (n < 0 || cfg[n].latent || cfg[n].kv_from >= 0) return fail(FC_E_FORMAT, "config.json: %s.kv_from names no earlier layer with keys of its own", mx.c_str());
                if (cfg[n].KV != c.KV || cfg[n].dim != c.dim || cfg[n].vdim != c.vdim || cfg[n].rot != c.rot || cfg[n].base != c.base)
                    return fail(FC_E_DIM, "config.json: %s does not have the sizes and rotation of the layer whose keys it uses", mx.c_str());
                c.kv_from = n;
                --n_own_layers;
            }
        }
        if (!e.has("mlp")) continue;
        const Json *mlp = e.find("mlp"), *kind = mlp->find("kind"), *router = mlp->find("router");
        if (!kind || kind->str != "moe") return fail(FC_E_FORMAT, "config.json: %s: feed-forward kind '%s' is not known", at.c_str(), kind ? kind->str.c_str() : "");
        FC_TRY(want_int(mlp->find("expert"), "ff", at + ".mlp.expert", &c.ff));
        FC_TRY(want_int(router, "experts", at + ".mlp.router", &c.experts));
        FC_TRY(want_int(router, "top", at + ".mlp.router", &c.top));
        if (router->has("groups")) {
            FC_TRY(want_int(router->find("groups"), "count", at + ".mlp.router.groups", &c.groups));
            FC_TRY(want_int(router->find("groups"), "keep", at + ".mlp.router.groups", &c.keep));
        }
        if (c.experts % c.groups || c.keep > c.groups || c.top > c.experts / c.groups * c.keep)
            return fail(FC_E_DIM, "config.json: %s: %d of %d experts cannot be chosen from %d of %d equal groups", at.c_str(), c.top, c.experts, c.keep, c.groups);
        if ((int64_t)c.experts * width * pad_to(c.ff, 64) >= (int64_t)1 << 35) return fail(FC_E_SHAPE, "%s: experts of more than 2^35 weights", at.c_str());
        if (c.top > kMaxTop) return fail(FC_E_SHAPE, "%s: a token uses at most %d experts", at.c_str(), kMaxTop);
    }
    return FC_OK;
}

// --------------------------------------------------------------------------------------------- loading
// Looks up and checks every tensor of a layer; with `w` uploads them.
int Zogevik::load_layer(const ModelDir& md, int i, Layer* w) {
    const LayerCfg& c = cfg[i];
    const int d = width;
    const int64_t qn = (int64_t)c.H * (c.dim + (c.latent ? c.rot : 0)), kn = (int64_t)c.KV * c.dim, vn = (int64_t)c.KV * c.vdim, on = (int64_t)c.H * c.vdim;
    const std::string p = "l" + std::to_string(i) + ".";
    const TensorView *n1, *n2 = nullptr, *q, *o, *dkv = nullptr, *cn = nullptr, *uk = nullptr, *uv = nullptr, *qnorm = nullptr, *k = nullptr, *v = nullptr, *knorm = nullptr, *router = nullptr;
    std::vector<const TensorView*> up(c.ff ? c.experts : 0), down(up.size());
    auto get = [&](const std::string& name, std::initializer_list<int64_t> shape, const TensorView** out) { return find_tensor(md, p + name, shape, out); };
    FC_TRY(get("norm1", {d}, &n1));
    FC_TRY(get("mix.q", {qn, d}, &q));
    FC_TRY(get("mix.o", {d, on}, &o));
    if (c.latent) {
        FC_TRY(get("mix.dkv", {c.rank + c.rot, d}, &dkv));
        FC_TRY(get("mix.dkv.norm", {c.rank}, &cn));
        FC_TRY(get("mix.uk", {(int64_t)c.H * c.dim, c.rank}, &uk));
        FC_TRY(get("mix.uv", {on, c.rank}, &uv));
    } else {
        FC_TRY(get("mix.q.norm", {qn}, &qnorm));
        if (c.kv_from < 0) {
            FC_TRY(get("mix.k", {kn, d}, &k));
            FC_TRY(get("mix.v", {vn, d}, &v));
            FC_TRY(get("mix.k.norm", {kn}, &knorm));
        }
    }
    if (c.ff) {
        FC_TRY(get("norm2", {d}, &n2));
        FC_TRY(get("mlp.router", {c.experts, d}, &router));
        for (int e = 0; e < c.experts; ++e) {
            FC_TRY(get("mlp.e" + std::to_string(e) + ".up", {c.ff, d}, &up[e]));
            FC_TRY(get("mlp.e" + std::to_string(e) + ".down", {d, c.ff}, &down[e]));
        }
    }
    if (!w) return FC_OK;

    w->latent = c.latent; w->kv_from = c.kv_from; w->ff = c.ff;
    std::vector<double> f(c.rot / 2);
    for (int r = 0; r < c.rot / 2; ++r) f[r] = std::pow(c.base, -2.0 * r / c.rot);
    double* freq = nullptr;
    FC_TRY(arena.alloc_n(&freq, f.size()));
    FC_CUDA(cudaMemcpy(freq, f.data(), f.size() * sizeof(double), cudaMemcpyHostToDevice));
    Rot rot;
    rot.dims = c.rot; rot.neighbours = c.latent; rot.freq = freq;
    std::vector<std::pair<int, Part>> in = {{0, {q, (int)qn}}};
    w->n_in = (int)qn;
    if (c.latent) {
        LatentAttn& t = w->lat;
        t.H = c.H; t.dim = c.dim; t.vdim = c.vdim; t.rank = c.rank;
        t.dp = pad_to(c.dim, 16); t.vp = pad_to(c.vdim, 16); t.lat = pad_to(c.rank, 64); t.rot_p = pad_to(c.rot, 16);
        t.scale = (float)c.scale; t.eps = (float)eps; t.window = c.window; t.rot = rot;
        float* dev = nullptr;
        FC_TRY(upload_vec(arena, *cn, &dev, st)); t.c_norm = dev;
        // a head's rows begin at a multiple of 16, so that its columns in the expanded rows do
        std::vector<std::pair<int, Part>> pk, pv;
        for (int h = 0; h < c.H; ++h) { pk.push_back({h * t.dp, {uk, c.dim, h * c.dim}}); pv.push_back({h * t.vp, {uv, c.vdim, h * c.vdim}}); }
        FC_TRY(upload_rows(arena, pk, c.H * t.dp, c.rank, "mix.uk", &w->uk, st));
        FC_TRY(upload_rows(arena, pv, c.H * t.vp, c.rank, "mix.uv", &w->uv, st));
        FC_TRY(map_of(w->uk, &w->m_uk));
        FC_TRY(map_of(w->uv, &w->m_uv));
        t.uk = w->uk.w; t.uv = w->uv.w;
        w->row = t.row();
        in.push_back({w->n_in, {dkv, c.rank + c.rot}});
        w->n_in += c.rank + c.rot;
    } else {
        RotAttn& t = w->att;
        t.H = c.H; t.KV = c.KV; t.dim = c.dim; t.vdim = c.vdim; t.kp = pad_to(c.dim, 16); t.vp = pad_to(c.vdim, 16);
        t.scale = (float)c.scale; t.eps = (float)eps; t.window = c.window; t.rot = rot; t.has_sink = true; t.own_kv = c.kv_from < 0;
        float* dev = nullptr;
        FC_TRY(upload_vec(arena, *qnorm, &dev, st)); t.q_norm = dev;
        w->row = c.KV * t.kp; w->vrow = c.KV * t.vp;
        if (t.own_kv) {
            FC_TRY(upload_vec(arena, *knorm, &dev, st)); t.k_norm = dev;
            in.push_back({w->n_in, {k, (int)kn}}); w->n_in += (int)kn;
            in.push_back({w->n_in, {v, (int)vn}}); w->n_in += (int)vn;
        }
    }
    w->proj = pad_to(w->n_in, 8);
    FC_TRY(upload_rows(arena, in, w->n_in, d, "mixer projections", &w->in, st));
    FC_TRY(upload_rows(arena, {{0, {o, d}}}, d, (int)on, "mix.o", &w->o, st));
    FC_TRY(map_of(w->in, &w->m_in));
    FC_TRY(map_of(w->o, &w->m_o));
    FC_TRY(upload_vec(arena, *n1, &w->norm1, st));
    if (!c.ff) return FC_OK;
    FC_TRY(upload_vec(arena, *n2, &w->norm2, st));
    BMat r;
    FC_TRY(upload_rows(arena, {{0, {router, c.experts}}}, c.experts, d, "mlp.router", &r, st));
    w->router.experts = c.experts; w->router.top = c.top; w->router.groups = c.groups; w->router.keep = c.keep;
    w->router.w = r.w; w->router.ld = r.K_pad;
    std::vector<std::pair<int, Part>> pu, pd;
    for (int e = 0; e < c.experts; ++e) { pu.push_back({e * c.ff, {up[e], c.ff}}); pd.push_back({e * d, {down[e], d}}); }
    FC_TRY(upload_rows(arena, pu, c.experts * c.ff, d, "experts' first matrices", &w->up, st));
    FC_TRY(upload_rows(arena, pd, c.experts * d, c.ff, "experts' second matrices", &w->down, st));
    FC_TRY(map_of(w->up, &w->m_up));
    return map_of(w->down, &w->m_down);
}

int Zogevik::tensors(const ModelDir& md, bool upload) {
    const TensorView* t;
    FC_TRY(find_tensor(md, "embed.norm", {width}, &t));
    for (int i = 0; i < n_layers && !upload; ++i) FC_TRY(load_layer(md, i, nullptr));
    if (!upload) return FC_OK;
    FC_TRY(upload_vec(arena, *t, &embed_norm, st));
    for (int i = 0; i < n_layers; ++i) {
        layers.push_back(std::make_unique<Layer>());
        Layer& w = *layers.back();
        FC_TRY(load_layer(md, i, &w));
        const LayerCfg& c = cfg[i];
        max_proj = std::max(max_proj, w.proj);
        max_att = std::max(max_att, w.o.K_pad);
        max_q = std::max(max_q, w.q_row());
        weight_bytes += 2LL * width * (w.n_in + c.H * c.vdim);
        if (c.latent) {
            max_k = std::max(max_k, c.H * w.lat.dp);
            max_v = std::max(max_v, c.H * w.lat.vp);
            max_span = std::max(max_span, std::min(c.window, ctx));
            weight_bytes += 2LL * c.H * (c.dim + c.vdim) * c.rank;
        }
        if (c.ff) {
            max_top = std::max(max_top, c.top);
            max_experts = std::max(max_experts, c.experts);
            max_hid = std::max(max_hid, w.down.K_pad);
            max_ff_top = std::max(max_ff_top, w.down.K_pad * c.top);
            weight_bytes += 2LL * width * (c.experts + 2 * c.top * c.ff);
        }
    }
    return FC_OK;
}

int Zogevik::workspace(int R) {
    const size_t RR = R, e = el(), d = width, dp = head.K_pad, slots = RR * std::max(max_top, 1);
    Arena& a = ws_arena;
    FC_TRY(zeroed_n(a, &x, RR * d));
    FC_TRY(zeroed_n(a, &proj, RR * max_proj));
    FC_TRY(zeroed_n(a, &outs, kOutSplits * RR * d));
    FC_TRY(zeroed(a, &q, RR * max_q * e));
    FC_TRY(zeroed(a, &att, RR * max_att * e));
    const size_t span = std::min<size_t>(ctx, RR + max_span) + 128;
    if (max_k) {
        FC_TRY(zeroed(a, &kx, span * max_k * e));
        FC_TRY(zeroed(a, &vx, span * max_v * e));
    }
    if (max_top) {
        FC_TRY(zeroed_n(a, &y, slots * d));
        FC_TRY(zeroed_n(a, &weight, slots));
        FC_TRY(zeroed_n(a, &expert, slots));
        FC_TRY(zeroed_n(a, &index, slots));
        FC_TRY(zeroed_n(a, &counts, (size_t)n_layers * max_experts));
        FC_TRY(zeroed_n(a, &n_table, 1));
        FC_TRY(zeroed_n(a, &table, slots / kRaggedRowsF32 + max_experts + 1));
        FC_TRY(zeroed(a, &rows, slots * dp * e));
        FC_TRY(zeroed(a, &hid, slots * max_hid * e));
    }
    if (f32) return FC_OK;
    for (auto& w : layers) {
        FC_TRY(tc::encode_bf16(&w->a_att, att, RR, w->o.K_pad, w->o.K_pad, kGemmBoxRows));
        if (!w->ff) continue;
        FC_TRY(tc::encode_bf16(&w->a_rows, rows, slots, dp, dp, kGemmBoxRows));
        FC_TRY(tc::encode_bf16(&w->a_hid, hid, slots, w->down.K_pad, w->down.K_pad, kGemmBoxRows));
    }
    return FC_OK;
}

// ---------------------------------------------------------------------- a portion of tokens
// K slices of the output product: enough that its tiles (round robin over the SMs) come out even.
static int out_splits(const BMat& o, int M) {
    const int tiles = ((o.N + 127) / 128) * ((M + 255) / 256), kb = o.K_pad / 64;
    int best = 1;
    double least = 1e30;
    for (int s = 1; s <= std::min(kOutSplits, kb); ++s) {
        const double cost = ((tiles * s + 147) / 148) * ((kb + s - 1) / s + 4.0) * (1.0 + 0.05 * (s - 1));
        if (cost < least) { least = cost; best = s; }
    }
    return best;
}
// One operand and one weight map in every slot.
static GemmMaps maps_of(const CUtensorMap& a, const CUtensorMap& b, const CUtensorMap& b2) {
    GemmMaps m;
    for (int i = 0; i < 3; ++i) { m.a[i] = a; m.b[i] = i == 1 ? b2 : b; }
    return m;
}

// Layer l's mixer for M rows whose operand is in the planes; what it adds to the residual is described by `add`.
int Zogevik::mixer(fc_decoder_cache* sc, int l, int M, PostNorm* add) {
    auto* s = static_cast<ZogevikCache*>(sc);
    const Layer& w = *layers[l];
    const int R = ws_rows, dp = head.K_pad, d = width, pos0 = s->host_pos, len = pos0 + M;
    const float factor = f32 ? 1.0f : kLog2e;
    if (f32) {
        GemmF32 p = {};
        p.a = (const float*)planes; p.lda = dp; p.y = proj; p.ldy = w.proj;
        FC_TRY(launch_gemm_bf16w_f32(w.in, 0, w.n_in, p, M, st));
    } else {
        GemmGroup g = {};
        GemmSeg& q1 = g.seg[g.n_seg++];
        q1.kb = dp / 64; q1.n = w.n_in; q1.y = proj; q1.ldy = w.proj;
        FC_TRY(launch_gemm_bf16_group(maps_of(a_head, w.m_in, w.m_in), g, M, status, st));
    }
    Flash f;
    if (w.latent) {
        const LatentAttn& t = w.lat;
        void* cache = s->kc[l];
        FC_TRY(launch_latent_prep(t, proj, w.proj, M, pos0, factor, q, cache, f32, st));
        // keys and values of every position the portion sees, from the cached latents
        const int base = std::max(0, pos0 - t.window + 1), n = len - base;
        if (f32) {
            GemmF32 p = {};
            p.a = (const float*)cache + (size_t)base * w.row; p.lda = w.row;
            p.y = (float*)kx; p.ldy = t.H * t.dp;
            FC_TRY(launch_gemm_bf16w_f32(w.uk, 0, t.H * t.dp, p, n, st));
            p.y = (float*)vx; p.ldy = t.H * t.vp;
            FC_TRY(launch_gemm_bf16w_f32(w.uv, 0, t.H * t.vp, p, n, st));
        } else {
            CUtensorMap a_lat;
            FC_TRY(tc::encode_bf16(&a_lat, cache, ctx, t.lat, w.row, kGemmBoxRows));
            GemmGroup g = {};
            for (int i = 0; i < 2; ++i) {
                GemmSeg& e = g.seg[g.n_seg++];
                e.b_map = i; e.a_row0 = base; e.kb = t.lat / 64;
                e.n = t.H * (i ? t.vp : t.dp); e.ldy = e.n; e.yb = (uint16_t*)(i ? vx : kx);
            }
            FC_TRY(launch_gemm_bf16_group(maps_of(a_lat, w.m_uk, w.m_uv), g, n, status, st));
        }
        f = latent_flash(t, kx, vx, n, base, cache, ctx);
    } else {
        const int from = w.kv_from < 0 ? l : w.kv_from;
        FC_TRY(launch_rot_prep(w.att, proj, w.proj, M, pos0, factor, q, s->kc[from], s->vc[from], f32, st));
        f = rot_flash(w.att, s->kc[from], s->vc[from], ctx);
    }
    if (f32) FC_TRY(launch_flash_f32(f, (const float*)q, M, pos0, (float*)att, w.o.K_pad, st));
    else FC_TRY(launch_flash_tc(f, q, M, pos0, att, w.o.K_pad, status, st));
    add->y = outs; add->part_rows = R; add->norm_w = w.norm1; add->n_parts = f32 ? 1 : out_splits(w.o, M);
    if (f32) {
        GemmF32 p = {};
        p.a = (const float*)att; p.lda = w.o.K_pad; p.y = outs; p.ldy = d;
        return launch_gemm_bf16w_f32(w.o, 0, d, p, M, st);
    }
    GemmGroup g = {};
    const int kb = w.o.K_pad / 64, n = add->n_parts;
    for (int i = 0; i < n; ++i) {
        GemmSeg& e = g.seg[g.n_seg++];
        e.kb0 = kb * i / n; e.kb = kb * (i + 1) / n - e.kb0; e.n = d; e.y = outs + (size_t)i * R * d; e.ldy = d;
    }
    return launch_gemm_bf16_group(maps_of(w.a_att, w.m_o, w.m_o), g, M, status, st);
}

// Layer l's feed-forward for M rows of the residual (and their operand).
int Zogevik::experts(int l, int M, PostNorm* add) {
    const Layer& w = *layers[l];
    const int dp = head.K_pad, d = width, tile = f32 ? kRaggedRowsF32 : kRaggedRows, entries = max_row_tiles(w.router, M, tile);
    RouteRows p = {};
    p.r = w.router; p.x = x; p.M = M; p.d = d; p.expert = expert; p.index = index; p.counts = counts + (size_t)l * max_experts; p.weight = weight;
    p.rows = rows; p.ld = dp; p.table = table; p.n_table = n_table; p.tile_rows = tile;
    FC_TRY(launch_route_rows(p, planes, f32, st));
    Ragged up = {table, n_table, w.ff}, down = {table, n_table, d};
    add->y = y; add->n_parts = w.router.top; add->index = index; add->weight = weight; add->norm_w = w.norm2;
    if (f32) {
        GemmF32 q1 = {};
        q1.a = (const float*)rows; q1.lda = dp; q1.y = (float*)hid; q1.ldy = w.down.K_pad; q1.epi = ROW_GELU;
        FC_TRY(launch_gemm_bf16w_f32_ragged(w.up, w.ff, q1, up, entries, st));
        GemmF32 q2 = {};
        q2.a = (const float*)hid; q2.lda = w.down.K_pad; q2.y = y; q2.ldy = d;
        return launch_gemm_bf16w_f32_ragged(w.down, d, q2, down, entries, st);
    }
    GemmSeg a = {}, b = {};
    a.kb = dp / 64; a.n = w.ff; a.yb = (uint16_t*)hid; a.ldy = w.down.K_pad; a.epi = ROW_GELU;
    FC_TRY(launch_gemm_bf16_ragged(maps_of(w.a_rows, w.m_up, w.m_up), a, up, entries, status, st));
    b.kb = w.down.K_pad / 64; b.n = d; b.y = y; b.ldy = d;
    return launch_gemm_bf16_ragged(maps_of(w.a_hid, w.m_down, w.m_down), b, down, entries, status, st);
}

int Zogevik::portion(fc_decoder_cache* s, int M, float* layers_out) {
    const int d = width;
    PostNormRows p = {};
    p.embed.table = embed.w; p.embed.vocab = vocab; p.embed.ld = embed.K_pad;
    p.ids = ids_d; p.x = x; p.eps = (float)eps; p.M = M; p.d = d; p.ld = head.K_pad; p.plane = planes; p.error_flag = status + 1;
    p.add.norm_w = embed_norm;
    FC_TRY(launch_post_norm_rows(p, f32, st));
    if (max_top) FC_CUDA(cudaMemsetAsync(counts, 0, (size_t)n_layers * max_experts * sizeof(int), st));
    for (int l = 0; l < n_layers; ++l) {
        p.add = PostNorm();
        FC_TRY(mixer(s, l, M, &p.add));
        FC_TRY(launch_post_norm_rows(p, f32, st));
        if (layers[l]->ff) {
            p.add = PostNorm();
            FC_TRY(experts(l, M, &p.add));
            FC_TRY(launch_post_norm_rows(p, f32, st));
        }
        if (layers_out) FC_CUDA(cudaMemcpyAsync(layers_out + (size_t)l * M * d, x, (size_t)M * d * 4, cudaMemcpyDeviceToHost, st));
    }
    return FC_OK;
}

int Zogevik::final_rows(const int* idx, int n) {
    PostNormRows p = {};
    p.x = x; p.row_idx = idx; p.out_norm_w = final_norm; p.eps = (float)eps; p.M = n; p.d = width; p.ld = head.K_pad; p.plane = planes;
    return launch_post_norm_rows(p, f32, st);
}

// ------------------------------------------------------------------------------ decode step
fc_decoder_cache* Zogevik::make_cache() { return new ZogevikCache(); }

AttnDecode ZogevikCache::attend(int l) const {
    const Layer& w = layer(l);
    AttnDecode a;
    a.H = w.H(); a.f32 = m->f32; a.window = w.window(); a.max_splits = max_splits; a.reach = std::min(w.window(), m->ctx);
    a.part = part; a.part_ml = part_ml; a.state = state;
    a.k_ld = w.row;
    if (w.latent) {
        a.KV = 1; a.kw = w.row; a.vw = w.lat.rank;
        a.kc = kc[l]; a.q = q;
    } else {
        const RotAttn& t = w.att;
        const int from = w.kv_from < 0 ? l : w.kv_from;
        a.KV = t.KV; a.kw = t.kp; a.vw = t.vdim; a.k_head = t.kp; a.v_ld = w.vrow; a.v_head = t.vp;
        a.kc = kc[from]; a.vc = vc[from]; a.prep = t; a.q = proj; a.has_sink = t.has_sink; a.out = att; a.counter = counter;
    }
    // splits of a tile each, but no more CTAs than two per SM
    a.max_splits = std::max(1, std::min(max_splits, 296 / attn_decode_blocks(a)));
    return a;
}

int ZogevikCache::create() {
    auto* n = static_cast<Zogevik*>(m);
    Arena& a = arena;
    const int d = n->width;
    int blocks = 1, q_max = 1, part_max = 1, heads = 1, att_max = 1;
    for (int l = 0; l < n->n_layers; ++l) {
        const Layer& w = *n->layers[l];
        void *k = nullptr, *v = nullptr;
        // rows a kernel may touch before they are written must hold finite values: the caches start as zero
        if (w.kv_from < 0) FC_TRY(n->zeroed(a, &k, (size_t)n->ctx * w.row * n->el()));
        if (w.kv_from < 0 && !w.latent) FC_TRY(n->zeroed(a, &v, (size_t)n->ctx * w.vrow * n->el()));
        kc.push_back(k);
        vc.push_back(v);
        blocks = std::max(blocks, attn_decode_blocks(attend(l)));
        heads = std::max(heads, w.H());
        att_max = std::max(att_max, w.H() * w.vdim());
        part_max = std::max(part_max, w.H() * pad_to(w.latent ? w.lat.rank : w.att.vdim, 4));
        if (w.latent) q_max = std::max(q_max, w.H() * w.row);
    }
    max_splits = kMaxSplitsRow;
    FC_TRY(a.alloc_n(&x[0], (size_t)d));
    FC_TRY(a.alloc_n(&x[1], (size_t)d));
    FC_TRY(a.alloc_n(&proj, (size_t)n->max_proj));
    FC_TRY(a.alloc_n(&q, (size_t)q_max));
    FC_TRY(a.alloc_n(&att, (size_t)att_max));
    FC_TRY(a.alloc_n(&outs, (size_t)kOutSplits * d));
    FC_TRY(a.alloc_n(&hid, (size_t)std::max(n->max_ff_top, 1)));
    FC_TRY(a.alloc_n(&y, (size_t)d));
    FC_TRY(a.alloc_n(&z, (size_t)std::max(n->max_experts, 1)));
    FC_TRY(a.alloc_n(&weight, (size_t)std::max(n->max_top, 1)));
    FC_TRY(n->zeroed_n(a, &expert, (size_t)std::max(n->max_top, 1)));
    FC_TRY(a.alloc_n(&part, (size_t)max_splits * part_max));
    FC_TRY(a.alloc_n(&part_ml, (size_t)max_splits * heads * 2));
    return n->zeroed_n(a, &counter, (size_t)blocks);
}

int Zogevik::step(fc_decoder_cache* sc, bool with_head) {
    auto* s = static_cast<ZogevikCache*>(sc);
    const int d = width;
    int cur = 0;                                            // which of the two residual buffers holds it
    GemvGroup base = {};
    base.eps = (float)eps; base.d = d; base.state = s->state; base.ctx = ctx;
    auto add = [](GemvGroup& g, const uint16_t* w, int ldw, int n, int K, int src, float* y) -> GemvSeg& {
        GemvSeg& q1 = g.seg[g.n_seg++];
        q1.w = w; q1.n = n; q1.ldw = ldw; q1.K_pad = pad_to(K, 64); q1.K = K; q1.src = src; q1.y = y;
        return q1;
    };
    PostNorm prev;
    prev.norm_w = embed_norm;
    for (int l = 0; l < n_layers; ++l) {
        const Layer& w = *layers[l];
        GemvGroup g = base;
        g.mode = 3;
        g.post = prev;
        if (!l) {
            g.embed.table = embed.w; g.embed.vocab = vocab; g.embed.ld = embed.K_pad;
            g.queue = s->queue;
        }
        g.x_in = s->x[cur]; g.x_out = s->x[cur ^ 1];
        cur ^= 1;
        add(g, w.in.w, w.in.K_pad, w.n_in, d, 0, s->proj);
        FC_TRY(launch_gemv_bf16_group(g, st));
        const AttnDecode a = s->attend(l);
        if (w.latent) FC_TRY(launch_latent_absorb(w.lat, s->proj, s->q, s->kc[l], f32, s->state, st));
        FC_TRY(launch_attn_decode_rows(a, st));
        if (w.latent) FC_TRY(launch_latent_expand(w.lat, a, s->att, st));
        GemvGroup o = base;
        const int kb = w.o.K_pad / 64, n = std::max(1, std::min(kOutSplits, (kb + 31) / 32));      // K slices of about 2048
        for (int i = 0; i < n; ++i) {
            const int k0 = kb * i / n * 64, k1 = std::min(w.o.K, kb * (i + 1) / n * 64);
            o.x[i] = s->att + k0;
            add(o, w.o.w + k0, w.o.K_pad, d, k1 - k0, i, s->outs + (size_t)i * d);
        }
        FC_TRY(launch_gemv_bf16_group(o, st));
        prev = PostNorm();
        prev.y = s->outs; prev.n_parts = n; prev.part_rows = 1; prev.norm_w = w.norm1;
        if (!w.ff) continue;
        // logits on the residual; the first product chooses from them; rows of the second run through the chosen experts
        GemvGroup r = base, up = base, down = base;
        r.mode = 3; r.post = prev; r.x_in = s->x[cur]; r.x_out = s->x[cur ^ 1];
        cur ^= 1;
        add(r, w.router.w, w.router.ld, w.router.experts, d, 0, s->z);
        FC_TRY(launch_gemv_bf16_group(r, st));
        up.x[0] = s->x[cur];
        up.router = w.router; up.z = s->z;
        up.expert = down.expert = s->expert; up.weight = down.weight = s->weight;
        GemvSeg& u = add(up, w.up.w, w.up.K_pad, w.ff, d, 0, s->hid);
        u.epi = ROW_GELU; u.reps = w.router.top; u.w_step = (size_t)w.ff * w.up.K_pad; u.y_step = w.down.K_pad;
        FC_TRY(launch_gemv_bf16_group(up, st));
        down.x[0] = s->hid;
        GemvSeg& v = add(down, w.down.w, w.down.K_pad, d, w.ff, 0, s->y);
        v.reps = w.router.top; v.sum = 1; v.w_step = (size_t)d * w.down.K_pad; v.x_step = w.down.K_pad;
        FC_TRY(launch_gemv_bf16_group(down, st));
        prev = PostNorm();
        prev.y = s->y; prev.n_parts = 1; prev.part_rows = 1; prev.norm_w = w.norm2;
    }
    if (!with_head) return FC_OK;
    GemvGroup g = base;
    g.mode = 4;
    g.post = prev;
    g.x_in = s->x[cur];
    g.norm_w = final_norm;
    add(g, head.w, head.K_pad, vocab, d, 0, s->logits);
    return launch_gemv_bf16_group(g, st);
}
