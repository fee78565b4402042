// Gadilix.cpp -- config parsing, construction and the per-layer step of the Gadilix stack (see Gadilix.hpp).
#include "Gadilix.hpp"

#include <algorithm>
#include <cmath>
#include <cstring>
#include <stdexcept>

namespace koifish {

#define KF_TRY(expr)                                                                       \
    do {                                                                                   \
        int _rc = (expr);                                                                  \
        if (_rc != KF_OK) {                                                                \
            *hFishErr = std::string(#expr) + " -> " + kf_status_string(_rc);               \
            return _rc;                                                                    \
        }                                                                                  \
    } while (0)

// ------------------------------------------------------------------------------------------------------------ config
static int need_int(const JSON& j, const char* key, const std::string& where) {
    const JSON* p = j.find(key);
    if (!p || !p->is_number()) throw std::runtime_error("config: " + where + "." + key + " is missing");
    return p->as_int();
}
static double need_num(const JSON& j, const char* key, const std::string& where) {
    const JSON* p = j.find(key);
    if (!p || !p->is_number()) throw std::runtime_error("config: " + where + "." + key + " is missing");
    return p->as_double(0.0);
}
static const JSON* present(const JSON& j, const char* key) {  // the value of a key that is there and not null
    const JSON* p = j.find(key);
    return (p && !p->is_null()) ? p : nullptr;
}
// two layers that share tensors agree in everything that sizes them
static bool same_sizes(const LAYER_CARD& a, const LAYER_CARD& b) {
    const MIXER_CARD &x = a.mixer, &y = b.mixer;
    const MOE_CARD &e = a.mlp, &g = b.mlp;
    return x.heads == y.heads && x.kv_heads == y.kv_heads && x.dim == y.dim && x.vdim == y.vdim && e.present == g.present && e.experts == g.experts && e.top == g.top &&
           e.ff == g.ff && e.shared_ff == g.shared_ff;
}

// config.json: {"architecture": "Gadilix", "vocab", "width", "norm": {"eps"}, "residual_mult",
//   "layers": [{"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "mask": {"size", "pool"}},
//               "mlp": null | {"kind": "moe", "expert": {"ff"}, "router": {"experts", "top"}, "shared": {"ff"}}, "weights_of": j}]}
// Keys that may be left out or null: residual_mult (1), kv_heads (= heads), vdim (= dim), scale (1 / sqrt(dim)), mask (every earlier
// position), mask.pool (no pooled blocks), mlp, mlp.shared, weights_of.
static void ParseGadilix(const JSON& h, MODEL_CARD& c) {
    c.vocab         = need_int(h, "vocab", "config");
    c.n_embd        = need_int(h, "width", "config");
    c.norm_rms_eps  = (float)need_num(h.at("norm"), "eps", "norm");
    c.norm_groups   = 1;
    c.residual_mult = present(h, "residual_mult") ? (float)need_num(h, "residual_mult", "config") : 1.f;
    const JSON& ls  = h.at("layers");
    if (!ls.is_array() || ls.arr.empty()) throw std::runtime_error("config: layers must be a non-empty list");
    const int L = (int)ls.arr.size();
    std::vector<int> of(L, -1);
    for (int i = 0; i < L; i++) {
        const JSON& l = ls.arr[i];
        const std::string where = "layers[" + std::to_string(i) + "]", wm = where + ".mixer";
        LAYER_CARD lc;
        MIXER_CARD& m = lc.mixer;
        m.type        = l.at("type").as_string();
        if (m.type != "attention") throw std::runtime_error("config: " + where + ": unknown mixer type '" + m.type + "'");
        const JSON& x = l.at("mixer");
        m.heads = need_int(x, "heads", wm), m.kv_heads = present(x, "kv_heads") ? need_int(x, "kv_heads", wm) : m.heads;
        m.dim = need_int(x, "dim", wm), m.vdim = present(x, "vdim") ? need_int(x, "vdim", wm) : m.dim;
        if (m.heads < 1 || m.kv_heads < 1 || m.heads % m.kv_heads || m.dim < 1 || m.dim > 512 || m.vdim < 1 || m.vdim > 512)
            throw std::runtime_error("config: " + wm + ": kv_heads must divide heads, 1 <= dim, vdim <= 512");
        m.scale = present(x, "scale") ? (float)need_num(x, "scale", wm) : 1.0f / std::sqrt((float)m.dim);
        if (const JSON* k = present(x, "mask")) {
            m.window = need_int(*k, "size", wm + ".mask");
            if (present(*k, "pool")) m.pool = need_int(*k, "pool", wm + ".mask");
            if (m.window < 1 || m.pool < 0) throw std::runtime_error("config: " + wm + ".mask: size must be positive, pool not negative");
        }
        if (const JSON* f = present(l, "mlp")) {
            const std::string kind = f->at("kind").as_string(), wf = where + ".mlp";
            if (kind != "moe") throw std::runtime_error("config: " + wf + ".kind '" + kind + "' is not built");
            MOE_CARD& e = lc.mlp;
            e.present = e.table_route = true;
            e.experts = need_int(f->at("router"), "experts", wf + ".router"), e.top = need_int(f->at("router"), "top", wf + ".router");
            e.ff = need_int(f->at("expert"), "ff", wf + ".expert");
            if (const JSON* sh = present(*f, "shared")) {
                e.shared_ff = need_int(*sh, "ff", wf + ".shared");
                if (e.shared_ff < 1) throw std::runtime_error("config: " + wf + ".shared.ff must be positive");
            }
            if (e.experts < 1 || e.experts > 8192 || e.top < 1 || e.top > e.experts || e.ff < 1)
                throw std::runtime_error("config: " + wf + ": 1 <= top <= experts <= 8192, expert.ff must be positive");
        }
        if (present(l, "weights_of")) of[i] = need_int(l, "weights_of", where);
        c.layers.push_back(lc);
    }
    for (int i = 0; i < L; i++) {  // follow the references to the layer that has the tensors
        if (of[i] < 0) {
            if (of[i] != -1) throw std::runtime_error("config: layers[" + std::to_string(i) + "].weights_of is not a layer");
            continue;
        }
        int j = i, hops = 0;
        while (of[j] >= 0) {
            if (of[j] >= L || ++hops > L) throw std::runtime_error("config: layers[" + std::to_string(i) + "].weights_of does not lead to a layer with tensors");
            j = of[j];
        }
        if (!same_sizes(c.layers[i], c.layers[j]))
            throw std::runtime_error("config: layers[" + std::to_string(i) + "] runs on the tensors of layers[" + std::to_string(j) + "] but has other sizes");
        c.layers[i].owner = j;
    }
    c.n_layers = L;
    if (c.vocab < 1 || c.n_embd < 1) throw std::runtime_error("config: vocab, width must be positive");
    c.n_head = c.n_head_kv = 1, c.head_dim = c.n_embd, c.n_ff = 0, c.tie_word_embeddings = false;
}

// ------------------------------------------------------------------------------------------------------------ build
namespace {
struct Builder {
    Fish& f;
    int next_id = 0;
    void Tensor(const std::string& name, int rows, int cols, hGTensor& out, int id_limit = 0) {
        out = std::make_shared<GTensor>(f.ctx, name, rows, cols);  // bf16 as stored, or a table of ids
        out->id_limit      = id_limit;
        f.tensors[name]    = out;
        f.tensor_ids[name] = next_id++;
    }
    template <typename T>
    int Buf(T** p, size_t bytes) {
        void* d = nullptr;
        int rc  = kf_malloc(f.ctx, std::max<size_t>(bytes, 16), &d);
        if (rc) return rc;
        f.owned.push_back(d);
        *p = (T*)d;
        return KF_OK;
    }
};
struct GdxExtra : GeNeuron {  // what belongs to no layer
    GroupNorm embed_norm;
    kf_table_route* routes = nullptr;  // device, one entry per layer with experts of its own
    std::vector<kf_table_route> host_routes;
    std::vector<hGTensor> route_tables;
    int max_experts = 1, max_top = 1;
};
// pooled rows of a slot, and the window / pool that the kernels see: a window longer than the ring means the ring was cut to max_seq rows --
// then every position lies in every window, nothing is ever masked and no block is ever behind the window
struct RingPlan {
    int ring, pooled, window, pool;
};
RingPlan PlanRing(const MIXER_CARD& m, int max_seq, long long step) {
    RingPlan r;
    r.ring   = m.window > 0 ? (int)std::min<long long>(max_seq, std::max(m.window, m.pool) + step - 1) : max_seq;
    r.window = m.window > 0 && m.window < max_seq ? m.window : 0;
    r.pool   = r.window > 0 && m.pool > 0 && m.pool < max_seq ? m.pool : 0;
    r.pooled = r.pool > 0 ? max_seq / r.pool : 0;
    return r;
}
}  // namespace

static int OwnerOf(const MODEL_CARD& c, int i) { return c.layers[i].owner >= 0 ? c.layers[i].owner : i; }

static int BuildGadilix(Fish& f) {
    std::string* hFishErr = &f.error;
    const MODEL_CARD& c   = f.config;
    if (f.tp_world != 1) {
        f.error = "the Gadilix stack runs on one GPU (no tensor-parallel shard plan)";
        return KF_ERR_UNSUPPORTED;
    }
    Builder b{f};
    const int E = c.n_embd, L = c.n_layers;
    const bool f32   = c.compute_f32;
    const size_t asz = f32 ? 4 : 2;
    auto ex = std::make_unique<GdxExtra>();
    ex->hFish = &f, ex->name = "model";
    f.embed.hFish = &f, f.embed.name = "embed";
    b.Tensor("embed", c.vocab, E, f.embed.w);
    ex->embed_norm.hFish = &f, ex->embed_norm.eps = c.norm_rms_eps;
    b.Tensor("embed.norm", 1, 1, ex->embed_norm.w);
    f.cls.hFish = &f, f.cls.name = "head";
    f.cls.norm.hFish = &f, f.cls.norm.rms_eps = c.norm_rms_eps;
    b.Tensor("final.norm", 1, 1, f.cls.norm.w);
    f.cls.proj.hFish = &f, f.cls.proj.nIn = E, f.cls.proj.nOut = c.vocab;
    b.Tensor("head", c.vocab, E, f.cls.proj.w);

    f.max_tokens = std::max(std::max(64, c.max_batch), c.max_prefill);
    f.logit_rows = c.logit_rows_cfg > 0 ? std::min(c.logit_rows_cfg, f.max_tokens) : std::max(64, c.max_batch);
    const size_t T = f.max_tokens;
    auto hs    = std::make_shared<HybridScratch>();
    f.hscratch = hs;
    size_t maxU = 1, maxY = 1, maxA = 1, maxTop = 1, maxFF = 1, maxSF = 1;
    f.states.layers.resize(L);
    f.states.max_seq = c.max_seq_len, f.states.f32 = f32;
    for (int i = 0; i < L; i++) {
        const LAYER_CARD& lc = c.layers[i];
        const MIXER_CARD& m  = lc.mixer;
        // cache and state: one entry per layer, also for a layer that shares its tensors
        SeqStateCache::Layer& sl = f.states.layers[i];
        const RingPlan rp = PlanRing(m, c.max_seq_len, (long long)T);
        sl.ring = rp.ring, sl.row_dim = m.kv_heads * (m.dim + m.vdim), sl.row_stride = (size_t)(rp.ring + rp.pooled) * sl.row_dim;
        sl.tail_stride = (size_t)E;
        // zeroed once: a reader may load rows of positions that the sequence has not written (masked, but they must hold numbers)
        KF_TRY(b.Buf((char**)&sl.rows, (size_t)c.max_batch * sl.row_stride * asz));
        KF_TRY(kf_memset(f.ctx, sl.rows, 0, (size_t)c.max_batch * sl.row_stride * asz));
        KF_TRY(b.Buf(&sl.tail, (size_t)c.max_batch * sl.tail_stride * 4));
        KF_TRY(kf_memset(f.ctx, sl.tail, 0, (size_t)c.max_batch * sl.tail_stride * 4));
        f.states.total_bytes += (size_t)c.max_batch * (sl.row_stride * asz + sl.tail_stride * 4);
        if (lc.owner >= 0) {  // runs on the block of its owner
            f.blocks.push_back(nullptr);
            continue;
        }
        const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
        auto blk   = std::make_unique<GdxBlock>();
        blk->hFish = &f, blk->name = p;
        blk->norm1.hFish = &f, blk->norm1.eps = c.norm_rms_eps;
        b.Tensor(p + "norm1", 1, 1, blk->norm1.w);
        b.Tensor(p + "shift", 1, E, blk->shift);
        auto a = std::make_unique<PooledAttention>();
        a->hFish = &f, a->name = mp, a->card = m;
        const int nq = m.heads * m.dim, nk = m.kv_heads * m.dim, nv = m.kv_heads * m.vdim, no = m.heads * m.vdim;
        b.Tensor(mp + "q", nq, E, a->q), b.Tensor(mp + "k", nk, E, a->k), b.Tensor(mp + "v", nv, E, a->v);
        b.Tensor(mp + "q.norm", 1, m.dim, a->qn), b.Tensor(mp + "k.norm", 1, m.dim, a->kn);
        b.Tensor(mp + "g", m.heads, E, a->g), b.Tensor(mp + "o", E, no, a->o);
        blk->cat.Plan({a->q, a->k, a->v, a->g});
        KF_TRY(b.Buf((char**)&blk->cat.w, (size_t)blk->cat.rows * E * 2));
        KF_TRY(kf_memset(f.ctx, blk->cat.w, 0, (size_t)blk->cat.rows * E * 2));
        maxU = std::max<size_t>(maxU, blk->cat.rows), maxA = std::max<size_t>(maxA, no), maxY = std::max<size_t>(maxY, nq / 2 + 1);  // maxY: the bf16 query of the panel kernel
        blk->attn = std::move(a);
        if (lc.mlp.present) {
            const MOE_CARD& mc = lc.mlp;
            blk->norm2.hFish = &f, blk->norm2.eps = c.norm_rms_eps;
            b.Tensor(p + "norm2", 1, 1, blk->norm2.w);
            auto e = std::make_unique<MoE>();
            e->hFish = &f, e->name = p + "mlp", e->card = mc;
            b.Tensor(p + "mlp.table", c.vocab, mc.top, e->table, mc.experts);
            e->gate.resize(mc.experts), e->up.resize(mc.experts), e->down.resize(mc.experts);
            for (int k = 0; k < mc.experts; k++) {
                const std::string ep = p + "mlp.e" + std::to_string(k) + ".";
                b.Tensor(ep + "gate", mc.ff, E, e->gate[k]), b.Tensor(ep + "up", mc.ff, E, e->up[k]), b.Tensor(ep + "down", E, mc.ff, e->down[k]);
            }
            if (mc.shared_ff > 0) {
                b.Tensor(p + "mlp.shared.gate", mc.shared_ff, E, e->sh_gate), b.Tensor(p + "mlp.shared.up", mc.shared_ff, E, e->sh_up);
                b.Tensor(p + "mlp.shared.down", E, mc.shared_ff, e->sh_down);
            }
            KF_TRY(b.Buf(&e->tables, (size_t)3 * mc.experts * sizeof(void*)));
            // dispatch tables of its own: all layers' tables are made at once, ahead of the first layer
            kf_table_route& r = e->route;
            const size_t TT = T * mc.top;
            r.experts = mc.experts, r.top = mc.top;
            KF_TRY(b.Buf(&r.idx, TT * 4));
            KF_TRY(b.Buf(&r.wgt, TT * 4));
            KF_TRY(b.Buf(&r.offsets, ((size_t)mc.experts + 1) * 4));
            KF_TRY(b.Buf(&r.entry_slot, TT * 4));
            KF_TRY(b.Buf(&r.slot_row, TT * 4));
            KF_TRY(b.Buf(&r.slot_group, TT * 4));
            KF_TRY(b.Buf(&r.work, (TT + mc.experts) * 4));
            ex->host_routes.push_back(r), ex->route_tables.push_back(e->table);
            ex->max_experts = std::max(ex->max_experts, mc.experts), ex->max_top = std::max(ex->max_top, mc.top);
            maxTop = std::max<size_t>(maxTop, mc.top), maxFF = std::max<size_t>(maxFF, (size_t)mc.top * mc.ff), maxSF = std::max<size_t>(maxSF, mc.shared_ff);
            blk->moe = std::move(e);
        }
        f.blocks.push_back(std::move(blk));
    }
    KF_TRY(b.Buf(&ex->routes, std::max<size_t>(1, ex->host_routes.size()) * sizeof(kf_table_route)));
    f.blocks.push_back(std::move(ex));  // kept behind the layers' blocks
    // activations: fp32 residual stream; matmul inputs in the activation type
    KF_TRY(kf_malloc(f.ctx, T * E * 4, &f.x));
    KF_TRY(b.Buf((char**)&hs->hact, T * E * asz));
    KF_TRY(b.Buf(&hs->sub, T * E * 4));
    KF_TRY(b.Buf(&hs->u, T * maxU * 4));
    KF_TRY(b.Buf(&hs->y, T * maxY * 4));
    KF_TRY(b.Buf((char**)&hs->act, T * maxA * asz));
    KF_TRY(b.Buf((char**)&hs->h1, T * maxFF * asz));
    KF_TRY(b.Buf(&hs->yslots, T * maxTop * E * 4));
    KF_TRY(b.Buf((char**)&hs->hs, T * maxSF * asz));
    KF_TRY(b.Buf(&hs->shared, T * E * 4));
    KF_TRY(b.Buf((char**)&hs->head_in, (size_t)f.logit_rows * E * asz));
    KF_TRY(kf_malloc(f.ctx, (size_t)f.logit_rows * c.vocab * 2, &f.logits));
    KF_TRY(kf_malloc(f.ctx, (size_t)f.logit_rows * c.vocab * 4, (void**)&f.logits_f32));
    KF_TRY(kf_malloc(f.ctx, T * 4, (void**)&f.d_tokens));
    KF_TRY(kf_malloc(f.ctx, T * 4, (void**)&f.d_pos));
    KF_TRY(kf_malloc(f.ctx, T * 4, (void**)&f.d_next));
    KF_TRY(kf_malloc(f.ctx, T * 4, (void**)&f.d_slot));
    KF_TRY(kf_malloc(f.ctx, T * 4, (void**)&f.d_sel));
    KF_TRY(kf_host_alloc(T * 4 * 5, (void**)&f.h_stage));
    KF_TRY(kf_host_alloc((size_t)f.logit_rows * c.vocab * 2, (void**)&f.h_logits));
    KF_TRY(kf_host_alloc((size_t)f.logit_rows * c.vocab * 4, (void**)&f.h_logits_f32));
    KF_TRY(kf_ctx_sync(f.ctx));
    f.attn_hint = c.max_seq_len - 1;
    return KF_OK;
}

static GdxBlock* BlockOf(Fish& f, int layer) { return static_cast<GdxBlock*>(f.blocks[OwnerOf(f.config, layer)].get()); }
static GdxExtra* ExtraOf(Fish& f) { return static_cast<GdxExtra*>(f.blocks[f.config.n_layers].get()); }

static int PrepareGadilix(Fish& f) {
    GdxExtra* ex = ExtraOf(f);
    for (int i = 0; i < f.config.n_layers; i++) {
        if (f.config.layers[i].owner >= 0) continue;
        GdxBlock* b = BlockOf(f, i);
        int rc = b->cat.Fill(f.ctx);
        if (!rc && b->moe) rc = b->moe->Prepare();
        if (rc) return rc;
    }
    for (size_t k = 0; k < ex->host_routes.size(); k++) ex->host_routes[k].table = (const int32_t*)ex->route_tables[k]->data;
    int rc = ex->host_routes.empty() ? KF_OK : kf_h2d(f.ctx, ex->routes, ex->host_routes.data(), ex->host_routes.size() * sizeof(kf_table_route));
    return rc ? rc : kf_ctx_sync(f.ctx);
}

// ------------------------------------------------------------------------------------------------------------ step
static int Lin(Fish& f, float* y, int ldy, const hGTensor& w, const void* x, int ldx, int M) {
    kf_tensor_desc d = w->Desc();
    return kf_linear_g(f.ctx, y, ldy, &d, x, f.config.compute_f32 ? 1 : 0, ldx, M);
}
static int LinStacked(Fish& f, float* y, const StackedLinear& s, const void* x, int M) {
    kf_tensor_desc d = {};
    d.data_dev = s.w, d.rows = s.rows, d.cols = s.cols, d.type = KF_T_BF16, d.group = 128;
    return kf_linear_g(f.ctx, y, s.rows, &d, x, f.config.compute_f32 ? 1 : 0, s.cols, M);
}

int PooledAttention::cuInfer(int M, float* u, int ldu, int off, int off_g, int layer) {
    Fish& f = *hFish;
    std::string* hFishErr = &f.error;
    HybridScratch& s = *f.hscratch;
    const MODEL_CARD& c = f.config;
    const MIXER_CARD& m = c.layers[layer].mixer;  // this run's window and scale; the sizes are the owner's
    const int ak = c.compute_f32 ? 1 : 0, no = m.heads * m.vdim;
    SeqStateCache::Layer& sl = f.states.layers[layer];
    const RingPlan rp = PlanRing(m, c.max_seq_len, f.max_tokens);
    // panels of one sequence with head sizes the tensor-core kernel takes go there; everything else (decode, other sizes, 32-bit) to the general kernel
    const bool tile = !ak && f.panel_consecutive && f.seq_mode == 0 && M >= 16 && m.dim == m.vdim && (m.dim == 64 || m.dim == 128);
    // per-head norms; this step's keys and values join the ring; blocks that it completes get their mean rows
    KF_TRY(kf_qk_heads_prepare(f.ctx, u + off, ldu, m.heads, m.kv_heads, m.dim, m.vdim, qn->data, kn->data, c.norm_rms_eps, 0, nullptr, 1.f, 0, sl.rows, ak,
                               sl.row_stride, rp.ring, rp.pool, f.seq_mode || M == 1, tile ? s.y : nullptr, f.d_pos, f.d_slot, M));
    if (tile)
        KF_TRY(kf_attn_pooled_prefill(f.ctx, s.act, no, s.y, sl.rows, sl.row_stride, rp.ring, nullptr, f.d_pos, f.d_slot, M, m.heads, m.kv_heads, m.dim, m.scale, 0.f,
                                      rp.window, rp.pool, u + off_g, ldu, 1.f));
    else
        KF_TRY(kf_attn_window_ex(f.ctx, s.act, ak, no, u + off, ldu, sl.rows, ak, sl.row_stride, rp.ring, nullptr, f.d_pos, f.d_slot, M, m.heads, m.kv_heads, m.dim,
                                 m.vdim, m.scale, 0.f, rp.window, f.attn_hint + 1, 1.f, rp.pool, u + off_g, ldu));
    KF_TRY(Lin(f, s.sub, c.n_embd, o, s.act, no, M));
    return KF_OK;
}

static int ForwardGadilix(Fish& f, int M, bool want_logits) {
    std::string* hFishErr = &f.error;
    HybridScratch& s = *f.hscratch;
    const MODEL_CARD& c = f.config;
    const int E = c.n_embd, ak = c.compute_f32 ? 1 : 0, L = c.n_layers;
    float* x = (float*)f.x;
    GdxExtra* ex = ExtraOf(f);
    // every token of the step belongs to a sequence of its own: the shift of a layer's input rides on the norm ahead of it; otherwise a token's
    // predecessor is another row of the step and the shift is a launch of its own
    const bool single = f.seq_mode || M == 1;
    auto shift_of = [&](int layer) -> const void* { return single && layer < L ? BlockOf(f, layer)->shift->data : nullptr; };
    auto tail_of  = [&](int layer) -> float* { return layer < L ? f.states.layers[layer].tail : nullptr; };
    if (!ex->host_routes.empty()) KF_TRY(kf_moe_route_table(f.ctx, ex->routes, (int)ex->host_routes.size(), ex->max_experts, ex->max_top, f.d_tokens, M));
    kf_tensor_desc de = f.embed.w->Desc();
    KF_TRY(kf_embed_norm(f.ctx, x, single ? s.hact : nullptr, ak, &de, f.d_tokens, ex->embed_norm.w->data, 0.f, 1, M, ex->embed_norm.eps, shift_of(0), tail_of(0), E,
                         f.d_pos, f.d_slot));
    for (int i = 0; i < L; i++) {
        GdxBlock* blk = BlockOf(f, i);
        if (!single) KF_TRY(kf_token_shift(f.ctx, s.hact, ak, x, E, blk->shift->data, tail_of(i), E, f.d_pos, f.d_slot, 1, M, E));
        // one matmul for everything that reads the shifted input: q | k | v | gate logits
        KF_TRY(LinStacked(f, s.u, blk->cat, s.hact, M));
        KF_TRY(blk->attn->cuInfer(M, s.u, blk->cat.rows, blk->cat.off[0], blk->cat.off[3], i));
        // x += m norm1(sub); hact = the new x for the feed-forward, or the next layer's shifted input
        const void* next = shift_of(i + 1);
        const bool last  = i + 1 == L;
        if (!blk->moe) {
            KF_TRY(kf_postnorm_residual_ex(f.ctx, x, single && !last ? s.hact : nullptr, ak, s.sub, E, 1.f, nullptr, 0, 0.f, blk->norm1.w->data, 0.f, 1, c.residual_mult,
                                           M, E, blk->norm1.eps, next, tail_of(i + 1), E, f.d_pos, f.d_slot));
            continue;
        }
        KF_TRY(kf_postnorm_residual_ex(f.ctx, x, s.hact, ak, s.sub, E, 1.f, nullptr, 0, 0.f, blk->norm1.w->data, 0.f, 1, c.residual_mult, M, E, blk->norm1.eps, nullptr,
                                       nullptr, 0, nullptr, nullptr));
        const MoE& e = *blk->moe;
        KF_TRY(blk->moe->Experts(M, e.route.offsets, e.route.slot_row, e.route.slot_group));
        // x += m norm2(sum of the experts); the next layer's shifted input on the way
        KF_TRY(kf_experts_postnorm_residual(f.ctx, x, single && !last ? s.hact : nullptr, ak, s.yslots, e.route.entry_slot, e.route.wgt,
                                            e.card.shared_ff > 0 ? s.shared : nullptr, e.card.top, blk->norm2.w->data, 0.f, 1, c.residual_mult, M, E, blk->norm2.eps, next,
                                            tail_of(i + 1), E, f.d_pos, f.d_slot));
    }
    if (want_logits && f.n_rows > 0) {
        const int R = f.n_rows;
        KF_TRY(kf_group_rmsnorm_wadd(f.ctx, s.head_in, ak, E, nullptr, 0.f, x, E, nullptr, 0, nullptr, 0, f.cls.norm.w->data, 2, 0.f, 1.f, f.d_sel, R, E, 1,
                                     c.norm_rms_eps));
        KF_TRY(Lin(f, f.logits_f32, c.vocab, f.cls.proj.w, s.head_in, E, R));
        KF_TRY(kf_f32_to_bf16(f.ctx, f.logits, f.logits_f32, (size_t)R * c.vocab));
    }
    return KF_OK;
}

const ARCH_ENTRY* GadilixArch() {
    static const ARCH_ENTRY e = {"GADILIX", ParseGadilix, BuildGadilix, ForwardGadilix, PrepareGadilix};
    return &e;
}

}  // namespace koifish
