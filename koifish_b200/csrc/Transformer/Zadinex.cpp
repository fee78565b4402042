// Zadinex.cpp -- config parsing, construction and the per-layer step of the Zadinex stack (see Zadinex.hpp).
#include "Zadinex.hpp"

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
constexpr int kDecayRank = 32;

// config.json: {"architecture": "Zadinex", "vocab", "width", "norm": {"eps"},
//   "layers": [{"type": "wkv", "mixer": {"heads", "dim", "w_rank"}} |
//              {"type": "attention", "mixer": {"heads", "kv_heads", "dim", "vdim", "scale", "v_mix", "rot": {"base", "dims"}}},
//              each with "mlp": null | {"kind": "dense", "ff"} |
//                               {"kind": "moe", "expert": {"ff", "limit"},
//                                "router": {"experts", "identity", "top", "groups": {"count", "keep"}}}]}
// Keys that may be left out or null: w_rank (the rows of the checkpoint's mix.w1, else 32), kv_heads (= heads), vdim (= dim), scale
// (1 / sqrt(dim)), v_mix (false), rot (no rotation), rot.dims (= dim), mlp, expert.limit (no clamp), identity (0), groups (one).
static void ParseZadinex(const JSON& h, MODEL_CARD& c) {
    c.vocab        = need_int(h, "vocab", "config");
    c.n_embd       = need_int(h, "width", "config");
    c.norm_rms_eps = (float)need_num(h.at("norm"), "eps", "norm");
    c.norm_groups  = 1;
    const JSON& ls = h.at("layers");
    if (!ls.is_array() || ls.arr.empty()) throw std::runtime_error("config: layers must be a non-empty list");
    const JSON* shapes = h.find("tensor_shapes");
    int blend_width = 0;  // kv_heads x vdim of the layers that blend their values
    for (size_t i = 0; i < ls.arr.size(); i++) {
        const JSON& l = ls.arr[i];
        const std::string where = "layers[" + std::to_string(i) + "]", wm = where + ".mixer";
        LAYER_CARD lc;
        MIXER_CARD& m = lc.mixer;
        m.type        = l.at("type").as_string();
        const JSON& x = l.at("mixer");
        if (m.type == "wkv") {
            m.heads = need_int(x, "heads", wm), m.dim = need_int(x, "dim", wm), m.vdim = m.dim, m.kv_heads = m.heads;
            m.rank_a = present(x, "w_rank") ? need_int(x, "w_rank", wm) : kDecayRank;
            if (!present(x, "w_rank") && shapes)
                if (const JSON* t = shapes->find("l" + std::to_string(i) + ".mix.w1"))
                    if (t->is_array() && !t->arr.empty()) m.rank_a = t->arr[0].as_int();
            if (m.heads < 1 || m.dim < 1 || m.dim > 512 || m.rank_a < 1) throw std::runtime_error("config: " + wm + ": heads, w_rank must be positive, 1 <= dim <= 512");
        } else if (m.type == "attention") {
            m.heads = need_int(x, "heads", wm), m.kv_heads = present(x, "kv_heads") ? need_int(x, "kv_heads", wm) : m.heads;
            m.dim = need_int(x, "dim", wm), m.vdim = present(x, "vdim") ? need_int(x, "vdim", wm) : m.dim;
            m.scale = present(x, "scale") ? (float)need_num(x, "scale", wm) : 1.0f / std::sqrt((float)m.dim);
            m.v_mix = present(x, "v_mix") && present(x, "v_mix")->as_bool(false);
            if (m.heads < 1 || m.kv_heads < 1 || m.heads % m.kv_heads || m.dim < 1 || m.dim > 1024 || m.vdim < 1 || m.vdim > 512)
                throw std::runtime_error("config: " + wm + ": kv_heads must divide heads, 1 <= dim <= 1024, 1 <= vdim <= 512");
            if (const JSON* t = present(x, "rot")) {
                m.rot_dims = present(*t, "dims") ? need_int(*t, "dims", wm + ".rot") : m.dim;
                m.rot_base = need_num(*t, "base", wm + ".rot");
                if (m.rot_dims < 0 || m.rot_dims > m.dim || m.rot_dims % 2 || (m.rot_dims > 0 && !(m.rot_base > 0.0)))
                    throw std::runtime_error("config: " + wm + ".rot: dims must be even and at most dim, base positive");
            }
            if (m.v_mix) {
                if (blend_width && blend_width != m.kv_heads * m.vdim)
                    throw std::runtime_error("config: " + wm + ": layers with v_mix must agree in kv_heads x vdim");
                blend_width = m.kv_heads * m.vdim;
            }
        } else {
            throw std::runtime_error("config: " + where + ": unknown mixer type '" + m.type + "'");
        }
        if (const JSON* f = present(l, "mlp")) {
            const std::string kind = f->at("kind").as_string(), wf = where + ".mlp";
            MOE_CARD& e = lc.mlp;
            e.present = true;
            if (kind == "dense") {
                e.dense = true, e.ff = need_int(*f, "ff", wf);
                if (e.ff < 1) throw std::runtime_error("config: " + wf + ".ff must be positive");
            } else if (kind == "moe") {
                const JSON &r = f->at("router"), &x1 = f->at("expert");
                e.softmax_groups = true, e.glu_alpha = 1.702f, e.glu_shift = 1.f;
                e.experts = need_int(r, "experts", wf + ".router"), e.top = need_int(r, "top", wf + ".router");
                e.pass = present(r, "identity") ? need_int(r, "identity", wf + ".router") : 0;
                e.ff = need_int(x1, "ff", wf + ".expert"), e.limit = present(x1, "limit") ? (float)need_num(x1, "limit", wf + ".expert") : 0.f;
                if (const JSON* g = present(r, "groups"))
                    e.groups = need_int(*g, "count", wf + ".router.groups"), e.keep = need_int(*g, "keep", wf + ".router.groups");
                const int outs = e.experts + e.pass;
                if (e.experts < 1 || e.pass < 0 || e.ff < 1 || e.limit < 0.f || e.groups < 1 || e.groups > 64 || outs % e.groups || e.keep < 1 || e.keep > e.groups ||
                    e.top < 1 || e.top > e.keep * (outs / e.groups))
                    throw std::runtime_error("config: " + wf + ".router: groups.count (<= 64) must divide experts + identity, 1 <= keep <= count, 1 <= top <= keep * "
                                             "(experts + identity) / count, expert.ff positive");
            } else {
                throw std::runtime_error("config: " + wf + ".kind '" + kind + "' is not built");
            }
        }
        c.layers.push_back(lc);
    }
    c.n_layers = (int)c.layers.size();
    if (c.vocab < 1 || c.n_embd < 1) throw std::runtime_error("config: vocab, width must be positive");
    c.n_head = c.n_head_kv = 1, c.head_dim = c.n_embd, c.n_ff = 0, c.tie_word_embeddings = false;
}

// ------------------------------------------------------------------------------------------------------------ build
namespace {
struct Builder {
    Fish& f;
    int next_id = 0;
    void Tensor(const std::string& name, int rows, int cols, hGTensor& out) {
        out = std::make_shared<GTensor>(f.ctx, name, rows, cols);  // bf16 as stored
        f.tensors[name]    = out;
        f.tensor_ids[name] = next_id++;
    }
    void Norm(const std::string& name, TanhNorm& n) {
        n.hFish = &f, n.name = name;
        Tensor(name, 1, f.config.n_embd, n.w), Tensor(name + ".b", 1, f.config.n_embd, n.b), Tensor(name + ".alpha", 1, 1, n.alpha);
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
    int Stack(StackedLinear& s, const std::vector<hGTensor>& parts) {
        s.Plan(parts);
        int rc = Buf((char**)&s.w, (size_t)s.rows * s.cols * 2);
        return rc ? rc : kf_memset(f.ctx, s.w, 0, (size_t)s.rows * s.cols * 2);
    }
};
struct ZdxExtra : GeNeuron {  // what belongs to no layer
    TanhNorm final_norm;
};
constexpr int kMixes = 5;
}  // namespace

static ZdxBlock* BlockOf(Fish& f, int layer) { return static_cast<ZdxBlock*>(f.blocks[layer].get()); }
static ZdxExtra* ExtraOf(Fish& f) { return static_cast<ZdxExtra*>(f.blocks[f.config.n_layers].get()); }

static int BuildZadinex(Fish& f) {
    std::string* hFishErr = &f.error;
    const MODEL_CARD& c   = f.config;
    if (f.tp_world != 1) {
        f.error = "the Zadinex stack runs on one GPU (no tensor-parallel shard plan)";
        return KF_ERR_UNSUPPORTED;
    }
    Builder b{f};
    const int E = c.n_embd, L = c.n_layers;
    const bool f32   = c.compute_f32;
    const size_t asz = f32 ? 4 : 2;
    auto ex   = std::make_unique<ZdxExtra>();
    ex->hFish = &f, ex->name = "model";
    f.embed.hFish = &f, f.embed.name = "embed";
    b.Tensor("embed", c.vocab, E, f.embed.w);
    b.Norm("final.norm", ex->final_norm);
    f.cls.hFish = &f, f.cls.name = "head";
    f.cls.proj.hFish = &f, f.cls.proj.nIn = E, f.cls.proj.nOut = c.vocab;
    b.Tensor("head", c.vocab, E, f.cls.proj.w);

    f.max_tokens = std::max(std::max(64, c.max_batch), c.max_prefill);
    f.logit_rows = c.logit_rows_cfg > 0 ? std::min(c.logit_rows_cfg, f.max_tokens) : std::max(64, c.max_batch);
    const size_t T = f.max_tokens;
    auto hs    = std::make_shared<HybridScratch>();
    f.hscratch = hs;
    size_t maxU = 1, maxV = 1, maxY = 1, maxL = 1, maxA = 1, maxMid = 1, maxVF = 1, maxE = 1, maxTop = 1, maxH1 = 1;
    bool blending = false;
    f.states.layers.resize(L);
    f.states.max_seq = c.max_seq_len, f.states.f32 = f32;
    for (int i = 0; i < L; i++) {
        const LAYER_CARD& lc = c.layers[i];
        const MIXER_CARD& m  = lc.mixer;
        const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
        auto blk   = std::make_unique<ZdxBlock>();
        blk->hFish = &f, blk->name = p;
        b.Norm(p + "norm1", blk->norm1);
        b.Tensor(p + "ls1", 1, E, blk->ls1);
        SeqStateCache::Layer& sl = f.states.layers[i];
        if (m.type == "wkv") {
            auto t = std::make_unique<TimeMix>();
            t->hFish = &f, t->name = mp, t->card = m;
            const int n = m.heads * m.dim;
            static const char* kMu[kMixes] = {"mu.r", "mu.k", "mu.v", "mu.g", "mu.w"};
            for (int q = 0; q < kMixes; q++) b.Tensor(mp + kMu[q], 1, E, t->mu[q]);
            b.Tensor(mp + "r", n, E, t->r), b.Tensor(mp + "k", n, E, t->k), b.Tensor(mp + "v", n, E, t->v), b.Tensor(mp + "g", n, E, t->g);
            b.Tensor(mp + "w1", m.rank_a, E, t->w1), b.Tensor(mp + "w2", n, m.rank_a, t->w2), b.Tensor(mp + "w0", 1, n, t->w0);
            b.Tensor(mp + "u", m.heads, m.dim, t->u), b.Tensor(mp + "norm", 1, n, t->norm), b.Tensor(mp + "o", E, n, t->o);
            KF_TRY(b.Stack(t->mus, {t->mu[0], t->mu[1], t->mu[2], t->mu[3], t->mu[4]}));
            sl.state_stride = (size_t)m.heads * m.dim * m.dim, sl.tail_stride = (size_t)E;
            KF_TRY(b.Buf(&sl.state, (size_t)c.max_batch * sl.state_stride * 4));
            KF_TRY(b.Buf(&sl.tail, (size_t)c.max_batch * sl.tail_stride * 4));
            KF_TRY(kf_memset(f.ctx, sl.tail, 0, (size_t)c.max_batch * sl.tail_stride * 4));
            f.states.total_bytes += (size_t)c.max_batch * (sl.state_stride + sl.tail_stride) * 4;
            maxU = std::max<size_t>(maxU, (size_t)4 * n), maxV = std::max<size_t>(maxV, m.rank_a), maxL = std::max<size_t>(maxL, n), maxY = std::max<size_t>(maxY, n);
            maxA = std::max<size_t>(maxA, n), maxMid = std::max<size_t>(maxMid, (size_t)kMixes * E);
            blk->wkv = std::move(t);
        } else {
            auto a = std::make_unique<BlendedAttention>();
            a->hFish = &f, a->name = mp, a->card = m;
            const int nq = m.heads * m.dim, nk = m.kv_heads * m.dim, nv = m.kv_heads * m.vdim, no = m.heads * m.vdim;
            b.Tensor(mp + "q", nq, E, a->q), b.Tensor(mp + "k", nk, E, a->k), b.Tensor(mp + "v", nv, E, a->v);
            if (m.v_mix) {
                b.Tensor(mp + "vmix", 1, 1, a->vmix);  // stored, and unused, in the first blending layer too
                a->blend_source = !blending, blending = true;
                maxVF = std::max<size_t>(maxVF, nv);
            }
            b.Tensor(mp + "sink", 1, m.heads, a->sink), b.Tensor(mp + "o", E, no, a->o);
            if (m.rot_dims > 0) {
                float amp = 1.f;
                const std::vector<double> fr = StretchedFrequencies(m.rot_dims, m.rot_base, 0.0, 0.0, 0.0, 0.0, &amp);
                KF_TRY(b.Buf(&a->inv_freq, fr.size() * sizeof(double)));
                KF_TRY(kf_h2d(f.ctx, a->inv_freq, fr.data(), fr.size() * sizeof(double)));
                KF_TRY(kf_ctx_sync(f.ctx));  // fr leaves scope
            }
            KF_TRY(b.Stack(blk->cat, {a->q, a->k, a->v}));
            sl.row_dim = nk + nv, sl.row_stride = (size_t)c.max_seq_len * sl.row_dim;
            // zeroed once: a reader may load rows of positions that the sequence has not written (masked, but they must hold numbers)
            KF_TRY(b.Buf((char**)&sl.rows, (size_t)c.max_batch * sl.row_stride * asz));
            KF_TRY(kf_memset(f.ctx, sl.rows, 0, (size_t)c.max_batch * sl.row_stride * asz));
            f.states.total_bytes += (size_t)c.max_batch * sl.row_stride * asz;
            maxU = std::max<size_t>(maxU, blk->cat.rows), maxA = std::max<size_t>(maxA, no), maxY = std::max<size_t>(maxY, nq / 2 + 1);  // maxY: the bf16 query of the panel kernel
            blk->attn = std::move(a);
        }
        if (lc.mlp.present) {
            b.Norm(p + "norm2", blk->norm2);
            b.Tensor(p + "ls2", 1, E, blk->ls2);
        }
        if (lc.mlp.present && lc.mlp.dense) {
            auto e = std::make_unique<GeluFF>();
            e->hFish = &f, e->name = p + "mlp", e->card = lc.mlp;
            b.Tensor(p + "mlp.gate", lc.mlp.ff, E, e->gate), b.Tensor(p + "mlp.up", lc.mlp.ff, E, e->up), b.Tensor(p + "mlp.down", E, lc.mlp.ff, e->down);
            KF_TRY(b.Stack(e->cat, {e->gate, e->up}));
            maxU = std::max<size_t>(maxU, e->cat.rows), maxH1 = std::max<size_t>(maxH1, lc.mlp.ff);
            blk->dense = std::move(e);
        } else if (lc.mlp.present) {
            const MOE_CARD& mc = lc.mlp;
            auto e = std::make_unique<MoE>();
            e->hFish = &f, e->name = p + "mlp", e->card = mc;
            b.Tensor(p + "mlp.router", mc.experts + mc.pass, E, e->router), b.Tensor(p + "mlp.correction", 1, mc.experts + mc.pass, e->router_b);
            e->gate.resize(mc.experts), e->up.resize(mc.experts), e->down.resize(mc.experts);
            for (int k = 0; k < mc.experts; k++) {
                const std::string ep = p + "mlp.e" + std::to_string(k) + ".";
                b.Tensor(ep + "gate", mc.ff, E, e->gate[k]), b.Tensor(ep + "up", mc.ff, E, e->up[k]), b.Tensor(ep + "down", E, mc.ff, e->down[k]);
            }
            KF_TRY(b.Buf(&e->tables, (size_t)3 * mc.experts * sizeof(void*)));
            maxE = std::max<size_t>(maxE, mc.experts + mc.pass), maxTop = std::max<size_t>(maxTop, mc.top), maxH1 = std::max<size_t>(maxH1, (size_t)mc.top * mc.ff);
            maxU = std::max<size_t>(maxU, mc.experts + mc.pass);
            blk->moe = std::move(e);
        }
        f.blocks.push_back(std::move(blk));
    }
    f.blocks.push_back(std::move(ex));  // kept behind the layers' blocks
    // activations: fp32 residual stream; matmul inputs in the activation type
    KF_TRY(kf_malloc(f.ctx, T * E * 4, &f.x));
    KF_TRY(b.Buf((char**)&hs->hact, T * E * asz));
    KF_TRY(b.Buf(&hs->sub, T * E * 4));
    KF_TRY(b.Buf(&hs->u, T * maxU * 4));
    KF_TRY(b.Buf(&hs->v, T * maxV * 4));
    KF_TRY(b.Buf(&hs->y, T * maxY * 4));
    KF_TRY(b.Buf(&hs->lat, T * maxL * 4));
    KF_TRY(b.Buf(&hs->vfirst, T * maxVF * 4));
    KF_TRY(b.Buf((char**)&hs->act, T * maxA * asz));
    KF_TRY(b.Buf((char**)&hs->mid, T * maxMid * asz));
    const size_t TT = T * maxTop;
    KF_TRY(b.Buf(&hs->idx, TT * 4));
    KF_TRY(b.Buf(&hs->wgt, TT * 4));
    KF_TRY(b.Buf(&hs->offsets, (maxE + 1) * 4));
    KF_TRY(b.Buf(&hs->entry_slot, TT * 4));
    KF_TRY(b.Buf(&hs->slot_row, TT * 4));
    KF_TRY(b.Buf(&hs->slot_group, TT * 4));
    KF_TRY(b.Buf(&hs->work, (2 * TT + maxE) * 4));
    KF_TRY(b.Buf((char**)&hs->h1, T * maxH1 * asz));
    KF_TRY(b.Buf(&hs->yslots, TT * E * 4));
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

static int PrepareZadinex(Fish& f) {
    for (int i = 0; i < f.config.n_layers; i++) {
        ZdxBlock* b = BlockOf(f, i);
        int rc = b->wkv ? b->wkv->mus.Fill(f.ctx) : b->cat.Fill(f.ctx);
        if (!rc && b->dense) rc = b->dense->cat.Fill(f.ctx);
        if (!rc && b->moe) rc = b->moe->Prepare();
        if (rc) return rc;
    }
    return KF_OK;
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

int TimeMix::cuInfer(int M, int layer) {
    Fish& f = *hFish;
    std::string* hFishErr = &f.error;
    HybridScratch& s = *f.hscratch;
    const MIXER_CARD& m = card;
    const MODEL_CARD& c = f.config;
    const int E = c.n_embd, n = m.heads * m.dim, ak = c.compute_f32 ? 1 : 0;
    const int nseq = f.seq_mode ? M : 1, T = f.seq_mode ? 1 : M;
    SeqStateCache::Layer& sl = f.states.layers[layer];
    const size_t plane = (size_t)M * E * (ak ? 4 : 2), Mn = (size_t)M * n;
    const char* mixed = (const char*)s.mid;
    float *R = s.u, *K = R + Mn, *V = K + Mn, *G = V + Mn, *Z = s.lat;
    // every projection reads its own mix; the decay's low-rank middle leaves through tanh in fp32
    const kf_tensor_desc w[kMixes] = {r->Desc(), k->Desc(), v->Desc(), g->Desc(), w1->Desc()};
    float* y[kMixes]       = {R, K, V, G, s.v};
    const void* x[kMixes]  = {mixed, mixed + plane, mixed + 2 * plane, mixed + 3 * plane, mixed + 4 * plane};
    const int act[kMixes]  = {0, 0, 0, 0, 3};
    KF_TRY(kf_linear_batch(f.ctx, kMixes, y, w, x, act, ak, E, M));
    kf_tensor_desc d2 = w2->Desc();
    KF_TRY(kf_linear_g(f.ctx, Z, n, &d2, s.v, 1, m.rank_a, M));  // fp32 activations: the decay's logarithm is formed in 32-bit
    KF_TRY(kf_wkv_scan(f.ctx, s.y, n, R, n, K, n, V, n, Z, n, w0->data, u->data, sl.state, sl.state_stride, f.d_pos, f.d_slot, nseq, T, m.heads, m.dim, m.dim));
    // every head over its rms, times the weight, times silu(g)
    KF_TRY(kf_group_rmsnorm_wadd(f.ctx, s.act, ak, n, nullptr, 0.f, s.y, n, G, n, nullptr, 4, norm->data, 0, 0.f, 1.f, nullptr, M, n, m.heads, c.norm_rms_eps));
    KF_TRY(Lin(f, s.sub, E, o, s.act, n, M));
    return KF_OK;
}

int BlendedAttention::cuInfer(int M, float* u, int ldu, int layer) {
    Fish& f = *hFish;
    std::string* hFishErr = &f.error;
    HybridScratch& s = *f.hscratch;
    const MIXER_CARD& m = card;
    const MODEL_CARD& c = f.config;
    const int ak = c.compute_f32 ? 1 : 0, no = m.heads * m.vdim;
    SeqStateCache::Layer& sl = f.states.layers[layer];
    const int ring = c.max_seq_len;  // every position keeps its row
    // panels of one sequence with head sizes the tensor-core kernel takes go there; everything else (decode, other sizes, 32-bit) to the general kernel
    const bool tile = !ak && f.panel_consecutive && f.seq_mode == 0 && M >= 16 && (m.dim == 64 || m.dim == 128) && (m.vdim == 32 || m.vdim == 64 || m.vdim == 128);
    KF_TRY(kf_qk_heads_prepare_ex(f.ctx, u, ldu, m.heads, m.kv_heads, m.dim, m.vdim, nullptr, nullptr, 1, c.norm_rms_eps, m.rot_dims, inv_freq, 1.f, 1,
                                  m.v_mix ? s.vfirst : nullptr, m.kv_heads * m.vdim, m.v_mix && !blend_source ? vmix->data : nullptr, sl.rows, ak, sl.row_stride, ring, 0,
                                  f.seq_mode || M == 1, tile ? s.y : nullptr, f.d_pos, f.d_slot, M));
    if (tile)
        KF_TRY(kf_attn_window_prefill_ex(f.ctx, s.act, no, s.y, sl.rows, sl.row_stride, ring, sink->data, f.d_pos, f.d_slot, M, m.heads, m.kv_heads, m.dim, m.vdim, m.scale,
                                         0.f, 0, 1.f));
    else
        KF_TRY(kf_attn_window(f.ctx, s.act, ak, no, u, ldu, sl.rows, ak, sl.row_stride, ring, sink->data, f.d_pos, f.d_slot, M, m.heads, m.kv_heads, m.dim, m.vdim,
                              m.scale, 0.f, 0, f.attn_hint + 1, 1.f));
    KF_TRY(Lin(f, s.sub, c.n_embd, o, s.act, no, M));
    return KF_OK;
}

int GeluFF::cuInfer(int M) {
    Fish& f = *hFish;
    std::string* hFishErr = &f.error;
    HybridScratch& s = *f.hscratch;
    const int ak = f.config.compute_f32 ? 1 : 0, F = card.ff;
    KF_TRY(LinStacked(f, s.u, cat, s.hact, M));
    KF_TRY(kf_bias_act(f.ctx, s.h1, ak, F, s.u + cat.off[0], cat.rows, nullptr, 1, s.u + cat.off[1], cat.rows, M, F));  // gelu(gate) * up
    KF_TRY(Lin(f, s.sub, f.config.n_embd, down, s.h1, F, M));
    return KF_OK;
}

static int ForwardZadinex(Fish& f, int M, bool want_logits) {
    std::string* hFishErr = &f.error;
    HybridScratch& s = *f.hscratch;
    const MODEL_CARD& c = f.config;
    const int E = c.n_embd, ak = c.compute_f32 ? 1 : 0, L = c.n_layers;
    // every token of the step belongs to a sequence of its own: the token mixes of a layer's input ride on the step ahead of it; otherwise a
    // token's predecessor is another row of the step and the mixes are a launch of their own
    const bool single = f.seq_mode || M == 1;
    const MoE* added_moe = nullptr;     // what the next step adds to x: this layer's experts,
    const float* added   = nullptr;     // ... or this sublayer result,
    const hGTensor* scale = nullptr;    // ... times this
    const bool want = want_logits && f.n_rows > 0;
    auto step_of = [&](const TanhNorm* n, void* out) {
        kf_dyt_step d = {};
        d.res = (float*)f.x, d.rows = M, d.dim = E, d.scale_bf16 = scale ? (*scale)->data : nullptr, d.out = out, d.out_f32 = ak;
        if (n) d.w_bf16 = n->w->data, d.b_bf16 = n->b->data, d.alpha_bf16 = n->alpha->data;
        return d;
    };
    auto with_mixes = [&](kf_dyt_step& d, int layer) {
        SeqStateCache::Layer& sl = f.states.layers[layer];
        d.out = s.mid, d.n_mix = kMixes, d.mu_bf16 = BlockOf(f, layer)->wkv->mus.w, d.plane = (size_t)M * E;
        d.tail = sl.tail, d.tail_stride = sl.tail_stride, d.pos = f.d_pos, d.slot = f.d_slot;
    };
    auto add = [&](const kf_dyt_step& d) {
        if (added_moe) return kf_dyt_experts(f.ctx, &d, s.yslots, s.entry_slot, s.wgt, s.hact, added_moe->card.top);
        return kf_dyt_residual(f.ctx, &d, added, E);
    };
    kf_tensor_desc de = f.embed.w->Desc();
    for (int i = 0; i < L; i++) {
        ZdxBlock* blk = BlockOf(f, i);
        // x takes what the layer before left (or the embedding row); the mixer's input n1(x), or its token mixes, on the way
        const bool apart = blk->wkv && !single;
        kf_dyt_step d = step_of(apart ? nullptr : &blk->norm1, s.hact);
        if (blk->wkv && single) with_mixes(d, i);
        if (i == 0) KF_TRY(kf_dyt_embed(f.ctx, &d, &de, f.d_tokens));
        else KF_TRY(add(d));
        if (apart) {
            kf_dyt_step t = step_of(&blk->norm1, nullptr);
            with_mixes(t, i);
            KF_TRY(kf_dyt_token_mix(f.ctx, &t, 1, M));
        }
        if (blk->wkv) {
            KF_TRY(blk->wkv->cuInfer(M, i));
        } else {
            KF_TRY(LinStacked(f, s.u, blk->cat, s.hact, M));  // q | k | v
            KF_TRY(blk->attn->cuInfer(M, s.u, blk->cat.rows, i));
        }
        added = s.sub, added_moe = nullptr, scale = &blk->ls1;
        if (!blk->dense && !blk->moe) continue;
        KF_TRY(add(step_of(&blk->norm2, s.hact)));
        scale = &blk->ls2;
        if (blk->dense) {
            KF_TRY(blk->dense->cuInfer(M));
        } else {
            const int outs = blk->moe->card.experts + blk->moe->card.pass;
            KF_TRY(Lin(f, s.u, outs, blk->moe->router, s.hact, E, M));
            KF_TRY(blk->moe->Route(M, s.u, outs, 0));
            KF_TRY(blk->moe->Experts(M, s.offsets, s.slot_row, s.slot_group));
            added_moe = blk->moe.get();  // combined by the step that adds it
        }
    }
    if (want) {
        const int R = f.n_rows;
        kf_dyt_step d = step_of(&ExtraOf(f)->final_norm, s.head_in);
        d.rows = R, d.row_idx = f.d_sel;
        KF_TRY(add(d));
        KF_TRY(Lin(f, f.logits_f32, c.vocab, f.cls.proj.w, s.head_in, E, R));
        KF_TRY(kf_f32_to_bf16(f.ctx, f.logits, f.logits_f32, (size_t)R * c.vocab));
    }
    return KF_OK;
}

const ARCH_ENTRY* ZadinexArch() {
    static const ARCH_ENTRY e = {"ZADINEX", ParseZadinex, BuildZadinex, ForwardZadinex, PrepareZadinex};
    return &e;
}

}  // namespace koifish
