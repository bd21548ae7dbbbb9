// fekopel_model.cpp — see fekopel_model.h
#include "fekopel_model.h"

#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstdlib>
#include <cstring>

#include "seq_cache.h"

#define FK_OP(name, expr)                        \
    do {                                         \
        ggb_prof_start(name);                    \
        const int rc__ = (expr);                 \
        ggb_prof_stop(name);                     \
        if (rc__ != 0) return fail(rc__, #expr); \
    } while (0)

#define FK_TRY(expr)                             \
    do {                                         \
        const int rc__ = (expr);                 \
        if (rc__ != 0) return fail(rc__, #expr); \
    } while (0)

static const float kSinkScore = 0.f; // of the term that "attention" adds to the soft-max's denominator

int fekopel_model::fail(int rc, const std::string &what) {
    if (err_.empty() || rc != GGB_ERR_ARG) err_ = what + ": " + ggb_last_error();
    return rc;
}

// ------------------------------------------------------------------------------------------------ configuration
int fk_parse_config(const json_value &j, const safetensors_file *file, fk_config *c, std::string *err) {
    auto bad = [&](const std::string &m) {
        if (err) *err = "config.json: " + m;
        return -1;
    };
    // a size the configuration leaves out: dimension `axis` of a tensor, 0 when there is neither
    auto shape_of = [&](const std::string &name, size_t axis) -> long long {
        const st_tensor *t = file ? file->find(name) : nullptr;
        return t && t->shape.size() > axis ? (long long)t->shape[axis] : 0;
    };
    auto object = [](const json_value *v) { return v && v->kind == json_value::OBJ ? v : nullptr; };
    c->vocab = (int)j.integer("vocab", shape_of("embed", 0));
    c->width = (int)j.integer("width", shape_of("embed", 1));
    if (c->vocab <= 0 || c->width <= 0) return bad("vocab and width must be positive");
    if (const json_value *n = object(j.get("norm"))) c->eps = (float)n->number("eps", 1e-5);
    const json_value *layers = j.get("layers");
    if (!layers || layers->kind != json_value::ARR || layers->arr.empty()) return bad("'layers' must be a list");
    for (size_t i = 0; i < layers->arr.size(); i++) {
        const json_value &L = layers->arr[i];
        const std::string where = "layer " + std::to_string(i) + ": ", l0 = "l" + std::to_string(i) + ".", p = l0 + "mix.", q = l0 + "mlp.";
        const std::string type = L.string("type", "");
        if (type != "attention" && type != "attention_2") return bad(where + "unknown mixer type '" + type + "'");
        const json_value *m = object(L.get("mixer"));
        if (!m) return bad(where + "no 'mixer'");
        fk_layer_cfg l;
        fk_mixer_cfg &a = l.mix;
        a.gated = type == "attention_2";
        a.heads = (int)m->integer("heads", 0);
        a.kv_heads = (int)m->integer("kv_heads", a.heads);
        a.dim = (int)m->integer("dim", a.heads > 0 ? shape_of(p + "q", 0) / a.heads : 0);
        a.vdim = (int)m->integer("vdim", a.kv_heads > 0 && shape_of(p + "v", 0) ? shape_of(p + "v", 0) / a.kv_heads : a.dim);
        if (a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dim <= 0 || a.vdim <= 0)
            return bad(where + "mixer sizes must be positive and kv_heads must divide heads");
        if (a.vdim % 2) return bad(where + "vdim must be even");
        if (a.vdim > 256) return bad(where + "vdim above 256 is not built");
        if (a.dim > 512) return bad(where + "dim above 512 is not built");
        a.scale = (float)m->number("scale", 1.0 / std::sqrt((double)a.dim));
        if (const json_value *k = object(m->get("mask"))) {
            a.window = k->integer("size", 0);
            if (a.window < 0) return bad(where + "mask.size must be positive");
        }
        if (a.gated) {
            if (const json_value *k = object(m->get("mask"))) a.keep_first = k->integer("keep_first", 0);
            if (a.keep_first < 0) return bad(where + "mask.keep_first must not be negative");
            if (a.window == 0) a.keep_first = 0; // everything is visible already
            a.softcap = (float)m->number("softcap", 0.0);
            if (a.softcap < 0.f) return bad(where + "softcap must be positive");
            if (const json_value *ro = object(m->get("rot"))) {
                a.rot.dims = (int)ro->integer("dims", a.dim);
                a.rot.base = ro->number("base", 10000.0);
                if (a.rot.dims < 0 || a.rot.dims > a.dim || a.rot.dims % 2) return bad(where + "rot.dims must be even and at most dim");
                if (!(a.rot.base > 0.0)) return bad(where + "rot.base must be positive");
            }
        }
        if (const json_value *f = object(L.get("mlp"))) {
            const std::string kind = f->string("kind", "moe");
            if (kind != "moe") return bad(where + "unknown mlp kind '" + kind + "'");
            fk_moe_cfg &x = l.moe;
            const json_value *e = object(f->get("expert")), *r = object(f->get("router")), *s = object(f->get("shared"));
            if (!r) return bad(where + "a mixture of experts needs a 'router'");
            x.ff = (int)(e ? e->integer("ff", shape_of(q + "e0.up", 0)) : shape_of(q + "e0.up", 0));
            x.experts = (int)r->integer("experts", shape_of(q + "router", 0));
            x.top = (int)r->integer("top", 0);
            x.scale = (float)r->number("scale", 1.0);
            if (x.ff <= 0 || x.experts <= 0 || x.top <= 0 || x.top > x.experts) return bad(where + "experts, ff and top must be positive and top at most experts");
            if (x.experts > 4096 || x.top > GGB_RESIDUAL_MAX_TOP) return bad(where + "more than 4096 experts or 64 a token are not built");
            if (const json_value *g = object(r->get("groups"))) {
                x.groups = (int)g->integer("count", 1);
                x.keep = (int)g->integer("keep", x.groups);
            }
            if (x.groups <= 0 || x.experts % x.groups || x.keep <= 0 || x.keep > x.groups || x.top > x.keep * (x.experts / x.groups))
                return bad(where + "groups.count must divide the experts and the groups that stay must hold 'top' experts");
            if (s) {
                x.shared_ff = (int)s->integer("ff", shape_of(q + "shared.up", 0));
                if (x.shared_ff <= 0) return bad(where + "shared.ff must be positive");
            }
        }
        c->layers.push_back(l);
    }
    const int n = (int)c->layers.size();
    if (const json_value *lp = object(j.get("loop"))) {
        c->loop_start = (int)lp->integer("start", 0);
        c->loop_stop = (int)lp->integer("stop", n);
        c->loop_times = (int)lp->integer("times", shape_of("loop.step", 0) ? shape_of("loop.step", 0) : 1);
        if (c->loop_start < 0 || c->loop_stop <= c->loop_start || c->loop_stop > n || c->loop_times < 1)
            return bad("loop needs 0 <= start < stop <= layers and times >= 1");
    }
    c->runs.clear();
    for (int i = 0; i < n;) {
        if (c->loop_times > 0 && i == c->loop_start) {
            for (int t = 0; t < c->loop_times; t++)
                for (int k = c->loop_start; k < c->loop_stop; k++) c->runs.push_back(fk_run{k, k == c->loop_start ? t : -1});
            i = c->loop_stop;
        } else {
            c->runs.push_back(fk_run{i++, -1});
        }
    }
    return 0;
}

void fk_lookback(const fk_config &c, int64_t *lookback, int64_t *keep_first) {
    *lookback = *keep_first = 0;
    for (const fk_layer_cfg &l : c.layers) {
        if (l.mix.window <= 0) {
            *lookback = *keep_first = 0;
            return;
        }
        *lookback = std::max(*lookback, l.mix.window);
        *keep_first = std::max(*keep_first, l.mix.keep_first);
    }
}

// ------------------------------------------------------------------------------------------------ weights
int fekopel_model::upload_matrix(const std::vector<float> &host, void **dev) {
    const size_t n = host.size();
    void *d = nullptr;
    FK_TRY(ggb_buffer_alloc(std::max<size_t>(n, 8) * ggb_dtype_size(dt_), &d));
    owned_.push_back(d);
    if (dt_ == GGB_TYPE_BF16) {
        std::vector<uint16_t> h(n);
        for (size_t i = 0; i < n; i++) h[i] = f32_to_bf16(host[i]);
        FK_TRY(ggb_upload(d, h.data(), n * 2));
        FK_TRY(ggb_sync());
    } else {
        FK_TRY(ggb_upload(d, host.data(), n * 4));
        FK_TRY(ggb_sync());
    }
    weight_bytes_ += n * ggb_dtype_size(dt_);
    *dev = d;
    return 0;
}

int fekopel_model::upload_f32(const std::vector<float> &host, float **dev) {
    void *d = nullptr;
    FK_TRY(ggb_buffer_alloc(std::max<size_t>(host.size(), 4) * 4, &d));
    owned_.push_back(d);
    FK_TRY(ggb_upload(d, host.data(), host.size() * 4));
    FK_TRY(ggb_sync());
    weight_bytes_ += host.size() * 4;
    *dev = (float *)d;
    return 0;
}

int fekopel_model::load(const safetensors_file *file, uint64_t seed) {
    const fk_config &c = cfg_;
    const int64_t W = c.width, V = c.vocab;
    weight_source src{file, seed, &err_};
    std::vector<float> a, b;
#define FK_GET(...)                                   \
    do {                                              \
        if (src.get(__VA_ARGS__)) return GGB_ERR_ARG; \
    } while (0)
#define FK_F32(name, n, amp, mean, dst)    \
    do {                                   \
        FK_GET(name, 1, n, amp, mean, &a); \
        FK_TRY(upload_f32(a, dst));        \
    } while (0)
#define FK_NORM(name, w, bias)                      \
    do {                                            \
        FK_F32(name, W, 0.1f, 1.0f, w);             \
        FK_F32((name) + ".b", W, 0.1f, 0.f, bias);  \
    } while (0)
    const float aw = std::sqrt(3.0f / (float)W);
    auto amp = [](int64_t fan_in) { return std::sqrt(3.0f / (float)fan_in); };
    FK_GET("embed", V, W, 1.7f, 0.f, &a);
    FK_TRY(upload_matrix(a, &embed_));
    FK_GET("head", V, W, aw, 0.f, &a);
    FK_TRY(upload_matrix(a, &head_));
    FK_NORM(std::string("final.norm"), &final_norm_, &final_normb_);
    if (c.loop_times > 0) {
        FK_GET("loop.step", c.loop_times, W, 0.5f, 0.f, &a);
        FK_TRY(upload_f32(a, &loop_step_));
    }
    lw_.assign(c.layers.size(), fk_layer_w());
    // stacks `name` (rows x W) below what `stack` already holds; returns the row it starts at
    std::vector<float> stack;
    auto push = [&](const std::string &name, int64_t rows, int64_t *at) -> int {
        if (at) *at = (int64_t)(stack.size() / (size_t)W);
        if (src.get(name, rows, W, aw, 0.f, &b)) return GGB_ERR_ARG;
        stack.insert(stack.end(), b.begin(), b.end());
        return 0;
    };
    int hmax = 1;
    for (size_t li = 0; li < c.layers.size(); li++) {
        const fk_mixer_cfg &A = c.layers[li].mix;
        const fk_moe_cfg &E = c.layers[li].moe;
        fk_layer_w &w = lw_[li];
        const std::string p = "l" + std::to_string(li) + ".", m = p + "mix.", f = p + "mlp.";
        const int64_t H = A.heads, G = A.kv_heads, D = A.dim, Dv = A.vdim;
        hmax = std::max(hmax, A.heads);
        FK_NORM(p + "norm1", &w.norm1, &w.norm1b);
        stack.clear();
        FK_TRY(push(m + "q", H * D, nullptr));
        FK_TRY(push(m + "k", G * D, &w.o_k));
        FK_TRY(push(m + "v", G * Dv, &w.o_v));
        if (A.gated) {
            FK_TRY(push(m + "g", H * Dv, &w.o_g));
            FK_F32(m + "q.norm", D, 0.1f, 1.0f, &w.q_norm);
            FK_F32(m + "k.norm", D, 0.1f, 1.0f, &w.k_norm);
        }
        w.n_proj = ((int64_t)(stack.size() / (size_t)W) + 31) / 32 * 32; // whole tiles for the tensor-core product
        stack.resize((size_t)(w.n_proj * W), 0.f);
        FK_TRY(upload_matrix(stack, &w.proj));
        FK_GET(m + "o", W, H * Dv, amp(H * Dv), 0.f, &a);
        FK_TRY(upload_matrix(a, &w.o));
        if (E.experts > 0) {
            FK_NORM(p + "norm2", &w.norm2, &w.norm2b);
            std::vector<float> up, dn;
            up.reserve((size_t)E.experts * (size_t)E.ff * (size_t)W);
            dn.reserve((size_t)E.experts * (size_t)E.ff * (size_t)W);
            for (int e = 0; e < E.experts; e++) {
                const std::string q = f + "e" + std::to_string(e) + ".";
                FK_GET(q + "up", E.ff, W, aw, 0.f, &a);
                up.insert(up.end(), a.begin(), a.end());
                FK_GET(q + "down", W, E.ff, amp(E.ff), 0.f, &a);
                dn.insert(dn.end(), a.begin(), a.end());
            }
            FK_TRY(upload_matrix(up, &w.e_up));
            FK_TRY(upload_matrix(dn, &w.e_down));
            std::vector<float> rt;
            FK_GET(f + "router", E.experts, W, aw, 0.f, &rt);
            if (E.shared_ff > 0) {
                FK_GET(f + "shared.up", E.shared_ff, W, aw, 0.f, &a);
                FK_TRY(upload_matrix(a, &w.s_up));
                FK_GET(f + "shared.down", W, E.shared_ff, amp(E.shared_ff), 0.f, &a);
                FK_TRY(upload_matrix(a, &w.s_down));
                FK_GET(f + "shared.sg", 1, W, aw, 0.f, &a);
                rt.insert(rt.end(), a.begin(), a.end()); // the gate reads what the router reads: one more row
            }
            FK_TRY(upload_f32(rt, &w.router));
        }
    }
#undef FK_GET
#undef FK_F32
#undef FK_NORM
    FK_TRY(upload_f32(std::vector<float>((size_t)hmax, kSinkScore), &sinks_));
    fk_lookback(c, &lookback_, &keep_first_);
    return 0;
}

lm_model *fekopel_model::create(const std::string &dir, const json_value &cfg, const lm_load_options &opt, std::string *err) {
    fekopel_model *m = new fekopel_model();
    safetensors_file file;
    m->dt_ = opt.dtype;
    if (opt.max_portion > 0) m->max_T_ = opt.max_portion;
    int rc = 0;
    if (!ggb_dtype_size(m->dt_)) rc = -1, m->err_ = "Fekopel runs in bfloat16 or float32";
    if (!rc && !opt.random_weights) rc = file.open(dir + "/model.safetensors", &m->err_);
    if (!rc) rc = fk_parse_config(cfg, opt.random_weights ? nullptr : &file, &m->cfg_, &m->err_);
    if (!rc) rc = m->load(opt.random_weights ? nullptr : &file, opt.seed);
    if (rc) {
        if (err) *err = m->err_;
        delete m;
        return nullptr;
    }
    return m;
}

fekopel_model::~fekopel_model() {
    ggb_sync();
    for (step_graph &g : graphs_) ggb_graph_free(g.graph);
    for (void *p : owned_) ggb_buffer_free(p);
}

std::vector<int64_t> fekopel_model::cache_row_elems() const {
    std::vector<int64_t> v;
    for (const fk_run &r : cfg_.runs) {
        const fk_mixer_cfg &a = cfg_.layers[(size_t)r.layer].mix;
        v.push_back(ggb_window_cache_ld(a.kv_heads, a.dim, a.vdim));
    }
    return v;
}

// ------------------------------------------------------------------------------------------------ buffers
int fekopel_model::alloc_scratch() {
    const fk_config &c = cfg_;
    const int64_t T = max_T_, W = c.width;
    int64_t npr = 0, nq = 0, nao = 0, slots = 0, ffs = 0, sff = 0, ints = 0, nz = 0;
    int hmax = 1;
    for (size_t li = 0; li < c.layers.size(); li++) {
        const fk_mixer_cfg &A = c.layers[li].mix;
        const fk_moe_cfg &E = c.layers[li].moe;
        npr = std::max(npr, lw_[li].n_proj);
        nq = std::max(nq, (int64_t)A.heads * A.dim);
        nao = std::max(nao, (int64_t)A.heads * A.vdim);
        hmax = std::max(hmax, A.heads);
        if (E.experts > 0) {
            slots = std::max(slots, T * E.top);
            ffs = std::max(ffs, T * E.top * E.ff);
            sff = std::max(sff, T * E.shared_ff);
            ints = std::max(ints, (int64_t)ggb_moe_group_ints(T * E.top, E.experts));
            nz = std::max(nz, (int64_t)E.experts + 1);
        }
    }
    const size_t es = ggb_dtype_size(dt_);
    auto alloc = [&](size_t bytes, void **p) -> int {
        FK_TRY(ggb_buffer_alloc(std::max<size_t>(bytes, 16), p));
        owned_.push_back(*p);
        return 0;
    };
#define FK_ALLOC(ptr, bytes) FK_TRY(alloc((size_t)(bytes), (void **)&(ptr)))
    FK_ALLOC(ids_, T * 4);
    FK_ALLOC(want_, T * 4);
    FK_ALLOC(pos0_, 16);
    FK_ALLOC(x_, T * W * 4);
    FK_ALLOC(h_, T * W * es);
    FK_ALLOC(pr_, T * npr * 4);
    FK_ALLOC(qr_, T * nq * 4);
    FK_ALLOC(ao_, T * nao * es);
    FK_ALLOC(wa_, ggb_window_attn_scratch_bytes(hmax));
    FK_ALLOC(ya_, T * W * 4);
    FK_ALLOC(y2_, slots * W * 4);
    FK_ALLOC(ys_, (sff > 0 ? T * W : 0) * 4);
    FK_ALLOC(act_, ffs * es);
    FK_ALLOC(acts_, sff * es);
    FK_ALLOC(route_z_, T * nz * 4);
    FK_ALLOC(route_i_, slots * 4);
    FK_ALLOC(route_w_, slots * 4);
    FK_ALLOC(group_ws_, ints * 4);
    FK_ALLOC(hw_, T * W * es);
    FK_ALLOC(logits_, T * (int64_t)c.vocab * 4);
#undef FK_ALLOC
    return 0;
}

int fekopel_model::bind_cache(paged_cache *cache, int64_t max_positions) {
    cache_ = cache;
    max_pos_ = max_positions;
    if ((int)cfg_.runs.size() != cache->n_layers()) return fail(GGB_ERR_ARG, "the cache has another number of layers than the model has layer runs");
    for (size_t li = 0; li < cfg_.layers.size(); li++) {
        const rot_spec &r = cfg_.layers[li].mix.rot;
        if (r.dims <= 0) continue;
        const std::string k = r.key();
        if (!rot_tables_.count(k)) {
            float *d = nullptr;
            FK_TRY(upload_f32(rot_table(r, max_positions), &d));
            rot_tables_[k] = d;
        }
        lw_[li].cs = rot_tables_[k];
    }
    return alloc_scratch();
}

// ------------------------------------------------------------------------------------------------ one portion
int fekopel_model::emit(int T, const int32_t *table, int n_want) {
    const fk_config &c = cfg_;
    const int64_t W = c.width, t = T;
    const int B = cache_->page_size();
    // a sublayer's output waits for the next pass over the residual: that pass adds it (for a mixture of experts it takes the weighted
    // sum), adds what a pass of the looped block starts with, and norms the row for the next sublayer
    bool started = false;
    const float *y = nullptr;
    const fk_moe_cfg *slots = nullptr;
    int64_t ldz = 0;
    auto residual = [&](const fk_run *begins, const float *nw, const float *nb, const int32_t *rows, int64_t n, float *x_out, void *h) -> int {
        const bool again = begins && begins->pass > 0, shared = slots && slots->shared_ff > 0;
        const void *emb = !started || again ? embed_ : nullptr;
        FK_OP("op_residual", ggb_op_residual_layer_norm(dt_, started ? x_ : nullptr, y, slots ? y2_ : nullptr, group_ws_, route_w_, t, slots ? slots->top : 0,
                                                        slots ? slots->experts : 0, shared ? ys_ : nullptr, shared ? route_z_ + slots->experts : nullptr, ldz, emb, ids_,
                                                        begins && begins->pass >= 0 ? loop_step_ + (int64_t)begins->pass * W : nullptr, nw, nb, c.eps, W, n, rows,
                                                        x_out, h));
        return 0;
    };
    auto taken = [&]() { started = true, y = nullptr, slots = nullptr; };
    for (size_t ri = 0; ri < c.runs.size(); ri++) {
        const fk_run &r = c.runs[ri];
        const fk_mixer_cfg &A = c.layers[(size_t)r.layer].mix;
        const fk_moe_cfg &E = c.layers[(size_t)r.layer].moe;
        const fk_layer_w &w = lw_[(size_t)r.layer];
        const int64_t N = w.n_proj, HV = (int64_t)A.heads * A.vdim;
        FK_TRY(residual(&r, w.norm1, w.norm1b, nullptr, t, x_, h_));
        taken();
        void *cache = cache_->layer((int)ri);
        FK_OP("op_linear", ggb_op_linear(dt_, w.proj, N, W, h_, W, t, pr_, N));
        FK_OP("op_attn_prep", ggb_op_head_qkv_store(dt_, pr_, pr_ + w.o_k, pr_ + w.o_v, N, t, A.heads, A.kv_heads, A.dim, A.vdim, w.q_norm, w.k_norm, c.eps,
                                                    A.rot.dims, 1, w.cs, A.scale, pos0_, table, B, cache, qr_));
        FK_OP("op_attn", ggb_op_masked_attn_gated(dt_, qr_, cache, table, B, pos0_, t, A.heads, A.kv_heads, A.dim, A.vdim, A.window, A.keep_first, A.softcap,
                                                  A.gated ? nullptr : sinks_, A.gated ? pr_ + w.o_g : nullptr, N, ao_, wa_));
        FK_OP("op_linear", ggb_op_linear(dt_, w.o, W, HV, ao_, HV, t, ya_, W));
        y = ya_;
        if (E.experts > 0) {
            FK_TRY(residual(nullptr, w.norm2, w.norm2b, nullptr, t, x_, h_));
            taken();
            const int extra = E.shared_ff > 0 ? 1 : 0;
            ldz = E.experts + extra;
            FK_OP("op_moe", ggb_op_moe_route_softmax_groups(dt_, h_, W, t, w.router, nullptr, E.experts, extra, E.top, E.groups, E.keep, E.scale, route_z_, route_i_,
                                                            route_w_, group_ws_));
            // a step of few slots: the router has listed them
            if (!ggb_moe_step_form(t * E.top)) FK_OP("op_moe", ggb_op_moe_group(route_i_, t, E.top, E.experts, group_ws_));
            if (extra) {
                FK_OP("op_moe_linear", ggb_op_moe_linear_shared(dt_, w.e_up, E.ff, W, h_, W, 1, t, E.top, E.experts, group_ws_, GGB_ACT_GELU_ERF, act_, E.ff, w.s_up,
                                                                E.shared_ff, W, h_, W, acts_));
                FK_OP("op_moe_linear", ggb_op_moe_linear_shared(dt_, w.e_down, W, E.ff, act_, E.ff, 0, t, E.top, E.experts, group_ws_, GGB_ACT_NONE, y2_, W, w.s_down, W,
                                                                E.shared_ff, acts_, E.shared_ff, ys_));
            } else {
                FK_OP("op_moe_linear", ggb_op_moe_linear(dt_, w.e_up, E.ff, W, h_, W, 1, t, E.top, E.experts, group_ws_, GGB_ACT_GELU_ERF, act_, E.ff));
                FK_OP("op_moe_linear", ggb_op_moe_linear(dt_, w.e_down, W, E.ff, act_, E.ff, 0, t, E.top, E.experts, group_ws_, GGB_ACT_NONE, y2_, W));
            }
            slots = &E;
        }
        if (capture_ && cap_) FK_TRY(residual(nullptr, nullptr, nullptr, nullptr, t, cap_ + ri * (size_t)max_T_ * (size_t)W, nullptr));
    }
    if (n_want > 0) { // the last sublayer's output enters on the way: only the wanted rows are computed
        FK_TRY(residual(nullptr, final_norm_, final_normb_, want_, n_want, nullptr, hw_));
        FK_OP("op_linear", ggb_op_linear(dt_, head_, c.vocab, W, hw_, W, n_want, logits_, c.vocab));
    }
    return 0;
}

int fekopel_model::forward(const lm_portion &p, const int32_t *want, int n_want) {
    if (!cache_) return fail(GGB_ERR_ARG, "forward before bind_cache");
    if (p.T <= 0 || p.T > max_T_ || n_want < 0 || n_want > p.T || p.pos0 < 0 || p.pos0 + p.T > max_pos_) {
        err_ = "forward: a portion of " + std::to_string(p.T) + " tokens at position " + std::to_string(p.pos0) + " does not fit";
        return GGB_ERR_ARG;
    }
    for (int i = 0; i < p.T; i++)
        if (p.tokens[i] < 0 || p.tokens[i] >= cfg_.vocab) {
            err_ = "forward: token " + std::to_string(p.tokens[i]) + " is outside the vocabulary";
            return GGB_ERR_ARG;
        }
    const int32_t pos0 = (int32_t)p.pos0;
    FK_TRY(ggb_upload(ids_, p.tokens, (size_t)p.T * 4));
    FK_TRY(ggb_upload(pos0_, &pos0, 4));
    if (n_want) FK_TRY(ggb_upload(want_, want, (size_t)n_want * 4));
    const int64_t l0 = ggb_launch_count();
    if (capture_) {
        if (!cap_) {
            void *d = nullptr;
            FK_TRY(ggb_buffer_alloc(cfg_.runs.size() * (size_t)max_T_ * (size_t)cfg_.width * 4, &d));
            owned_.push_back(d);
            cap_ = (float *)d;
        }
        cap_T_ = p.T;
    }
    if (p.T == 1 && use_graphs_ && !capture_ && !getenv("GGB_NO_STEP_GRAPH")) {
        ggb_graph *g = nullptr;
        for (const step_graph &sg : graphs_)
            if (sg.table == p.block_table_dev && sg.n_want == n_want) g = sg.graph;
        if (!g) {
            FK_TRY(ggb_capture_begin());
            const int rc = emit(1, p.block_table_dev, n_want);
            const int rc2 = ggb_capture_end(&g);
            if (rc) return rc;
            if (rc2) return fail(rc2, "ggb_capture_end");
            if (graphs_.size() >= 32) {
                ggb_graph_free(graphs_.front().graph);
                graphs_.erase(graphs_.begin());
            }
            graphs_.push_back(step_graph{p.block_table_dev, n_want, g});
        }
        FK_TRY(ggb_graph_launch(g));
    } else {
        FK_TRY(emit(p.T, p.block_table_dev, n_want));
    }
    kernels_last_ = (int)(ggb_launch_count() - l0);
    return 0;
}

int fekopel_model::get_capture(int run, float *host, int64_t n) const {
    if (!cap_ || run < 0 || run >= (int)cfg_.runs.size() || n > (int64_t)cap_T_ * cfg_.width) return GGB_ERR_ARG;
    return ggb_download(host, cap_ + (size_t)run * (size_t)max_T_ * (size_t)cfg_.width, (size_t)n * 4);
}

namespace {
struct register_fekopel {
    register_fekopel() { lm_register("Fekopel", &fekopel_model::create); }
} g_register_fekopel;
} // namespace
