// tezesun_model.cpp — see tezesun_model.h
#include "tezesun_model.h"

#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstdlib>
#include <cstring>

#include "seq_cache.h"

#define TZ_OP(name, expr)                        \
    do {                                         \
        ggb_prof_start(name);                    \
        const int rc__ = (expr);                 \
        ggb_prof_stop(name);                     \
        if (rc__ != 0) return fail(rc__, #expr); \
    } while (0)

#define TZ_TRY(expr)                             \
    do {                                         \
        const int rc__ = (expr);                 \
        if (rc__ != 0) return fail(rc__, #expr); \
    } while (0)

static const double kDecayRate = 8.0; // log a = -8 r softplus(lam)

int tezesun_model::fail(int rc, const std::string &what) {
    if (err_.empty() || rc != GGB_ERR_ARG) err_ = what + ": " + ggb_last_error();
    return rc;
}

// ------------------------------------------------------------------------------------------------ configuration
static int parse_rot(const json_value *ro, int head_dims, rot_spec *rot, std::string *why) {
    if (!ro || ro->kind != json_value::OBJ) return 0;
    rot->dims = (int)ro->integer("dims", head_dims);
    rot->base = ro->number("base", 10000.0);
    if (rot->dims < 0 || rot->dims > head_dims || rot->dims % 2) return *why = "rot.dims must be even and at most the rotated size", -1;
    if (!(rot->base > 0.0)) return *why = "rot.base must be positive", -1;
    const json_value *s = ro->get("scaling");
    if (s && s->kind == json_value::OBJ) {
        rot->scaled = true;
        rot->factor = s->number("factor", 1.0);
        rot->original = s->number("original", 0.0);
        rot->fast = s->number("fast", 32.0);
        rot->slow = s->number("slow", 1.0);
        if (!(rot->factor > 0.0) || !(rot->original > 0.0) || !(rot->fast > 0.0) || !(rot->slow > 0.0))
            return *why = "rot.scaling needs factor, original, fast and slow above 0", -1;
    }
    return 0;
}

int tz_parse_config(const json_value &j, const safetensors_file *file, tz_config *c, std::string *err) {
    auto bad = [&](const std::string &m) {
        if (err) *err = "config.json: " + m;
        return -1;
    };
    c->vocab = (int)j.integer("vocab", 0);
    c->width = (int)j.integer("width", 0);
    if (c->vocab <= 0 || c->width <= 0) return bad("vocab and width must be positive");
    if (const json_value *n = j.get("norm")) c->eps = (float)n->number("eps", 1e-6);
    c->logit_scale = j.number("logit_scale", 1.0);
    const json_value *layers = j.get("layers");
    if (!layers || layers->kind != json_value::ARR || layers->arr.empty()) return bad("'layers' must be a list");
    for (size_t i = 0; i < layers->arr.size(); i++) {
        const json_value &L = layers->arr[i];
        const std::string where = "layer " + std::to_string(i) + ": ", p = "l" + std::to_string(i) + ".mix.";
        const std::string type = L.string("type", "");
        const json_value *m = L.get("mixer");
        if (!m || m->kind != json_value::OBJ) return bad(where + "no 'mixer'");
        tz_layer_cfg l;
        std::string why;
        if (type == "attention") {
            l.type = 0;
            tz_attn_cfg &a = l.attn;
            a.heads = (int)m->integer("heads", 0);
            a.kv_heads = (int)m->integer("kv_heads", a.heads);
            a.dim = (int)m->integer("dim", 0);
            a.vdim = (int)m->integer("vdim", a.dim);
            if (a.heads <= 0 || a.kv_heads <= 0 || a.heads % a.kv_heads || a.dim <= 0 || a.vdim <= 0)
                return bad(where + "mixer sizes must be positive and kv_heads must divide heads");
            if (a.dim % 2 || a.vdim % 2) return bad(where + "dim and vdim must be even");
            if (a.vdim > 256) return bad(where + "vdim above 256 is not built");
            a.scale = (float)m->number("scale", 1.0 / std::sqrt((double)a.dim));
            a.softcap = (float)m->number("softcap", 0.0);
            if (a.softcap < 0.f) return bad(where + "softcap must be positive");
            if (!m->get("diff")) return bad(where + "no 'diff'");
            a.diff = m->number("diff", 0.0);
            const json_value *k = m->get("mask");
            if (k && k->kind == json_value::OBJ) {
                a.window = k->integer("size", 0);
                a.keep_first = k->integer("keep_first", 0);
                if (a.window < 0 || a.keep_first < 0) return bad(where + "mask.size and mask.keep_first must not be negative");
                if (a.window == 0) a.keep_first = 0; // everything is visible already
            }
            if (parse_rot(m->get("rot"), a.dim, &a.rot, &why)) return bad(where + why);
        } else if (type == "latent_attention") {
            l.type = 1;
            tz_latent_cfg &a = l.latent;
            a.heads = (int)m->integer("heads", 0);
            a.dim = (int)m->integer("dim", 0);
            a.rot_dim = (int)m->integer("rot_dim", 0);
            a.vdim = (int)m->integer("vdim", a.dim);
            a.kv_rank = (int)m->integer("kv_rank", 0);
            a.q_rank = (int)m->integer("q_rank", 0);
            if (a.q_rank == 0 && file) { // not configured: as many as the file's down-projection has rows
                const st_tensor *t = file->find(p + "dq");
                if (t && t->shape.size() == 2) a.q_rank = (int)t->shape[0];
            }
            if (a.heads <= 0 || a.dim <= 0 || a.rot_dim < 0 || a.vdim <= 0 || a.kv_rank <= 0 || a.q_rank <= 0)
                return bad(where + "heads, dim, vdim, kv_rank and q_rank must be positive");
            if (a.kv_rank > 1024) return bad(where + "kv_rank above 1024 is not built");
            if (a.dim > 1024) return bad(where + "dim above 1024 is not built");
            a.scale = (float)m->number("scale", 1.0 / std::sqrt((double)(a.dim + a.rot_dim)));
            if (parse_rot(m->get("rot"), a.rot_dim, &a.rot, &why)) return bad(where + why);
        } else if (type == "rglru") {
            l.type = 2;
            tz_rglru_cfg &r = l.rec;
            r.width = (int)m->integer("width", 0);
            r.blocks = (int)m->integer("blocks", 1);
            r.conv = (int)m->integer("conv", 1);
            if (r.width <= 0 || r.blocks <= 0 || r.width % r.blocks) return bad(where + "blocks must divide width");
            if (r.conv < 1 || r.conv > 8) return bad(where + "conv must be between 1 and 8 taps");
        } else {
            return bad(where + "unknown mixer type '" + type + "'");
        }
        const json_value *f = L.get("mlp");
        if (f && f->kind == json_value::OBJ) {
            const std::string kind = f->string("kind", "");
            if (kind != "dense") return bad(where + "unknown mlp kind '" + kind + "'");
            l.ff = (int)f->integer("ff", 0);
            if (l.ff <= 0) return bad(where + "ff must be positive");
        }
        c->layers.push_back(l);
    }
    return 0;
}

void tz_lookback(const tz_config &c, int64_t *lookback, int64_t *keep_first) {
    *lookback = *keep_first = 0;
    for (const tz_layer_cfg &l : c.layers) {
        if (l.type == 2) continue; // no rows per position
        if (l.type == 1 || l.attn.window <= 0) {
            *lookback = *keep_first = 0;
            return;
        }
        *lookback = std::max(*lookback, l.attn.window);
        *keep_first = std::max(*keep_first, l.attn.keep_first);
    }
}

// ------------------------------------------------------------------------------------------------ weights
int tezesun_model::upload_matrix(const std::vector<float> &host, void **dev) {
    const size_t n = host.size();
    void *d = nullptr;
    TZ_TRY(ggb_buffer_alloc(std::max<size_t>(n, 8) * ggb_dtype_size(dt_), &d));
    owned_.push_back(d);
    if (dt_ == GGB_TYPE_BF16) {
        std::vector<uint16_t> h(n);
        for (size_t i = 0; i < n; i++) h[i] = f32_to_bf16(host[i]);
        TZ_TRY(ggb_upload(d, h.data(), n * 2));
        TZ_TRY(ggb_sync());
    } else {
        TZ_TRY(ggb_upload(d, host.data(), n * 4));
        TZ_TRY(ggb_sync());
    }
    weight_bytes_ += n * ggb_dtype_size(dt_);
    *dev = d;
    return 0;
}

int tezesun_model::upload_f32(const std::vector<float> &host, float **dev) {
    void *d = nullptr;
    TZ_TRY(ggb_buffer_alloc(std::max<size_t>(host.size(), 4) * 4, &d));
    owned_.push_back(d);
    TZ_TRY(ggb_upload(d, host.data(), host.size() * 4));
    TZ_TRY(ggb_sync());
    weight_bytes_ += host.size() * 4;
    *dev = (float *)d;
    return 0;
}

static double softplus(double z) { return z > 30.0 ? z : std::log1p(std::exp(z)); }

int tezesun_model::load(const safetensors_file *file, uint64_t seed) {
    const tz_config &c = cfg_;
    const int64_t W = c.width, V = c.vocab;
    weight_source src{file, seed, &err_};
    std::vector<float> a, b;
#define TZ_GET(...)                                   \
    do {                                              \
        if (src.get(__VA_ARGS__)) return GGB_ERR_ARG; \
    } while (0)
#define TZ_F32(name, n, amp, mean, dst)    \
    do {                                   \
        TZ_GET(name, 1, n, amp, mean, &a); \
        TZ_TRY(upload_f32(a, dst));        \
    } while (0)
    const float aw = std::sqrt(3.0f / (float)W);
    auto amp = [](int64_t fan_in) { return std::sqrt(3.0f / (float)fan_in); };
    TZ_GET("embed", V, W, 1.7f, 0.f, &a);
    TZ_TRY(upload_matrix(a, &embed_));
    TZ_GET("head", V, W, aw, 0.f, &a);
    TZ_TRY(upload_matrix(a, &head_));
    TZ_GET("final.norm", 1, W, 0.1f, 1.0f, &a);
    for (float &v : a) v = (float)((double)v * c.logit_scale); // the logits' factor rides on the last norm
    TZ_TRY(upload_f32(a, &final_norm_));
    lw_.assign(c.layers.size(), tz_layer_w());
    // stacks `name` (rows x W) below what `stack` already holds; returns the row it starts at
    std::vector<float> stack;
    auto push = [&](const std::string &name, int64_t rows, int64_t *at) -> int {
        if (at) *at = (int64_t)(stack.size() / (size_t)W);
        if (src.get(name, rows, W, aw, 0.f, &b)) return GGB_ERR_ARG;
        stack.insert(stack.end(), b.begin(), b.end());
        return 0;
    };
    int64_t st = 0;
    auto take = [&](int64_t n) {
        const int64_t at = st;
        st += (n + 3) / 4 * 4;
        return at;
    };
    int n_cache = 0;
    for (size_t li = 0; li < c.layers.size(); li++) {
        const tz_layer_cfg &l = c.layers[li];
        tz_layer_w &w = lw_[li];
        const std::string p = "l" + std::to_string(li) + ".", q = p + "mix.";
        TZ_F32(p + "norm1", W, 0.1f, 1.0f, &w.norm1);
        TZ_F32(p + "ls1", W, 0.1f, 0.5f, &w.ls1);
        TZ_F32(p + "shift", W, 0.3f, 0.3f, &w.shift);
        w.s_h = take(W);
        stack.clear();
        if (l.type == 0) {
            const tz_attn_cfg &A = l.attn;
            const int64_t H = A.heads, G = A.kv_heads, D = A.dim, Dv = A.vdim;
            TZ_TRY(push(q + "q", 2 * H * D, nullptr));
            TZ_TRY(push(q + "k", 2 * G * D, &w.o1));
            TZ_TRY(push(q + "v", G * Dv, &w.o2));
            TZ_TRY(push(q + "g", H * Dv, &w.o3));
            double s[2];
            for (int k = 0; k < 2; k++) {
                const std::string n = std::to_string(k + 1);
                TZ_GET(q + "lq" + n, 1, D, 0.1f, 0.f, &a);
                TZ_GET(q + "lk" + n, 1, D, 0.1f, 0.f, &b);
                s[k] = 0.0;
                for (int64_t i = 0; i < D; i++) s[k] += (double)a[(size_t)i] * (double)b[(size_t)i];
            }
            w.lambda = (float)(std::exp(s[0]) - std::exp(s[1]) + A.diff);
            w.k_o = H * Dv;
            w.cache_index = n_cache++;
        } else if (l.type == 1) {
            const tz_latent_cfg &A = l.latent;
            const int64_t H = A.heads, D = A.dim, Dr = A.rot_dim, Dv = A.vdim, R = A.kv_rank, Rq = A.q_rank;
            TZ_TRY(push(q + "dq", Rq, nullptr));
            TZ_TRY(push(q + "dkv", R + Dr, &w.o1));
            TZ_F32(q + "dq.norm", Rq, 0.1f, 1.0f, &w.dq_norm);
            TZ_F32(q + "dkv.norm", R, 0.1f, 1.0f, &w.dkv_norm);
            TZ_GET(q + "uq", H * (D + Dr), Rq, amp(Rq), 0.f, &a);
            TZ_TRY(upload_matrix(a, &w.uq));
            // keys' and values' up-projections below one another: one product when they are materialised
            TZ_GET(q + "uk", H * D, R, amp(R), 0.f, &a);
            TZ_GET(q + "uv", H * Dv, R, amp(R), 0.f, &b);
            a.insert(a.end(), b.begin(), b.end());
            TZ_TRY(upload_matrix(a, &w.ukv));
            w.uk = w.ukv;
            w.uv = (char *)w.ukv + (size_t)(H * D * R) * ggb_dtype_size(dt_);
            w.k_o = H * Dv;
            w.cache_index = n_cache++;
        } else {
            const tz_rglru_cfg &R = l.rec;
            const int64_t C = R.width, nb = R.blocks, d = C / nb;
            TZ_TRY(push(q + "x", C, nullptr));
            TZ_TRY(push(q + "y", C, &w.o1));
            TZ_F32(q + "x.b", C, 0.1f, 0.f, &w.xb);
            TZ_F32(q + "y.b", C, 0.1f, 0.f, &w.yb);
            TZ_GET(q + "conv", C, R.conv, 0.5f, 0.f, &a);
            TZ_TRY(upload_f32(a, &w.conv));
            TZ_F32(q + "conv.b", C, 0.1f, 0.f, &w.conv_b);
            // per block the rows of both gates below one another
            std::vector<float> ra, ri, rab, rib, w2, w3, b2;
            TZ_GET(q + "ra", nb * d, d, amp(d), 0.f, &ra);
            TZ_GET(q + "ri", nb * d, d, amp(d), 0.f, &ri);
            TZ_GET(q + "ra.b", 1, C, 1.0f, -1.0f, &rab);
            TZ_GET(q + "ri.b", 1, C, 1.0f, 0.f, &rib);
            const bool split = ggb_rglru_split_fits(dt_, 1 << 20, (int)d) != 0;
            for (int64_t k = 0; k < nb; k++)
                for (int g = 0; g < 2; g++) {
                    const std::vector<float> &m = g ? ri : ra, &mb = g ? rib : rab;
                    b2.insert(b2.end(), mb.begin() + (ptrdiff_t)(k * d), mb.begin() + (ptrdiff_t)((k + 1) * d));
                    for (int64_t n = k * d; n < (k + 1) * d; n++) {
                        const auto r0 = m.begin() + (ptrdiff_t)(n * d), r1 = r0 + (ptrdiff_t)d;
                        w2.insert(w2.end(), r0, r1);
                        for (int rep = 0; split && rep < 3; rep++) w3.insert(w3.end(), r0, r1);
                    }
                }
            TZ_TRY(upload_matrix(w2, &w.w_ri));
            if (split) TZ_TRY(upload_matrix(w3, &w.w_ri3));
            TZ_TRY(upload_f32(b2, &w.b_ri));
            TZ_GET(q + "lam", 1, C, 1.0f, -2.0f, &a);
            for (float &v : a) v = (float)(-kDecayRate * softplus((double)v));
            TZ_TRY(upload_f32(a, &w.rate));
            w.k_o = C;
            w.s_hist = take((int64_t)ggb_rglru_history_rows(R.conv) * C);
            w.s_S = take(C);
        }
        w.n_proj = ((int64_t)(stack.size() / (size_t)W) + 31) / 32 * 32; // whole tiles for the tensor-core product
        stack.resize((size_t)(w.n_proj * W), 0.f);
        TZ_TRY(upload_matrix(stack, &w.proj));
        TZ_GET(q + "o", W, w.k_o, amp(w.k_o), 0.f, &a);
        TZ_TRY(upload_matrix(a, &w.o));
        if (l.ff > 0) {
            TZ_F32(p + "ls2", W, 0.1f, 0.5f, &w.ls2);
            TZ_GET(p + "mlp.up", l.ff, W, aw, 0.f, &a);
            TZ_TRY(upload_matrix(a, &w.up));
            TZ_GET(p + "mlp.down", W, l.ff, amp(l.ff), 0.f, &a);
            TZ_TRY(upload_matrix(a, &w.down));
            TZ_GET(p + "mlp.act", 1, 2, 0.5f, 0.f, &a);
            w.act_p = (float)softplus((double)a[0]);
            w.act_n = (float)(0.5 + softplus((double)a[1]));
        }
    }
#undef TZ_GET
#undef TZ_F32
    state_elems_ = st;
    tz_lookback(c, &lookback_, &keep_first_);
    return 0;
}

lm_model *tezesun_model::create(const std::string &dir, const json_value &cfg, const lm_load_options &opt, std::string *err) {
    tezesun_model *m = new tezesun_model();
    safetensors_file file;
    m->dt_ = opt.dtype;
    if (opt.max_portion > 0) m->max_T_ = opt.max_portion;
    int rc = 0;
    if (!ggb_dtype_size(m->dt_)) rc = -1, m->err_ = "Tezesun runs in bfloat16 or float32";
    if (!rc && !opt.random_weights) rc = file.open(dir + "/model.safetensors", &m->err_);
    if (!rc) rc = tz_parse_config(cfg, opt.random_weights ? nullptr : &file, &m->cfg_, &m->err_);
    if (!rc) rc = m->load(opt.random_weights ? nullptr : &file, opt.seed);
    if (rc) {
        if (err) *err = m->err_;
        delete m;
        return nullptr;
    }
    return m;
}

tezesun_model::~tezesun_model() {
    ggb_sync();
    for (step_graph &g : graphs_) ggb_graph_free(g.graph);
    for (void *p : owned_) ggb_buffer_free(p);
}

std::vector<int64_t> tezesun_model::cache_row_elems() const {
    std::vector<int64_t> v;
    for (const tz_layer_cfg &l : cfg_.layers) {
        if (l.type == 0) v.push_back(ggb_window_cache_ld(l.attn.kv_heads, 2 * l.attn.dim, l.attn.vdim));
        if (l.type == 1) v.push_back(ggb_latent_cache_ld(l.latent.kv_rank, l.latent.rot_dim));
    }
    return v;
}

// ------------------------------------------------------------------------------------------------ buffers
int tezesun_model::alloc_scratch() {
    const tz_config &c = cfg_;
    const int64_t T = max_T_, W = c.width;
    int64_t npr = 0, nq = 0, nao = 0, nqa = 0, nhr = 0, ncq = 0, nrec = 0, nsplit = 0, nbmax = 0, ff = 0, ldkv = 0, nkvf = 0, rmax = 0;
    int hmax = 1;
    const size_t es = ggb_dtype_size(dt_);
    kv_rows_ = max_pos_;
    bool expand = false;
    for (size_t li = 0; li < c.layers.size(); li++) {
        const tz_layer_cfg &l = c.layers[li];
        npr = std::max(npr, lw_[li].n_proj);
        nao = std::max(nao, lw_[li].k_o);
        ff = std::max(ff, (int64_t)l.ff);
        if (l.type == 0) {
            nq = std::max(nq, 2 * (int64_t)l.attn.heads * l.attn.dim);
            hmax = std::max(hmax, l.attn.heads);
        } else if (l.type == 1) {
            const tz_latent_cfg &A = l.latent;
            nq = std::max(nq, (int64_t)A.heads * (A.dim + A.rot_dim));
            nqa = std::max(nqa, (int64_t)A.heads * (std::max(A.kv_rank, A.dim) + A.rot_dim));
            nhr = std::max(nhr, (int64_t)A.heads * (A.kv_rank + 2));
            ncq = std::max(ncq, (int64_t)A.q_rank);
            if (materialise(A, (int)T)) {
                expand = true;
                ldkv = std::max(ldkv, ggb_window_cache_ld(A.heads, A.dim + A.rot_dim, A.vdim));
                nkvf = std::max(nkvf, (int64_t)A.heads * (A.dim + A.vdim));
                rmax = std::max(rmax, (int64_t)A.kv_rank);
            }
        } else {
            nrec = std::max(nrec, (int64_t)l.rec.width);
            if (ggb_rglru_split_fits(dt_, T, l.rec.width / l.rec.blocks)) nsplit = std::max(nsplit, (int64_t)l.rec.width * 3);
            nbmax = std::max(nbmax, (int64_t)l.rec.blocks);
        }
    }
    part_rows_ = std::max<int64_t>(T, 320);
    // the materialised form of the latent attention: as many positions as a modest buffer holds, the absorbed form beyond them
    if (!expand) kv_rows_ = 0;
    else kv_rows_ = std::min<int64_t>(kv_rows_, ((int64_t)768 << 20) / (ldkv * (int64_t)es + nkvf * 4 + rmax * (int64_t)es));
    auto alloc = [&](size_t bytes, void **p) -> int {
        TZ_TRY(ggb_buffer_alloc(std::max<size_t>(bytes, 16), p));
        owned_.push_back(*p);
        return 0;
    };
#define TZ_ALLOC(ptr, bytes) TZ_TRY(alloc((size_t)(bytes), (void **)&(ptr)))
    TZ_ALLOC(ids_, T * 4);
    TZ_ALLOC(want_, T * 4);
    TZ_ALLOC(pos0_, 16);
    TZ_ALLOC(xa_, T * W * 4);
    TZ_ALLOC(xb_, T * W * 4);
    TZ_ALLOC(h_, T * W * es);
    TZ_ALLOC(hs_, T * W * es);
    TZ_ALLOC(pr_, T * npr * 4);
    TZ_ALLOC(q_, T * nq * 4);
    TZ_ALLOC(qa_, T * nqa * 4);
    TZ_ALLOC(cq_, T * ncq * es);
    TZ_ALLOC(part_, (nhr ? part_rows_ * nhr : 0) * 4);
    TZ_ALLOC(wa_, ggb_window_attn_scratch_bytes(2 * hmax));
    TZ_ALLOC(ao_, T * nao * es);
    TZ_ALLOC(u_, T * nrec * 4);
    TZ_ALLOC(z_, T * 2 * nrec * 4);
    TZ_ALLOC(split_, T * nsplit * 2);
    TZ_ALLOC(offsets_, (nbmax + 1) * 4);
    TZ_ALLOC(gu_, T * ff * 4);
    TZ_ALLOC(act_, T * ff * es);
    TZ_ALLOC(ya_, T * W * 4);
    TZ_ALLOC(yb_, T * W * 4);
    TZ_ALLOC(hw_, T * W * es);
    TZ_ALLOC(logits_, T * (int64_t)c.vocab * 4);
    if (kv_rows_ > 0) {
        TZ_ALLOC(crows_, kv_rows_ * rmax * es);
        TZ_ALLOC(kvf_, kv_rows_ * nkvf * 4);
        TZ_ALLOC(kv_, kv_rows_ * ldkv * es);
        const int64_t np = kv_rows_ / cache_->page_size() + 2;
        TZ_ALLOC(page_iota_, np * 4);
        std::vector<int32_t> pi((size_t)np);
        for (int64_t i = 0; i < np; i++) pi[(size_t)i] = (int32_t)i;
        TZ_TRY(ggb_upload(page_iota_, pi.data(), (size_t)np * 4));
        TZ_TRY(ggb_sync());
    }
#undef TZ_ALLOC
    return 0;
}

int tezesun_model::bind_cache(paged_cache *cache, int64_t max_positions) {
    cache_ = cache;
    max_pos_ = max_positions;
    if ((int)cache_row_elems().size() != cache->n_layers()) return fail(GGB_ERR_ARG, "the cache has another number of layers than the model");
    if (cache->state_elems() < state_elems_) return fail(GGB_ERR_ARG, "the cache keeps less state per sequence than the model needs");
    for (size_t li = 0; li < cfg_.layers.size(); li++) {
        const tz_layer_cfg &l = cfg_.layers[li];
        if (l.type == 2) continue;
        const rot_spec &r = l.type == 0 ? l.attn.rot : l.latent.rot;
        if (r.dims <= 0) continue;
        const std::string k = r.key();
        if (!rot_tables_.count(k)) {
            float *d = nullptr;
            TZ_TRY(upload_f32(rot_table(r, max_positions), &d));
            rot_tables_[k] = d;
        }
        lw_[li].cs = rot_tables_[k];
    }
    return alloc_scratch();
}

// The absorbed form scores against the latent (2 R + Dr multiply-adds per key and head); the materialised form multiplies the
// visible latents by [W_uk; W_uv] once per portion (a tensor-core product) and then pays D + Dr + Dv per key and head in the
// window attention kernel.  Portions take the second when heads are short beside the latent; steps always take the first.
bool tezesun_model::materialise(const tz_latent_cfg &a, int T) const {
    return T >= 64 && a.vdim % 2 == 0 && a.vdim <= 256 && 8 * (int64_t)(a.dim + a.rot_dim + a.vdim) <= 5 * (2 * (int64_t)a.kv_rank + a.rot_dim) &&
           !getenv("GGB_LATENT_ABSORBED");
}

// ------------------------------------------------------------------------------------------------ one portion
int tezesun_model::emit_latent(const tz_latent_cfg &A, const tz_layer_w &w, int T, int64_t pos0, int ns, const int32_t *table) {
    const int64_t t = T, N = w.n_proj;
    const int B = cache_->page_size(), H = A.heads, D = A.dim, Dr = A.rot_dim, Dv = A.vdim, R = A.kv_rank, Rq = A.q_rank, rd = A.rot.dims;
    void *cache = cache_->layer(w.cache_index);
    TZ_OP("op_attn_prep", ggb_op_latent_prep(dt_, pr_, Rq, w.dq_norm, cq_, pr_ + w.o1, N, t, R, Dr, rd, 1, w.dkv_norm, cfg_.eps, w.cs, pos0_, table, B, cache));
    const int64_t nq = (int64_t)H * (D + Dr);
    TZ_OP("op_linear", ggb_op_linear(dt_, w.uq, nq, Rq, cq_, Rq, t, q_, nq));
    const int64_t n_vis = pos0 + T;
    if (kv_rows_ >= n_vis && materialise(A, T)) {
        TZ_OP("op_attn_expand", ggb_op_latent_expand_rot(dt_, cache, table, B, 0, n_vis, R, H, D, Dr, Dv, w.ukv, crows_, kvf_, kv_,
                                                         ggb_window_cache_ld(H, D + Dr, Dv)));
        TZ_OP("op_attn_prep", ggb_op_latent_q_rotate(q_, nq, t, H, D, Dr, rd, 1, w.cs, pos0_, A.scale, qa_));
        TZ_OP("op_attn_latent", ggb_op_window_attn(dt_, qa_, kv_, page_iota_, B, pos0_, t, H, H, D + Dr, Dv, 0, nullptr, ao_, nullptr));
    } else {
        TZ_OP("op_attn_prep", ggb_op_latent_q_absorb_halves(dt_, q_, nq, t, H, D, Dr, rd, w.cs, pos0_, w.uk, R, A.scale, qa_));
        TZ_OP("op_attn_latent", ggb_op_latent_attn(dt_, qa_, cache, table, B, pos0_, t, H, R, Dr, ns, part_));
        TZ_OP("op_attn_out", ggb_op_latent_attn_out_gated(dt_, part_, ns, nullptr, w.uv, t, H, R, Dv, nullptr, 0, ao_));
    }
    return 0;
}

int tezesun_model::emit_rglru(const tz_rglru_cfg &R, const tz_layer_w &w, int T, float *state) {
    const int64_t t = T, N = w.n_proj;
    const int nb = R.blocks, d = R.width / R.blocks;
    float *hist = R.conv > 1 ? state + w.s_hist : nullptr, *S = state + w.s_S;
    const float *x = pr_, *y = pr_ + w.o1;
    if (ggb_rglru_step_form(t, d)) {
        TZ_OP("op_recurrence", ggb_op_rglru_step(dt_, x, y, N, t, nb, d, w.conv, w.conv_b, R.conv, w.xb, w.yb, w.w_ri, w.b_ri, w.rate, pos0_, hist, S, ao_));
        return 0;
    }
    void *split = w.w_ri3 && ggb_rglru_split_fits(dt_, t, d) ? split_ : nullptr;
    TZ_OP("op_conv", ggb_op_rglru_conv(x, N, t, nb, d, w.conv, w.conv_b, R.conv, w.xb, pos0_, hist, u_, split, offsets_));
    TZ_OP("op_gates", ggb_op_rglru_gates(dt_, u_, split, offsets_, t, nb, d, w.w_ri, w.w_ri3, z_));
    TZ_OP("op_recurrence", ggb_op_rglru_scan(dt_, z_, u_, y, N, t, nb, d, w.yb, w.b_ri, w.rate, S, ao_));
    return 0;
}

int tezesun_model::emit(int T, int64_t pos0, int ns, const int32_t *table, float *state, int n_want) {
    const tz_config &c = cfg_;
    const int64_t W = c.width, t = T;
    const int B = cache_->page_size();
    // the residual of layer i is in `x`; a layer's two outputs wait in ya_ and yb_ for the next pass
    float *x = nullptr, *x_next = xa_;
    const float *ya = nullptr, *yb = nullptr, *ls1 = nullptr, *ls2 = nullptr;
    for (size_t li = 0; li < c.layers.size(); li++) {
        const tz_layer_cfg &l = c.layers[li];
        const tz_layer_w &w = lw_[li];
        const int64_t N = w.n_proj;
        // one pass: the layer before enters the residual (the first one starts it from the embedding rows), norm, token shift
        TZ_OP("op_residual", ggb_op_shift_norm(dt_, x, x ? nullptr : embed_, ids_, ya, ls1, yb, ls2, w.norm1, c.eps, w.shift, state + w.s_h, W, t, nullptr,
                                               x_next, h_, hs_));
        x = x_next;
        x_next = x == xa_ ? xb_ : xa_;
        // the feed-forward's first product reads h, every projection of the mixer reads the shifted h
        if (l.ff > 0)
            TZ_OP("op_linear", ggb_op_linear_pair(dt_, w.up, l.ff, W, h_, W, w.proj, N, W, hs_, W, t, gu_, l.ff, act_, w.act_p, w.act_n, pr_, N));
        else
            TZ_OP("op_linear", ggb_op_linear(dt_, w.proj, N, W, hs_, W, t, pr_, N));
        if (l.type == 0) {
            const tz_attn_cfg &A = l.attn;
            void *cache = cache_->layer(w.cache_index);
            TZ_OP("op_attn_prep", ggb_op_diff_qkv_store(dt_, pr_, pr_ + w.o1, pr_ + w.o2, N, t, A.heads, A.kv_heads, A.dim, A.vdim, A.rot.dims, 0, w.cs, A.scale,
                                                        pos0_, table, B, cache, q_));
            TZ_OP("op_attn", ggb_op_diff_attn(dt_, q_, cache, table, B, pos0_, t, A.heads, A.kv_heads, A.dim, A.vdim, A.window, A.keep_first, A.softcap,
                                              w.lambda, (float)(1.0 - A.diff), c.eps, pr_ + w.o3, N, ao_, wa_));
        } else if (l.type == 1) {
            const int rc = emit_latent(l.latent, w, T, pos0, ns, table);
            if (rc) return rc;
        } else {
            const int rc = emit_rglru(l.rec, w, T, state);
            if (rc) return rc;
        }
        if (l.ff > 0)
            TZ_OP("op_linear", ggb_op_linear_pair(dt_, w.down, W, l.ff, act_, l.ff, w.o, W, w.k_o, ao_, w.k_o, t, yb_, W, nullptr, 0.f, 0.f, ya_, W));
        else
            TZ_OP("op_linear", ggb_op_linear(dt_, w.o, W, w.k_o, ao_, w.k_o, t, ya_, W));
        ya = ya_, ls1 = w.ls1;
        yb = l.ff > 0 ? yb_ : nullptr, ls2 = w.ls2;
        if (capture_ && cap_)
            TZ_OP("op_rows", ggb_op_shift_norm(dt_, x, nullptr, nullptr, ya, ls1, yb, ls2, nullptr, c.eps, nullptr, nullptr, W, t, nullptr,
                                               cap_ + li * (size_t)max_T_ * (size_t)W, nullptr, nullptr));
    }
    if (n_want > 0) { // the last layer enters on the way: only the wanted rows are computed
        TZ_OP("op_residual", ggb_op_shift_norm(dt_, x, nullptr, nullptr, ya, ls1, yb, ls2, final_norm_, c.eps, nullptr, nullptr, W, n_want, want_, nullptr, hw_,
                                               nullptr));
        TZ_OP("op_linear", ggb_op_linear(dt_, head_, c.vocab, W, hw_, W, n_want, logits_, c.vocab));
    }
    return 0;
}

int tezesun_model::forward(const lm_portion &p, const int32_t *want, int n_want) {
    if (!cache_) return fail(GGB_ERR_ARG, "forward before bind_cache");
    if (p.T <= 0 || p.T > max_T_ || n_want < 0 || n_want > p.T || p.pos0 < 0 || p.pos0 + p.T > max_pos_ || !p.state_dev) {
        err_ = "forward: a portion of " + std::to_string(p.T) + " tokens at position " + std::to_string(p.pos0) + " does not fit";
        return GGB_ERR_ARG;
    }
    for (int i = 0; i < p.T; i++)
        if (p.tokens[i] < 0 || p.tokens[i] >= cfg_.vocab) {
            err_ = "forward: token " + std::to_string(p.tokens[i]) + " is outside the vocabulary";
            return GGB_ERR_ARG;
        }
    const int32_t pos0 = (int32_t)p.pos0;
    TZ_TRY(ggb_upload(ids_, p.tokens, (size_t)p.T * 4));
    TZ_TRY(ggb_upload(pos0_, &pos0, 4));
    if (n_want) TZ_TRY(ggb_upload(want_, want, (size_t)n_want * 4));
    // splits of a latent layer's visible positions: enough CTAs for a short portion, one split once the tokens fill the GPU
    int64_t ns = 1;
    for (const tz_layer_cfg &l : cfg_.layers)
        if (l.type == 1) {
            const int64_t n_vis = p.pos0 + p.T;
            ns = std::min<int64_t>((n_vis + (p.T <= 8 ? 31 : 127)) / (p.T <= 8 ? 32 : 128), std::max<int64_t>(1, 296 / p.T));
            ns = std::max<int64_t>(1, std::min<int64_t>(ns, 64));
        }
    if (p.T == 1) { // powers of two: the captured one-token step changes rarely
        int64_t q = 1;
        while (q < ns) q *= 2;
        ns = q;
    }
    while (ns > 1 && ns * p.T > part_rows_) ns--;
    const int64_t l0 = ggb_launch_count();
    if (capture_) {
        if (!cap_) {
            void *d = nullptr;
            TZ_TRY(ggb_buffer_alloc(cfg_.layers.size() * (size_t)max_T_ * (size_t)cfg_.width * 4, &d));
            owned_.push_back(d);
            cap_ = (float *)d;
        }
        cap_T_ = p.T;
    }
    if (p.T == 1 && use_graphs_ && !capture_ && !getenv("GGB_NO_STEP_GRAPH")) {
        ggb_graph *g = nullptr;
        for (const step_graph &sg : graphs_)
            if (sg.table == p.block_table_dev && sg.state == p.state_dev && sg.n_split == (int)ns && sg.n_want == n_want) g = sg.graph;
        if (!g) {
            TZ_TRY(ggb_capture_begin());
            const int rc = emit(1, p.pos0, (int)ns, p.block_table_dev, p.state_dev, n_want);
            const int rc2 = ggb_capture_end(&g);
            if (rc) return rc;
            if (rc2) return fail(rc2, "ggb_capture_end");
            if (graphs_.size() >= 32) {
                ggb_graph_free(graphs_.front().graph);
                graphs_.erase(graphs_.begin());
            }
            graphs_.push_back(step_graph{p.block_table_dev, p.state_dev, (int)ns, n_want, g});
        }
        TZ_TRY(ggb_graph_launch(g));
    } else {
        TZ_TRY(emit(p.T, p.pos0, (int)ns, p.block_table_dev, p.state_dev, n_want));
    }
    kernels_last_ = (int)(ggb_launch_count() - l0);
    return 0;
}

int tezesun_model::get_capture(int layer, float *host, int64_t n) const {
    if (!cap_ || layer < 0 || layer >= (int)cfg_.layers.size() || n > (int64_t)cap_T_ * cfg_.width) return GGB_ERR_ARG;
    return ggb_download(host, cap_ + (size_t)layer * (size_t)max_T_ * (size_t)cfg_.width, (size_t)n * 4);
}

namespace {
struct register_tezesun {
    register_tezesun() { lm_register("Tezesun", &tezesun_model::create); }
} g_register_tezesun;
} // namespace
