// tezesun_model.h — the Tezesun decoder: layers whose mixer and feed-forward read one normed input side by side, each output
// with a weight per channel, x += mixer(shift(h)) * ls1 + ff(h) * ls2 with h = norm(x); what the mixer reads is h blended
// channel by channel with the h of the token before (token shift).  Three kinds of mixer in any order: "attention"
// (differential attention: two soft-max maps per head over the same values, their difference normed per head; soft-capped scores,
// a sliding window that keeps the first tokens, rotary neighbour pairs with a frequency blend, an output gate per element),
// "latent_attention" (queries and keys / values through normed latents, one shared rotated key part in the halves layout, causal)
// and "rglru" (a gated diagonal linear recurrence behind a short convolution, beside a gelu branch).  The feed-forward is dense with
// an xIELU.  Every size and constant comes from config.json or a tensor's shape.
//
// What a sequence carries: cache rows [k of both maps | v] of attention layers and [latent | rotated key part] of latent layers in
// the engine's paged cache, and one block of fp32 state in the cache's per-sequence storage: every layer's previous h, and per rglru
// layer the convolution's last inputs and the state S.  When every caching layer has a window, pages behind the widest one go
// back to the pool while the sequence lives, except those of the kept first tokens.
//
// The class lowers a portion of tokens to ggb_op_* operators (dense.cu, window_attention.cu, latent_attention.cu, rglru.cu), as the
// other designs do; positions, page tables and state are read on the device, so the one-token step is captured into a CUDA
// graph per sequence slot and replayed.
#pragma once

#include <map>
#include <string>
#include <vector>

#include "ggml_b200.h"
#include "lm_model.h"
#include "lm_weights.h"
#include "rotary.h"
#include "safetensors.h"

struct tz_attn_cfg {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0; // dim: of one map
    int64_t window = 0, keep_first = 0;             // window 0: every earlier position
    float scale = 1.0f;
    float softcap = 0.0f; // 0: scores as they are
    double diff = 0.0;
    rot_spec rot; // dims 0: none
};

struct tz_latent_cfg {
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, q_rank = 0, kv_rank = 0;
    float scale = 1.0f;
    rot_spec rot;
};

struct tz_rglru_cfg {
    int width = 0, blocks = 0, conv = 1;
};

struct tz_layer_cfg {
    int type = 0; // 0 attention, 1 latent_attention, 2 rglru
    tz_attn_cfg attn;
    tz_latent_cfg latent;
    tz_rglru_cfg rec;
    int ff = 0; // 0: no feed-forward
};

struct tz_config {
    int vocab = 0, width = 0;
    float eps = 1e-6f;
    double logit_scale = 1.0;
    std::vector<tz_layer_cfg> layers;
};
// file: where sizes that a configuration leaves to a tensor's shape are read from (may be null)
int tz_parse_config(const json_value &j, const safetensors_file *file, tz_config *c, std::string *err);
// widest window over all caching layers and the most kept first tokens; 0 when some layer sees everything or none caches
void tz_lookback(const tz_config &c, int64_t *lookback, int64_t *keep_first);

struct tz_layer_w {
    float *norm1 = nullptr, *ls1 = nullptr, *ls2 = nullptr, *shift = nullptr;
    void *proj = nullptr; // every matrix that reads the mixer's input, stacked (rows padded to a multiple of 32)
    int64_t n_proj = 0;
    int64_t o1 = 0, o2 = 0, o3 = 0; // rows of the 2nd, 3rd, 4th matrix: attention q k v g, latent dq dkv, rglru x y
    void *o = nullptr;
    int64_t k_o = 0;                // columns of o
    const float *cs = nullptr;      // rotary table
    float lambda = 0.f;             // attention
    float *dq_norm = nullptr, *dkv_norm = nullptr; // latent
    void *uq = nullptr, *ukv = nullptr, *uk = nullptr, *uv = nullptr; // uk and uv lie inside ukv
    float *conv = nullptr, *conv_b = nullptr, *xb = nullptr, *yb = nullptr, *b_ri = nullptr, *rate = nullptr; // rglru
    void *w_ri = nullptr, *w_ri3 = nullptr;
    void *up = nullptr, *down = nullptr;
    float act_p = 0.f, act_n = 0.f; // xIELU factors
    int cache_index = -1;
    int64_t s_h = 0, s_hist = 0, s_S = 0; // offsets (fp32 numbers) into the sequence's state block
};

class tezesun_model : public lm_model {
  public:
    static lm_model *create(const std::string &dir, const json_value &cfg, const lm_load_options &opt, std::string *err);
    ~tezesun_model() override;

    const char *architecture() const override { return "Tezesun"; }
    int vocab() const override { return cfg_.vocab; }
    int dtype() const override { return dt_; }
    std::vector<int64_t> cache_row_elems() const override;
    int64_t state_elems() const override { return state_elems_; }
    int64_t cache_lookback() const override { return lookback_; }
    int64_t cache_keep_first() const override { return keep_first_; }
    int bind_cache(paged_cache *cache, int64_t max_positions) override;
    int max_portion() const override { return max_T_; }
    int forward(const lm_portion &p, const int32_t *want, int n_want) override;
    const float *logits_dev() const override { return logits_; }
    std::string last_error() const override { return err_; }
    int set_capture(bool on) override {
        capture_ = on;
        return 0;
    }
    int set_use_graphs(bool on) override {
        use_graphs_ = on;
        return 0;
    }
    int get_capture(int layer, float *host, int64_t n) const override;
    size_t weight_bytes() const override { return weight_bytes_; }
    int kernels_last_forward() const override { return kernels_last_; }
    const tz_config &config() const { return cfg_; }

  private:
    tezesun_model() {}
    int load(const safetensors_file *file, uint64_t seed);
    int alloc_scratch();
    bool materialise(const tz_latent_cfg &a, int T) const;
    int emit(int T, int64_t pos0, int n_split, const int32_t *table_dev, float *state, int n_want);
    int emit_latent(const tz_latent_cfg &a, const tz_layer_w &w, int T, int64_t pos0, int n_split, const int32_t *table);
    int emit_rglru(const tz_rglru_cfg &r, const tz_layer_w &w, int T, float *state);
    int upload_matrix(const std::vector<float> &host, void **dev);
    int upload_f32(const std::vector<float> &host, float **dev);
    int fail(int rc, const std::string &what);

    tz_config cfg_;
    int dt_ = GGB_TYPE_BF16;
    int max_T_ = 1024;
    std::string err_;
    std::vector<tz_layer_w> lw_;
    void *embed_ = nullptr, *head_ = nullptr;
    float *final_norm_ = nullptr; // times logit_scale
    size_t weight_bytes_ = 0;
    int64_t state_elems_ = 0, lookback_ = 0, keep_first_ = 0;
    std::vector<void *> owned_;
    paged_cache *cache_ = nullptr;
    int64_t max_pos_ = 0, part_rows_ = 0, kv_rows_ = 0;
    std::map<std::string, float *> rot_tables_;
    int32_t *ids_ = nullptr, *pos0_ = nullptr, *want_ = nullptr, *page_iota_ = nullptr, *offsets_ = nullptr;
    float *xa_ = nullptr, *xb_ = nullptr, *pr_ = nullptr, *q_ = nullptr, *qa_ = nullptr, *part_ = nullptr, *wa_ = nullptr, *u_ = nullptr,
          *z_ = nullptr, *gu_ = nullptr, *ya_ = nullptr, *yb_ = nullptr, *kvf_ = nullptr, *logits_ = nullptr, *cap_ = nullptr;
    void *h_ = nullptr, *hs_ = nullptr, *ao_ = nullptr, *cq_ = nullptr, *split_ = nullptr, *act_ = nullptr, *crows_ = nullptr, *kv_ = nullptr,
         *hw_ = nullptr;
    bool capture_ = false, use_graphs_ = true;
    int cap_T_ = 0, kernels_last_ = 0;
    struct step_graph {
        const int32_t *table;
        const float *state;
        int n_split, n_want;
        ggb_graph *graph;
    };
    std::vector<step_graph> graphs_;
};
