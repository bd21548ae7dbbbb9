// fekopel_model.h — the Fekopel decoder: pre-norm layers with layer norms (weight and bias) and two kinds of mixer in any order, both
// grouped-query soft-max attention with q and k normed per head.  "attention" knows no positions: unit q and k, a sliding window,
// a soft-max with one more term of score 0 in its denominator (a sink without a value).  "attention_2" has norms with weights, rotary
// positions in the halves layout on a part of each head, soft-capped scores, a window that keeps the first positions visible and a
// sigmoid gate per element.  The feed-forward is a mixture of gelu experts (soft-max router over all experts, groups, a factor) beside
// an expert that every token uses under a sigmoid gate of its own.  A block of consecutive layers may run several times with the
// same weights; every pass starts by adding the embedding row again (not the first) and a learned vector of the pass.  Every size
// and constant comes from config.json or a tensor's shape.
//
// What a sequence carries: rows [k | v] of every layer RUN in the engine's paged cache (a layer that runs three times owns three
// arrays), no other state.  When every layer has a window, pages behind the widest one go back to the pool while the sequence lives,
// except those of the kept first positions.
//
// The class lowers a portion of tokens to ggb_op_* operators (residual.cu, dense.cu, window_attention.cu, moe.cu), as the other
// designs do; positions and page tables are read on the device, so the one-token step is captured into a CUDA graph per sequence slot
// and replayed.
#pragma once

#include <map>
#include <string>
#include <vector>

#include "ggml_b200.h"
#include "lm_model.h"
#include "lm_weights.h"
#include "rotary.h"
#include "safetensors.h"

struct fk_mixer_cfg {
    bool gated = false; // attention_2; else attention
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0;
    int64_t window = 0, keep_first = 0; // window 0: every earlier position
    float scale = 1.0f;
    float softcap = 0.0f; // 0: scores as they are
    rot_spec rot;         // dims 0: none
};

struct fk_moe_cfg {
    int experts = 0, top = 0, ff = 0; // experts 0: the layer has no feed-forward
    int groups = 1, keep = 1;
    float scale = 1.0f;
    int shared_ff = 0; // 0: no shared expert
};

struct fk_layer_cfg {
    fk_mixer_cfg mix;
    fk_moe_cfg moe;
};

struct fk_run {
    int layer = 0;
    int pass = -1; // number of the looped block's pass that begins with this run, -1: none begins here
};

struct fk_config {
    int vocab = 0, width = 0;
    float eps = 1e-5f;
    int loop_start = 0, loop_stop = 0, loop_times = 0; // times 0: no looped block
    std::vector<fk_layer_cfg> layers;
    std::vector<fk_run> runs; // every layer run in order (a looped layer appears once per pass); run i owns cache array i
};
// file: where sizes that the configuration leaves out are read from (may be null)
int fk_parse_config(const json_value &j, const safetensors_file *file, fk_config *c, std::string *err);
// what the farthest-looking layer sees: the widest window (0: some layer sees everything) and the most kept first positions
void fk_lookback(const fk_config &c, int64_t *lookback, int64_t *keep_first);

struct fk_layer_w {
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
    void *proj = nullptr; // q | k | v (| g) stacked (rows padded to a multiple of 32)
    int64_t n_proj = 0, o_k = 0, o_v = 0, o_g = 0;
    float *q_norm = nullptr, *k_norm = nullptr;
    const float *cs = nullptr;
    void *o = nullptr;
    float *router = nullptr; // the shared expert's gate is one more row
    void *e_up = nullptr, *e_down = nullptr, *s_up = nullptr, *s_down = nullptr;
};

class fekopel_model : public lm_model {
  public:
    static lm_model *create(const std::string &dir, const json_value &cfg, const lm_load_options &opt, std::string *err);
    ~fekopel_model() override;

    const char *architecture() const override { return "Fekopel"; }
    int vocab() const override { return cfg_.vocab; }
    int dtype() const override { return dt_; }
    std::vector<int64_t> cache_row_elems() const override;
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
    int get_capture(int run, float *host, int64_t n) const override; // the residual after layer run `run`
    size_t weight_bytes() const override { return weight_bytes_; }
    int kernels_last_forward() const override { return kernels_last_; }

  private:
    fekopel_model() {}
    int load(const safetensors_file *file, uint64_t seed);
    int alloc_scratch();
    int emit(int T, const int32_t *table_dev, int n_want);
    int upload_matrix(const std::vector<float> &host, void **dev);
    int upload_f32(const std::vector<float> &host, float **dev);
    int fail(int rc, const std::string &what);

    fk_config cfg_;
    int dt_ = GGB_TYPE_BF16;
    int max_T_ = 1024;
    std::string err_;
    std::vector<fk_layer_w> lw_;
    void *embed_ = nullptr, *head_ = nullptr;
    float *final_norm_ = nullptr, *final_normb_ = nullptr, *loop_step_ = nullptr, *sinks_ = nullptr;
    size_t weight_bytes_ = 0;
    int64_t lookback_ = 0, keep_first_ = 0;
    std::vector<void *> owned_;
    paged_cache *cache_ = nullptr;
    int64_t max_pos_ = 0;
    std::map<std::string, float *> rot_tables_;
    int32_t *ids_ = nullptr, *pos0_ = nullptr, *want_ = nullptr, *route_i_ = nullptr, *group_ws_ = nullptr;
    float *x_ = nullptr, *pr_ = nullptr, *qr_ = nullptr, *wa_ = nullptr, *ya_ = nullptr, *y2_ = nullptr, *ys_ = nullptr, *route_z_ = nullptr,
          *route_w_ = nullptr, *logits_ = nullptr, *cap_ = nullptr;
    void *h_ = nullptr, *ao_ = nullptr, *act_ = nullptr, *acts_ = nullptr, *hw_ = nullptr;
    bool capture_ = false, use_graphs_ = true;
    int cap_T_ = 0, kernels_last_ = 0;
    struct step_graph {
        const int32_t *table;
        int n_want;
        ggb_graph *graph;
    };
    std::vector<step_graph> graphs_;
};
