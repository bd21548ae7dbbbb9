// residual.cu — the pass between two sublayers of a pre-norm decoder whose norms subtract the mean: what the sublayer before
// computed enters the residual, rows that a looped block starts from are added, and the layer norm in front of the next sublayer
// is taken, in one launch over the row.  Residual, sums, mean and variance are fp32; the variance is the mean of the squared
// deviations (a second pass over the row in shared memory, nothing is cancelled).
//
// Compiled with -fmad=false: multiply-adds are spelled fmaf().
#include <cuda_bf16.h>

#include "common.cuh"
#include "dense.cuh"

namespace {

constexpr int kMaxSlots = GGB_RESIDUAL_MAX_TOP;

template <typename E> struct residual_args {
    const float *x; // the residual, or null: it starts at zero
    const float *y; // a sublayer's output, or null
    const float *y2, *wt; // a mixture of experts whose weighted sum has not been taken: slot rows, weights, the slots' rows
    const int32_t *inv;
    int top;
    const float *ys, *gate; // an expert every token uses: its output times sigmoid(gate[t * ldg]); gate null: times one
    int64_t ldg;
    const E *table; // the tokens' embedding rows, added after the above, and one more row for all tokens
    const int32_t *ids;
    const float *add;
    const float *nw, *nb;
    float eps;
    int64_t W;
    const int32_t *rows;
    float *x_out;
    E *h;
};

// one CTA per row; a thread owns the same columns in every loop, so that x_out may be x
template <typename E, int V, int TB>
__global__ void __launch_bounds__(TB) residual_layer_norm_kernel(residual_args<E> p) {
    extern __shared__ __align__(16) float rl_row[]; // [W]
    __shared__ float red[32], s_wt[kMaxSlots];
    __shared__ int64_t s_off[kMaxSlots];
    const int64_t b = blockIdx.x, t = p.rows ? p.rows[b] : b, W = p.W;
    if (p.y2) { // the token's slots, looked up once: the loads below then depend on nothing
        if ((int)threadIdx.x < p.top) {
            s_wt[threadIdx.x] = p.wt[t * p.top + threadIdx.x];
            s_off[threadIdx.x] = (int64_t)p.inv[t * p.top + threadIdx.x] * W;
        }
        __syncthreads();
    }
    const float gs = p.ys && p.gate ? 1.0f / (1.0f + expf(-p.gate[t * p.ldg])) : 1.0f;
    const E *er = p.table ? p.table + (int64_t)p.ids[t] * W : nullptr;
    float sum = 0.f;
    for (int64_t i = (int64_t)threadIdx.x * V; i < W; i += (int64_t)TB * V) {
        float x[V], v[V];
#pragma unroll
        for (int c = 0; c < V; c++) x[c] = 0.f;
        if (p.x) load_vec<V>(p.x + t * W + i, x);
        if (p.y) {
            load_vec<V>(p.y + t * W + i, v);
#pragma unroll
            for (int c = 0; c < V; c++) x[c] += v[c];
        }
        if (p.y2) {
            float s[V];
#pragma unroll
            for (int c = 0; c < V; c++) s[c] = 0.f;
#pragma unroll 4
            for (int k = 0; k < p.top; k++) {
                load_vec<V>(p.y2 + s_off[k] + i, v);
#pragma unroll
                for (int c = 0; c < V; c++) s[c] = fmaf(s_wt[k], v[c], s[c]);
            }
            if (p.ys) {
                load_vec<V>(p.ys + t * W + i, v);
#pragma unroll
                for (int c = 0; c < V; c++) s[c] = fmaf(gs, v[c], s[c]);
            }
#pragma unroll
            for (int c = 0; c < V; c++) x[c] += s[c];
        }
        if (er) {
#pragma unroll
            for (int c = 0; c < V; c++) x[c] += to_f32(er[i + c]);
        }
        if (p.add) {
            load_vec<V>(p.add + i, v);
#pragma unroll
            for (int c = 0; c < V; c++) x[c] += v[c];
        }
        if (p.x_out) store_vec<V>(p.x_out + b * W + i, x);
#pragma unroll
        for (int c = 0; c < V; c++) {
            rl_row[i + c] = x[c];
            sum += x[c];
        }
    }
    if (!p.h) return;
    const float mean = block_sum_any(sum, red) / (float)W;
    float ss = 0.f;
    for (int64_t i = (int64_t)threadIdx.x * V; i < W; i += (int64_t)TB * V)
#pragma unroll
        for (int c = 0; c < V; c++) {
            const float d = rl_row[i + c] - mean;
            ss = fmaf(d, d, ss);
        }
    const float r = 1.0f / sqrtf(block_sum_any(ss, red) / (float)W + p.eps);
    for (int64_t i = (int64_t)threadIdx.x * V; i < W; i += (int64_t)TB * V) {
        float w[V], o[V];
        load_vec<V>(p.nw + i, w);
        load_vec<V>(p.nb + i, o);
#pragma unroll
        for (int c = 0; c < V; c++) o[c] = fmaf((rl_row[i + c] - mean) * r, w[c], o[c]);
        store_vec<V>(p.h + b * W + i, o);
    }
}

template <typename E> int residual_launch(const residual_args<E> &p, int64_t T) {
    const int64_t W = p.W;
    const size_t smem = (size_t)W * 4;
    const bool vec = W % 4 == 0 && (((uintptr_t)p.x | (uintptr_t)p.y | (uintptr_t)p.y2 | (uintptr_t)p.ys | (uintptr_t)p.add | (uintptr_t)p.nw | (uintptr_t)p.nb |
                                     (uintptr_t)p.x_out | (uintptr_t)p.h) & 15) == 0;
    const int64_t per_pass = W / (vec ? 4 : 1);
    // a step of few tokens is a chain of latencies on a nearly empty GPU: a wide CTA covers the row in one pass
    const int tb = per_pass <= 128 ? 128 : T <= 64 && per_pass >= 1024 ? 1024 : T <= 64 && per_pass >= 512 ? 512 : 256;
#define RL_LAUNCH(V, TB)                                                                                                        \
    {                                                                                                                           \
        auto k = residual_layer_norm_kernel<E, V, TB>;                                                                          \
        if (smem > 48 * 1024) GGB_CUDA(cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));         \
        k<<<(unsigned)T, TB, smem, ggb_cuda_stream()>>>(p);                                                                     \
    }
#define RL_TB(V)                                                                                                                \
    {                                                                                                                           \
        if (tb == 128) RL_LAUNCH(V, 128)                                                                                        \
        else if (tb == 256) RL_LAUNCH(V, 256)                                                                                   \
        else if (tb == 512) RL_LAUNCH(V, 512)                                                                                   \
        else RL_LAUNCH(V, 1024)                                                                                                 \
    }
    if (vec) RL_TB(4) else RL_TB(1)
#undef RL_TB
#undef RL_LAUNCH
    GGB_LAUNCH_CHECK();
    return GGB_OK;
}

} // namespace

extern "C" {

int ggb_op_residual_layer_norm(int dt, const float *x, const float *y, const float *y2, const int32_t *ws, const float *wt, int64_t T_slots, int top, int n_exp,
                               const float *ys, const float *gate, int64_t ldg, const void *table, const int32_t *ids, const float *add, const float *nw,
                               const float *nb, float eps, int64_t W, int64_t T, const int32_t *rows, float *x_out, void *h) {
    GGB_REQUIRE_INIT();
    GGB_CHECK_ARG(dt == GGB_TYPE_BF16 || dt == GGB_TYPE_F32, "dtype %d is neither bf16 nor f32", dt);
    GGB_CHECK_ARG((x || (table && ids)) && W > 0 && T > 0 && (x_out || h) && (!h || (nw && nb)), "residual_layer_norm: bad arguments");
    GGB_CHECK_ARG((!table || ids) && !(y && y2) && (!ys || y2) && (!gate || (ys && ldg > 0)), "residual_layer_norm: an input without its companions");
    GGB_CHECK_ARG(!y2 || (ws && wt && top > 0 && top <= kMaxSlots && n_exp > 0 && T_slots >= 1), "residual_layer_norm: expert slots without their lists (at most %d a token)",
                  kMaxSlots);
    GGB_CHECK_ARG(!(rows && x_out && x_out == x), "residual_layer_norm: chosen rows go to another buffer");
    GGB_CHECK_ARG((size_t)W * 4 <= 200 * 1024, "residual_layer_norm: width %lld does not fit shared memory", (long long)W);
    const int32_t *inv = y2 ? ws + n_exp + 1 + T_slots * top : nullptr;
#define RL_CASE(E)                                                                                                                                         \
    return residual_launch<E>(residual_args<E>{x, y, y2, wt, inv, top, ys, gate, ldg, (const E *)table, ids, add, nw, nb, eps, W, rows, x_out, (E *)h}, T);
    if (dt == GGB_TYPE_BF16) RL_CASE(__nv_bfloat16)
    RL_CASE(float)
#undef RL_CASE
}

} // extern "C"
