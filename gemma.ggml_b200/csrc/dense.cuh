// dense.cuh — what the bf16 / fp32 operator files (dense.cu, latent_attention.cu, moe.cu) share.
#pragma once

#include <cuda_bf16.h>
#include <stdint.h>

#include "common.cuh"

// Sorted-slot description of one mixture-of-experts layer on the device (built by ggb_op_moe_group): slot s of token t
// (s < top) is row `inv[t * top + s]` of the sorted order, in which the slots of expert e are rows
// [offsets[e], offsets[e + 1]); row i of the sorted order belongs to token row_src[i].  The grouped products walk a list
// of 64-row tiles, none of which crosses an expert.
struct ggb_moe_groups {
    const int32_t *offsets = nullptr;     // [E + 1]
    const int32_t *row_src = nullptr;     // [n] A row of a sorted row, or null: A is already in sorted order
    const int32_t *tile_expert = nullptr; // [max_tiles]
    const int32_t *tile_row0 = nullptr;   // [max_tiles]
    const int32_t *n_tiles = nullptr;     // [1]
};

int ggb_linear_grouped_launch(int dt, const void *w, int64_t N, int64_t K, const void *a, int64_t lda, int max_tiles, float *c,
                              void *c_act, int64_t ldc, int act, const ggb_moe_groups &grp);

// the tcgen05 GEMM of prefill.cu on plain bf16 matrices: C[T][N] (fp32) = A[T][K] W[N][K]^T; with c_act it leaves as bf16 act(C)
// instead (GGB_ACT_*, ldc %% 8 == 0)
bool ggb_gemm_dense_bf16_fits(int64_t N, int64_t K, int64_t T, int64_t ldc);
int ggb_gemm_dense_bf16(const void *w, int64_t N, int64_t K, const void *a, int64_t T, float *c, int64_t ldc, void *c_act = nullptr, int act = 0);

// the grouped tcgen05 form: w [n_exp][N][K] bf16, a rows in sorted-slot order, offsets [n_exp + 1] on the device;
// c fp32 or (c_act) bf16 act(c)
bool ggb_gemm_grouped_bf16_fits(int64_t N, int64_t K, int64_t ldc);
int ggb_gemm_grouped_bf16(const void *w, int64_t N, int64_t K, const void *a, int64_t n_rows, int n_exp, const int32_t *offsets, float *c,
                          void *c_act, int act, int64_t ldc);

// norms on both sides of a sublayer (ggb_op_norm_add_norm); with inv / wt the sublayer's output is the weighted sum of
// the token's `top` expert slots, gathered on the way in (moe.cu)
int ggb_norm_add_norm_launch(int dt, const float *a, const float *bias, const int32_t *inv, const float *wt, int top, const float *wa, float eps,
                             int64_t E, int64_t T, float *x, const float *wy, void *y);

#ifdef __CUDACC__
__device__ __forceinline__ float gelu_tanh_f32(float z) {
    return 0.5f * z * (1.0f + tanhf(0.79788456080286535588f * (z + 0.044715f * z * z * z)));
}
// z times the normal distribution function at z
__device__ __forceinline__ float gelu_erf_f32(float z) { return 0.5f * z * (1.0f + erff(z * 0.70710678118654752440f)); }
// the activations of a product that is not gated (GGB_ACT_*)
__device__ __forceinline__ float act_f32(float v, int act) {
    if (act == GGB_ACT_RELU2) return v > 0.f ? v * v : 0.f;
    if (act == GGB_ACT_GELU_ERF) return gelu_erf_f32(v);
    return v;
}
__device__ __forceinline__ float to_f32(float v) { return v; }
__device__ __forceinline__ float to_f32(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename E> __device__ __forceinline__ E from_f32(float v);
template <> __device__ __forceinline__ float from_f32<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 from_f32<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

__device__ __forceinline__ float block_sum_any(float v, float *red) { // all threads get the sum; blockDim.x a multiple of 32, at most 1024
    v = warp_sum_f32(v);
    __syncthreads(); // `red` may still be read by the previous call
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float tot = 0.f;
    for (int i = 0; i < (int)(blockDim.x >> 5); i++) tot += red[i];
    return tot;
}

// V numbers (V = 4: a 16-byte store in fp32, 8 bytes in bf16) rounded into the matrices' type
template <int V, typename E> __device__ __forceinline__ void store_vec(E *dst, const float (&v)[V]) {
    if (V == 4 && sizeof(E) == 2) {
        union {
            uint2 u;
            __nv_bfloat16 h[4];
        } p;
#pragma unroll
        for (int c = 0; c < V; c++) p.h[c] = __float2bfloat16_rn(v[c]);
        *reinterpret_cast<uint2 *>(dst) = p.u;
    } else if (V == 4) {
        *reinterpret_cast<float4 *>(dst) = make_float4(v[0], v[1 % V], v[2 % V], v[3 % V]);
    } else {
        dst[0] = from_f32<E>(v[0]);
    }
}
// V fp32 numbers
template <int V> __device__ __forceinline__ void load_vec(const float *src, float (&v)[V]) {
    if (V == 4) {
        const float4 v4 = *reinterpret_cast<const float4 *>(src);
        v[0] = v4.x, v[1 % V] = v4.y, v[2 % V] = v4.z, v[3 % V] = v4.w;
    } else {
        v[0] = src[0];
    }
}
#endif
