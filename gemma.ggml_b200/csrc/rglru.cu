// rglru.cu — a gated diagonal linear recurrence (real-gated linear recurrent unit) behind a short causal convolution:
//
//   u_t = conv_b + sum_j conv_w[:, j] (x + x_b)_(t - taps + 1 + j)         per channel, zeros before the sequence's start
//   r_t = sigmoid(W_r[b] u_t[b] + r_b),  i_t = sigmoid(W_i[b] u_t[b] + i_b)  channels cut into blocks b of d, square matrices
//   log a_t = rate r_t  (rate = -8 softplus(lam), per channel);  S <- a_t S + sqrt(1 - a_t^2) i_t u_t
//   out_t = S gelu_tanh(y_t + y_b)
//
// Everything from u on is fp32; the matrices are in the storage type and u enters the gates' products with all its bits.
// What a sequence carries: S and the last inputs of the convolution.  Those lie in a ring indexed by position,
// hist[p mod L] with L = taps - 1 + 8: a step of up to 8 tokens writes other slots than it reads, so the CTAs of one launch
// need no order among themselves.
//
// steps (T <= 8, rglru_step_kernel): one launch.  A CTA owns a slice of a block's channels, computes u of the whole block
// (cheap, repeated by the CTAs of the block), then a warp takes a channel: its two matrix rows against u in shared memory,
// the gates of the tokens on different lanes, the recurrence by shuffles.
// portions: convolution -> gates -> scan.  The gates are block-diagonal products: on the tensor cores for aligned bf16
// matrices, with u written as the sum of three bf16 numbers (exact to fp32 rounding; a row is [high | middle | low], the matrix
// row three times the same, the accumulator fp32), otherwise a shared-memory tile kernel in fp32.  The scan cuts time into
// pieces: every piece's (product of a, local S) first, then the pieces' prefix, then the outputs, all in one pass over memory.
//
// Compiled with -fmad=false: multiply-adds are spelled fmaf().
#include <algorithm>

#include "common.cuh"
#include "dense.cuh"

namespace {

constexpr int kMaxTaps = 8, kStepT = 8, kConvTokens = 32;

__device__ __forceinline__ float sigmoid_f32(float z) { return __frcp_rn(1.0f + expf(-z)); }

// decay and input of one (token, channel): a = exp(rate r), in = sqrt(1 - a^2) i u
__device__ __forceinline__ void rglru_terms(float zr, float zi, float u, float rate, float *a, float *in) {
    const float la = rate * sigmoid_f32(zr);
    *a = expf(la);
    *in = sqrtf(-expm1f(2.0f * la)) * sigmoid_f32(zi) * u;
}

struct rglru_conv_args {
    const float *x, *w, *wb, *xb; // x rows of stride ld; w [C][taps]; biases [C]
    int64_t ld;
    int taps, L;
    float *hist; // [L][C]
};

// the taps - 1 inputs before position p0, oldest first
__device__ __forceinline__ void load_history(const rglru_conv_args &c, int64_t C, int64_t ch, int p0, float (&win)[kMaxTaps]) {
    const int nt = c.taps - 1;
#pragma unroll
    for (int j = 0; j < kMaxTaps - 1; j++) {
        const int p = p0 - nt + j;
        win[j] = (j < nt && p >= 0) ? c.hist[(int64_t)(p % c.L) * C + ch] : 0.f;
    }
}
// one output from the window and the current input; the window moves on
__device__ __forceinline__ float conv_tap(const float (&wt)[kMaxTaps], float (&win)[kMaxTaps], int nt, float xv, float bias) {
    float acc = bias;
#pragma unroll
    for (int j = 0; j < kMaxTaps - 1; j++)
        if (j < nt) acc = fmaf(wt[j], win[j], acc);
#pragma unroll
    for (int j = 0; j < kMaxTaps; j++)
        if (j == nt) acc = fmaf(wt[j], xv, acc);
#pragma unroll
    for (int j = 0; j < kMaxTaps - 1; j++) {
        if (j + 1 < nt) win[j] = win[j + 1];
        else if (j + 1 == nt) win[j] = xv;
    }
    return acc;
}

// ------------------------------------------------------------------------------------------------ steps
template <typename E, int TT>
__global__ void __launch_bounds__(256) rglru_step_kernel(rglru_conv_args cv, const float *__restrict__ y, const float *__restrict__ yb, int T, int d,
                                                         int per_cta, const E *__restrict__ w_ri, const float *__restrict__ b_ri,
                                                         const float *__restrict__ rate, const int32_t *__restrict__ pos0, float *state,
                                                         E *__restrict__ out, int vec) {
    extern __shared__ __align__(16) float us[]; // [TT][d]
    const int b = blockIdx.y, tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int64_t C = (int64_t)gridDim.y * d;
    const int k_lo = blockIdx.x * per_cta, k_hi = min(d, k_lo + per_cta);
    const int p0 = *pos0;
    const int nt = cv.taps - 1;
    for (int k = tid; k < d; k += 256) {
        const int64_t c = (int64_t)b * d + k;
        float wt[kMaxTaps], win[kMaxTaps];
#pragma unroll
        for (int j = 0; j < kMaxTaps; j++) wt[j] = j < cv.taps ? cv.w[c * cv.taps + j] : 0.f;
        load_history(cv, C, c, p0, win);
        const float xb = cv.xb[c], wb = cv.wb[c];
        const bool own = k >= k_lo && k < k_hi;
#pragma unroll
        for (int t = 0; t < TT; t++) {
            float u = 0.f;
            if (t < T) {
                const float xv = cv.x[t * cv.ld + c] + xb;
                u = conv_tap(wt, win, nt, xv, wb);
                if (own && nt > 0) cv.hist[(int64_t)((p0 + t) % cv.L) * C + c] = xv;
            }
            us[t * d + k] = u;
        }
    }
    __syncthreads();
    for (int k = k_lo + warp; k < k_hi; k += 8) {
        const int64_t c = (int64_t)b * d + k;
        const E *wr = w_ri + ((int64_t)b * 2 * d + k) * d, *wi = wr + (int64_t)d * d;
        float zr[TT], zi[TT];
#pragma unroll
        for (int t = 0; t < TT; t++) zr[t] = zi[t] = 0.f;
        if (vec) {
            constexpr int VE = 16 / (int)sizeof(E);
#pragma unroll 2
            for (int q = lane * VE; q < d; q += 32 * VE) {
                const uint4 rv = ldg_stream_u4(wr + q), iv = ldg_stream_u4(wi + q);
                const E *re = reinterpret_cast<const E *>(&rv), *ie = reinterpret_cast<const E *>(&iv);
#pragma unroll
                for (int t = 0; t < TT; t++)
#pragma unroll
                    for (int v = 0; v < VE; v += 4) {
                        const float4 u4 = *reinterpret_cast<const float4 *>(us + t * d + q + v);
                        zr[t] = fmaf(to_f32(re[v]), u4.x, zr[t]), zi[t] = fmaf(to_f32(ie[v]), u4.x, zi[t]);
                        zr[t] = fmaf(to_f32(re[v + 1]), u4.y, zr[t]), zi[t] = fmaf(to_f32(ie[v + 1]), u4.y, zi[t]);
                        zr[t] = fmaf(to_f32(re[v + 2]), u4.z, zr[t]), zi[t] = fmaf(to_f32(ie[v + 2]), u4.z, zi[t]);
                        zr[t] = fmaf(to_f32(re[v + 3]), u4.w, zr[t]), zi[t] = fmaf(to_f32(ie[v + 3]), u4.w, zi[t]);
                    }
            }
        } else {
            for (int q = lane; q < d; q += 32) {
                const float rv = to_f32(wr[q]), iv = to_f32(wi[q]);
#pragma unroll
                for (int t = 0; t < TT; t++) zr[t] = fmaf(rv, us[t * d + q], zr[t]), zi[t] = fmaf(iv, us[t * d + q], zi[t]);
            }
        }
        float my_r = 0.f, my_i = 0.f; // lane t keeps token t
#pragma unroll
        for (int t = 0; t < TT; t++) {
            const float sr = warp_sum_f32(zr[t]), si = warp_sum_f32(zi[t]);
            if (lane == t) my_r = sr, my_i = si;
        }
        float a = 0.f, in = 0.f;
        if (lane < T) rglru_terms(my_r + b_ri[(int64_t)b * 2 * d + k], my_i + b_ri[(int64_t)b * 2 * d + d + k], us[lane * d + k], rate[c], &a, &in);
        float S = state[c], mine = 0.f;
#pragma unroll
        for (int t = 0; t < TT; t++)
            if (t < T) {
                S = fmaf(__shfl_sync(0xffffffffu, a, t), S, __shfl_sync(0xffffffffu, in, t));
                if (lane == t) mine = S;
            }
        if (lane < T) out[(int64_t)lane * C + c] = from_f32<E>(mine * gelu_tanh_f32(y[(int64_t)lane * cv.ld + c] + yb[c]));
        __syncwarp();
        if (lane == 0) state[c] = S;
    }
}

// ------------------------------------------------------------------------------------------------ portions: convolution
// grid (channel blocks, token chunks); a thread owns one channel of one chunk.  Chunk 0 alone reads the ring and, having the
// old inputs in registers, alone writes it.  With `split` u also leaves as three bf16 numbers per channel.
__global__ void __launch_bounds__(128) rglru_conv_kernel(rglru_conv_args cv, int64_t T, int nb, int d, const int32_t *__restrict__ pos0,
                                                         float *__restrict__ u, __nv_bfloat16 *__restrict__ split, int32_t *__restrict__ offsets) {
    const int64_t C = (int64_t)nb * d, c = (int64_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (split && blockIdx.x == 0 && blockIdx.y == 0)
        for (int e = threadIdx.x; e <= nb; e += blockDim.x) offsets[e] = (int32_t)(e * T); // block e's rows of the split form
    if (c >= C) return;
    const int64_t t0 = (int64_t)blockIdx.y * kConvTokens, t1 = min(T, t0 + kConvTokens);
    const int p0 = *pos0;
    const int nt = cv.taps - 1;
    const float xb = cv.xb[c], wb = cv.wb[c];
    float wt[kMaxTaps], win[kMaxTaps];
#pragma unroll
    for (int j = 0; j < kMaxTaps; j++) wt[j] = j < cv.taps ? cv.w[c * cv.taps + j] : 0.f;
    if (t0 == 0) {
        load_history(cv, C, c, p0, win);
    } else {
#pragma unroll
        for (int j = 0; j < kMaxTaps - 1; j++) win[j] = j < nt ? cv.x[(t0 - nt + j) * cv.ld + c] + xb : 0.f; // kConvTokens > taps
    }
    const int64_t b = c / d, k = c - b * d;
    constexpr int kAhead = 8; // inputs of eight tokens in flight together
    for (int64_t tb = t0; tb < t1; tb += kAhead) {
        float xv[kAhead];
#pragma unroll
        for (int s = 0; s < kAhead; s++) xv[s] = cv.x[min(tb + s, t1 - 1) * cv.ld + c] + xb;
#pragma unroll
        for (int s = 0; s < kAhead; s++) {
            const int64_t t = tb + s;
            if (t >= t1) break;
            const float v = conv_tap(wt, win, nt, xv[s], wb);
            u[t * C + c] = v;
            if (split) {
                __nv_bfloat16 *row = split + (b * T + t) * 3 * d + k;
                const __nv_bfloat16 hi = __float2bfloat16_rn(v);
                const float r1 = v - __bfloat162float(hi);
                const __nv_bfloat16 mid = __float2bfloat16_rn(r1);
                row[0] = hi;
                row[d] = mid;
                row[2 * d] = __float2bfloat16_rn(r1 - __bfloat162float(mid));
            }
        }
    }
    if (t0 == 0)
        for (int64_t s = max((int64_t)0, T - nt); s < T; s++) cv.hist[((p0 + (int)s) % cv.L) * C + c] = cv.x[s * cv.ld + c] + xb;
}

// ------------------------------------------------------------------------------------------------ portions: gates in fp32
// z[b][t][n] = sum_k w[b][n][k] u[t][b d + k], n < 2d (the rows of W_r, then of W_i): 64 x 64 tile per CTA, 4 x 4 per thread
template <typename E>
__global__ void __launch_bounds__(256) rglru_gates_kernel(const float *__restrict__ u, int64_t T, int nb, int d, const E *__restrict__ w,
                                                          float *__restrict__ z) {
    constexpr int BM = 64, BN = 64, BK = 16;
    __shared__ float sa[BK][BM + 4], sb[BK][BN + 4];
    const int b = blockIdx.z, N = 2 * d, n0 = blockIdx.x * BN;
    const int64_t m0 = (int64_t)blockIdx.y * BM, C = (int64_t)nb * d;
    const int tid = threadIdx.x, tx = tid & 15, ty = tid >> 4, lr = tid >> 2, lk = (tid & 3) * 4;
    const float *arow = m0 + lr < T ? u + (m0 + lr) * C + (int64_t)b * d : nullptr;
    const E *wrow = n0 + lr < N ? w + ((int64_t)b * N + n0 + lr) * d : nullptr;
    float acc[4][4];
#pragma unroll
    for (int i = 0; i < 4; i++)
#pragma unroll
        for (int j = 0; j < 4; j++) acc[i][j] = 0.f;
    for (int k0 = 0; k0 < d; k0 += BK) {
#pragma unroll
        for (int v = 0; v < 4; v++) {
            const int k = k0 + lk + v;
            sa[lk + v][lr] = (arow && k < d) ? arow[k] : 0.f;
            sb[lk + v][lr] = (wrow && k < d) ? to_f32(wrow[k]) : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int kk = 0; kk < BK; kk++) {
            const float4 av = *reinterpret_cast<const float4 *>(&sa[kk][ty * 4]), bv = *reinterpret_cast<const float4 *>(&sb[kk][tx * 4]);
            const float ar[4] = {av.x, av.y, av.z, av.w}, br[4] = {bv.x, bv.y, bv.z, bv.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(ar[i], br[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int64_t m = m0 + ty * 4 + i;
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int n = n0 + tx * 4 + j;
            if (m < T && n < N) z[((int64_t)b * T + m) * N + n] = acc[i][j];
        }
    }
}

// ------------------------------------------------------------------------------------------------ portions: scan
// CH channels per CTA; 32 / CH pieces of time per warp, TP tokens a piece, so a sweep covers pieces * TP tokens.  A thread
// keeps its piece's decays and inputs in registers between the local pass and the outputs.
constexpr int kScanWarps = 16, kScanTP = 8;

template <typename E, int CH>
__global__ void __launch_bounds__(32 * kScanWarps) rglru_scan_kernel(const float *__restrict__ z, const float *__restrict__ u, const float *__restrict__ y,
                                                                     int64_t ld, int64_t T, int nb, int d, const float *__restrict__ yb,
                                                                     const float *__restrict__ b_ri, const float *__restrict__ rate, float *state,
                                                                     E *__restrict__ out) {
    constexpr int NP = kScanWarps * 32 / CH; // pieces of a sweep
    __shared__ float sA[NP][CH], sB[NP][CH], carry[CH];
    const int cl = threadIdx.x % CH, piece = threadIdx.x / CH;
    const int64_t C = (int64_t)nb * d, c = (int64_t)blockIdx.x * CH + cl;
    const bool live = c < C;
    const int64_t b = live ? c / d : 0, k = live ? c - b * d : 0;
    const float br = live ? b_ri[b * 2 * d + k] : 0.f, bi = live ? b_ri[b * 2 * d + d + k] : 0.f, rt = live ? rate[c] : 0.f, ybc = live ? yb[c] : 0.f;
    if (piece == 0) carry[cl] = live ? state[c] : 0.f;
    __syncthreads();
    for (int64_t tb = 0; tb < T; tb += (int64_t)NP * kScanTP) {
        const int64_t t0 = tb + (int64_t)piece * kScanTP;
        float a[kScanTP], in[kScanTP], zr[kScanTP], zi[kScanTP], uv[kScanTP], yv[kScanTP];
#pragma unroll
        for (int s = 0; s < kScanTP; s++) { // a piece's loads are independent and in flight together
            const int64_t t = t0 + s;
            const bool on = live && t < T;
            const int64_t zo = on ? (b * T + t) * 2 * d + k : 0;
            zr[s] = on ? z[zo] : 0.f;
            zi[s] = on ? z[zo + d] : 0.f;
            uv[s] = on ? u[t * C + c] : 0.f;
            yv[s] = on ? y[t * ld + c] : 0.f;
        }
        float A = 1.f, B = 0.f;
#pragma unroll
        for (int s = 0; s < kScanTP; s++) {
            a[s] = 1.f, in[s] = 0.f; // past the end: nothing changes
            if (live && t0 + s < T) rglru_terms(zr[s] + br, zi[s] + bi, uv[s], rt, &a[s], &in[s]);
            A *= a[s];
            B = fmaf(a[s], B, in[s]);
        }
        sA[piece][cl] = A;
        sB[piece][cl] = B;
        __syncthreads();
        float S = carry[cl];
        for (int p = 0; p < piece; p++) S = fmaf(sA[p][cl], S, sB[p][cl]);
#pragma unroll
        for (int s = 0; s < kScanTP; s++) {
            S = fmaf(a[s], S, in[s]);
            if (live && t0 + s < T) out[(t0 + s) * C + c] = from_f32<E>(S * gelu_tanh_f32(yv[s] + ybc));
        }
        __syncthreads(); // every piece has read the carry
        if (piece == NP - 1) carry[cl] = S;
        __syncthreads();
    }
    if (piece == 0 && live) state[c] = carry[cl];
}

} // namespace

extern "C" {

#define GGB_CHECK_DT(dt) GGB_CHECK_ARG((dt) == GGB_TYPE_BF16 || (dt) == GGB_TYPE_F32, "dtype %d is neither bf16 nor f32", (int)(dt))

int ggb_rglru_history_rows(int taps) { return taps > 1 ? taps - 1 + kStepT : 0; }

int ggb_rglru_step_form(int64_t T, int d) { return T <= kStepT && (int64_t)kStepT * d * 4 <= 160 * 1024; }

int ggb_rglru_split_fits(int dt, int64_t T, int d) {
    return dt == GGB_TYPE_BF16 && T >= 64 && d % 64 == 0 && ggb_gemm_grouped_bf16_fits(2 * (int64_t)d, 3 * (int64_t)d, 2 * (int64_t)d);
}

static bool rglru_conv_ok(const float *x, int64_t ld, int64_t T, int nb, int d, const float *cw, const float *cb, int taps, const float *xb, const float *hist) {
    return x && cw && cb && xb && T > 0 && nb > 0 && d > 0 && ld >= (int64_t)nb * d && taps >= 1 && taps <= kMaxTaps && (taps == 1 || hist);
}

int ggb_op_rglru_step(int dt, const float *x, const float *y, int64_t ld, int64_t T, int nb, int d, const float *conv_w, const float *conv_b, int taps,
                      const float *xb, const float *yb, const void *w_ri, const float *b_ri, const float *rate, const int32_t *pos0, float *hist,
                      float *state, void *out) {
    GGB_REQUIRE_INIT();
    GGB_CHECK_DT(dt);
    GGB_CHECK_ARG(rglru_conv_ok(x, ld, T, nb, d, conv_w, conv_b, taps, xb, hist) && y && yb && w_ri && b_ri && rate && pos0 && state && out &&
                      nb <= 65535 && ggb_rglru_step_form(T, d),
                  "rglru_step: bad arguments (%lld tokens, at most %d; taps %d, at most %d)", (long long)T, kStepT, taps, kMaxTaps);
    const rglru_conv_args cv{x, conv_w, conv_b, xb, ld, taps, ggb_rglru_history_rows(taps), hist};
    // channels per CTA: 8 (one a warp) while every CTA then finds an SM with room, more for wide models
    int per = 8;
    while (per < 64 && (int64_t)nb * ((d + per - 1) / per) > 4 * (int64_t)ggb_sm_count()) per *= 2;
    const dim3 grid((unsigned)((d + per - 1) / per), (unsigned)nb);
    const int ve = dt == GGB_TYPE_BF16 ? 8 : 4;
    const int vec = d % ve == 0 && ((uintptr_t)w_ri & 15) == 0;
    const int tt = T <= 1 ? 1 : T <= 2 ? 2 : T <= 4 ? 4 : 8;
    const size_t smem = (size_t)tt * d * 4;
#define RS_LAUNCH(E, TT)                                                                                                                       \
    {                                                                                                                                          \
        auto kf = rglru_step_kernel<E, TT>;                                                                                                    \
        if (smem > 48 * 1024) GGB_CUDA(cudaFuncSetAttribute(kf, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));                       \
        kf<<<grid, 256, smem, ggb_cuda_stream()>>>(cv, y, yb, (int)T, d, per, (const E *)w_ri, b_ri, rate, pos0, state, (E *)out, vec);         \
    }
#define RS_T(E)                        \
    {                                  \
        if (tt == 1) RS_LAUNCH(E, 1)   \
        else if (tt == 2) RS_LAUNCH(E, 2) \
        else if (tt == 4) RS_LAUNCH(E, 4) \
        else RS_LAUNCH(E, 8)           \
    }
    if (dt == GGB_TYPE_BF16) RS_T(__nv_bfloat16) else RS_T(float)
#undef RS_T
#undef RS_LAUNCH
    GGB_LAUNCH_CHECK();
    return GGB_OK;
}

int ggb_op_rglru_conv(const float *x, int64_t ld, int64_t T, int nb, int d, const float *conv_w, const float *conv_b, int taps, const float *xb,
                      const int32_t *pos0, float *hist, float *u, void *split, int32_t *offsets) {
    GGB_REQUIRE_INIT();
    GGB_CHECK_ARG(rglru_conv_ok(x, ld, T, nb, d, conv_w, conv_b, taps, xb, hist) && pos0 && u && (!split || offsets) && (int64_t)nb * T < (1ll << 31),
                  "rglru_conv: bad arguments (taps %d, at most %d)", taps, kMaxTaps);
    const rglru_conv_args cv{x, conv_w, conv_b, xb, ld, taps, std::max(1, ggb_rglru_history_rows(taps)), hist};
    const int64_t C = (int64_t)nb * d;
    const dim3 grid((unsigned)((C + 127) / 128), (unsigned)((T + kConvTokens - 1) / kConvTokens));
    rglru_conv_kernel<<<grid, 128, 0, ggb_cuda_stream()>>>(cv, T, nb, d, pos0, u, (__nv_bfloat16 *)split, offsets);
    GGB_LAUNCH_CHECK();
    return GGB_OK;
}

int ggb_op_rglru_gates(int dt, const float *u, const void *split, const int32_t *offsets, int64_t T, int nb, int d, const void *w_ri, const void *w_ri3,
                       float *z) {
    GGB_REQUIRE_INIT();
    GGB_CHECK_DT(dt);
    GGB_CHECK_ARG(u && w_ri && z && T > 0 && nb > 0 && d > 0 && nb <= 65535, "rglru_gates: bad arguments");
    if (split && w_ri3 && ggb_rglru_split_fits(dt, T, d)) { // every block is a group of T rows of its own
        GGB_CHECK_ARG(offsets != nullptr, "rglru_gates: the split form needs its offsets");
        return ggb_gemm_grouped_bf16(w_ri3, 2 * (int64_t)d, 3 * (int64_t)d, split, T, nb, offsets, z, nullptr, GGB_ACT_NONE, 2 * (int64_t)d);
    }
    const dim3 grid((unsigned)((2 * d + 63) / 64), (unsigned)((T + 63) / 64), (unsigned)nb);
    if (dt == GGB_TYPE_BF16) rglru_gates_kernel<<<grid, 256, 0, ggb_cuda_stream()>>>(u, T, nb, d, (const __nv_bfloat16 *)w_ri, z);
    else rglru_gates_kernel<<<grid, 256, 0, ggb_cuda_stream()>>>(u, T, nb, d, (const float *)w_ri, z);
    GGB_LAUNCH_CHECK();
    return GGB_OK;
}

int ggb_op_rglru_scan(int dt, const float *z, const float *u, const float *y, int64_t ld, int64_t T, int nb, int d, const float *yb, const float *b_ri,
                      const float *rate, float *state, void *out) {
    GGB_REQUIRE_INIT();
    GGB_CHECK_DT(dt);
    GGB_CHECK_ARG(z && u && y && yb && b_ri && rate && state && out && T > 0 && nb > 0 && d > 0 && ld >= (int64_t)nb * d, "rglru_scan: bad arguments");
    const int64_t C = (int64_t)nb * d;
#define SC_LAUNCH(E, CH) rglru_scan_kernel<E, CH><<<(unsigned)((C + CH - 1) / CH), 32 * kScanWarps, 0, ggb_cuda_stream()>>>(z, u, y, ld, T, nb, d, yb, b_ri, rate, state, (E *)out);
    // fewer channels per CTA while that brings more SMs to work
#define SC_CH(E)                                               \
    {                                                          \
        if (C >= 32 * (int64_t)ggb_sm_count()) { SC_LAUNCH(E, 32) } \
        else if (C >= 12 * (int64_t)ggb_sm_count()) { SC_LAUNCH(E, 16) } \
        else { SC_LAUNCH(E, 8) }                               \
    }
    if (dt == GGB_TYPE_BF16) SC_CH(__nv_bfloat16) else SC_CH(float)
#undef SC_CH
#undef SC_LAUNCH
    GGB_LAUNCH_CHECK();
    return GGB_OK;
}

} // extern "C"
