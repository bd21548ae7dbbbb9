// window_attention.cu — grouped-query soft-max attention over a sliding window of a paged cache, with rotary positions
// on queries and keys and with rotated values: the value of position j is cached turned by j, the weighted sum of a head
// is turned back by the reader's position i, so that what a head adds depends on i - j only.
//
// The cache row of a position holds [k (G * D) | v (G * Dv)] in the storage type; page tables and positions are read
// on the device (a captured one-token step replays anywhere).  Scores, soft-max and the weighted sum are fp32.
//
// qkv_store: one CTA per token: root mean square over the whole q and the whole k projection, weights, rotation, store.
// window_attn, both forms: lane = key for the scores, lane = pair of value coordinates for the weighted sum, running
// maximum and sum in registers.
//   portions (window_attn_tile_kernel): a CTA owns 32 consecutive tokens of one head, 4 per warp.  Their windows
//   overlap almost wholly, so every tile of 32 cache rows is staged once in shared memory as fp32 (row pitch odd in words:
//   lane = row reads are conflict-free) and serves all 32 queries; a K word read feeds 4 multiply-adds.
//   steps of few tokens (window_attn_kernel): 8 warps split one (token, head)'s keys, rows straight from the cache
//   (several loads in flight), parts merged through shared memory.
//
// The same kernels serve other masks and layouts, all arguments: the visible range of a query is a sliding window or the
// chunk of consecutive positions it lies in (chunks counted from position 0), a score may pass a soft cap
// cap * tanh(s / cap) before the soft-max, and the rotary pairs of q and k are neighbours (2i, 2i + 1) or halves
// (i, i + rot_dims / 2).  A window may keep the first positions of the sequence visible (keep_first): their tiles come
// first, then those of the window.
//
// MAPS 2 is differential attention: a head has two query / key maps over the same values, each with a soft-max of its own;
// the head's output is a1 - lambda a2, divided by its root mean square, scaled, and gated element by element.  One CTA runs
// both maps of a head, so every value row is read once for both, and the combination is the epilogue of the kernel that
// holds the sums.
//
// One-map heads have two more choices at their end: a sink per head (one more exp(sink) in the soft-max's denominator that no
// value goes with) and the gate per element.  head_qkv_store divides every head of q and k by its own root mean square.
//
// Compiled with -fmad=false: multiply-adds are spelled fmaf().
#include <algorithm>

#include "common.cuh"
#include "dense.cuh"

namespace {

constexpr int kMaxDvRegs = 8; // value coordinates per lane: Dv <= 32 * kMaxDvRegs
constexpr int kWarps = 8;
constexpr int kMaxSplit = 16; // CTAs that share one (token, head) of a short step

// what becomes of a head's weighted sums.  MAPS 1: the sum over l, or over l + exp(sink[head]) with a sink.  MAPS 2: o = a1 -
// lambda a2; o <- o / sqrt(mean(o^2) + eps) * scale.  Then, with a gate, times sigmoid(gate[token][head * Dv + c])
struct finish_args {
    float lambda = 0.f, scale = 1.f, eps = 0.f;
    const float *gate = nullptr; // fp32 rows of stride ldg, or null
    int64_t ldg = 0;
    const float *sink = nullptr; // a score per head, or null
};

// the first position the query at position i sees: everything (size <= 0), the last `size` positions, or its chunk
__device__ __forceinline__ int64_t first_visible(int64_t i, int64_t size, int chunked) {
    if (size <= 0) return 0;
    return chunked ? i - i % size : max((int64_t)0, i - size + 1);
}
__device__ __forceinline__ float soft_cap(float s, float cap) { return cap > 0.f ? cap * tanhf(s / cap) : s; }

template <typename E>
__global__ void __launch_bounds__(256) window_qkv_store_kernel(const float *__restrict__ q, const float *__restrict__ k, const float *__restrict__ v,
                                                               int64_t ld, int H, int G, int D, int Gv, int Dv, const float *__restrict__ qn_w,
                                                               const float *__restrict__ kn_w, float eps, int rot_dims, int rot_halves,
                                                               const float *__restrict__ cs_k, const float *__restrict__ cs_v, float scale,
                                                               const int32_t *__restrict__ pos0, const int32_t *__restrict__ table, int B,
                                                               E *__restrict__ cache, int64_t cache_ld, float *__restrict__ q_out) {
    __shared__ float red[2][8];
    const int64_t t = blockIdx.x;
    const int64_t pos = (int64_t)*pos0 + t;
    const float *qr = q + t * ld, *kr = k + t * ld, *vr = v + t * ld;
    const int nq = H * D, nk = G * D, nv = Gv * Dv;
    float rq = 1.f, rk = 1.f;
    if (qn_w || kn_w) {
        float sq = 0.f, sk = 0.f;
        for (int i = threadIdx.x; i < nq; i += blockDim.x) sq = fmaf(qr[i], qr[i], sq);
        for (int i = threadIdx.x; i < nk; i += blockDim.x) sk = fmaf(kr[i], kr[i], sk);
        sq = warp_sum_f32(sq);
        sk = warp_sum_f32(sk);
        if ((threadIdx.x & 31) == 0) {
            red[0][threadIdx.x >> 5] = sq;
            red[1][threadIdx.x >> 5] = sk;
        }
        __syncthreads();
        float tq = 0.f, tk = 0.f;
#pragma unroll
        for (int i = 0; i < 8; i++) {
            tq += red[0][i];
            tk += red[1][i];
        }
        if (qn_w) rq = 1.0f / sqrtf(tq / (float)nq + eps);
        if (kn_w) rk = 1.0f / sqrtf(tk / (float)nk + eps);
    }
    E *row = cache + ((int64_t)table[pos / B] * B + pos % B) * cache_ld;
    const float *ck = cs_k ? cs_k + pos * (rot_dims / 2) * 2 : nullptr;
    // pairs of q and k: pair m of a head is (2m, 2m + 1), or with rot_halves (m, m + rot_dims / 2) for the rotated pairs and
    // the neighbours behind them for the rest; pair m < rot_dims / 2 turns by the table's entry m
    for (int p = threadIdx.x; p < (nq + nk) / 2; p += blockDim.x) {
        const bool is_q = p < nq / 2;
        const int e = is_q ? 2 * p : 2 * p - nq; // even coordinate inside the projection
        const float *src = is_q ? qr : kr;
        const float *nw = is_q ? qn_w : kn_w;
        const float r = is_q ? rq : rk;
        const int d = e % D, m = d / 2;
        const bool turn = ck && d < rot_dims;
        int e0 = e, e1 = e + 1;
        if (rot_halves) {
            if (turn) e0 = e - d + m, e1 = e0 + rot_dims / 2;
            else e0 = e - d + rot_dims + 2 * (m - rot_dims / 2), e1 = e0 + 1;
        }
        float u = src[e0], w = src[e1];
        if (nw) {
            u = u * r * nw[e0];
            w = w * r * nw[e1];
        }
        if (turn) {
            const float c = ck[d], s = ck[d + 1]; // pair m: [cos, sin]
            const float u2 = u * c - w * s, w2 = w * c + u * s;
            u = u2;
            w = w2;
        }
        if (is_q) {
            q_out[t * nq + e0] = u * scale;
            q_out[t * nq + e1] = w * scale;
        } else {
            row[e0] = from_f32<E>(u);
            row[e1] = from_f32<E>(w);
        }
    }
    const float *cv = cs_v ? cs_v + pos * (Dv / 2) * 2 : nullptr;
    for (int p = threadIdx.x; p < nv / 2; p += blockDim.x) {
        const int e = 2 * p, d = e % Dv;
        float u = vr[e], w = vr[e + 1];
        if (cv) {
            const float c = cv[d], s = cv[d + 1];
            const float u2 = u * c - w * s, w2 = w * c + u * s;
            u = u2;
            w = w2;
        }
        row[nk + e] = from_f32<E>(u);
        row[nk + e + 1] = from_f32<E>(w);
    }
}

// the same with a norm per head: a warp takes one head of q, k or v of one token (rows y * 8 + warp of H + 2 G).  q and k are divided
// by the root mean square over the head's D numbers, times a weight of D numbers that all heads share (null: none), before the rotation.
template <typename E>
__global__ void __launch_bounds__(256) head_qkv_store_kernel(const float *__restrict__ q, const float *__restrict__ k, const float *__restrict__ v, int64_t ld,
                                                             int H, int G, int D, int Dv, const float *__restrict__ qn_w, const float *__restrict__ kn_w,
                                                             float eps, int rot_dims, int rot_halves, const float *__restrict__ cs, float scale,
                                                             const int32_t *__restrict__ pos0, const int32_t *__restrict__ table, int B,
                                                             E *__restrict__ cache, int64_t cache_ld, float *__restrict__ q_out) {
    const int lane = threadIdx.x & 31, item = (int)blockIdx.y * 8 + (int)(threadIdx.x >> 5);
    if (item >= H + 2 * G) return;
    const int64_t t = blockIdx.x, pos = (int64_t)*pos0 + t;
    E *row = cache + ((int64_t)table[pos / B] * B + pos % B) * cache_ld;
    if (item >= H + G) { // a value head
        const int g = item - H - G;
        const float *src = v + t * ld + (int64_t)g * Dv;
        E *dst = row + (int64_t)G * D + (int64_t)g * Dv;
        for (int c = lane; c < Dv; c += 32) dst[c] = from_f32<E>(src[c]);
        return;
    }
    const bool is_q = item < H;
    const float *src = is_q ? q + t * ld + (int64_t)item * D : k + t * ld + (int64_t)(item - H) * D;
    const float *nw = is_q ? qn_w : kn_w;
    float ss = 0.f;
    for (int d = lane; d < D; d += 32) ss = fmaf(src[d], src[d], ss);
    const float r = 1.0f / sqrtf(warp_sum_f32(ss) / (float)D + eps);
    float *qd = q_out + (t * H + item) * D;
    E *kd = row + (int64_t)(item - H) * D;
    auto normed = [&](int d) { return nw ? src[d] * r * nw[d] : src[d] * r; };
    auto put = [&](int d, float x) {
        if (is_q) qd[d] = x * scale;
        else kd[d] = from_f32<E>(x);
    };
    const int half = rot_dims / 2;
    const float *ct = cs + pos * rot_dims;
    for (int m = lane; m < half; m += 32) {
        const int d0 = rot_halves ? m : 2 * m, d1 = rot_halves ? m + half : 2 * m + 1;
        const float u = normed(d0), w = normed(d1), c = ct[2 * m], s = ct[2 * m + 1];
        put(d0, u * c - w * s);
        put(d1, w * c + u * s);
    }
    for (int d = rot_dims + lane; d < D; d += 32) put(d, normed(d));
}

template <typename E> struct RowVec { // 16 bytes of a cache row
    static constexpr int n = 16 / (int)sizeof(E);
    uint4 raw;
    __device__ __forceinline__ float at(int i) const { return to_f32(reinterpret_cast<const E *>(&raw)[i]); }
};

// what a head's weighted sum becomes: divided by the soft-max sum, turned back by the reader's position, gated, stored
template <typename E, int NP = kMaxDvRegs / 2>
__device__ __forceinline__ void window_finish(const float *acc, float m, float l, int64_t i, int64_t t, int h, int lane, int Dv,
                                              const float *__restrict__ cs_v, const finish_args &fa, E *orow) {
    float inv = 1.0f / l;
    if (fa.sink) { // sum and weighted sum are relative to the running maximum m (finite: a query sees itself)
        const float s0 = fa.sink[h], M = fmaxf(m, s0), f = expf(m - M);
        inv = f / (l * f + expf(s0 - M));
    }
    const float *gr = fa.gate ? fa.gate + t * fa.ldg + (int64_t)h * Dv : nullptr;
    const float *cv = cs_v ? cs_v + i * (Dv / 2) * 2 : nullptr;
#pragma unroll
    for (int r = 0; r < NP; r++) {
        const int c = 2 * lane + 64 * r;
        if (c < Dv) {
            float u = acc[2 * r] * inv, w = acc[2 * r + 1] * inv;
            if (cv) { // turned back: by -i
                const float cs = cv[c], sn = cv[c + 1];
                const float u2 = u * cs + w * sn, w2 = w * cs - u * sn;
                u = u2;
                w = w2;
            }
            if (gr) {
                u = u / (1.0f + expf(-gr[c]));
                w = w / (1.0f + expf(-gr[c + 1]));
            }
            orow[c] = from_f32<E>(u);
            orow[c + 1] = from_f32<E>(w);
        }
    }
}

// the same for the two maps of a differential head (all lanes of the warp take part)
template <typename E, int NP = kMaxDvRegs / 2>
__device__ __forceinline__ void diff_finish(const float *acc1, float l1, const float *acc2, float l2, int64_t t, int h, int lane, int Dv,
                                            const finish_args &da, E *orow) {
    const float i1 = 1.0f / l1, i2 = da.lambda / l2;
    float o[2 * NP], ss = 0.f;
#pragma unroll
    for (int r = 0; r < NP; r++) {
        const bool in = 2 * lane + 64 * r < Dv;
#pragma unroll
        for (int u = 2 * r; u < 2 * r + 2; u++) {
            o[u] = in ? acc1[u] * i1 - acc2[u] * i2 : 0.f;
            ss = fmaf(o[u], o[u], ss);
        }
    }
    const float f = da.scale / sqrtf(warp_sum_f32(ss) / (float)Dv + da.eps);
    const float *gr = da.gate ? da.gate + t * da.ldg + (int64_t)h * Dv : nullptr;
#pragma unroll
    for (int r = 0; r < NP; r++) {
        const int c = 2 * lane + 64 * r;
        if (c < Dv) {
            float u = o[2 * r] * f, w = o[2 * r + 1] * f;
            if (gr) {
                u = u / (1.0f + expf(-gr[c]));
                w = w / (1.0f + expf(-gr[c + 1]));
            }
            orow[c] = from_f32<E>(u);
            orow[c + 1] = from_f32<E>(w);
        }
    }
}

constexpr int kPartW = 2 + 32 * kMaxDvRegs; // one part: running maximum, sum, weighted sum as the lanes hold it

// The key tiles of one query: first those of the kept positions [0, n_keep), n_keep <= jlo, then those of [jlo, i].
struct key_tiles {
    int64_t jlo, n_keep;
    int n_kt; // tiles of the kept positions
    __device__ __forceinline__ key_tiles(int64_t jlo_, int64_t keep) : jlo(jlo_), n_keep(min(keep, jlo_)), n_kt((int)((n_keep + 31) / 32)) {}
    __device__ __forceinline__ int64_t first(int64_t n) const { return n < n_kt ? 32 * n : jlo + 32 * (n - n_kt); }
    __device__ __forceinline__ int64_t last(int64_t n, int64_t i) const { return n < n_kt ? n_keep - 1 : i; } // last position a tile may hold
};

// The CTA (token blockIdx.x, head blockIdx.y, split blockIdx.z of gridDim.z) takes the key tiles whose number is
// split * 8 + warp modulo 8 * splits, one warp a tile.  One split: the result goes to `out`; several: the CTA's merged
// part goes to `part` and window_merge_kernel finishes.
template <typename E, int MAPS>
__global__ void __launch_bounds__(32 * kWarps) window_attn_kernel(const float *__restrict__ q, const E *__restrict__ cache, int64_t cache_ld,
                                                                  const int32_t *__restrict__ table, int B, const int32_t *__restrict__ pos0,
                                                                  int64_t T, int H, int G, int D, int Dv, int64_t window, int chunked, int64_t keep,
                                                                  float cap, const float *__restrict__ cs_v, finish_args da, E *__restrict__ out,
                                                                  int vec, float *__restrict__ part_out) {
    extern __shared__ __align__(16) float wa_smem[]; // q: [kWarps][MAPS][Dp]; merge: [kWarps][MAPS][kPartW]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int h = blockIdx.y, g = h / (H / G);
    const int Dp = (D + 3) & ~3;
    const int64_t t = blockIdx.x;
    const bool active = t < T;
    float *sq = wa_smem + warp * MAPS * Dp;
    if (active)
        for (int d = lane; d < MAPS * Dp; d += 32) {
            const int mp = d / Dp, dd = d - mp * Dp;
            sq[d] = dd < D ? q[((t * H + h) * MAPS + mp) * D + dd] : 0.f;
        }
    __syncwarp();
    const int64_t i = (int64_t)*pos0 + (active ? t : 0);
    const key_tiles kt(first_visible(i, window, chunked), keep);
    const int nreg = (Dv + 63) / 64; // pairs of coordinates per lane: c = 2 * lane + 64 * r
    float acc[MAPS][kMaxDvRegs], m[MAPS], l[MAPS];
#pragma unroll
    for (int a = 0; a < MAPS; a++) {
        m[a] = -INFINITY, l[a] = 0.f;
#pragma unroll
        for (int r = 0; r < kMaxDvRegs; r++) acc[a][r] = 0.f;
    }
    const int64_t koff = (int64_t)g * MAPS * D, voff = (int64_t)G * MAPS * D + (int64_t)g * Dv;
    if (active) {
        const int64_t step = kWarps * (int64_t)gridDim.z;
        for (int64_t n = (int64_t)blockIdx.z * kWarps + warp;; n += step) {
            const int64_t j0 = kt.first(n), j_last = kt.last(n, i);
            if (j0 > j_last) break; // only behind the last tile of the window: the kept tiles hold a position each
            const int64_t j = j0 + lane;
            float s[MAPS];
#pragma unroll
            for (int a = 0; a < MAPS; a++) s[a] = -INFINITY;
            // the lane's row of the cache, looked up once: the weighted sum below gets the other lanes' rows by shuffle
            const int64_t jc = min(j, j_last);
            const int64_t my_row = (int64_t)table[jc / B] * B + jc % B;
            if (j <= j_last) {
#pragma unroll
                for (int a = 0; a < MAPS; a++) {
                    const E *kr = cache + my_row * cache_ld + koff + a * D;
                    const float *qa = sq + a * Dp;
                    float a0 = 0.f, a1 = 0.f;
                    if (vec) {
                        constexpr int VN = RowVec<E>::n;
#pragma unroll 8
                        for (int d = 0; d < D; d += VN) {
                            RowVec<E> kv;
                            kv.raw = *reinterpret_cast<const uint4 *>(kr + d);
#pragma unroll
                            for (int u = 0; u < VN; u += 2) {
                                a0 = fmaf(kv.at(u), qa[d + u], a0);
                                a1 = fmaf(kv.at(u + 1), qa[d + u + 1], a1);
                            }
                        }
                    } else {
                        for (int d = 0; d < D; d++) a0 = fmaf(to_f32(kr[d]), qa[d], a0);
                    }
                    s[a] = soft_cap(a0 + a1, cap);
                }
            }
            float p[MAPS];
#pragma unroll
            for (int a = 0; a < MAPS; a++) {
                const float m_new = fmaxf(m[a], warp_max_f32(s[a])); // finite: key j0 of the tile is always visible
                p[a] = j <= j_last ? expf(s[a] - m_new) : 0.f;
                const float corr = expf(m[a] - m_new); // m = -inf at the first tile: 0
                l[a] = l[a] * corr + warp_sum_f32(p[a]);
#pragma unroll
                for (int r = 0; r < kMaxDvRegs; r++) acc[a][r] *= corr;
                m[a] = m_new;
            }
            const int n_keys = (int)min((int64_t)32, j_last - j0 + 1);
            // rows in groups of 8: the loads of a group are independent and in flight together (a row past the last
            // visible one repeats it with weight 0)
            for (int jb = 0; jb < n_keys; jb += 8) {
                const E *vrow[8];
                float pj[MAPS][8];
#pragma unroll
                for (int u = 0; u < 8; u++) {
                    const int jj = min(jb + u, n_keys - 1);
#pragma unroll
                    for (int a = 0; a < MAPS; a++) {
                        const float pv = __shfl_sync(0xffffffffu, p[a], jj);
                        pj[a][u] = jb + u < n_keys ? pv : 0.f;
                    }
                    vrow[u] = cache + __shfl_sync(0xffffffffu, my_row, jj) * cache_ld + voff;
                }
#pragma unroll
                for (int r = 0; r < kMaxDvRegs / 2; r++) {
                    const int c = 2 * lane + 64 * r;
                    if (r < nreg && c < Dv) {
                        float v0[8], v1[8];
#pragma unroll
                        for (int u = 0; u < 8; u++) {
                            v0[u] = to_f32(vrow[u][c]);
                            v1[u] = to_f32(vrow[u][c + 1]);
                        }
#pragma unroll
                        for (int u = 0; u < 8; u++)
#pragma unroll
                            for (int a = 0; a < MAPS; a++) {
                                acc[a][2 * r] = fmaf(pj[a][u], v0[u], acc[a][2 * r]);
                                acc[a][2 * r + 1] = fmaf(pj[a][u], v1[u], acc[a][2 * r + 1]);
                            }
                    }
                }
            }
        }
    }
    { // merge the warps' parts: [m, l, acc...] per warp and map
        __syncthreads();
        float *part = wa_smem + kWarps * MAPS * Dp;
        const int pw = MAPS * kPartW;
#pragma unroll
        for (int a = 0; a < MAPS; a++) {
            float *pa = part + warp * pw + a * kPartW;
            if (lane == 0) {
                pa[0] = m[a];
                pa[1] = l[a];
            }
#pragma unroll
            for (int r = 0; r < kMaxDvRegs; r++) pa[2 + r * 32 + lane] = acc[a][r];
        }
        __syncthreads();
        if (warp != 0) return;
#pragma unroll
        for (int a = 0; a < MAPS; a++) {
            const float *pa = part + a * kPartW;
            float M = -INFINITY;
            for (int w = 0; w < kWarps; w++) M = fmaxf(M, pa[w * pw]);
            l[a] = 0.f;
#pragma unroll
            for (int r = 0; r < kMaxDvRegs; r++) acc[a][r] = 0.f;
            for (int w = 0; w < kWarps; w++) {
                const float mw = pa[w * pw];
                if (mw == -INFINITY) continue; // a warp without keys
                const float f = expf(mw - M);
                l[a] = fmaf(pa[w * pw + 1], f, l[a]);
#pragma unroll
                for (int r = 0; r < kMaxDvRegs; r++) acc[a][r] = fmaf(pa[w * pw + 2 + r * 32 + lane], f, acc[a][r]);
            }
            m[a] = M;
        }
    }
    if (gridDim.z > 1) { // M = -inf, l = 0 when the split had no tile
        float *po = part_out + ((t * H + h) * gridDim.z + blockIdx.z) * (MAPS * kPartW);
#pragma unroll
        for (int a = 0; a < MAPS; a++) {
            if (lane == 0) {
                po[a * kPartW] = m[a];
                po[a * kPartW + 1] = l[a];
            }
#pragma unroll
            for (int r = 0; r < kMaxDvRegs; r++) po[a * kPartW + 2 + r * 32 + lane] = acc[a][r];
        }
        return;
    }
    E *orow = out + (t * H + h) * Dv;
    if (MAPS == 1) window_finish(acc[0], m[0], l[0], i, t, h, lane, Dv, cs_v, da, orow);
    else diff_finish(acc[0], l[0], acc[MAPS - 1], l[MAPS - 1], t, h, lane, Dv, da, orow);
}

// one warp per (token, head): the splits' parts merged, then as above
template <typename E, int MAPS>
__global__ void __launch_bounds__(32) window_merge_kernel(const float *__restrict__ part, int n_split, const int32_t *__restrict__ pos0, int H, int Dv,
                                                         const float *__restrict__ cs_v, finish_args da, E *__restrict__ out) {
    const int64_t t = blockIdx.x;
    const int h = blockIdx.y, lane = threadIdx.x;
    constexpr int pw = MAPS * kPartW;
    float m[MAPS], l[MAPS], acc[MAPS][kMaxDvRegs];
#pragma unroll
    for (int a = 0; a < MAPS; a++) {
        const float *pp = part + (t * H + h) * n_split * pw + a * kPartW;
        float M = -INFINITY;
#pragma unroll 4
        for (int s = 0; s < n_split; s++) M = fmaxf(M, pp[s * pw]);
        m[a] = M;
        l[a] = 0.f;
#pragma unroll
        for (int r = 0; r < kMaxDvRegs; r++) acc[a][r] = 0.f;
#pragma unroll 4
        for (int s = 0; s < n_split; s++) { // a split without keys holds m = -inf and zeros: its weight is 0; the loads do not wait for it
            const float f = expf(pp[s * pw] - M);
            l[a] = fmaf(pp[s * pw + 1], f, l[a]);
#pragma unroll
            for (int r = 0; r < kMaxDvRegs; r++) acc[a][r] = fmaf(pp[s * pw + 2 + r * 32 + lane], f, acc[a][r]);
        }
    }
    E *orow = out + (t * H + h) * Dv;
    if (MAPS == 1) window_finish(acc[0], m[0], l[0], (int64_t)*pos0 + t, t, h, lane, Dv, cs_v, da, orow);
    else diff_finish(acc[0], l[0], acc[MAPS - 1], l[MAPS - 1], t, h, lane, Dv, da, orow);
}

// ---- portions: 32 tokens of one head per CTA, tiles of 32 cache rows staged in shared memory
constexpr int kQT = 32, kQPW = kQT / kWarps; // queries per CTA and per warp

// NP: groups of 64 value coordinates (a pair per lane) the lanes accumulate, Dv <= 64 NP.  VEC: rows are staged and K rows
// read in 16-byte pieces; the K pitch kp is then a multiple of 4 words with kp / 4 odd (the eight lanes of a quarter warp, a
// row each, cover all 32 banks) and the V pitch vp a multiple of 4; otherwise kp is odd and vp even (float2 reads).
// MAPS 2: a query has two rows of q, a cache row two key parts; the value part of a tile serves both maps.
template <typename E, int NP, bool VEC, int MAPS>
__global__ void __launch_bounds__(32 * kWarps) window_attn_tile_kernel(const float *__restrict__ q, const E *__restrict__ cache, int64_t cache_ld,
                                                                       const int32_t *__restrict__ table, int B, const int32_t *__restrict__ pos0,
                                                                       int64_t T, int H, int G, int D, int Dv, int kp, int vp, int64_t window,
                                                                       int chunked, int64_t keep, float cap, const float *__restrict__ cs_v,
                                                                       finish_args da, E *__restrict__ out) {
    extern __shared__ __align__(16) float wa_smem[];
    const int Dp = (D + 3) & ~3;
    float *sq = wa_smem;               // [kQT][MAPS][Dp]
    float *sk = sq + kQT * MAPS * Dp;  // [MAPS][32][kp]
    float *sv = sk + MAPS * 32 * kp;   // [32][vp]
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int h = blockIdx.y, g = h / (H / G);
    const int64_t t0 = (int64_t)blockIdx.x * kQT;
    const int nq = (int)min((int64_t)kQT, T - t0);
    const int64_t i0 = (int64_t)*pos0 + t0;          // position of the CTA's first query
    const int64_t i_last = i0 + nq - 1;
    for (int e = threadIdx.x; e < kQT * MAPS * Dp; e += blockDim.x) {
        const int row = e / Dp, d = e - row * Dp, qi = row / MAPS;
        sq[e] = (qi < nq && d < D) ? q[((t0 + qi) * H + h) * MAPS * D + (row - qi * MAPS) * D + d] : 0.f;
    }
    // the window's tiles start at the first query's first key: never later than a later query's
    const key_tiles kt(first_visible(i0, window, chunked), keep);
    float acc[kQPW][MAPS][2 * NP], m[kQPW][MAPS], l[kQPW][MAPS];
    int64_t lo[kQPW];
#pragma unroll
    for (int a = 0; a < kQPW; a++) {
        lo[a] = first_visible(i0 + warp * kQPW + a, window, chunked);
#pragma unroll
        for (int mp = 0; mp < MAPS; mp++) {
            m[a][mp] = -INFINITY;
            l[a][mp] = 0.f;
#pragma unroll
            for (int r = 0; r < 2 * NP; r++) acc[a][mp][r] = 0.f;
        }
    }
    const int64_t koff = (int64_t)g * MAPS * D, voff = (int64_t)G * MAPS * D + (int64_t)g * Dv;
    const int row_elems = MAPS * D + Dv;
    for (int64_t n = 0;; n++) {
        const int64_t j0 = kt.first(n), j_last = kt.last(n, i_last);
        if (j0 > j_last) break;
        __syncthreads(); // the previous tile has been consumed (and sq is written, the first time)
        const int n_rows = (int)min((int64_t)32, j_last - j0 + 1);
        // a warp stages rows warp, warp + 8, ...: 16-byte pieces of the K part and of the V part, converted to fp32
        for (int rr = warp; rr < 32; rr += kWarps) {
            const int64_t j = j0 + min(rr, n_rows - 1); // a row past the last one repeats it (masked below, weight 0)
            const E *row = cache + ((int64_t)table[j / B] * B + j % B) * cache_ld;
            if (VEC) {
                constexpr int VN = RowVec<E>::n;
                const int nk1 = D / VN, nk = MAPS * nk1, nv = Dv / VN;
                for (int vi = lane; vi < nk + nv; vi += 32) {
                    const bool is_k = vi < nk;
                    const int c = (is_k ? vi : vi - nk) * VN;
                    RowVec<E> x;
                    x.raw = *reinterpret_cast<const uint4 *>(row + (is_k ? koff : voff) + c);
                    float *dst1 = sv + rr * vp + c;
                    if (is_k) {
                        const int mp = MAPS == 1 ? 0 : vi >= nk1;
                        dst1 = sk + (mp * 32 + rr) * kp + c - mp * D;
                    }
                    float4 *dst = reinterpret_cast<float4 *>(dst1);
#pragma unroll
                    for (int u = 0; u < VN; u += 4) dst[u / 4] = make_float4(x.at(u), x.at(u + 1), x.at(u + 2), x.at(u + 3));
                }
            } else {
                for (int c = lane; c < row_elems; c += 32) {
                    if (c < MAPS * D) {
                        const int mp = MAPS == 1 ? 0 : c >= D;
                        sk[(mp * 32 + rr) * kp + c - mp * D] = to_f32(row[koff + c]);
                    } else {
                        sv[rr * vp + c - MAPS * D] = to_f32(row[voff + c - MAPS * D]);
                    }
                }
            }
        }
        __syncthreads();
        // scores of the warp's queries against key j0 + lane
        float p[kQPW][MAPS];
        const int64_t j = j0 + lane;
        const bool in_tile = lane < n_rows;
#pragma unroll
        for (int mp = 0; mp < MAPS; mp++) {
            float s[kQPW];
#pragma unroll
            for (int a = 0; a < kQPW; a++) s[a] = 0.f;
            const float *kr = sk + (mp * 32 + lane) * kp;
            const float *qw = sq + (warp * kQPW * MAPS + mp) * Dp; // query a of the warp: qw + a * MAPS * Dp
            const int D4 = D & ~3;
#pragma unroll 2
            for (int d = 0; d < D4; d += 4) {
                float k0, k1, k2, k3;
                if (VEC) {
                    const float4 kv = *reinterpret_cast<const float4 *>(kr + d);
                    k0 = kv.x, k1 = kv.y, k2 = kv.z, k3 = kv.w;
                } else {
                    k0 = kr[d], k1 = kr[d + 1], k2 = kr[d + 2], k3 = kr[d + 3];
                }
#pragma unroll
                for (int a = 0; a < kQPW; a++) {
                    const float4 qv = *reinterpret_cast<const float4 *>(qw + a * MAPS * Dp + d);
                    s[a] = fmaf(k0, qv.x, s[a]);
                    s[a] = fmaf(k1, qv.y, s[a]);
                    s[a] = fmaf(k2, qv.z, s[a]);
                    s[a] = fmaf(k3, qv.w, s[a]);
                }
            }
            for (int d = D4; d < D; d++)
#pragma unroll
                for (int a = 0; a < kQPW; a++) s[a] = fmaf(kr[d], qw[a * MAPS * Dp + d], s[a]);
#pragma unroll
            for (int a = 0; a < kQPW; a++) {
                const int64_t i = i0 + warp * kQPW + a;
                const bool live = warp * kQPW + a < nq;
                const bool vis = live && in_tile && j <= i && (j >= lo[a] || j < keep);
                const float sa = vis ? soft_cap(s[a], cap) : -INFINITY;
                const float m_new = fmaxf(m[a][mp], warp_max_f32(sa));
                // a query none of whose keys lie in this tile keeps m = -inf: nothing to rescale, nothing to add
                const float corr = m_new == -INFINITY ? 1.f : expf(m[a][mp] - m_new);
                p[a][mp] = vis ? expf(sa - m_new) : 0.f;
                l[a][mp] = l[a][mp] * corr + warp_sum_f32(p[a][mp]);
#pragma unroll
                for (int r = 0; r < 2 * NP; r++) acc[a][mp][r] *= corr;
                m[a][mp] = m_new;
            }
        }
#pragma unroll 2
        for (int jj = 0; jj < n_rows; jj++) {
            float pj[kQPW][MAPS];
#pragma unroll
            for (int a = 0; a < kQPW; a++)
#pragma unroll
                for (int mp = 0; mp < MAPS; mp++) pj[a][mp] = __shfl_sync(0xffffffffu, p[a][mp], jj);
#pragma unroll
            for (int r = 0; r < NP; r++) {
                const int c = 2 * lane + 64 * r;
                if (c < Dv) {
                    const float2 vv = *reinterpret_cast<const float2 *>(sv + jj * vp + c);
#pragma unroll
                    for (int a = 0; a < kQPW; a++)
#pragma unroll
                        for (int mp = 0; mp < MAPS; mp++) {
                            acc[a][mp][2 * r] = fmaf(pj[a][mp], vv.x, acc[a][mp][2 * r]);
                            acc[a][mp][2 * r + 1] = fmaf(pj[a][mp], vv.y, acc[a][mp][2 * r + 1]);
                        }
                }
            }
        }
    }
#pragma unroll
    for (int a = 0; a < kQPW; a++) {
        const int qi = warp * kQPW + a;
        if (qi >= nq) continue;
        E *orow = out + ((t0 + qi) * H + h) * Dv;
        if (MAPS == 1) window_finish<E, NP>(acc[a][0], m[a][0], l[a][0], i0 + qi, t0 + qi, h, lane, Dv, cs_v, da, orow);
        else diff_finish<E, NP>(acc[a][0], l[a][0], acc[a][MAPS - 1], l[a][MAPS - 1], t0 + qi, h, lane, Dv, da, orow);
    }
}

} // namespace

extern "C" {

int64_t ggb_window_cache_ld(int G, int D, int Dv) { return (((int64_t)G * (D + Dv)) + 7) / 8 * 8; }

int ggb_op_window_qkv_store(int dt, const float *q, const float *k, const float *v, int64_t ld, int64_t T, int H, int G, int D, int Dv,
                            const float *qn_w, const float *kn_w, float eps, int rot_dims, const float *cos_sin_k, const float *cos_sin_v,
                            float scale, const int32_t *pos0, const int32_t *block_table, int block_size, void *cache, float *q_out) {
    return ggb_op_masked_qkv_store(dt, q, k, v, ld, T, H, G, D, Dv, qn_w, kn_w, eps, rot_dims, 0, cos_sin_k, cos_sin_v, scale, pos0, block_table,
                                   block_size, cache, q_out);
}

// H query heads of size D over Gk key heads, Gv value heads of size Dv
static int qkv_store_launch(int dt, const float *q, const float *k, const float *v, int64_t ld, int64_t T, int H, int Gk, int D, int Gv, int Dv,
                            const float *qn_w, const float *kn_w, float eps, int rot_dims, int rot_halves, const float *cos_sin_k,
                            const float *cos_sin_v, float scale, const int32_t *pos0, const int32_t *block_table, int block_size, int64_t cld,
                            void *cache, float *q_out) {
    GGB_REQUIRE_INIT();
    GGB_CHECK_ARG(dt == GGB_TYPE_BF16 || dt == GGB_TYPE_F32, "window_qkv_store: dtype %d is neither bf16 nor f32", dt);
    GGB_CHECK_ARG(q && k && v && pos0 && block_table && cache && q_out && T > 0 && H > 0 && Gk > 0 && H % Gk == 0 && Gv > 0 && block_size > 0,
                  "window_qkv_store: bad arguments");
    GGB_CHECK_ARG(D > 0 && D % 2 == 0 && Dv > 0 && Dv % 2 == 0 && rot_dims >= 0 && rot_dims <= D && rot_dims % 2 == 0 && (!rot_dims || cos_sin_k),
                  "window_qkv_store: head sizes %d / %d and %d rotated dimensions must be even", D, Dv, rot_dims);
    if (dt == GGB_TYPE_BF16)
        window_qkv_store_kernel<<<(unsigned)T, 256, 0, ggb_cuda_stream()>>>(q, k, v, ld, H, Gk, D, Gv, Dv, qn_w, kn_w, eps, rot_dims, rot_halves,
                                                                            rot_dims ? cos_sin_k : nullptr, cos_sin_v, scale, pos0, block_table,
                                                                            block_size, (__nv_bfloat16 *)cache, cld, q_out);
    else
        window_qkv_store_kernel<<<(unsigned)T, 256, 0, ggb_cuda_stream()>>>(q, k, v, ld, H, Gk, D, Gv, Dv, qn_w, kn_w, eps, rot_dims, rot_halves,
                                                                            rot_dims ? cos_sin_k : nullptr, cos_sin_v, scale, pos0, block_table,
                                                                            block_size, (float *)cache, cld, q_out);
    GGB_LAUNCH_CHECK();
    return GGB_OK;
}

int ggb_op_masked_qkv_store(int dt, const float *q, const float *k, const float *v, int64_t ld, int64_t T, int H, int G, int D, int Dv,
                            const float *qn_w, const float *kn_w, float eps, int rot_dims, int rot_halves, const float *cos_sin_k,
                            const float *cos_sin_v, float scale, const int32_t *pos0, const int32_t *block_table, int block_size, void *cache,
                            float *q_out) {
    return qkv_store_launch(dt, q, k, v, ld, T, H, G, D, G, Dv, qn_w, kn_w, eps, rot_dims, rot_halves, cos_sin_k, cos_sin_v, scale, pos0, block_table,
                            block_size, ggb_window_cache_ld(G, D, Dv), cache, q_out);
}

int ggb_op_head_qkv_store(int dt, const float *q, const float *k, const float *v, int64_t ld, int64_t T, int H, int G, int D, int Dv, const float *qn_w,
                          const float *kn_w, float eps, int rot_dims, int rot_halves, const float *cos_sin, float scale, const int32_t *pos0,
                          const int32_t *block_table, int block_size, void *cache, float *q_out) {
    GGB_REQUIRE_INIT();
    GGB_CHECK_ARG(dt == GGB_TYPE_BF16 || dt == GGB_TYPE_F32, "head_qkv_store: dtype %d is neither bf16 nor f32", dt);
    GGB_CHECK_ARG(q && k && v && pos0 && block_table && cache && q_out && T > 0 && H > 0 && G > 0 && H % G == 0 && block_size > 0 && D > 0 && Dv > 0,
                  "head_qkv_store: bad arguments");
    GGB_CHECK_ARG(rot_dims >= 0 && rot_dims <= D && rot_dims % 2 == 0 && (!rot_dims || cos_sin), "head_qkv_store: %d of %d dimensions cannot turn", rot_dims, D);
    const int64_t cld = ggb_window_cache_ld(G, D, Dv);
    const dim3 grid((unsigned)T, (unsigned)((H + 2 * G + 7) / 8));
    if (dt == GGB_TYPE_BF16)
        head_qkv_store_kernel<<<grid, 256, 0, ggb_cuda_stream()>>>(q, k, v, ld, H, G, D, Dv, qn_w, kn_w, eps, rot_dims, rot_halves, cos_sin, scale, pos0,
                                                                   block_table, block_size, (__nv_bfloat16 *)cache, cld, q_out);
    else
        head_qkv_store_kernel<<<grid, 256, 0, ggb_cuda_stream()>>>(q, k, v, ld, H, G, D, Dv, qn_w, kn_w, eps, rot_dims, rot_halves, cos_sin, scale, pos0,
                                                                   block_table, block_size, (float *)cache, cld, q_out);
    GGB_LAUNCH_CHECK();
    return GGB_OK;
}

int ggb_op_diff_qkv_store(int dt, const float *q, const float *k, const float *v, int64_t ld, int64_t T, int H, int G, int D, int Dv, int rot_dims,
                          int rot_halves, const float *cos_sin_k, float scale, const int32_t *pos0, const int32_t *block_table, int block_size,
                          void *cache, float *q_out) {
    return qkv_store_launch(dt, q, k, v, ld, T, 2 * H, 2 * G, D, G, Dv, nullptr, nullptr, 0.f, rot_dims, rot_halves, cos_sin_k, nullptr, scale, pos0,
                            block_table, block_size, ggb_window_cache_ld(G, 2 * D, Dv), cache, q_out);
}

size_t ggb_window_attn_scratch_bytes(int H) { return (size_t)(kQT - 1) * (size_t)H * kMaxSplit * kPartW * 4; }

int ggb_op_window_attn(int dt, const float *q, const void *cache, const int32_t *block_table, int block_size, const int32_t *pos0, int64_t T,
                       int H, int G, int D, int Dv, int64_t window, const float *cos_sin_v, void *out, float *scratch) {
    return ggb_op_masked_attn(dt, q, cache, block_table, block_size, pos0, T, H, G, D, Dv, window, 0, 0.f, cos_sin_v, out, scratch);
}

} // extern "C"

template <int MAPS>
static int masked_attn_launch(int dt, const float *q, const void *cache, const int32_t *block_table, int block_size, const int32_t *pos0, int64_t T,
                              int H, int G, int D, int Dv, int64_t window, int chunked, int64_t keep, float softcap, const float *cos_sin_v,
                              const finish_args &da, void *out, float *scratch) {
    GGB_REQUIRE_INIT();
    GGB_CHECK_ARG(softcap >= 0.f && (chunked == 0 || chunked == 1), "masked_attn: the soft cap must not be negative");
    GGB_CHECK_ARG(dt == GGB_TYPE_BF16 || dt == GGB_TYPE_F32, "window_attn: dtype %d is neither bf16 nor f32", dt);
    GGB_CHECK_ARG(q && cache && block_table && pos0 && out && T > 0 && H > 0 && G > 0 && H % G == 0 && block_size > 0 && D > 0 && Dv > 0 &&
                      Dv % 2 == 0 && Dv <= 32 * kMaxDvRegs && keep >= 0,
                  "window_attn: bad arguments (value size %d, even and at most %d)", Dv, 32 * kMaxDvRegs);
    const int64_t cld = ggb_window_cache_ld(G, MAPS * D, Dv);
    const int Dp = (D + 3) & ~3;
    const int es = dt == GGB_TYPE_BF16 ? 2 : 4, vn = 16 / es;
    const int vec = D % vn == 0 && ((uintptr_t)cache % 16 == 0); // rows are 8 numbers apart at least: 16-byte aligned in both types
    cudaStream_t st = ggb_cuda_stream();
    if (T >= kQT) { // a portion: tiles of cache rows staged once for 32 queries
        // 16-byte pieces need every head's keys and values to start on one: D, Dv and G * D whole pieces
        const bool tv = vec && Dv % vn == 0 && ((int64_t)G * D) % vn == 0;
        int kp = D | 1, vp = Dv + 2;
        if (tv) {
            kp = (D + 3) & ~3;
            if ((kp / 4) % 2 == 0) kp += 4;
            vp = (Dv + 3) & ~3;
        }
        const size_t smem = ((size_t)kQT * MAPS * Dp + 32 * (size_t)MAPS * (size_t)kp + 32 * (size_t)vp) * 4;
        GGB_CHECK_ARG(smem <= 200 * 1024, "window_attn: head sizes %d / %d do not fit shared memory", D, Dv);
        const dim3 grid((unsigned)((T + kQT - 1) / kQT), (unsigned)H);
#define WT_LAUNCH(ET, NP, VEC)                                                                                               \
    {                                                                                                                        \
        auto kfn = window_attn_tile_kernel<ET, NP, VEC, MAPS>;                                                               \
        if (smem > 48 * 1024) GGB_CUDA(cudaFuncSetAttribute(kfn, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));    \
        kfn<<<grid, 32 * kWarps, smem, st>>>(q, (const ET *)cache, cld, block_table, block_size, pos0, T, H, G, D, Dv, kp, vp, \
                                             window, chunked, keep, softcap, cos_sin_v, da, (ET *)out);                      \
    }
#define WT_NP(ET, VEC)                             \
    {                                              \
        if (Dv <= 64) WT_LAUNCH(ET, 1, VEC)        \
        else if (Dv <= 128) WT_LAUNCH(ET, 2, VEC)  \
        else WT_LAUNCH(ET, 4, VEC)                 \
    }
        if (dt == GGB_TYPE_BF16) {
            if (tv) WT_NP(__nv_bfloat16, true) else WT_NP(__nv_bfloat16, false)
        } else {
            if (tv) WT_NP(float, true) else WT_NP(float, false)
        }
#undef WT_NP
#undef WT_LAUNCH
    } else {
        const size_t smem = (size_t)kWarps * MAPS * ((size_t)Dp + kPartW) * 4;
        GGB_CHECK_ARG(smem <= 48 * 1024, "window_attn: key size %d does not fit shared memory", D);
        // a warp a tile: as many splits as the longest visible range has groups of 8 tiles (the range is bounded by the
        // window; without one, by what the scratch was sized for)
        int n_split = 1;
        if (scratch && window > 0) n_split = (int)std::min<int64_t>(kMaxSplit, ((window + 62) / 32 + (keep + 31) / 32 + kWarps - 1) / kWarps);
        else if (scratch) n_split = kMaxSplit / 2;
        const dim3 grid((unsigned)T, (unsigned)H, (unsigned)n_split);
#define WS_LAUNCH(ET)                                                                                                                        \
    window_attn_kernel<ET, MAPS><<<grid, 32 * kWarps, smem, st>>>(q, (const ET *)cache, cld, block_table, block_size, pos0, T, H, G, D, Dv, window,  \
                                                                  chunked, keep, softcap, cos_sin_v, da, (ET *)out, vec, scratch);            \
    if (n_split > 1) {                                                                                                                       \
        GGB_LAUNCH_CHECK();                                                                                                                  \
        window_merge_kernel<ET, MAPS><<<dim3((unsigned)T, (unsigned)H), 32, 0, st>>>(scratch, n_split, pos0, H, Dv, cos_sin_v, da, (ET *)out); \
    }
        if (dt == GGB_TYPE_BF16) { WS_LAUNCH(__nv_bfloat16) } else { WS_LAUNCH(float) }
#undef WS_LAUNCH
    }
    GGB_LAUNCH_CHECK();
    return GGB_OK;
}

extern "C" {

int ggb_op_masked_attn(int dt, const float *q, const void *cache, const int32_t *block_table, int block_size, const int32_t *pos0, int64_t T,
                       int H, int G, int D, int Dv, int64_t window, int chunked, float softcap, const float *cos_sin_v, void *out,
                       float *scratch) {
    return masked_attn_launch<1>(dt, q, cache, block_table, block_size, pos0, T, H, G, D, Dv, window, chunked, 0, softcap, cos_sin_v, finish_args{}, out,
                                 scratch);
}

int ggb_op_masked_attn_keep(int dt, const float *q, const void *cache, const int32_t *block_table, int block_size, const int32_t *pos0, int64_t T,
                            int H, int G, int D, int Dv, int64_t window, int64_t keep_first, float softcap, void *out, float *scratch) {
    return masked_attn_launch<1>(dt, q, cache, block_table, block_size, pos0, T, H, G, D, Dv, window, 0, keep_first, softcap, nullptr, finish_args{}, out,
                                 scratch);
}

int ggb_op_masked_attn_gated(int dt, const float *q, const void *cache, const int32_t *block_table, int block_size, const int32_t *pos0, int64_t T,
                             int H, int G, int D, int Dv, int64_t window, int64_t keep_first, float softcap, const float *sink, const float *gate,
                             int64_t ldg, void *out, float *scratch) {
    GGB_CHECK_ARG(!gate || ldg >= (int64_t)H * Dv, "masked_attn_gated: a gate row holds a number per output");
    finish_args fa;
    fa.sink = sink, fa.gate = gate, fa.ldg = ldg;
    return masked_attn_launch<1>(dt, q, cache, block_table, block_size, pos0, T, H, G, D, Dv, window, 0, keep_first, softcap, nullptr, fa, out, scratch);
}

int ggb_op_diff_attn(int dt, const float *q, const void *cache, const int32_t *block_table, int block_size, const int32_t *pos0, int64_t T, int H,
                     int G, int D, int Dv, int64_t window, int64_t keep_first, float softcap, float lambda, float out_scale, float eps,
                     const float *gate, int64_t ldg, void *out, float *scratch) {
    GGB_CHECK_ARG(!gate || ldg >= (int64_t)H * Dv, "diff_attn: a gate row holds a number per output");
    return masked_attn_launch<2>(dt, q, cache, block_table, block_size, pos0, T, H, G, D, Dv, window, 0, keep_first, softcap, nullptr,
                                 finish_args{lambda, out_scale, eps, gate, ldg, nullptr}, out, scratch);
}

} // extern "C"
