// Sliding-window grouped-query attention over the paged cache, floating point (bf16, or fp32 in the 32-bit mode):
//   q, k = rms norm over the whole projection, before the split into heads
//   s    = softcap * tanh(scale * (q . k) / softcap) + bias[head][i - j]          0 <= i - j < window
//   p    = exp(s) / (sink + sum exp(s)),   out = (sum p v) * logistic(gate)
// Norms, softcap, bias, sink (a score of 0, or one learned score per head) and gate are optional; the first `keep` positions may
// stay visible behind the window; a call may use another layer's keys and values. A distance bias and the window are one
// table per layer (-inf outside the window), so that a masked key costs nothing extra. Scores, weights and sums are fp32.
//
// Cache pages hold 64 tokens, K [page][G][64][dkp] and V transposed [page][G][dv][64] (as the int8 cache does).
//   one token per sequence : attn_decode_mma_kernel (bf16), else attn_row_kernel<FUSED>: norms, append and attention in one
//                            launch, keys split over CTAs
//   prompts, bf16          : attn_prepare_kernel, then attn_window_prefill_kernel on tcgen05
//   prompts, otherwise     : attn_prepare_kernel, then attn_row_kernel row by row
// Where softcap and bias bound the scores, the tensor-core forms use a constant softmax shift; otherwise (no softcap, no bias)
// their ONLINE variants keep a running maximum, which starts at the sink's score.
#include <cmath>
#include <vector>

#include "float_common.cuh"
#include "kv_cache.h"
#include "tc_common.cuh"

namespace flexllm {

using namespace tc;

namespace {

constexpr int PG = 64;                     // tokens per page
constexpr int TILE_PAGES = 4;              // pages per key tile of the row kernel
constexpr int TILE_KEYS = TILE_PAGES * PG;
constexpr long kDecodeCtas = 1776;         // CTAs the decode form aims at: four waves of three per SM

// Start position of sequence b; a value that would leave the page-table row is clamped and reported.
__device__ __forceinline__ int start_pos(const AttnCall& c, int b, int* error_flag) {
    int pos = c.ctx[b];
    if (pos < 0 || pos + c.Sc - 1 > c.max_pos) {
        if (error_flag) atomicOr(error_flag, 2);
        pos = pos < 0 ? 0 : c.max_pos - (c.Sc - 1);
    }
    return pos;
}

// Logical pages that a range of positions reads: the pages of the kept first positions, then those of the window.
struct KeyPages {
    int keep, lo, n;
    __device__ __forceinline__ KeyPages(const AttnShape& s, int first, int last) {        // positions [first, last]
        lo = max(0, first - s.window + 1) / PG;
        keep = min((s.keep + PG - 1) / PG, lo);
        n = keep + last / PG - lo + 1;
    }
    __device__ __forceinline__ int at(int i) const { return i < keep ? i : lo + i - keep; }
};
__device__ __forceinline__ bool sees(const AttnShape& s, int pos, int key) { return key <= pos && (pos - key < s.window || key < s.keep); }
// Score of the sink of head h (-inf: none).
__device__ __forceinline__ float sink_score(const AttnCall& c, int h) {
    return c.s.sink == 2 ? c.sinks[h] : c.s.sink ? 0.0f : -INFINITY;
}

// This thread's share (NT threads) of the sum of squares of n elements at a 16-byte aligned address.
template <int NT, class T> __device__ __forceinline__ float share_sumsq(const T* p, int n, int tid) {
    float s = 0.0f;
    const int nv = n >> 3;
    for (int i = tid; i < nv; i += NT) {
        float f[8];
        load8(p + 8 * i, f);
#pragma unroll
        for (int e = 0; e < 8; e++) s = __fmaf_rn(f[e], f[e], s);
    }
    for (int i = (nv << 3) + tid; i < n; i += NT) { const float v = to_f(p[i]); s = __fmaf_rn(v, v, s); }
    return s;
}
// Normed elements e0 .. e0+7 of a head whose first element is j0 of the projection at src (j0 + e0 is 8-aligned when dk is a
// multiple of 8); zero from dk on.
template <class T> __device__ __forceinline__ void normed8(const T* src, const float* gain, int j0, int e0, int dk, float r, float (&f)[8]) {
    if ((dk & 7) == 0) {
        load8(src + j0 + e0, f);
        if (!gain) return;
        const float4 a = load4(gain + j0 + e0), b = load4(gain + j0 + e0 + 4);
        f[0] = (f[0] * r) * a.x; f[1] = (f[1] * r) * a.y; f[2] = (f[2] * r) * a.z; f[3] = (f[3] * r) * a.w;
        f[4] = (f[4] * r) * b.x; f[5] = (f[5] * r) * b.y; f[6] = (f[6] * r) * b.z; f[7] = (f[7] * r) * b.w;
    } else {
#pragma unroll
        for (int e = 0; e < 8; e++) f[e] = e0 + e < dk ? (gain ? (to_f(src[j0 + e0 + e]) * r) * gain[j0 + e0 + e] : to_f(src[j0 + e0 + e])) : 0.0f;
    }
}
// Reciprocal root mean squares of the q and k projections of a row (1 without norms).
template <class T> __device__ __forceinline__ float2 qk_rms(const AttnCall& c, const T* row, int tid, float* red) {
    if (!c.q_gain) return make_float2(1.0f, 1.0f);
    const int nq = c.s.H * c.s.dk, nk = c.s.G * c.s.dk;
    const float2 ss = block_sum2<256>(share_sumsq<256>(row + c.s.q_off, nq, tid), share_sumsq<256>(row + c.s.k_off, nk, tid), red);
    return make_float2(1.0f / sqrtf(ss.x / (float)nq + c.eps), 1.0f / sqrtf(ss.y / (float)nk + c.eps));
}
template <class T> __device__ __forceinline__ void store8(T* p, const float (&f)[8]) {
    store4(p, make_float4(f[0], f[1], f[2], f[3]));
    store4(p + 4, make_float4(f[4], f[5], f[6], f[7]));
}

// ---------------------------------------------------------------------------------------------------------------
// Norm of q and k over their whole projections, q to the scratch, k rows and v columns to the pages.
// CTAs 0 .. B*Sc-1: one row each. The rest: one (page, V head, sequence) each, transposing through shared memory.
template <class T>
__global__ void __launch_bounds__(256) attn_prepare_kernel(const AttnCall c, int v_pages, int* error_flag) {
    __shared__ float red[16];
    __shared__ T tile[PG][PG + 2];
    pdl_sync();
    const AttnShape& s = c.s;
    const int rows = c.B * c.Sc, tid = threadIdx.x;
    if ((int)blockIdx.x < rows) {
        const int m = blockIdx.x, b = m / c.Sc;
        const int pos = start_pos(c, b, error_flag) + m % c.Sc;
        const T* src = (const T*)c.proj + (long)m * s.ld;
        const float2 rms = qk_rms(c, src, tid, red);
        const float rq = rms.x, rk = rms.y;
        T* q = (T*)c.q + (long)m * s.H * s.dkp;
        const int nv = s.dkp >> 3;                                  // 8-element blocks per head
        for (int i = tid; i < s.H * nv; i += 256) {
            const int h = i / nv, e0 = (i - h * nv) * 8;
            float f[8];
            normed8(src + s.q_off, c.q_gain, h * s.dk, e0, s.dk, rq, f);
            store8(q + (long)i * 8, f);
        }
        if (s.k_off < 0) return;
        const long page = c.page_table[(long)b * c.max_pages + pos / PG];
        T* kp = (T*)c.k_pool + (page * s.G * PG + (pos & (PG - 1))) * s.dkp;
        for (int i = tid; i < s.G * nv; i += 256) {
            const int g = i / nv, e0 = (i - g * nv) * 8;
            float f[8];
            normed8(src + s.k_off, c.k_gain, g * s.dk, e0, s.dk, rk, f);
            store8(kp + (long)g * PG * s.dkp + e0, f);
        }
        return;
    }
    int id = blockIdx.x - rows;
    const int pi = id % v_pages; id /= v_pages;
    const int g = id % s.G, b = id / s.G;
    const int p0 = start_pos(c, b, error_flag);
    const int page_i = p0 / PG + pi;
    const int lo = max(p0, page_i * PG), hi = min(p0 + c.Sc, (page_i + 1) * PG);     // positions [lo, hi)
    if (lo >= hi) return;
    const long page = c.page_table[(long)b * c.max_pages + page_i];
    T* vp = (T*)c.v_pool + (page * s.G + g) * (long)s.dv * PG;
    const T* src = (const T*)c.proj + ((long)b * c.Sc + (lo - p0)) * s.ld + s.v_off + g * s.dv;
    const int n = hi - lo, slot0 = lo & (PG - 1);
    for (int d0 = 0; d0 < s.dv; d0 += PG) {
        const int nd = min(PG, s.dv - d0);
        for (int i = tid; i < n * PG; i += 256) {
            const int t = i >> 6, d = i & (PG - 1);
            if (d < nd) tile[t][d] = src[(long)t * s.ld + d0 + d];
        }
        __syncthreads();
        for (int i = tid; i < nd * PG; i += 256) {
            const int d = i >> 6, t = i & (PG - 1);
            if (t < n) vp[(long)(d0 + d) * PG + slot0 + t] = tile[t][d];
        }
        __syncthreads();
    }
}

// ---------------------------------------------------------------------------------------------------------------
// One query row (position) x one key/value head per CTA, its keys split over gridDim.x CTAs.
// RC: query heads handled at a time; L lanes share a key (8 elements each, WIDE: several times 8).
struct RowSmem { long q, sc, o, m, l, al, total; };
__host__ __device__ inline RowSmem row_smem(int R, int dkp, int dv) {
    RowSmem r;
    r.q = 0;                                    // [R][dkp]
    r.sc = r.q + (long)R * dkp;                 // [R][TILE_KEYS]
    r.o = r.sc + (long)R * TILE_KEYS;           // [R][dv]
    r.m = r.o + (((long)R * dv + 3) & ~3L);
    r.l = r.m + R; r.al = r.l + R;
    r.total = r.al + R;
    return r;
}

template <class T, int RC, bool FUSED, bool WIDE>
__global__ void __launch_bounds__(256) attn_row_kernel(const AttnCall c, int L, int* error_flag) {
    constexpr bool FAST = sizeof(T) == 2;
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[16];
    __shared__ int last_sm;
    const AttnShape& s = c.s;
    const int R = s.H / s.G;
    const RowSmem o = row_smem(R, s.dkp, s.dv);
    float *q_sm = sm + o.q, *s_sm = sm + o.sc, *o_sm = sm + o.o, *m_sm = sm + o.m, *l_sm = sm + o.l, *al_sm = sm + o.al;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int split = blockIdx.x, n_split = gridDim.x, g = blockIdx.y, row = blockIdx.z;
    pdl_sync();
    const int b = row / c.Sc;
    const int pos = start_pos(c, b, error_flag) + row % c.Sc;
    const int32_t* pt = c.page_table + (long)b * c.max_pages;
    const T* prow = (const T*)c.proj + (long)row * s.ld;
    const long kh = (long)PG * s.dkp, vh = (long)PG * s.dv;          // one head of a page
    if (FUSED) {
        const float2 rms = qk_rms(c, prow, tid, red);
        const float rq = rms.x, rk = rms.y;
        for (int i = tid; i < R * s.dkp; i += 256) {
            const int r = i / s.dkp, e = i - r * s.dkp, j = (g * R + r) * s.dk + e;
            q_sm[i] = e < s.dk ? (to_f(prow[s.q_off + j]) * rq) * (c.q_gain ? c.q_gain[j] : 1.0f) : 0.0f;
        }
        if (s.k_off >= 0 && split == n_split - 1) {               // the split that holds the newest key appends it
            const long page = pt[pos / PG];
            const int slot = pos & (PG - 1);
            T* kp = (T*)c.k_pool + (page * s.G + g) * kh + (long)slot * s.dkp;
            for (int e = tid; e < s.dkp; e += 256) {
                const int j = g * s.dk + e;
                kp[e] = from_f<T>(e < s.dk ? (to_f(prow[s.k_off + j]) * rk) * (c.k_gain ? c.k_gain[j] : 1.0f) : 0.0f);
            }
            T* vp = (T*)c.v_pool + (page * s.G + g) * vh + slot;
            for (int d = tid; d < s.dv; d += 256) vp[(long)d * PG] = prow[s.v_off + g * s.dv + d];
        }
    } else {
        const T* q = (const T*)c.q + ((long)row * s.H + (long)g * R) * s.dkp;
        for (int i = tid; i < R * s.dkp; i += 256) q_sm[i] = to_f(q[i]);
    }
    for (int i = tid; i < R * s.dv; i += 256) o_sm[i] = 0.0f;
    for (int i = tid; i < R; i += 256) { m_sm[i] = sink_score(c, g * R + i); l_sm[i] = 0.0f; }
    __syncthreads();

    const KeyPages pages(s, pos, pos);
    const int n_pg = pages.n;
    const int n_tiles = (n_pg + TILE_PAGES - 1) / TILE_PAGES;
    const int t_beg = (int)((long)split * n_tiles / n_split), t_end = (int)((long)(split + 1) * n_tiles / n_split);
    const float* bias_g = c.bias ? c.bias + (long)g * (2 * kBiasPad + s.window) * R : nullptr;
    const float inv_cap = s.softcap > 0.0f ? s.scale / s.softcap : 0.0f;
    const int kpw = 32 / L, sub = lane / L, ln = lane % L;            // keys per warp step, this lane's key and part
    for (int t = t_beg; t < t_end; t++) {
        const int pg0 = t * TILE_PAGES, npg = min(TILE_PAGES, n_pg - t * TILE_PAGES);
        // ---- scores of the tile's keys
        for (int r0 = 0; r0 < R; r0 += RC) {
            float qr[RC][8];
            if (!WIDE)
#pragma unroll
                for (int r = 0; r < RC; r++)
#pragma unroll
                    for (int e = 0; e < 8; e++) qr[r][e] = (r0 + r < R && ln * 8 < s.dkp) ? q_sm[(r0 + r) * s.dkp + ln * 8 + e] : 0.0f;
#pragma unroll 2
            for (int k = warp * kpw + sub; k < npg * PG; k += 8 * kpw) {
                const int lp = pages.at(pg0 + (k >> 6));                         // logical page
                const T* kp = (const T*)c.k_pool + ((long)pt[lp] * s.G + g) * kh + (long)(k & (PG - 1)) * s.dkp;
                float acc[RC];
#pragma unroll
                for (int r = 0; r < RC; r++) acc[r] = 0.0f;
                if (WIDE) {
                    for (int e0 = ln * 8; e0 < s.dkp; e0 += L * 8) {
                        float kf[8];
                        load8(kp + e0, kf);
#pragma unroll
                        for (int r = 0; r < RC; r++)
                            if (r0 + r < R)
#pragma unroll
                                for (int e = 0; e < 8; e++) acc[r] = __fmaf_rn(q_sm[(r0 + r) * s.dkp + e0 + e], kf[e], acc[r]);
                    }
                } else if (ln * 8 < s.dkp) {
                    float kf[8];
                    load8(kp + ln * 8, kf);
#pragma unroll
                    for (int r = 0; r < RC; r++)
#pragma unroll
                        for (int e = 0; e < 8; e++) acc[r] = __fmaf_rn(qr[r][e], kf[e], acc[r]);
                }
                // the loop bound is the same for all lanes of a warp step: npg * 64 is a multiple of 8 * kpw
                for (int off = L >> 1; off > 0; off >>= 1)
#pragma unroll
                    for (int r = 0; r < RC; r++) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], off);
                const int key = lp * PG + (k & (PG - 1));
#pragma unroll
                for (int r = 0; r < RC; r++)
                    if (r0 + r < R && ln == (r & (L - 1))) {
                        float v = -INFINITY;
                        if (sees(s, pos, key)) {
                            if (s.softcap > 0.0f) {
                                const float z = acc[r] * inv_cap;
                                v = s.softcap * (FAST ? 1.0f - 2.0f * rcp_fast(1.0f + ex2_fast(z * (2.0f * kLog2e))) : tanhf(z));
                            } else {
                                v = acc[r] * s.scale;
                            }
                            if (bias_g) v += bias_g[(long)(pos - key + kBiasPad) * R + r0 + r];
                        }
                        s_sm[(r0 + r) * TILE_KEYS + k] = v;
                    }
            }
        }
        __syncthreads();
        // ---- running maximum, weights, sums: one warp per head
        for (int r = warp; r < R; r += 8) {
            float* sr = s_sm + r * TILE_KEYS;
            float mx = -INFINITY;
            for (int k = lane; k < npg * PG; k += 32) mx = fmaxf(mx, sr[k]);
            mx = warp_max(mx);
            const float m_old = m_sm[r], m_new = fmaxf(m_old, mx);
            const float ref = m_new == -INFINITY ? 0.0f : m_new;
            float sum = 0.0f;
            for (int k = lane; k < npg * PG; k += 32) {
                const float p = FAST ? ex2_fast((sr[k] - ref) * kLog2e) : expf(sr[k] - ref);
                sr[k] = p;
                sum += p;
            }
            sum = warp_sum(sum);
            __syncwarp();
            if (lane == 0) {
                const float al = m_old == -INFINITY ? 0.0f : expf(m_old - ref);
                al_sm[r] = al; m_sm[r] = m_new; l_sm[r] = __fmaf_rn(l_sm[r], al, sum);
            }
        }
        __syncthreads();
        // ---- values: 8 lanes share one row (dimension) of a V^T page, 8 tokens each
        const int dl = lane >> 3, tv = lane & 7;
        for (int r0 = 0; r0 < R; r0 += RC) {
            for (int db = warp * 4; db < s.dv; db += 32) {
                const int d = db + dl;
                float acc[RC];
#pragma unroll
                for (int r = 0; r < RC; r++) acc[r] = 0.0f;
                if (d < s.dv) {
#pragma unroll 4
                    for (int p = 0; p < npg; p++) {
                        float vf[8];
                        load8((const T*)c.v_pool + ((long)pt[pages.at(pg0 + p)] * s.G + g) * vh + (long)d * PG + tv * 8, vf);
#pragma unroll
                        for (int r = 0; r < RC; r++) {
                            if (r0 + r >= R) continue;
                            const float* pr = s_sm + (r0 + r) * TILE_KEYS + p * PG + tv * 8;
                            const float4 x = load4(pr), y = load4(pr + 4);
                            float t8 = acc[r];
                            t8 = __fmaf_rn(x.x, vf[0], t8); t8 = __fmaf_rn(x.y, vf[1], t8); t8 = __fmaf_rn(x.z, vf[2], t8); t8 = __fmaf_rn(x.w, vf[3], t8);
                            t8 = __fmaf_rn(y.x, vf[4], t8); t8 = __fmaf_rn(y.y, vf[5], t8); t8 = __fmaf_rn(y.z, vf[6], t8); t8 = __fmaf_rn(y.w, vf[7], t8);
                            acc[r] = t8;
                        }
                    }
                }
#pragma unroll
                for (int off = 4; off > 0; off >>= 1)
#pragma unroll
                    for (int r = 0; r < RC; r++) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], off);
                if (tv == 0 && d < s.dv)
#pragma unroll
                    for (int r = 0; r < RC; r++)
                        if (r0 + r < R) { float* op = o_sm + (r0 + r) * s.dv + d; *op = __fmaf_rn(*op, al_sm[r0 + r], acc[r]); }
            }
        }
        __syncthreads();
    }

    if (n_split > 1) {
        // partial (maximum, sum, values) per head; the last CTA of this (row, head) combines them in split order
        const long stride = (long)R * (s.dv + 2);
        float* part = c.ws + ((long)row * s.G + g) * n_split * stride;
        float* mine = part + split * stride;
        for (int i = tid; i < R; i += 256) { mine[i] = m_sm[i]; mine[R + i] = l_sm[i]; }
        for (int i = tid; i < R * s.dv; i += 256) mine[2 * R + i] = o_sm[i];
        __threadfence();
        __syncthreads();
        int* cnt = c.counters + (long)row * s.G + g;
        if (tid == 0) last_sm = atomicAdd(cnt, 1) == n_split - 1;
        __syncthreads();
        if (!last_sm) return;
        __threadfence();
        for (int r = tid; r < R; r += 256) {
            float m = sink_score(c, g * R + r);
            for (int k = 0; k < n_split; k++) m = fmaxf(m, __ldcg(part + k * stride + r));
            float l = 0.0f;
            for (int k = 0; k < n_split; k++) {
                const float mk = __ldcg(part + k * stride + r);
                const float w = mk == -INFINITY ? 0.0f : expf(mk - m);
                l = __fmaf_rn(__ldcg(part + k * stride + R + r), w, l);
            }
            m_sm[r] = m; l_sm[r] = l;
        }
        __syncthreads();
        for (int i = tid; i < R * s.dv; i += 256) {
            const int r = i / s.dv;
            float v = 0.0f;
            for (int k = 0; k < n_split; k++) {
                const float mk = __ldcg(part + k * stride + r);
                const float w = mk == -INFINITY ? 0.0f : expf(mk - m_sm[r]);
                v = __fmaf_rn(__ldcg(part + k * stride + 2 * R + i), w, v);
            }
            o_sm[i] = v;
        }
        if (tid == 0) *cnt = 0;
        __syncthreads();
    }
    T* out = (T*)c.out + (long)row * c.ldo + (long)g * R * s.dv;
    for (int i = tid; i < R * s.dv; i += 256) {
        const int r = i / s.dv;
        const float den = l_sm[r] + (s.sink ? expf(sink_score(c, g * R + r) - m_sm[r]) : 0.0f);
        float v = o_sm[i] / den;
        if (s.g_off >= 0) v *= sigmoid_f<FAST>(to_f(prow[s.g_off + (long)g * R * s.dv + i]));
        out[i] = from_f<T>(v);
    }
}

// ---------------------------------------------------------------------------------------------------------------
// Decoding, bf16, up to 8 query heads per key/value head: the fused form of the row kernel with warp-level bf16 MMAs.
// A CTA takes one (sequence, key/value head) and a share of its key tiles of 128 keys (two pages):
//   scores: warp w has keys 16 w .. 16 w + 15 of the tile on the 16-row side, the query heads on the 8-column side
//   values: dimensions on the 16-row side (V^T page rows), heads on the 8-column side, the tile's keys as the inner index,
//           cut into KS slices when there are fewer than 8 blocks of 16 dimensions (MPW blocks per warp)
// Every operand row is read with 16-byte loads: lane % 4 holds elements 8 c .. 8 c + 7 of each 32, i.e. the inner index is
// permuted, the same way in both operands. K of the next tile and V of this one are in flight during the arithmetic. Bounded
// scores (see the prompt kernel) need no running maximum and splits just add up; ONLINE (no softcap, no bias): the warps agree on
// a tile's maxima through shared memory, and a running maximum that grows by more than kSlack rescales sums and outputs.
struct DecodeArgs { AttnCall c; float a2, b2, shift2; int tiles_max; int* error_flag; };
constexpr float kSlack = 8.0f;             // log2 units by which a score may exceed the softmax shift of its row
constexpr float kNoScore = -1e30f;         // initial running maximum without a sink: below every score
constexpr int DT_KEYS = 128, DT_PS = DT_KEYS + 8;      // keys per tile, row pitch of the weights in shared memory

__host__ __device__ inline size_t decode_smem(int dkp, int dv, int KS, int tiles_max) {
    // page ids, q [8][dkp + 8], weights [2][8][DT_PS], sums [8][8], outputs [KS][8][dv]; ONLINE: maxima [2][8][8] before the outputs
    return (size_t)((2 * tiles_max + 3) & ~3) * 4 + 8 * (size_t)(dkp + 8) * 2 + 2 * 8 * DT_PS * 2 + (64 + 128) * 4 + (size_t)KS * 8 * dv * 4;
}

template <bool ONLINE, int DKC, int KS, int MPW>
__global__ void __launch_bounds__(256, DKC == 8 || MPW == 2 ? 1 : 2) attn_decode_mma_kernel(const __grid_constant__ DecodeArgs a) {
    constexpr int MTP = MPW == 2 ? 8 : 8 / KS;             // warps along the dimensions
    constexpr int NCH = 4 / KS;                            // 32-key chunks of a warp's slice
    extern __shared__ __align__(16) uint8_t raw[];
    __shared__ float red[16];
    __shared__ int last_sm;
    const AttnCall& c = a.c;
    const AttnShape& s = c.s;
    const int R = s.H / s.G;
    int* pt_sm = reinterpret_cast<int*>(raw);
    bf16* q_sm = reinterpret_cast<bf16*>(raw + (size_t)((2 * a.tiles_max + 3) & ~3) * 4);
    bf16* p_sm = q_sm + 8 * (s.dkp + 8);
    float* l_sm = reinterpret_cast<float*>(p_sm + 2 * 8 * DT_PS);
    float* mx_sm = l_sm + 64;
    float* o_sm = mx_sm + 128;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lc = lane & 3;
    const int split = blockIdx.x, n_split = gridDim.x, g = blockIdx.y, b = blockIdx.z;
    pdl_sync();
    const int pos = start_pos(c, b, a.error_flag);
    const KeyPages pages(s, pos, pos);
    const int n_pg = pages.n, n_tiles = (n_pg + 1) / 2;
    const int t_beg = (int)((long)split * n_tiles / n_split), t_end = (int)((long)(split + 1) * n_tiles / n_split);
    const int32_t* pt = c.page_table + (long)b * c.max_pages;
    const bf16* prow = (const bf16*)c.proj + (long)b * s.ld;
    const long kh = (long)PG * s.dkp, vh = (long)PG * s.dv;
    for (int i = tid; i < 2 * (t_end - t_beg); i += 256) pt_sm[i] = 2 * t_beg + i < n_pg ? pt[pages.at(2 * t_beg + i)] : -1;
    const int nv = s.dkp >> 3;
    const float2 rms = qk_rms(c, prow, tid, red);
    const float rq = rms.x, rk = rms.y;
    for (int i = tid; i < 8 * nv; i += 256) {
        const int r = i / nv, e0 = (i - r * nv) * 8;
        float f[8] = {0, 0, 0, 0, 0, 0, 0, 0};
        if (r < R) normed8(prow + s.q_off, c.q_gain, (g * R + r) * s.dk, e0, s.dk, rq, f);
        store8(q_sm + r * (s.dkp + 8) + e0, f);
    }
    if (s.k_off >= 0 && split == n_split - 1) {
        const long page = pt[pages.at(n_pg - 1)];
        const int slot = pos & (PG - 1);
        bf16* kp = (bf16*)c.k_pool + (page * s.G + g) * kh + (long)slot * s.dkp;
        for (int i = tid; i < nv; i += 256) {
            float f[8];
            normed8(prow + s.k_off, c.k_gain, g * s.dk, i * 8, s.dk, rk, f);
            store8(kp + i * 8, f);
        }
        bf16* vp = (bf16*)c.v_pool + (page * s.G + g) * vh + slot;
        for (int d = tid; d < s.dv; d += 256) vp[(long)d * PG] = prow[s.v_off + g * s.dv + d];
    }
    __syncthreads();

    uint4 qb[DKC];
#pragma unroll
    for (int ch = 0; ch < DKC; ch++) {
        const int e = ch * 32 + lc * 8;
        qb[ch] = e < s.dkp ? *reinterpret_cast<const uint4*>(q_sm + lr * (s.dkp + 8) + e) : make_uint4(0, 0, 0, 0);
    }
    uint4 kr[DKC][2];
    auto load_k = [&](int t) {
        const int page = pt_sm[2 * (t - t_beg) + (warp >> 2)];
        const bf16* kp = (const bf16*)c.k_pool + ((long)page * s.G + g) * kh + (long)((warp & 3) * 16 + lr) * s.dkp + lc * 8;
#pragma unroll
        for (int ch = 0; ch < DKC; ch++) {
            const bool in = page >= 0 && ch * 32 + lc * 8 < s.dkp;
#pragma unroll
            for (int h = 0; h < 2; h++)
                kr[ch][h] = in ? *reinterpret_cast<const uint4*>(kp + (long)h * 8 * s.dkp + ch * 32) : make_uint4(0, 0, 0, 0);
        }
    };
    const int mt = warp % MTP, slice = warp / MTP;
    const bool pv_on = slice < KS;
    float acc[MPW][4] = {};
    float lsum[2] = {0.0f, 0.0f}, m_run[2] = {kNoScore, kNoScore};
    const float* bias_g = ONLINE ? nullptr : c.bias + (long)g * (2 * kBiasPad + s.window) * R;
    const float badd = s.softcap * kLog2e - a.shift2;
    if (t_beg < t_end) load_k(t_beg);
    for (int t = t_beg; t < t_end; t++) {
        uint4 vr[MPW][NCH][2];
        if (pv_on) {
#pragma unroll
            for (int ch = 0; ch < NCH; ch++) {
                const int key = slice * (DT_KEYS / KS) + ch * 32;          // of the tile
                const int page = pt_sm[2 * (t - t_beg) + (key >> 6)];
                const bf16* vp = (const bf16*)c.v_pool + ((long)page * s.G + g) * vh + (key & 63) + lc * 8;
#pragma unroll
                for (int m = 0; m < MPW; m++)
#pragma unroll
                    for (int h = 0; h < 2; h++) {
                        const int d = (mt + 8 * m) * 16 + lr + 8 * h;
                        vr[m][ch][h] = page >= 0 && d < s.dv ? *reinterpret_cast<const uint4*>(vp + (long)d * PG) : make_uint4(0, 0, 0, 0);
                    }
            }
        }
        // biases of this thread's two keys and two heads (-inf: masked, or no such head)
        const int d0 = pos - (pages.at(2 * t + (warp >> 2)) * PG + (warp & 3) * 16 + lr);        // distance of this thread's first key
        float bi[2][2];
        if (!ONLINE)
#pragma unroll
        for (int h = 0; h < 2; h++)
#pragma unroll
            for (int u = 0; u < 2; u++)
                bi[h][u] = lc * 2 + u < R ? bias_g[(long)(d0 - 8 * h + kBiasPad) * R + lc * 2 + u] : -INFINITY;
        float sc[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
        for (int ch = 0; ch < DKC; ch++) {
            mma_bf16(sc, kr[ch][0].x, kr[ch][1].x, kr[ch][0].y, kr[ch][1].y, qb[ch].x, qb[ch].y);
            mma_bf16(sc, kr[ch][0].z, kr[ch][1].z, kr[ch][0].w, kr[ch][1].w, qb[ch].z, qb[ch].w);
        }
        if (t + 1 < t_end) load_k(t + 1);
        bf16* pb = p_sm + (t & 1) * 8 * DT_PS + warp * 16 + lr;
        if (ONLINE) {
            float* mx = mx_sm + (t & 1) * 64;
            const bool in0 = 2 * t + (warp >> 2) < n_pg && sees(s, pos, pos - d0), in1 = 2 * t + (warp >> 2) < n_pg && sees(s, pos, pos - d0 + 8);
            float tm[2];
#pragma unroll
            for (int u = 0; u < 2; u++) {
                const bool head = lc * 2 + u < R;
                sc[u] = in0 && head ? sc[u] * a.a2 : -INFINITY;
                sc[2 + u] = in1 && head ? sc[2 + u] * a.a2 : -INFINITY;
                tm[u] = fmaxf(sc[u], sc[2 + u]);
#pragma unroll
                for (int o = 4; o < 32; o <<= 1) tm[u] = fmaxf(tm[u], __shfl_xor_sync(0xffffffffu, tm[u], o));
            }
            if (lr == 0) *reinterpret_cast<float2*>(mx + warp * 8 + lc * 2) = make_float2(tm[0], tm[1]);
            __syncthreads();
            float al[2];
#pragma unroll
            for (int u = 0; u < 2; u++) {
                float v = mx[lc * 2 + u];
#pragma unroll
                for (int w = 1; w < 8; w++) v = fmaxf(v, mx[w * 8 + lc * 2 + u]);
                const float m_new = v > m_run[u] + kSlack ? v : m_run[u];
                al[u] = ex2_fast(m_run[u] - m_new);
                m_run[u] = m_new;
                lsum[u] *= al[u];
            }
#pragma unroll
            for (int m = 0; m < MPW; m++)
#pragma unroll
                for (int i = 0; i < 4; i++) acc[m][i] *= al[i & 1];
        }
#pragma unroll
        for (int h = 0; h < 2; h++)
#pragma unroll
            for (int u = 0; u < 2; u++) {
                const float s2 = ONLINE ? sc[2 * h + u] - m_run[u]
                                        : __fmaf_rn(a.b2, rcp_fast(1.0f + ex2_fast(sc[2 * h + u] * a.a2)), __fmaf_rn(bi[h][u], kLog2e, badd));
                const float p = ex2_fast(s2);
                lsum[u] += p;
                pb[(lc * 2 + u) * DT_PS + 8 * h] = __float2bfloat16_rn(p);
            }
        __syncthreads();
        if (pv_on) {
            const bf16* pr = p_sm + (t & 1) * 8 * DT_PS + lr * DT_PS + slice * (DT_KEYS / KS) + lc * 8;
#pragma unroll
            for (int ch = 0; ch < NCH; ch++) {
                const uint4 pw = *reinterpret_cast<const uint4*>(pr + ch * 32);
#pragma unroll
                for (int m = 0; m < MPW; m++) {
                    mma_bf16(acc[m], vr[m][ch][0].x, vr[m][ch][1].x, vr[m][ch][0].y, vr[m][ch][1].y, pw.x, pw.y);
                    mma_bf16(acc[m], vr[m][ch][0].z, vr[m][ch][1].z, vr[m][ch][0].w, vr[m][ch][1].w, pw.z, pw.w);
                }
            }
        }
    }
    // sums over the warps' keys, outputs over the slices
#pragma unroll
    for (int o = 4; o < 32; o <<= 1)
#pragma unroll
        for (int u = 0; u < 2; u++) lsum[u] += __shfl_xor_sync(0xffffffffu, lsum[u], o);
    if (lr == 0) { l_sm[warp * 8 + lc * 2] = lsum[0]; l_sm[warp * 8 + lc * 2 + 1] = lsum[1]; }
    if (pv_on)
#pragma unroll
        for (int m = 0; m < MPW; m++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const int d = (mt + 8 * m) * 16 + lr + 8 * (i >> 1);
                if (d < s.dv) o_sm[((long)slice * 8 + lc * 2 + (i & 1)) * s.dv + d] = acc[m][i];
            }
    __syncthreads();
    auto head_l = [&](int r) { float v = 0.0f; for (int w = 0; w < 8; w++) v += l_sm[w * 8 + r]; return v; };
    auto head_o = [&](int r, int d) { float v = 0.0f; for (int k = 0; k < KS; k++) v += o_sm[((long)k * 8 + r) * s.dv + d]; return v; };
    // ONLINE: the heads' running maxima, the same in all warps
    if (ONLINE && tid < 4) { mx_sm[lc * 2] = m_run[0]; mx_sm[lc * 2 + 1] = m_run[1]; }
    if (ONLINE) __syncthreads();
    const float sink = s.sink ? ex2_fast(-a.shift2) : 0.0f;
    const long stride = (long)R * (s.dv + (ONLINE ? 2 : 1)), o_at = ONLINE ? 2 * R : R;
    float* part = c.ws + ((long)b * s.G + g) * n_split * stride;
    if (n_split > 1) {
        float* mine = part + split * stride;
        for (int i = tid; i < R; i += 256) { mine[i] = head_l(i); if (ONLINE) mine[R + i] = mx_sm[i]; }
        for (int i = tid; i < R * s.dv; i += 256) mine[o_at + i] = head_o(i / s.dv, i % s.dv);
        __threadfence();
        __syncthreads();
        int* cnt = c.counters + (long)b * s.G + g;
        if (tid == 0) last_sm = atomicAdd(cnt, 1) == n_split - 1;
        __syncthreads();
        if (!last_sm) return;
        __threadfence();
        if (tid == 0) *cnt = 0;
    }
    bf16* out = (bf16*)c.out + (long)b * c.ldo + (long)g * R * s.dv;
    for (int i = tid; i < R * s.dv; i += 256) {
        const int r = i / s.dv;
        float l = sink, v = 0.0f;
        if (ONLINE) {
            const float snk = sink_score(c, g * R + r) * kLog2e;             // -inf without a sink
            float m = fmaxf(snk, kNoScore);
            if (n_split > 1) {
                for (int k = 0; k < n_split; k++) m = fmaxf(m, __ldcg(part + k * stride + R + r));
                l = ex2_fast(snk - m);
#pragma unroll 4
                for (int k = 0; k < n_split; k++) {
                    const float w = ex2_fast(__ldcg(part + k * stride + R + r) - m);
                    l = __fmaf_rn(__ldcg(part + k * stride + r), w, l);
                    v = __fmaf_rn(__ldcg(part + k * stride + o_at + i), w, v);
                }
            } else {
                m = fmaxf(m, mx_sm[r]);
                const float w = ex2_fast(mx_sm[r] - m);
                l = __fmaf_rn(head_l(r), w, ex2_fast(snk - m));
                v = head_o(r, i - r * s.dv) * w;
            }
        } else if (n_split > 1) {
#pragma unroll 4
            for (int k = 0; k < n_split; k++) { l += __ldcg(part + k * stride + r); v += __ldcg(part + k * stride + R + i); }
        } else {
            l += head_l(r); v = head_o(r, i - r * s.dv);
        }
        v /= l;
        if (s.g_off >= 0) v *= sigmoid_f<true>(to_f(prow[s.g_off + (long)g * R * s.dv + i]));
        out[i] = __float2bfloat16_rn(v);
    }
}

// ---------------------------------------------------------------------------------------------------------------
// Prompt attention on the tensor cores. A CTA takes TQ = 128 / R consecutive positions x the R query heads of one key/value
// head (row = position * R + head: the heads of a group share the K and V tiles, and a small window wastes few keys), and
// walks the key pages its window reaches (and those of the kept first positions). Scores bounded by softcap + max|bias| have a
// constant softmax shift (`shift2`) and the values accumulate in TMEM over all pages without rescaling. ONLINE (no softcap, no
// bias): a row's shift is its running maximum, lazily: only when a score exceeds it by more than kSlack does the row's warp wait
// for the products so far and rescale the accumulator in TMEM.
//   warps 0..3  softmax: one row per thread        warp 4  TMA: Q, then K and V pages        warp 5  MMA issue, TMEM
struct PrefillArgs {
    AttnCall c;
    int R, TQ, n_qt;                  // heads per group, positions per CTA, CTAs per (sequence, group)
    int kc, vrows;                    // 128-byte blocks of a Q/K row; rows of a V^T tile (dv rounded up to 16)
    float a2, b2, shift2;             // tanh argument factor and -2 softcap in log2 units; softmax shift
    int tmem_cols, o_col, p_bufs;
    bool online;
    int* error_flag;
};
constexpr int PF_S_COLS = 64;

struct PrefillSmem { uint32_t k, v, p, bias, bars, total; };
__host__ __device__ inline PrefillSmem prefill_smem(int kc, int vrows, int R, int TQ, int p_bufs, bool online) {
    PrefillSmem o;
    o.k = (uint32_t)kc * 16384u;                                   // Q first
    o.v = o.k + 2u * (uint32_t)kc * 8192u;
    o.p = o.v + 2u * (((uint32_t)vrows * 128u + 1023u) & ~1023u);
    o.bias = o.p + (uint32_t)p_bufs * 16384u;
    const uint32_t bias_floats = online ? 0u : (uint32_t)((TQ + 63) * R + 128);
    o.bars = o.bias + 2u * ((bias_floats * 4u + 15u) & ~15u);
    o.total = o.bars + 256u + 1024u;
    return o;
}

template <bool ONLINE>
__global__ void __launch_bounds__(192, 2) attn_window_prefill_kernel(const __grid_constant__ CUtensorMap tmapQ,
                                                                  const __grid_constant__ CUtensorMap tmapK,
                                                                  const __grid_constant__ CUtensorMap tmapV,
                                                                  const __grid_constant__ PrefillArgs a) {
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t base = (raw + 1023u) & ~1023u;
    uint8_t* base_ptr = smem_raw + (base - raw);
    const AttnShape& s = a.c.s;
    const int R = a.R, TQ = a.TQ;
    const PrefillSmem o = prefill_smem(a.kc, a.vrows, R, TQ, a.p_bufs, ONLINE);
    const uint32_t k_bytes = (uint32_t)a.kc * 8192u, v_bytes = (uint32_t)a.vrows * 128u, v_stride = (v_bytes + 1023u) & ~1023u;
    uint64_t* bars = reinterpret_cast<uint64_t*>(base_ptr + o.bars);
    const uint32_t bar_q = smem_u32(bars);
    const uint32_t bar_kf = bar_q + 8, bar_ke = bar_kf + 16, bar_vf = bar_ke + 16, bar_ve = bar_vf + 16;
    const uint32_t bar_sf = bar_ve + 16, bar_se = bar_sf + 16, bar_pf = bar_se + 16, bar_pe = bar_pf + 16, bar_o = bar_pe + 16;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 20);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;

    if (threadIdx.x == 0) {
        mbar_init(bar_q, 1); mbar_init(bar_o, 1);
        for (int i = 0; i < 2; i++) {
            mbar_init(bar_kf + 8 * i, 1); mbar_init(bar_ke + 8 * i, 1); mbar_init(bar_vf + 8 * i, 1); mbar_init(bar_ve + 8 * i, 1);
            mbar_init(bar_sf + 8 * i, 1); mbar_init(bar_se + 8 * i, 4); mbar_init(bar_pf + 8 * i, 4); mbar_init(bar_pe + 8 * i, 1);
        }
        *abort_flag = 0;
        fence_barrier_init();
    }
    if (warp == 5) { tmem_alloc(smem_u32(tmem_slot), a.tmem_cols); tmem_relinquish(); }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    pdl_sync();

    // the longest-running tiles (late positions) first
    const int qt = a.n_qt - 1 - (int)blockIdx.x, g = blockIdx.y, b = blockIdx.z;
    const int p0 = start_pos(a.c, b, a.error_flag);
    const int q0 = p0 + qt * TQ;                                         // first position of the tile
    const int q1 = min(p0 + a.c.Sc, q0 + TQ) - 1;                        // last one
    const KeyPages pages(s, q0, q1);
    const int n_kt = pages.n;
    const int32_t* pt = a.c.page_table + (long)b * a.c.max_pages;

    if (warp == 4) {
        if (lane == 0) {
            tma_prefetch_desc(&tmapQ); tma_prefetch_desc(&tmapK); tma_prefetch_desc(&tmapV);
            mbar_expect_tx(bar_q, (uint32_t)a.kc * (uint32_t)(TQ * R) * 128u);
            for (int i = 0; i < a.kc; i++) tma_load_3d(base + i * 16384u, &tmapQ, bar_q, i * 128, g * R, b * a.c.Sc + qt * TQ);
            bool ok = true;
            for (int j = 0; ok && j < n_kt; j++) {
                const int sb = j & 1;
                const uint32_t ph = (uint32_t)((j >> 1) & 1) ^ 1u;
                const int page = __ldg(pt + pages.at(j));
                if (!mbar_wait(bar_ke + 8 * sb, ph, abort_flag)) break;
                mbar_expect_tx(bar_kf + 8 * sb, k_bytes);
                for (int i = 0; i < a.kc; i++)
                    tma_load_2d(base + o.k + sb * k_bytes + i * 8192u, &tmapK, bar_kf + 8 * sb, i * 128, (page * s.G + g) * PG);
                if (!mbar_wait(bar_ve + 8 * sb, ph, abort_flag)) { ok = false; break; }
                mbar_expect_tx(bar_vf + 8 * sb, v_bytes);
                tma_load_2d(base + o.v + sb * v_stride, &tmapV, bar_vf + 8 * sb, 0, (page * s.G + g) * s.dv);
            }
        }
    } else if (warp == 5) {
        if (lane == 0) {
            const uint32_t idesc_qk = umma_idesc_bf16(128, PF_S_COLS), idesc_pv = umma_idesc_bf16(128, a.vrows);
            const int ksteps = (s.dkp + 15) / 16;
            bool ok = mbar_wait(bar_q, 0, abort_flag);
            auto issue_qk = [&](int j) {
                const int sb = j & 1;
                const uint32_t ph = (uint32_t)((j >> 1) & 1);
                if (!mbar_wait(bar_kf + 8 * sb, ph, abort_flag)) return false;
                if (!mbar_wait(bar_se + 8 * sb, ph ^ 1u, abort_flag)) return false;
                tc_fence_after();
                for (int k = 0; k < ksteps; k++) {
                    const uint32_t blk = k >> 2, off = 2 * (k & 3);
                    umma_bf16(tmem_base + sb * PF_S_COLS, umma_desc_k_sw128(base + blk * 16384u) + off,
                              umma_desc_k_sw128(base + o.k + sb * k_bytes + blk * 8192u) + off, idesc_qk, k > 0 ? 1u : 0u);
                }
                umma_commit(bar_sf + 8 * sb);
                umma_commit(bar_ke + 8 * sb);
                return true;
            };
            if (ok) ok = issue_qk(0);
            for (int j = 0; ok && j < n_kt; j++) {
                if (j + 1 < n_kt && !issue_qk(j + 1)) { ok = false; break; }
                const int sb = j & 1, pb = a.p_bufs == 2 ? sb : 0;
                if (!mbar_wait(bar_vf + 8 * sb, (uint32_t)((j >> 1) & 1), abort_flag)) { ok = false; break; }
                if (!mbar_wait(bar_pf + 8 * pb, (uint32_t)((a.p_bufs == 2 ? j >> 1 : j) & 1), abort_flag)) { ok = false; break; }
                tc_fence_after();
                const uint64_t pd = umma_desc_k_sw128(base + o.p + pb * 16384u), vd = umma_desc_k_sw128(base + o.v + sb * v_stride);
                for (int k = 0; k < 4; k++)
                    umma_bf16(tmem_base + a.o_col, pd + 2 * k, vd + 2 * k, idesc_pv, (j > 0 || k > 0) ? 1u : 0u);
                umma_commit(bar_pe + 8 * pb);
                umma_commit(bar_ve + 8 * sb);
            }
            if (ok) umma_commit(bar_o);
        }
    } else {
        const int rr = warp * 32 + lane;                       // row: position rr / R of the tile, head rr % R of the group
        const uint32_t lane_addr = (uint32_t)(warp * 32) << 16;
        const int n_bias = ONLINE ? 0 : (TQ + 63) * R;
        float* bias_sm = reinterpret_cast<float*>(base_ptr + o.bias);
        const int bias_stride = (n_bias + 128 + 3) & ~3;
        const float* bias_g = ONLINE ? nullptr : a.c.bias + (long)g * (2 * kBiasPad + s.window) * R;
        auto wait_bar = [&](uint32_t bar, uint32_t parity) {
            int got = (lane == 0) ? (mbar_wait(bar, parity, abort_flag) ? 1 : 0) : 1;
            return __shfl_sync(0xffffffffu, got, 0) != 0;
        };
        // biases of key tile j, in log2 units with the constants of the score formula folded in; masked keys stay -inf.
        // Entry (t + 63 - key) * R + r belongs to position t, head r: consecutive rows read consecutive words.
        const float badd = s.softcap * kLog2e - a.shift2;
        // The values of the next tile travel through registers, so that their latency hides behind this tile's arithmetic.
        constexpr int NB = 9;                                            // (TQ + 63) * R <= 1136 for R <= 16
        float nb[NB];
        auto fetch_bias = [&](int j) {
            const int dmin = q0 - pages.at(j) * PG - 63;                 // distance of the first entry
            const float* src = bias_g + (long)(dmin + kBiasPad) * R;
#pragma unroll
            for (int i = 0; i < NB; i++) nb[i] = rr + 128 * i < n_bias ? src[rr + 128 * i] : 0.0f;
        };
        auto stage_bias = [&](int j) {
            float* dst = bias_sm + (j & 1) * bias_stride;
#pragma unroll
            for (int i = 0; i < NB; i++)
                if (rr + 128 * i < n_bias) dst[rr + 128 * i] = __fmaf_rn(nb[i], kLog2e, badd);
        };
        float l = 0.0f;
        bool ok = true;
        // ---- ONLINE: this row's position, its softmax shift and, per tile, the keys it sees
        const int my_pos = q0 + rr / R;
        const float snk = ONLINE ? sink_score(a.c, g * R + rr % R) * kLog2e : 0.0f;
        float m = ONLINE ? fmaxf(snk, kNoScore) : 0.0f;
        if (ONLINE)
        for (int j = 0; j < n_kt; j++) {
            const int sb = j & 1, pb = a.p_bufs == 2 ? sb : 0;
            if (!wait_bar(bar_sf + 8 * sb, (uint32_t)((j >> 1) & 1))) { ok = false; break; }
            tc_fence_after();
            const uint32_t tS = tmem_base + sb * PF_S_COLS + lane_addr;
            uint32_t v[4][16];
#pragma unroll
            for (int cc = 0; cc < 4; cc++) tmem_ld_32x16(tS + 16 * cc, v[cc]);
            tmem_ld_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_se + 8 * sb);                 // the scores are in registers: the next product may start
            const int key0 = pages.at(j) * PG;
            const int hi = my_pos - key0, lo = hi - s.window + 1, kept = s.keep - key0;      // sees key c: c <= hi, c >= lo or c < kept
            const bool all = hi >= PG - 1 && (lo <= 0 || kept >= PG);
            float mx = -INFINITY;
#pragma unroll
            for (int cc = 0; cc < 4; cc++)
#pragma unroll
                for (int i = 0; i < 16; i++) v[cc][i] = __float_as_uint(__uint_as_float(v[cc][i]) * a.a2);
            if (!__all_sync(0xffffffffu, all))
#pragma unroll
                for (int cc = 0; cc < 4; cc++)
#pragma unroll
                    for (int i = 0; i < 16; i++) {
                        const int c = cc * 16 + i;
                        if (c > hi || (c < lo && c >= kept)) v[cc][i] = 0xff800000u;
                    }
#pragma unroll
            for (int cc = 0; cc < 4; cc++)
#pragma unroll
                for (int i = 0; i < 16; i++) mx = fmaxf(mx, __uint_as_float(v[cc][i]));
            const bool grow = mx > m + kSlack;
            if (__any_sync(0xffffffffu, grow)) {
                const float m_new = grow ? mx : m, al = ex2_fast(m - m_new);
                m = m_new;
                l *= al;
                if (j > 0) {
                    // the products up to tile j - 1 are in the accumulator; tile j's waits for this warp's weights
                    const int ob = a.p_bufs == 2 ? (j - 1) & 1 : 0;
                    if (!wait_bar(bar_pe + 8 * ob, (uint32_t)((a.p_bufs == 2 ? (j - 1) >> 1 : j - 1) & 1))) { ok = false; break; }
                    tc_fence_after();
                    for (int d0 = 0; d0 < a.vrows; d0 += 16) {
                        uint32_t w[16];
                        tmem_ld_32x16(tmem_base + a.o_col + d0 + lane_addr, w);
                        tmem_ld_wait();
#pragma unroll
                        for (int i = 0; i < 16; i++) w[i] = __float_as_uint(__uint_as_float(w[i]) * al);
                        tmem_st_32x16(tmem_base + a.o_col + d0 + lane_addr, w);
                    }
                    tmem_st_wait();
                    tc_fence_before();
                }
            }
            if (!wait_bar(bar_pe + 8 * pb, (uint32_t)((a.p_bufs == 2 ? j >> 1 : j) & 1) ^ 1u)) { ok = false; break; }
            uint8_t* prow = base_ptr + o.p + pb * 16384 + rr * 128;
#pragma unroll
            for (int cc = 0; cc < 4; cc++) {
                uint32_t pk[8];
#pragma unroll
                for (int i = 0; i < 16; i += 2) {
                    const float p0 = ex2_fast(__uint_as_float(v[cc][i]) - m), p1 = ex2_fast(__uint_as_float(v[cc][i + 1]) - m);
                    l += p0 + p1;
                    pk[i >> 1] = bf_pack(p0, p1);
                }
                *reinterpret_cast<uint4*>(prow + (((2 * cc) ^ (rr & 7)) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
                *reinterpret_cast<uint4*>(prow + (((2 * cc + 1) ^ (rr & 7)) << 4)) = make_uint4(pk[4], pk[5], pk[6], pk[7]);
            }
            fence_proxy_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_pf + 8 * pb);
        }
        if (!ONLINE) { fetch_bias(0); stage_bias(0); }
        if (!ONLINE)
        for (int j = 0; j < n_kt; j++) {
            const int sb = j & 1, pb = a.p_bufs == 2 ? sb : 0;
            named_sync<1, 128>();                                        // tile j's biases are in place; j - 1's reads are over
            if (j + 1 < n_kt) fetch_bias(j + 1);
            const float* bs = bias_sm + sb * bias_stride + rr + 63 * R;
            if (ok && !wait_bar(bar_sf + 8 * sb, (uint32_t)((j >> 1) & 1))) ok = false;
            if (ok && !wait_bar(bar_pe + 8 * pb, (uint32_t)((a.p_bufs == 2 ? j >> 1 : j) & 1) ^ 1u)) ok = false;
            if (!ok) continue;                                           // keep meeting the others at the barrier
            tc_fence_after();
            uint8_t* prow = base_ptr + o.p + pb * 16384 + rr * 128;
            const uint32_t tS = tmem_base + sb * PF_S_COLS + lane_addr;
            auto chunk = [&](const uint32_t (&v)[16], int cc) {
                uint32_t pk[8];
#pragma unroll
                for (int i = 0; i < 16; i += 2) {
                    // softcap * tanh(z) = softcap - 2 softcap / (1 + e^(2 z)), in log2 units; the two reciprocals of a pair
                    // come from one: 1/x = y / (x y). The clamp (tanh is 1 there) keeps the product finite.
                    const float e0 = 1.0f + ex2_fast(fminf(__uint_as_float(v[i]) * a.a2, 60.0f));
                    const float e1 = 1.0f + ex2_fast(fminf(__uint_as_float(v[i + 1]) * a.a2, 60.0f));
                    const float rc = rcp_fast(e0 * e1) * a.b2;
                    const float p0 = ex2_fast(__fmaf_rn(rc, e1, bs[-(cc * 16 + i) * R]));
                    const float p1 = ex2_fast(__fmaf_rn(rc, e0, bs[-(cc * 16 + i + 1) * R]));
                    l += p0 + p1;
                    pk[i >> 1] = bf_pack(p0, p1);
                }
                *reinterpret_cast<uint4*>(prow + (((2 * cc) ^ (rr & 7)) << 4)) = make_uint4(pk[0], pk[1], pk[2], pk[3]);
                *reinterpret_cast<uint4*>(prow + (((2 * cc + 1) ^ (rr & 7)) << 4)) = make_uint4(pk[4], pk[5], pk[6], pk[7]);
            };
            uint32_t va[16], vb[16];
            tmem_ld_32x16(tS, va);
            tmem_ld_wait();
            tmem_ld_32x16(tS + 16, vb);
            chunk(va, 0);
            tmem_ld_wait();
            tmem_ld_32x16(tS + 32, va);
            chunk(vb, 1);
            tmem_ld_wait();
            tmem_ld_32x16(tS + 48, vb);
            chunk(va, 2);
            tmem_ld_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_se + 8 * sb);                 // the scores are in registers: the next product may start
            chunk(vb, 3);
            fence_proxy_async_smem();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar_pf + 8 * pb);
            if (j + 1 < n_kt) stage_bias(j + 1);
        }
        if (ok) ok = wait_bar(bar_o, 0);
        if (ok) {
            tc_fence_after();
            const int t = rr / R, r = rr - t * R;
            const bool row_ok = rr < TQ * R && q0 + t <= q1;
            const float rl = 1.0f / (l + (ONLINE ? ex2_fast(snk - m) : s.sink ? ex2_fast(-a.shift2) : 0.0f));
            const long m = (long)b * a.c.Sc + qt * TQ + t;
            const long hcol = (long)(g * R + r) * s.dv;
            bf16* out = (bf16*)a.c.out + m * a.c.ldo + hcol;
            const bf16* gate = s.g_off >= 0 ? (const bf16*)a.c.proj + m * s.ld + s.g_off + hcol : nullptr;
            const bool vec = (s.dv & 7) == 0 && (a.c.ldo & 7) == 0;       // proj offsets and rows are multiples of 8
            for (int d0 = 0; d0 < a.vrows; d0 += 16) {
                uint32_t v[16];
                tmem_ld_32x16(tmem_base + a.o_col + d0 + lane_addr, v);
                tmem_ld_wait();
                if (!row_ok) continue;
#pragma unroll
                for (int h = 0; h < 2; h++) {
                    const int d = d0 + 8 * h;
                    if (d >= s.dv) continue;
                    float f[8], gf[8];
                    if (vec) {
                        if (gate) load8(gate + d, gf);
#pragma unroll
                        for (int e = 0; e < 8; e++) { f[e] = __uint_as_float(v[8 * h + e]) * rl; if (gate) f[e] *= sigmoid_f<true>(gf[e]); }
                        *reinterpret_cast<uint4*>(out + d) = make_uint4(bf_pack(f[0], f[1]), bf_pack(f[2], f[3]), bf_pack(f[4], f[5]), bf_pack(f[6], f[7]));
                    } else {
#pragma unroll
                        for (int e = 0; e < 8; e++)
                            if (d + e < s.dv) {
                                float x = __uint_as_float(v[8 * h + e]) * rl;
                                if (gate) x *= sigmoid_f<true>(to_f(gate[d + e]));
                                out[d + e] = __float2bfloat16_rn(x);
                            }
                    }
                }
            }
        }
    }

    tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        const unsigned long long t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 200000ull) { __nanosleep(1000); }
        if (threadIdx.x == 0 && a.error_flag) atomicOr(a.error_flag, 1);
        __syncthreads();
    }
    if (warp == 5) { tc_fence_after(); tmem_dealloc(tmem_base, a.tmem_cols); }
}

int set_smem(const void* kern, size_t bytes) {
    return bytes > 48 * 1024 ? cuda_status(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes)) : FLEXLLM_OK;
}

template <class T, int RC, bool FUSED, bool WIDE> int launch_row(const AttnCall& c, int splits, int L, cudaStream_t st) {
    const int R = c.s.H / c.s.G;
    const size_t smem = (size_t)row_smem(R, c.s.dkp, c.s.dv).total * 4;
    if (smem > 220 * 1024) return FLEXLLM_ENOTSUP;
    auto kern = attn_row_kernel<T, RC, FUSED, WIDE>;
    TRY_RC(set_smem((const void*)kern, smem));
    launch_k(kern, dim3(splits, c.s.G, c.B * c.Sc), dim3(256), smem, st, c, L, device_error_flag());
    return launch_status();
}

template <class T, bool FUSED> int run_row(const AttnCall& c, cudaStream_t st) {
    const AttnShape& s = c.s;
    const int R = s.H / s.G;
    const long ctas = (long)c.B * c.Sc * s.G;
    if (ctas / s.G > 65535) return FLEXLLM_ENOTSUP;
    const int reach = s.window < c.max_pos + 1 ? s.window : c.max_pos + 1;
    const int tiles = ((reach + 2 * PG - 2) / PG + attn_keep_pages(s.keep)) / TILE_PAGES + 1;
    long splits = 1;
    if (FUSED && c.ws) {
        splits = 2L * gemm_sm_count() / ctas;
        if (splits > tiles) splits = tiles;
        const long per = ctas * R * (s.dv + 2);
        if (splits * per > (long)c.ws_floats) splits = (long)c.ws_floats / per;
        if (splits < 1 || ctas > c.n_counters) splits = 1;
    }
    const int vecs = s.dkp / 8;
    const int L = vecs <= 8 ? 8 : vecs <= 16 ? 16 : 32;
#define FLEXLLM_ROW(RC_) return vecs > 32 ? launch_row<T, RC_, FUSED, true>(c, (int)splits, L, st) : launch_row<T, RC_, FUSED, false>(c, (int)splits, L, st)
    if (R == 1) FLEXLLM_ROW(1);
    if (R == 2) FLEXLLM_ROW(2);
    FLEXLLM_ROW(4);
#undef FLEXLLM_ROW
}

// Constants of the score formula in log2 units for the kernels that rely on bounded scores; false when the bound is missing
// (no softcap) or so wide that sums could vanish below the smallest floats.
bool bounded_scores(const AttnCall& c, float* a2, float* b2, float* shift2) {
    const AttnShape& s = c.s;
    if (s.softcap <= 0.0f || !c.bias || s.keep || s.sink == 2) return false;
    const float bound2 = (s.softcap + c.bias_max_abs) * kLog2e;
    *shift2 = bound2 > 100.0f ? bound2 - 100.0f : 0.0f;
    *a2 = s.scale / s.softcap * 2.0f * kLog2e; *b2 = -2.0f * s.softcap * kLog2e;
    return *shift2 <= (s.sink ? 80.0f : 20.0f);
}

template <bool ONLINE, int DKC, int KS, int MPW> int launch_decode(DecodeArgs& a, int splits, cudaStream_t st) {
    const AttnCall& c = a.c;
    const size_t smem = decode_smem(c.s.dkp, c.s.dv, KS, a.tiles_max);
    auto kern = attn_decode_mma_kernel<ONLINE, DKC, KS, MPW>;
    if (smem > 200 * 1024) return FLEXLLM_ENOTSUP;
    TRY_RC(set_smem((const void*)kern, smem));
    launch_k(kern, dim3(splits, c.s.G, c.B), dim3(256), smem, st, a);
    return launch_status();
}
template <bool ONLINE, int DKC> int pick_decode(DecodeArgs& a, int splits, cudaStream_t st) {
    const int dv = a.c.s.dv;
    if (dv <= 32) return launch_decode<ONLINE, DKC, 4, 1>(a, splits, st);
    if (dv <= 64) return launch_decode<ONLINE, DKC, 2, 1>(a, splits, st);
    if (dv <= 128) return launch_decode<ONLINE, DKC, 1, 1>(a, splits, st);
    return launch_decode<ONLINE, DKC, 1, 2>(a, splits, st);
}
template <bool ONLINE> int pick_decode_dk(DecodeArgs& a, int splits, cudaStream_t st) {
    if (a.c.s.dkp <= 64) return pick_decode<ONLINE, 2>(a, splits, st);
    if (a.c.s.dkp <= 128) return pick_decode<ONLINE, 4>(a, splits, st);
    return pick_decode<ONLINE, 8>(a, splits, st);
}
// Whether the ONLINE forms cover the scores; their factor to log2 units.
bool plain_scores(const AttnCall& c, float* a2) {
    *a2 = c.s.scale * kLog2e;
    return c.s.softcap <= 0.0f && !c.bias;
}
// FLEXLLM_ENOTSUP: the row kernel takes the call.
int run_decode(const AttnCall& c, cudaStream_t st) {
    const AttnShape& s = c.s;
    DecodeArgs a;
    a.c = c; a.error_flag = device_error_flag();
    const bool bounded = bounded_scores(c, &a.a2, &a.b2, &a.shift2);
    if (s.H / s.G > 8 || s.dkp > 256 || s.dv > 256 || c.B > 65535 || (!bounded && !plain_scores(c, &a.a2))) return FLEXLLM_ENOTSUP;
    const int reach = s.window < c.max_pos + 1 ? s.window : c.max_pos + 1;
    const int tiles = ((reach + 2 * PG - 2) / PG + attn_keep_pages(s.keep)) / 2 + 1;
    const long ctas = (long)c.B * s.G;
    long splits = (kDecodeCtas + ctas - 1) / ctas;
    if (splits > tiles / 2) splits = tiles / 2;
    const long per = ctas * (s.H / s.G) * (s.dv + 2);
    if (splits * per > (long)c.ws_floats) splits = (long)c.ws_floats / per;
    if (splits < 1 || ctas > c.n_counters || !c.ws) splits = 1;
    a.tiles_max = (int)((tiles + splits - 1) / splits + 1);
    return bounded ? pick_decode_dk<false>(a, (int)splits, st) : pick_decode_dk<true>(a, (int)splits, st);
}

// Whether the tensor-core kernel covers the call (bf16 only).
bool prefill_covers(const AttnCall& c, PrefillArgs* a) {
    const AttnShape& s = c.s;
    a->c = c;
    a->R = s.H / s.G; a->TQ = a->R <= 16 ? 128 / a->R : 0;
    if (a->R > 16 || s.dkp > 256 || s.dv > 256) return false;
    a->online = !bounded_scores(c, &a->a2, &a->b2, &a->shift2);
    if (a->online && !plain_scores(c, &a->a2)) return false;
    a->kc = (s.dkp + 63) / 64; a->vrows = (s.dv + 15) / 16 * 16;
    a->n_qt = (c.Sc + a->TQ - 1) / a->TQ;
    a->o_col = 2 * PF_S_COLS;
    int cols = 32;
    while (cols < a->o_col + a->vrows) cols *= 2;
    a->tmem_cols = cols;
    // two CTAs per SM where one P buffer makes that possible
    a->p_bufs = prefill_smem(a->kc, a->vrows, a->R, a->TQ, 2, a->online).total <= 113 * 1024 ? 2
              : prefill_smem(a->kc, a->vrows, a->R, a->TQ, 1, a->online).total <= 113 * 1024 ? 1 : 2;
    if (prefill_smem(a->kc, a->vrows, a->R, a->TQ, a->p_bufs, a->online).total > 227 * 1024) a->p_bufs = 1;
    a->error_flag = device_error_flag();
    return prefill_smem(a->kc, a->vrows, a->R, a->TQ, a->p_bufs, a->online).total <= 227 * 1024;
}

int run_prefill(const PrefillArgs& a, cudaStream_t st) {
    const AttnCall& c = a.c;
    const AttnShape& s = c.s;
    CUtensorMap tq, tk, tv;
    TRY_RC(make_tmap_rows3_u8(&tq, c.q, (uint64_t)c.B * c.Sc, (uint64_t)s.H, (uint64_t)s.dkp * 2, (uint32_t)a.TQ, (uint32_t)a.R));
    TRY_RC(cached_tmap_u8(&tk, c.k_pool, (uint64_t)c.n_pages * s.G * PG, (uint64_t)s.dkp * 2, PG, 0));
    TRY_RC(cached_tmap_u8(&tv, c.v_pool, (uint64_t)c.n_pages * s.G * s.dv, PG * 2, (uint32_t)a.vrows, 0));
    const size_t smem = prefill_smem(a.kc, a.vrows, a.R, a.TQ, a.p_bufs, a.online).total;
    auto kern = a.online ? attn_window_prefill_kernel<true> : attn_window_prefill_kernel<false>;
    TRY_RC(set_smem((const void*)kern, smem));
    launch_k(kern, dim3(a.n_qt, s.G, c.B), dim3(192), smem, st, tq, tk, tv, a);
    return launch_status();
}

template <class T> int run_tensor_decode(const AttnCall&, cudaStream_t) { return FLEXLLM_ENOTSUP; }
template <> int run_tensor_decode<bf16>(const AttnCall& c, cudaStream_t st) { return run_decode(c, st); }
template <class T> bool run_tensor_prefill(const AttnCall&, cudaStream_t, int*) { return false; }
template <> bool run_tensor_prefill<bf16>(const AttnCall& c, cudaStream_t st, int* rc) {
    PrefillArgs a;
    if (!prefill_covers(c, &a)) return false;
    *rc = run_prefill(a, st);
    return true;
}

int check_call(const AttnCall& c) {
    const AttnShape& s = c.s;
    FLEXLLM_REQUIRE(c.proj && !c.q_gain == !c.k_gain && c.k_pool && c.v_pool && c.page_table && c.ctx && c.out);
    FLEXLLM_REQUIRE(s.keep >= 0 && (!c.bias || s.keep == 0) && (s.sink != 2 || c.sinks) && (s.k_off >= 0 || !c.q_gain));
    FLEXLLM_REQUIRE(s.H > 0 && s.G > 0 && s.H % s.G == 0 && s.dk > 0 && s.dv > 0 && s.window > 0 && s.dkp % 8 == 0 && s.dkp >= s.dk);
    FLEXLLM_REQUIRE(s.ld % 8 == 0 && s.q_off % 8 == 0 && (s.k_off < 0 || (s.k_off % 8 == 0 && s.v_off % 8 == 0)) && (s.g_off < 0 || s.g_off % 8 == 0));
    FLEXLLM_REQUIRE(c.B > 0 && c.Sc > 0 && c.max_pos >= c.Sc - 1 && c.max_pos < c.max_pages * PG && c.n_pages > 0);
    return FLEXLLM_OK;
}

}  // namespace

size_t attn_window_ws_floats(int max_batch, int G, int R, int dv) {
    const size_t ctas = (size_t)max_batch * G;
    return ((size_t)kDecodeCtas + ctas) * R * (dv + 2);
}

void attn_layout(AttnShape* s, bool gate, bool own_kv) {
    s->dkp = (int)up_to(s->dk, 8);
    s->q_off = 0;
    s->k_off = s->v_off = -1;
    int end = (int)up_to((long)s->H * s->dk, 8);
    if (own_kv) {
        s->k_off = end;
        s->v_off = s->k_off + (int)up_to((long)s->G * s->dk, 8);
        end = s->v_off + (int)up_to((long)s->G * s->dv, 8);
    }
    s->g_off = gate ? end : -1;
    s->ld = gate ? end + up_to((long)s->H * s->dv, 8) : end;
}

// Row of the distance table for distance n: exact below half the rows, logarithmic up to bias_max from there on. A quotient
// of logarithms that is an integer in exact arithmetic must not fall below it by rounding.
static int distance_bucket(int n, int rows, int bias_max) {
    const int half = rows / 2;
    if (n < half) return n;
    if (half == 0 || bias_max <= half) return rows - 1;
    const double v = std::log((double)n / half) / std::log((double)bias_max / half) * (rows - half);
    const double b = half + std::floor(v + 1e-9);
    return b < rows - 1 ? (int)b : rows - 1;
}

void attn_bias_table(const AttnShape& s, const float* table, int rows, int bias_max, float* out) {
    const int R = s.H / s.G;
    const size_t n = 2 * (size_t)kBiasPad + s.window;
    for (size_t i = 0; i < (size_t)s.H * n; i++) out[i] = -INFINITY;
    for (int d = 0; d < s.window; d++) {
        const int bk = distance_bucket(d, rows, bias_max);
        for (int h = 0; h < s.H; h++) out[((h / R) * n + kBiasPad + d) * R + h % R] = table[(size_t)bk * s.H + h];
    }
}

template <class T> int attn_window(const AttnCall& c, cudaStream_t st) {
    TRY_RC(check_call(c));
    if (c.Sc == 1) {
        const int rc = run_tensor_decode<T>(c, st);
        return rc == FLEXLLM_ENOTSUP ? run_row<T, true>(c, st) : rc;
    }
    FLEXLLM_REQUIRE(c.q);
    const int v_pages = c.s.k_off >= 0 ? (c.Sc + PG - 2) / PG + 1 : 0;
    launch_k(attn_prepare_kernel<T>, dim3(c.B * c.Sc + c.B * c.s.G * v_pages), dim3(256), 0, st, c, v_pages, device_error_flag());
    TRY_RC(launch_status());
    int rc = FLEXLLM_OK;
    if (run_tensor_prefill<T>(c, st, &rc)) return rc;
    return run_row<T, false>(c, st);
}
template int attn_window<float>(const AttnCall&, cudaStream_t);
template int attn_window<bf16>(const AttnCall&, cudaStream_t);

}  // namespace flexllm

using namespace flexllm;

// ---- C ABI, see include/flexllm_b200.h
namespace {
bool make_shape(const flexllm_attn_window_shape* a, AttnShape* s) {
    if (!a || a->heads <= 0 || a->kv_heads <= 0 || a->heads % a->kv_heads || a->dim <= 0 || a->vdim <= 0 || a->window <= 0) return false;
    *s = AttnShape();
    s->H = a->heads; s->G = a->kv_heads; s->dk = a->dim; s->dv = a->vdim; s->window = a->window;
    if (a->sink < 0 || a->sink > 2 || a->keep_first < 0) return false;
    s->scale = a->scale; s->softcap = a->softcap; s->sink = a->sink; s->keep = a->keep_first;
    attn_layout(s, a->gate != 0, !a->shared_kv);
    return true;
}
struct WindowWs { size_t ws_floats, counters, q, total; };      // byte offsets of the counters and of the q scratch
WindowWs window_ws(const AttnShape& s, int B, int n) {
    WindowWs w;
    w.ws_floats = attn_window_ws_floats(B, s.G, s.H / s.G, s.dv);
    w.counters = (w.ws_floats * 4 + 255) / 256 * 256;
    w.q = w.counters + ((size_t)B * s.G * 4 + 255) / 256 * 256;
    w.total = w.q + (size_t)B * n * s.H * s.dkp * 4 + 256;
    return w;
}
}  // namespace

extern "C" long flexllm_attn_window_row(const flexllm_attn_window_shape* a) { AttnShape s; return make_shape(a, &s) ? s.ld : 0; }
extern "C" size_t flexllm_attn_window_bias_floats(const flexllm_attn_window_shape* a) { AttnShape s; return make_shape(a, &s) ? attn_bias_floats(s) : 0; }
extern "C" size_t flexllm_attn_window_workspace(const flexllm_attn_window_shape* a, int B, int n) {
    AttnShape s;
    return make_shape(a, &s) && B > 0 && n > 0 ? window_ws(s, B, n).total : 0;
}
extern "C" int flexllm_attn_window_bias(const flexllm_attn_window_shape* a, const float* table_host, int rows, int bias_max, float* bias, void* stream) {
    AttnShape s;
    FLEXLLM_REQUIRE(make_shape(a, &s) && table_host && rows > 0 && bias);
    std::vector<float> t(attn_bias_floats(s));
    attn_bias_table(s, table_host, rows, bias_max, t.data());
    FLEXLLM_CHECK_CUDA(cudaMemcpyAsync(bias, t.data(), t.size() * 4, cudaMemcpyHostToDevice, (cudaStream_t)stream));
    return cuda_status(cudaStreamSynchronize((cudaStream_t)stream));
}
extern "C" int flexllm_attn_window(int dtype, flexllm_kv_cache* kv, int layer, const flexllm_attn_window_shape* a, const void* proj,
                                   const float* q_gain, const float* k_gain, const float* bias, float bias_abs, const float* sinks,
                                   const int32_t* page_table, int max_pages, const int32_t* ctx, int max_ctx, int B, int n, void* out, long ldo, void* workspace,
                                   size_t workspace_bytes, void* stream) {
    AttnCall c = {};
    FLEXLLM_REQUIRE(make_shape(a, &c.s) && kv && layer >= 0 && layer < kv->layers && B > 0 && n > 0);
    FLEXLLM_REQUIRE(dtype == FLEXLLM_F32 || dtype == FLEXLLM_BF16);
    FLEXLLM_REQUIRE(kv->elem_bytes == (dtype == FLEXLLM_BF16 ? 2 : 4));
    const flexllm_kv_shape& ks = kv->shape[layer];
    FLEXLLM_REQUIRE(ks.hkv == c.s.G && ks.kdim == c.s.dkp && ks.vdim == c.s.dv && ldo >= (long)c.s.H * c.s.dv);
    const WindowWs w = window_ws(c.s, B, n);
    FLEXLLM_REQUIRE(workspace && aligned(workspace, 256) && workspace_bytes >= w.total && aligned(proj, 16) && aligned(out, 16));
    c.proj = proj; c.q_gain = q_gain; c.k_gain = k_gain; c.eps = a->eps; c.bias = bias; c.bias_max_abs = bias_abs; c.sinks = sinks;
    c.k_pool = kv->k + kv->k_off[layer]; c.v_pool = kv->v + kv->v_off[layer]; c.n_pages = kv->n_pages;
    c.page_table = page_table; c.max_pages = max_pages; c.ctx = ctx; c.max_pos = max_ctx; c.B = B; c.Sc = n;
    c.ws = (float*)workspace; c.ws_floats = w.ws_floats; c.counters = (int*)((char*)workspace + w.counters); c.n_counters = B * c.s.G;
    c.q = (char*)workspace + w.q; c.out = out; c.ldo = ldo;
    cudaStream_t st = (cudaStream_t)stream;
    FLEXLLM_CHECK_CUDA(cudaMemsetAsync(c.counters, 0, (size_t)c.n_counters * 4, st));
    return dtype == FLEXLLM_BF16 ? attn_window<bf16>(c, st) : attn_window<float>(c, st);
}
