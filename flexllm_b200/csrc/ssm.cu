// State-space mixer (the Mamba-2 form) between its two projections, over per-sequence states:
//   x | B | C <- silu(causal convolution)       dt <- softplus(dt + dt_bias)
//   S_t = exp(A dt) S_{t-1} + dt B_t x_t^T       y_t = S_t^T C_t + D x_t         (per head; A = -exp(A_log))
//   out = rms norm in parts of (y * silu(z)) * gain
// Decays, steps and states are fp32. x, B and C are rounded to the activation type after the convolution.
// ssm_conv_kernel, then
//   prompts, bf16   : ssm_chunk_kernel on warp MMAs (chunks of 64 tokens, state in registers)
//   otherwise       : ssm_scan_kernel token by token (decoding: one state read and write)
// both with the gate in their epilogue, then ssm_norm_kernel.
// A state row holds one value dimension: [head][value dimension][state]. The inputs of the convolution are kept in a ring of
// `taps` rows per sequence, position p in row p % taps. A sequence at position 0 starts from zero whatever its slot holds.
#include "float_common.cuh"

namespace flexllm {

namespace {

constexpr int kChunk = 64;                 // tokens per step of the chunked form
constexpr int kScanTile = 16;              // tokens staged at a time by the scan

__device__ __forceinline__ float silu_acc(float z) { return z / (1.0f + expf(-z)); }
template <bool FAST> __device__ __forceinline__ float silu_t(float z) { return FAST ? z * rcp_fast(1.0f + ex2_fast(-z * kLog2e)) : silu_acc(z); }
__device__ __forceinline__ float softplus_f(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

// Input of the convolution at position `at` (channel c), from this call's rows or, before its first position p0, the history.
template <class T> __device__ __forceinline__ const T* conv_row(const SsmCall& k, int b, int p0, int at) {
    if (at >= p0) return (const T*)k.proj + ((long)b * k.Sc + (at - p0)) * k.s.ld + k.s.x_off;
    return (const T*)k.conv_state + ((long)b * k.s.taps + at % k.s.taps) * k.s.ch;
}
__device__ __forceinline__ int first_pos(const SsmCall& k, int b) { return max(0, k.ctx[b]); }

// The last inputs of the call go to the history. Every CTA of sequence b takes a share (id of n); the convolution, which reads the
// older history, was an earlier launch.
template <class T> __device__ __forceinline__ void keep_history(const SsmCall& k, int b, int p0, int id, int n) {
    const SsmShape& s = k.s;
    const int rows = min(k.Sc, s.taps), vecs = s.ch >> 3;
    for (int i = id * blockDim.x + threadIdx.x; i < rows * vecs; i += n * blockDim.x) {
        const int r = i / vecs, c = (i - r * vecs) * 8, at = p0 + k.Sc - 1 - r;
        const T* src = conv_row<T>(k, b, p0, at) + c;
        T* dst = (T*)k.conv_state + ((long)b * s.taps + at % s.taps) * s.ch + c;
        const uint4* a = reinterpret_cast<const uint4*>(src);
        uint4* d = reinterpret_cast<uint4*>(dst);
        d[0] = a[0];
        if (sizeof(T) == 4) d[1] = a[1];
    }
}

// ---------------------------------------------------------------------------------------------------------------
// Convolution and silu: one thread has 8 channels of TT consecutive tokens. TAPS 0: any number of taps.
constexpr int kConvTokens = 8;
// 8 elements as they lie in memory
template <class T> struct Vec8;
template <> struct Vec8<bf16> {
    uint4 v;
    __device__ __forceinline__ void load(const bf16* p) { v = *reinterpret_cast<const uint4*>(p); }
    __device__ __forceinline__ void zero() { v = make_uint4(0, 0, 0, 0); }
    __device__ __forceinline__ void get(float (&f)[8]) const { unpack8(v, f); }
};
template <> struct Vec8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float* p) { a = load4(p); b = load4(p + 4); }
    __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ void get(float (&f)[8]) const { f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w; }
};
template <class T, int TAPS>
__global__ void __launch_bounds__(128) ssm_conv_kernel(const SsmCall k) {
    constexpr bool FAST = sizeof(T) == 2;
    pdl_sync();
    const SsmShape& s = k.s;
    const int c = (blockIdx.x * 128 + threadIdx.x) * 8, t0 = blockIdx.y * kConvTokens, b = blockIdx.z;
    if (c >= s.ch) return;
    const int p0 = first_pos(k, b), t1 = min(t0 + kConvTokens, k.Sc), taps = TAPS ? TAPS : s.taps;
    auto load = [&](int at, float (&f)[8]) {
        if (at >= 0) load8(conv_row<T>(k, b, p0, at) + c, f);
        else
#pragma unroll
            for (int e = 0; e < 8; e++) f[e] = 0.0f;
    };
    auto put = [&](int t, const float (&v)[8]) {
        T* o = (T*)k.xbc + ((long)b * k.Sc + t) * s.ch + c;
        store4(o, make_float4(silu_t<FAST>(v[0]), silu_t<FAST>(v[1]), silu_t<FAST>(v[2]), silu_t<FAST>(v[3])));
        store4(o + 4, make_float4(silu_t<FAST>(v[4]), silu_t<FAST>(v[5]), silu_t<FAST>(v[6]), silu_t<FAST>(v[7])));
    };
    float bias[8];
    load8(k.conv_b + c, bias);
    if constexpr (TAPS > 0) {
        float w[TAPS][8];
        Vec8<T> in[TAPS - 1 + kConvTokens];                 // all inputs are asked for before the first is used
#pragma unroll
        for (int j = 0; j < TAPS - 1 + kConvTokens; j++) {
            const int at = p0 + t0 - (TAPS - 1) + j;
            if (at >= 0 && at < p0 + t1) in[j].load(conv_row<T>(k, b, p0, at) + c); else in[j].zero();
        }
#pragma unroll
        for (int j = 0; j < TAPS; j++) load8(k.conv_w + (long)j * s.ch + c, w[j]);
#pragma unroll
        for (int t = 0; t < kConvTokens; t++) {
            if (t0 + t >= t1) break;
            float v[8];
#pragma unroll
            for (int e = 0; e < 8; e++) v[e] = bias[e];
#pragma unroll
            for (int j = 0; j < TAPS; j++) {
                float x[8];
                in[t + j].get(x);
#pragma unroll
                for (int e = 0; e < 8; e++) v[e] = __fmaf_rn(w[j][e], x[e], v[e]);
            }
            put(t0 + t, v);
        }
    } else {
        for (int t = t0; t < t1; t++) {
            float v[8];
#pragma unroll
            for (int e = 0; e < 8; e++) v[e] = bias[e];
            for (int j = 0; j < taps; j++) {
                float w[8], x[8];
                load8(k.conv_w + (long)j * s.ch + c, w);
                load(p0 + t - (taps - 1) + j, x);
#pragma unroll
                for (int e = 0; e < 8; e++) v[e] = __fmaf_rn(w[e], x[e], v[e]);
            }
            put(t, v);
        }
    }
}

// ---------------------------------------------------------------------------------------------------------------
// Recurrence token by token, TT tokens staged at a time: a CTA has 32 value dimensions of one head, 8 lanes share a state row (NV
// float4 each).
template <class T, int NV, int TT>
__global__ void __launch_bounds__(256) ssm_scan_kernel(const SsmCall k) {
    constexpr bool FAST = sizeof(T) == 2;
    constexpr int NW = 32 * NV;
    __shared__ __align__(16) float b_sm[TT][NW], c_sm[TT][NW];
    __shared__ float x_sm[TT][32], dt_sm[TT], dec_sm[TT];
    const SsmShape& s = k.s;
    const int tid = threadIdx.x, h = blockIdx.y, b = blockIdx.z, g = h / (s.H / s.G);
    const int pb = blockIdx.x * 32, pr = tid >> 3, p = pb + pr, ns = tid & 7;
    const bool on = p < s.P;
    pdl_sync();
    const int p0 = first_pos(k, b);
    float* st = k.state + (((long)b * s.H + h) * s.P + (on ? p : 0)) * s.Np;
    float4 S[NV];
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int n = 32 * i + 4 * ns;
        S[i] = on && p0 > 0 && n < s.Np ? load4(st + n) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const float A = k.A[h], Dh = k.D[h], dtb = k.dt_bias[h];
    const int xc = h * s.P8 + pb, bc = s.inner + g * s.N8, cc = bc + s.G * s.N8;       // first channels of x, B and C
    for (int t0 = 0; t0 < k.Sc; t0 += TT) {
        const int nt = min(TT, k.Sc - t0);
        if (t0) __syncthreads();
        for (int i = tid; i < nt * (2 * NW + 32); i += 256) {
            const int t = i / (2 * NW + 32), j = i - t * (2 * NW + 32);
            const int e = j < NW ? j : j < 2 * NW ? j - NW : j - 2 * NW;
            const bool in = j < 2 * NW ? e < s.N8 : pb + e < s.P8;
            const int c = (j < NW ? bc : j < 2 * NW ? cc : xc) + e;
            float v = 0.0f;
            if (in) v = to_f(((const T*)k.xbc)[((long)b * k.Sc + t0 + t) * s.ch + c]);
            if (j < NW) b_sm[t][e] = v; else if (j < 2 * NW) c_sm[t][e] = v; else x_sm[t][e] = v;
        }
        if (tid < nt) {
            const T* row = (const T*)k.proj + ((long)b * k.Sc + t0 + tid) * s.ld;
            const float dt = softplus_f(to_f(row[s.dt_off + h]) + dtb);
            dt_sm[tid] = dt;
            dec_sm[tid] = expf(A * dt);
        }
        __syncthreads();
        for (int t = 0; t < nt; t++) {
            const float x = x_sm[t][pr], dec = dec_sm[t], dx = dt_sm[t] * x;
            float y = 0.0f;
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const float4 bv = load4(&b_sm[t][32 * i + 4 * ns]), cv = load4(&c_sm[t][32 * i + 4 * ns]);
                S[i].x = __fmaf_rn(S[i].x, dec, bv.x * dx); S[i].y = __fmaf_rn(S[i].y, dec, bv.y * dx);
                S[i].z = __fmaf_rn(S[i].z, dec, bv.z * dx); S[i].w = __fmaf_rn(S[i].w, dec, bv.w * dx);
                y = __fmaf_rn(S[i].x, cv.x, y); y = __fmaf_rn(S[i].y, cv.y, y); y = __fmaf_rn(S[i].z, cv.z, y); y = __fmaf_rn(S[i].w, cv.w, y);
            }
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
            if (ns == 0 && p < s.P8) {
                const long row = (long)b * k.Sc + t0 + t;
                const int col = h * s.P8 + p;
                const float z = to_f(((const T*)k.proj)[row * s.ld + col]);
                ((T*)k.y)[row * s.inner + col] = from_f<T>(on ? __fmaf_rn(Dh, x, y) * silu_t<FAST>(z) : 0.0f);
            }
        }
    }
    if (on)
#pragma unroll
        for (int i = 0; i < NV; i++)
            if (32 * i + 4 * ns < s.Np) store4(st + 32 * i + 4 * ns, S[i]);
    keep_history<T>(k, b, p0, blockIdx.x + gridDim.x * blockIdx.y, gridDim.x * gridDim.y);
}

// ---------------------------------------------------------------------------------------------------------------
// RMS norm of a row in `parts` equal parts of its H * P true columns (a part may begin and end inside a head). One CTA per row;
// a part's sum is formed by its own warps, or a warp takes several parts.
template <class T>
__global__ void __launch_bounds__(256) ssm_norm_kernel(const SsmCall k) {
    extern __shared__ float rinv[];                          // [parts], then [8] partial sums
    pdl_sync();
    const SsmShape& s = k.s;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const long row = blockIdx.x;
    const T* y = (const T*)k.y + row * s.inner;
    T* out = (T*)k.out + row * s.inner;
    const int len = s.H * s.P / s.parts;
    const bool vec = s.P == s.P8 && (len & 7) == 0;
    auto part_sum = [&](int part, int first, int step) {      // this lane's share
        float ss = 0.0f;
        if (vec) {
            const T* p = y + (long)part * len;
            for (int i = first; i < len >> 3; i += step) {
                float f[8];
                load8(p + 8 * i, f);
#pragma unroll
                for (int e = 0; e < 8; e++) ss = __fmaf_rn(f[e], f[e], ss);
            }
        } else {
            for (int i = first; i < len; i += step) {
                const int t = part * len + i, h = t / s.P;
                const float v = to_f(y[h * s.P8 + t - h * s.P]);
                ss = __fmaf_rn(v, v, ss);
            }
        }
        return warp_sum(ss);
    };
    float* part = rinv + s.parts;
    const int wpp = s.parts <= 4 ? 8 / s.parts : 1;          // warps per part
    if (wpp > 1) {
        if (warp < wpp * s.parts) {
            const float v = part_sum(warp / wpp, (warp % wpp) * 32 + lane, 32 * wpp);
            if (lane == 0) part[warp] = v;
        }
        __syncthreads();
        if (tid < s.parts) {
            float v = 0.0f;
            for (int w = 0; w < wpp; w++) v += part[tid * wpp + w];
            rinv[tid] = 1.0f / sqrtf(v / (float)len + k.eps);
        }
    } else {
        for (int q = warp; q < s.parts; q += 8) {
            const float v = part_sum(q, lane, 32);
            if (lane == 0) rinv[q] = 1.0f / sqrtf(v / (float)len + k.eps);
        }
    }
    __syncthreads();
    for (int i = tid; i < s.inner >> 3; i += 256) {
        float f[8];
        load8(y + 8 * i, f);
        const float4 a = load4(k.gain + 8 * i), b = load4(k.gain + 8 * i + 4);
        const float gn[8] = {a.x, a.y, a.z, a.w, b.x, b.y, b.z, b.w};
        if (vec) {
            const float r = rinv[8 * i / len];
#pragma unroll
            for (int e = 0; e < 8; e++) f[e] = (f[e] * r) * gn[e];
        } else {
            const int h = 8 * i / s.P8, q0 = 8 * i - h * s.P8;
#pragma unroll
            for (int e = 0; e < 8; e++) f[e] = q0 + e < s.P ? (f[e] * rinv[(h * s.P + q0 + e) / len]) * gn[e] : 0.0f;
        }
        store4(out + 8 * i, make_float4(f[0], f[1], f[2], f[3]));
        store4(out + 8 * i + 4, make_float4(f[4], f[5], f[6], f[7]));
    }
}

// ---------------------------------------------------------------------------------------------------------------
// Recurrence in chunks of 64 tokens, bf16 operands. With cum_t the running sum of A dt inside the chunk,
//   y_t = exp(cum_t) C_t S_in + sum_{s <= t} [exp(cum_t - cum_s) dt_s (C_t B_s) + D (s == t)] x_s
//   S_out = exp(cum_end) S_in + sum_t exp(cum_end - cum_t) dt_t B_t x_t^T
// (cum is kept in log2 units). A CTA has up to 8 PT value dimensions of one head and walks the chunks; warp w has the tokens 16 w .. 16 w + 15 of the chunk and a
// quarter of the state's rows, which stay in its registers in fp32. B, C and x are bf16 as they come; every fp32 operand of a
// product (the weights of the second term, dt-weighted B, the state) enters as the sum of two bf16 numbers, which keeps 16 bits.
__device__ __forceinline__ void ldsm4(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void ldsm4t(uint32_t addr, uint32_t (&r)[4]) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
// 16 bytes global -> shared, zeros instead where !in
__device__ __forceinline__ void cp16(uint32_t dst, const void* src, bool in) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
// (x, y) as hi + lo, two bf16 pairs
__device__ __forceinline__ void split2(float x, float y, uint32_t* hi, uint32_t* lo) {
    const uint32_t h = bf_pack(x, y);
    *hi = h;
    *lo = bf_pack(x - bf_lo(h), y - bf_hi(h));
}

struct ChunkSmem { uint32_t c, b, x, s, f, total; };        // byte offsets; NB buffers of C, B and x
__host__ __device__ constexpr ChunkSmem chunk_smem(int NK, int PT, int NB) {
    ChunkSmem o{};
    const uint32_t rn = (uint32_t)(NK * 16 + 8) * 2, rp = (uint32_t)(PT * 8 + 8) * 2;       // row pitches
    o.c = 0;
    o.b = o.c + NB * kChunk * rn;
    o.x = o.b + NB * kChunk * rn;
    o.s = o.x + NB * kChunk * rp;                            // state, hi then lo: [NK * 16][PT * 8]
    o.f = o.s + 2 * NK * 16 * rp;                            // cum [64], dt [64], weight [64]
    o.total = o.f + 3 * kChunk * 4;
    return o;
}

template <int NK, int PT, int NB, int CTAS>
__global__ void __launch_bounds__(128, CTAS) ssm_chunk_kernel(const SsmCall k) {
    constexpr int MT = NK / 4;                               // 16-row blocks of the state per warp
    constexpr ChunkSmem o = chunk_smem(NK, PT, NB);
    constexpr uint32_t RN = (NK * 16 + 8) * 2, RP = (PT * 8 + 8) * 2;
    extern __shared__ __align__(16) uint8_t sm[];
    const SsmShape& s = k.s;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, lr = lane >> 2, lc = (lane & 3) * 2;
    const int h = blockIdx.y, b = blockIdx.z, g = h / (s.H / s.G), pb = blockIdx.x * PT * 8;
    const uint32_t base = (uint32_t)__cvta_generic_to_shared(sm);
    float *cum = reinterpret_cast<float*>(sm + o.f), *dts = cum + kChunk, *wts = dts + kChunk;
    const int np = min(PT * 8, s.P8 - pb);                   // value dimensions of this CTA (multiple of 8)
    pdl_sync();
    const int p0 = first_pos(k, b);
    const float A2 = k.A[h] * kLog2e, Dh = k.D[h], dtb = k.dt_bias[h];
    const int xc = h * s.P8 + pb, bc = s.inner + g * s.N8, cc = bc + s.G * s.N8;
    const bf16* xbc = (const bf16*)k.xbc + (long)b * k.Sc * s.ch;
    const bf16* proj = (const bf16*)k.proj + (long)b * k.Sc * s.ld;

    auto fetch = [&](int t0, int buf) {
        constexpr int VN = NK * 2, VP = PT;                  // 16-byte vectors per row
        for (int i = tid; i < kChunk * VN; i += 128) {
            const int t = i / VN, v = i - t * VN;
            const bool in = t0 + t < k.Sc && v * 8 < s.N8;
            const bf16* r = xbc + (long)(in ? t0 + t : 0) * s.ch + (in ? v * 8 : 0);
            const uint32_t d = (uint32_t)(buf * kChunk + t) * RN + v * 16;
            cp16(base + o.c + d, r + cc, in);
            cp16(base + o.b + d, r + bc, in);
        }
        for (int i = tid; i < kChunk * VP; i += 128) {
            const int t = i / VP, v = i - t * VP;
            const bool in = t0 + t < k.Sc && v * 8 < np;
            cp16(base + o.x + (uint32_t)(buf * kChunk + t) * RP + v * 16, xbc + (long)(in ? t0 + t : 0) * s.ch + xc + (in ? v * 8 : 0), in);
        }
        cp_commit();
    };
    auto raw_dt = [&](int t0) { return tid < kChunk && t0 + tid < k.Sc ? to_f(proj[(long)(t0 + tid) * s.ld + s.dt_off + h]) : 0.0f; };

    // state: rows n = 16 (MT warp + m) + lr (+ 8), columns p = 8 j + lc (+ 1)
    float S[MT][PT][4];
    float* st = k.state + ((long)b * s.H + h) * s.P * s.Np;
    auto st_at = [&](int m, int j, int i) -> float* {
        const int n = 16 * (MT * warp + m) + lr + 8 * (i >> 1), p = pb + 8 * j + lc + (i & 1);
        return n < s.Np && p < s.P && 8 * j < np ? st + (long)p * s.Np + n : nullptr;
    };
    auto stage_state = [&]() {
#pragma unroll
        for (int m = 0; m < MT; m++)
#pragma unroll
            for (int j = 0; j < PT; j++)
#pragma unroll
                for (int u = 0; u < 2; u++) {
                    uint32_t hi, lo;
                    split2(S[m][j][2 * u], S[m][j][2 * u + 1], &hi, &lo);
                    const uint32_t d = o.s + (uint32_t)(16 * (MT * warp + m) + lr + 8 * u) * RP + (8 * j + lc) * 2;
                    *reinterpret_cast<uint32_t*>(sm + d) = hi;
                    *reinterpret_cast<uint32_t*>(sm + d + NK * 16 * RP) = lo;
                }
    };
    fetch(0, 0);
    float dt_next = raw_dt(0);
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int j = 0; j < PT; j++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                const float* q = p0 > 0 ? st_at(m, j, i) : nullptr;
                S[m][j][i] = q ? *q : 0.0f;
            }
    stage_state();

    const int n_chunks = (k.Sc + kChunk - 1) / kChunk;
    for (int ch = 0; ch < n_chunks; ch++) {
        const int t0 = ch * kChunk, buf = NB == 2 ? ch & 1 : 0;
        if (tid < kChunk) dts[tid] = t0 + tid < k.Sc ? softplus_f(dt_next + dtb) : 0.0f;
        cp_wait<0>();
        __syncthreads();                                     // tiles, state and dt are in place; the other buffers are free
        if (ch + 1 < n_chunks) { if (NB == 2) fetch(t0 + kChunk, buf ^ 1); dt_next = raw_dt(t0 + kChunk); }
        float end;                                           // every warp: running sums in fp32
        {
            const float d0 = A2 * dts[2 * lane], d1 = A2 * dts[2 * lane + 1];
            float v = d0 + d1;
#pragma unroll
            for (int off = 1; off < 32; off <<= 1) { const float u = __shfl_up_sync(0xffffffffu, v, off); if (lane >= off) v += u; }
            end = __shfl_sync(0xffffffffu, v, 31);
            const float c0 = v - d1;
            if (warp == 0) { cum[2 * lane] = c0; cum[2 * lane + 1] = v; }
            if (warp == 1) { wts[2 * lane] = ex2_fast(end - c0) * dts[2 * lane]; wts[2 * lane + 1] = ex2_fast(end - v) * dts[2 * lane + 1]; }
        }
        __syncthreads();
        const uint32_t cB = base + o.c + buf * kChunk * RN, bB = base + o.b + buf * kChunk * RN, xB = base + o.x + buf * kChunk * RP;
        const uint32_t sB = base + o.s;
        // ---- output of this warp's 16 tokens (their gates are asked for here and used at the end)
        uint32_t z[PT][2];
#pragma unroll
        for (int j = 0; j < PT; j++)
#pragma unroll
            for (int u = 0; u < 2; u++) {
                const int t = t0 + 16 * warp + lr + 8 * u;
                z[j][u] = t < k.Sc && j * 8 < np ? *reinterpret_cast<const uint32_t*>(proj + (long)t * s.ld + xc + 8 * j + lc) : 0u;
            }
        float y[PT][4] = {};
        uint32_t cf[NK][4];
#pragma unroll
        for (int q = 0; q < NK; q++) {
            ldsm4(cB + (uint32_t)(16 * warp + (lane & 15)) * RN + (q * 16 + (lane >> 4) * 8) * 2, cf[q]);
            // (here and below) products into one accumulator lie PT apart, and nothing depends on the true sizes: straight-line
            // code in which loads and products of independent accumulators overlap; the padding of the tiles is zero
#pragma unroll
            for (int part = 0; part < 2; part++) {
                uint32_t f[PT / 2][4];
#pragma unroll
                for (int j = 0; j < PT; j += 2)
                    ldsm4t(sB + (uint32_t)(part * NK * 16 + q * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * RP + (j * 8 + (lane >> 4) * 8) * 2, f[j / 2]);
#pragma unroll
                for (int j = 0; j < PT; j += 2) {
                    mma_bf16(y[j], cf[q][0], cf[q][1], cf[q][2], cf[q][3], f[j / 2][0], f[j / 2][1]);
                    mma_bf16(y[j + 1], cf[q][0], cf[q][1], cf[q][2], cf[q][3], f[j / 2][2], f[j / 2][3]);
                }
            }
        }
        const int tr = 16 * warp + lr;                       // rows tr and tr + 8 of the chunk
        const float ct0 = cum[tr], ct1 = cum[tr + 8];
        {
            const float e0 = ex2_fast(ct0), e1 = ex2_fast(ct1);
#pragma unroll
            for (int j = 0; j < PT; j++) { y[j][0] *= e0; y[j][1] *= e0; y[j][2] *= e1; y[j][3] *= e1; }
        }
        for (int q = 0; q <= warp; q++) {                    // 16 source tokens at a time
            float gm[2][4] = {}, g2[2][4] = {};
#pragma unroll
            for (int n = 0; n < NK; n++) {
                uint32_t f[4];
                ldsm4(bB + (uint32_t)(16 * q + (lane & 7) + (lane >> 4) * 8) * RN + (n * 16 + ((lane >> 3) & 1) * 8) * 2, f);
                mma_bf16(n & 1 ? g2[0] : gm[0], cf[n][0], cf[n][1], cf[n][2], cf[n][3], f[0], f[1]);
                mma_bf16(n & 1 ? g2[1] : gm[1], cf[n][0], cf[n][1], cf[n][2], cf[n][3], f[2], f[3]);
            }
            uint32_t xf[PT / 2][4];
#pragma unroll
            for (int j = 0; j < PT; j += 2)
                ldsm4t(xB + (uint32_t)(16 * q + (lane & 7) + ((lane >> 3) & 1) * 8) * RP + (j * 8 + (lane >> 4) * 8) * 2, xf[j / 2]);
            uint32_t wf[2][4];                               // hi, lo
#pragma unroll
            for (int u = 0; u < 2; u++) {
                float w[4];
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const int sr = 16 * q + 8 * u + lc + (i & 1), t = tr + 8 * (i >> 1);
                    float v = sr <= t ? (gm[u][i] + g2[u][i]) * (ex2_fast((i >> 1 ? ct1 : ct0) - cum[sr]) * dts[sr]) : 0.0f;
                    if (sr == t) v += Dh;
                    w[i] = v;
                }
                split2(w[0], w[1], &wf[0][2 * u], &wf[1][2 * u]);
                split2(w[2], w[3], &wf[0][2 * u + 1], &wf[1][2 * u + 1]);
            }
#pragma unroll
            for (int part = 0; part < 2; part++)
#pragma unroll
                for (int j = 0; j < PT; j += 2) {
                    mma_bf16(y[j], wf[part][0], wf[part][1], wf[part][2], wf[part][3], xf[j / 2][0], xf[j / 2][1]);
                    mma_bf16(y[j + 1], wf[part][0], wf[part][1], wf[part][2], wf[part][3], xf[j / 2][2], xf[j / 2][3]);
                }
        }
        // ---- gate and store
#pragma unroll
        for (int j = 0; j < PT; j++)
            if (j * 8 < np)
#pragma unroll
                for (int u = 0; u < 2; u++) {
                    const int t = t0 + tr + 8 * u;
                    if (t < k.Sc)
                        *reinterpret_cast<uint32_t*>((bf16*)k.y + ((long)b * k.Sc + t) * s.inner + xc + 8 * j + lc) =
                            bf_pack(y[j][2 * u] * silu_t<true>(bf_lo(z[j][u])), y[j][2 * u + 1] * silu_t<true>(bf_hi(z[j][u])));
                }
        // ---- state after the chunk
        {
            const float e = ex2_fast(end);
#pragma unroll
            for (int m = 0; m < MT; m++)
#pragma unroll
                for (int j = 0; j < PT; j++)
#pragma unroll
                    for (int i = 0; i < 4; i++) S[m][j][i] *= e;
        }
#pragma unroll
        for (int q = 0; q < kChunk / 16; q++) {
            uint32_t xf[PT / 2][4];
#pragma unroll
            for (int j = 0; j < PT; j += 2)
                ldsm4t(xB + (uint32_t)(16 * q + (lane & 7) + ((lane >> 3) & 1) * 8) * RP + (j * 8 + (lane >> 4) * 8) * 2, xf[j / 2]);
            const float2 w0 = *reinterpret_cast<const float2*>(wts + 16 * q + lc), w1 = *reinterpret_cast<const float2*>(wts + 16 * q + lc + 8);
#pragma unroll
            for (int m = 0; m < MT; m++) {
                uint32_t f[4], wb[2][4];
                ldsm4t(bB + (uint32_t)(16 * q + (lane & 7) + (lane >> 4) * 8) * RN + (16 * (MT * warp + m) + ((lane >> 3) & 1) * 8) * 2, f);
#pragma unroll
                for (int i = 0; i < 4; i++) {
                    const float2 w = i < 2 ? w0 : w1;
                    split2(bf_lo(f[i]) * w.x, bf_hi(f[i]) * w.y, &wb[0][i], &wb[1][i]);
                }
#pragma unroll
                for (int part = 0; part < 2; part++)
#pragma unroll
                    for (int j = 0; j < PT; j += 2) {
                        mma_bf16(S[m][j], wb[part][0], wb[part][1], wb[part][2], wb[part][3], xf[j / 2][0], xf[j / 2][1]);
                        mma_bf16(S[m][j + 1], wb[part][0], wb[part][1], wb[part][2], wb[part][3], xf[j / 2][2], xf[j / 2][3]);
                    }
            }
        }
        __syncthreads();                                     // everyone has read the state (and this chunk's tiles)
        if (NB == 1 && ch + 1 < n_chunks) fetch(t0 + kChunk, 0);
        stage_state();
    }
#pragma unroll
    for (int m = 0; m < MT; m++)
#pragma unroll
        for (int j = 0; j < PT; j++)
#pragma unroll
            for (int i = 0; i < 4; i++) {
                float* q = st_at(m, j, i);
                if (q) *q = S[m][j][i];
            }
    keep_history<bf16>(k, b, p0, blockIdx.x + gridDim.x * blockIdx.y, gridDim.x * gridDim.y);
}

template <class T, int NV, int TT> int launch_scan(const SsmCall& c, cudaStream_t st) {
    launch_k(ssm_scan_kernel<T, NV, TT>, dim3((c.s.P8 + 31) / 32, c.s.H, c.B), dim3(256), 0, st, c);
    return launch_status();
}
template <class T, int TT> int run_scan(const SsmCall& c, cudaStream_t st) {
    if (c.s.N8 <= 32) return launch_scan<T, 1, TT>(c, st);
    if (c.s.N8 <= 64) return launch_scan<T, 2, TT>(c, st);
    if (c.s.N8 <= 128) return launch_scan<T, 4, TT>(c, st);
    return launch_scan<T, 8, TT>(c, st);
}

template <int NK, int PT, int NB, int CTAS> int launch_chunk(const SsmCall& c, cudaStream_t st) {
    constexpr size_t smem = chunk_smem(NK, PT, NB).total;
    auto kern = ssm_chunk_kernel<NK, PT, NB, CTAS>;
    FLEXLLM_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    launch_k(kern, dim3((c.s.P8 + PT * 8 - 1) / (PT * 8), c.s.H, c.B), dim3(128), smem, st, c);
    return launch_status();
}
template <class T> int run_chunks(const SsmCall&, cudaStream_t) { return FLEXLLM_ENOTSUP; }
template <> int run_chunks<bf16>(const SsmCall& c, cudaStream_t st) {
    if (c.Sc < kScanTile) return FLEXLLM_ENOTSUP;
    // 64 value dimensions per CTA do the least work; 32 when those would not fill the SMs
    const bool many = (long)c.B * c.s.H * ((c.s.P8 + 63) / 64) > gemm_sm_count();
    if (c.s.N8 <= 64) return many ? launch_chunk<4, 8, 1, 2>(c, st) : launch_chunk<4, 4, 2, 2>(c, st);
    if (c.s.N8 <= 128) return many ? launch_chunk<8, 8, 1, 2>(c, st) : launch_chunk<8, 4, 2, 2>(c, st);
    return launch_chunk<16, 4, 1, 2>(c, st);
}

template <class T> int run_conv(const SsmCall& c, cudaStream_t st) {
    const dim3 grid((c.s.ch + 1023) / 1024, (c.Sc + kConvTokens - 1) / kConvTokens, c.B);
    switch (c.s.taps) {
        case 2: launch_k(ssm_conv_kernel<T, 2>, grid, dim3(128), 0, st, c); break;
        case 3: launch_k(ssm_conv_kernel<T, 3>, grid, dim3(128), 0, st, c); break;
        case 4: launch_k(ssm_conv_kernel<T, 4>, grid, dim3(128), 0, st, c); break;
        default: launch_k(ssm_conv_kernel<T, 0>, grid, dim3(128), 0, st, c);
    }
    return launch_status();
}

}  // namespace

void ssm_layout(SsmShape* s) {
    s->P8 = (int)up_to(s->P, 8); s->N8 = (int)up_to(s->N, 8); s->Np = (int)up_to(s->N, 4);
    s->inner = s->H * s->P8;
    s->ch = s->inner + 2 * s->G * s->N8;
    s->x_off = s->inner;
    s->dt_off = s->inner + s->ch;
    s->ld = s->dt_off + up_to(s->H, 8);
}
bool ssm_supported(const SsmShape& s) { return s.N8 <= 256 && s.H <= 65535 && s.parts <= 4096; }

template <class T> int ssm_mixer(const SsmCall& c, cudaStream_t st) {
    const SsmShape& s = c.s;
    FLEXLLM_REQUIRE(s.H > 0 && s.P > 0 && s.N > 0 && s.G > 0 && s.H % s.G == 0 && s.taps > 0 && s.parts > 0 && (s.H * s.P) % s.parts == 0);
    FLEXLLM_REQUIRE(c.proj && c.conv_w && c.conv_b && c.dt_bias && c.A && c.D && c.gain && c.state && c.conv_state && c.ctx && c.y && c.out);
    FLEXLLM_REQUIRE(c.B > 0 && c.Sc > 0 && c.xbc);
    if (!ssm_supported(s) || c.B > 65535 || c.Sc > 65535 * kConvTokens) return FLEXLLM_ENOTSUP;
    TRY_RC(run_conv<T>(c, st));
    int rc = c.Sc == 1 ? run_scan<T, 1>(c, st) : run_chunks<T>(c, st);
    if (rc == FLEXLLM_ENOTSUP) rc = run_scan<T, kScanTile>(c, st);
    TRY_RC(rc);
    launch_k(ssm_norm_kernel<T>, dim3(c.B * c.Sc), dim3(256), (size_t)(s.parts + 8) * 4, st, c);
    return launch_status();
}
template int ssm_mixer<float>(const SsmCall&, cudaStream_t);
template int ssm_mixer<bf16>(const SsmCall&, cudaStream_t);

}  // namespace flexllm

using namespace flexllm;

// ---- C ABI, see include/flexllm_b200.h
namespace {
bool make_shape(const flexllm_ssm_shape* a, SsmShape* s) {
    if (!a || a->heads <= 0 || a->vdim <= 0 || a->state <= 0 || a->groups <= 0 || a->heads % a->groups || a->conv <= 0 || a->norm_groups <= 0 ||
        ((long)a->heads * a->vdim) % a->norm_groups) return false;
    *s = SsmShape();
    s->H = a->heads; s->P = a->vdim; s->N = a->state; s->G = a->groups; s->taps = a->conv; s->parts = a->norm_groups;
    ssm_layout(s);
    return true;
}
}  // namespace

extern "C" long flexllm_ssm_row(const flexllm_ssm_shape* a) { SsmShape s; return make_shape(a, &s) ? s.ld : 0; }
extern "C" long flexllm_ssm_channels(const flexllm_ssm_shape* a) { SsmShape s; return make_shape(a, &s) ? s.ch : 0; }
extern "C" size_t flexllm_ssm_state_floats(const flexllm_ssm_shape* a) { SsmShape s; return make_shape(a, &s) ? ssm_state_floats(s) : 0; }
extern "C" size_t flexllm_ssm_workspace(const flexllm_ssm_shape* a, int B, int n) {
    SsmShape s;
    return make_shape(a, &s) && B > 0 && n > 0 ? (size_t)B * n * (s.ch + s.inner) * 4 + 512 : 0;
}
extern "C" int flexllm_ssm(int dtype, const flexllm_ssm_shape* a, const void* proj, const float* conv_w, const float* conv_b, const float* dt_bias,
                           const float* A, const float* D, const float* gain, float* state, void* conv_state, const int32_t* ctx, int B, int n,
                           void* out, void* workspace, size_t workspace_bytes, void* stream) {
    SsmCall c = {};
    FLEXLLM_REQUIRE(make_shape(a, &c.s) && B > 0 && n > 0 && (dtype == FLEXLLM_F32 || dtype == FLEXLLM_BF16));
    FLEXLLM_REQUIRE(workspace && workspace_bytes >= flexllm_ssm_workspace(a, B, n) && aligned(workspace, 256) && aligned(proj, 16) && aligned(out, 16));
    c.proj = proj; c.conv_w = conv_w; c.conv_b = conv_b; c.dt_bias = dt_bias; c.A = A; c.D = D; c.gain = gain; c.eps = a->eps;
    c.state = state; c.conv_state = conv_state; c.ctx = ctx; c.B = B; c.Sc = n;
    c.xbc = workspace;
    c.y = (char*)workspace + up_to((long)B * n * c.s.ch * 4, 256);
    c.out = out;
    return dtype == FLEXLLM_BF16 ? ssm_mixer<bf16>(c, (cudaStream_t)stream) : ssm_mixer<float>(c, (cudaStream_t)stream);
}
