// Helpers of the floating-point model path (bf16 weights; activations T = bf16, or float when everything
// runs in 32 bits): conversions, the activation functions, block reductions, and the declarations shared by
// its translation units. The library is compiled with -fmad=false, so fused multiply-adds are spelled out.
#pragma once
#include <cuda_bf16.h>

#include "common.cuh"

namespace flexllm {

typedef __nv_bfloat16 bf16;

inline long up_to(long n, long a) { return (n + a - 1) / a * a; }

__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
template <class T> __device__ __forceinline__ T from_f(float v);
template <> __device__ __forceinline__ float from_f<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 from_f<bf16>(float v) { return __float2bfloat16_rn(v); }

// the two bf16 halves of a 32-bit word
__device__ __forceinline__ float bf_lo(uint32_t w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float bf_hi(uint32_t w) { return __uint_as_float(w & 0xffff0000u); }
__device__ __forceinline__ uint32_t bf_pack(float lo, float hi) {
    uint32_t r;
    asm("cvt.rn.bf16x2.f32 %0, %1, %2;" : "=r"(r) : "f"(hi), "f"(lo));
    return r;
}
__device__ __forceinline__ void unpack8(const uint4& v, float (&f)[8]) {
    f[0] = bf_lo(v.x); f[1] = bf_hi(v.x); f[2] = bf_lo(v.y); f[3] = bf_hi(v.y);
    f[4] = bf_lo(v.z); f[5] = bf_hi(v.z); f[6] = bf_lo(v.w); f[7] = bf_hi(v.w);
}
// 8 consecutive elements from 16-byte aligned memory
__device__ __forceinline__ void load8(const bf16* p, float (&f)[8]) { unpack8(*reinterpret_cast<const uint4*>(p), f); }
__device__ __forceinline__ void load8(const float* p, float (&f)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ float4 load4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 load4(const bf16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(bf_lo(v.x), bf_hi(v.x), bf_lo(v.y), bf_hi(v.y));
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(bf16* p, float4 v) { *reinterpret_cast<uint2*>(p) = make_uint2(bf_pack(v.x, v.y), bf_pack(v.z, v.w)); }

// warp-level product for the weight- and cache-streaming kernels: d [16 x 8] += a [16 x 16] b [16 x 8]
__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}

__device__ __forceinline__ float ex2_fast(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ float rcp_fast(float x) { float y; asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }

constexpr float kLog2e = 1.4426950408889634f;

// logistic function; FAST: hardware exponential and reciprocal (a few ulp), else the accurate library ones
template <bool FAST> __device__ __forceinline__ float sigmoid_f(float z) {
    if (FAST) return rcp_fast(1.0f + ex2_fast(-z * kLog2e));
    return 1.0f / (1.0f + expf(-z));
}
// tanh form of GELU: 0.5 z (1 + tanh u) = z * logistic(2 u), u = sqrt(2/pi) (z + 0.044715 z^3)
template <bool FAST> __device__ __forceinline__ float gelu_tanh_f(float z) {
    const float u = 0.7978845608028654f * __fmaf_rn(0.044715f * z, z * z, z);
    return z * sigmoid_f<FAST>(2.0f * u);
}

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Sums of two values over a block of NT threads; every thread gets both. red: 2 * NT / 32 floats.
template <int NT> __device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
    a = warp_sum(a); b = warp_sum(b);
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
    constexpr int NW = NT / 32;
    __syncthreads();
    if (l == 0) { red[w] = a; red[NW + w] = b; }
    __syncthreads();
    a = l < NW ? red[l] : 0.0f;
    b = l < NW ? red[NW + l] : 0.0f;
    return make_float2(warp_sum(a), warp_sum(b));
}

int* device_error_flag();
int gemm_sm_count();

// ---------------------------------------------------------------------------- linear layers
// y[m][n] = sum_k a[m][k] w[n][k] (+ bias[n]); a T [M][lda], w bf16 [N][ldw]. ldw and lda are multiples of 8 and at least
// K rounded up to 8; the columns from K on are zero in w and finite in a.
// act, applied to the sums: kActGeluGate: rows of w alternate in blocks of 16 (gate 0..15, up 0..15, gate 16..31, ...),
// y[m][f] = gelu_tanh(gate_f) * up_f, N = 2 F; kActRelu2: max(y, 0)^2.
enum { kActNone = 0, kActGeluGate = 1, kActRelu2 = 2 };
__device__ __forceinline__ float relu2_f(float v) { v = fmaxf(v, 0.0f); return v * v; }
struct LinearOut { float* f32; void* t; long ld; };      // exactly one of f32 / t (type T) is set
int linear_bf16(const bf16* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y, cudaStream_t st);
int linear_f32(const float* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y, cudaStream_t st);
// tensor-core kernels behind linear_bf16
int gemm_bf16_prefill(const bf16* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y, cudaStream_t st);
int gemm_bf16_decode(const bf16* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y, cudaStream_t st);

// ---------------------------------------------------------------------------- norms around a sublayer
// One pass over the rows of the residual stream, every step optional:
//   x (or the embedding of the row's token) -> x += rms(y) * gain_post -> [trace] -> x += embedding -> x += add_vec -> x stored
//   -> h = rms(x) * gain_pre
struct ResNormArgs {
    float* x; long ldx; int D; float eps;
    const int32_t* rows;                    // row r of the launch is row rows[r] of x (nullptr: r)
    int keep_x;                             // do not store x
    const int32_t* tok; int S, c0, Sc;      // token of row r: tok[(r / Sc) * S + c0 + r % Sc]
    const bf16* emb; long lde; float emb_scale; int V; int* error_flag;
    int emb_mode;                           // 0 none, 1 x starts as the embedding, 2 the embedding is added after the sublayer
    const float* y; long ldy; const float* gain_post;
    const float* add_vec;
    float* trace;                           // dense [rows][D]
    const float* gain_pre; void* h; long ldh;
};
template <class T> int res_norm(const ResNormArgs& a, int rows, cudaStream_t st);

// The same place in a model whose residual is a set of n streams mixed around every sublayer (hyper-connections), every step
// optional:
//   x_s (or the embedding of the row's token, in every stream) -> x_t <- sum_s mix[s][t] x_s + out[t] y -> [trace: sum of the streams]
//   -> x stored -> h = rms(u) * gain, u = sum_s in[s] x_s
constexpr int kMaxStreams = 8;
struct HyperNormArgs {
    float* x; long lds; int n, D; float eps;   // x [row][n][lds]
    const int32_t* rows;                    // row r of the launch is row rows[r] of x (nullptr: r)
    const int32_t* tok; int S, c0, Sc;      // token of row r: tok[(r / Sc) * S + c0 + r % Sc] ...
    const bf16* emb; long lde; float emb_scale; int V; int* error_flag;      // ... when emb is given
    const float* y; long ldy;               // sublayer output, nullptr: none
    const float *mix, *out;                 // [n][n] (from, to), [n]
    float* trace;                           // dense [rows][D]
    const float* in;                        // [n]
    const float* gain; void* h; long ldh;
};
template <class T> int hyper_norm(const HyperNormArgs& a, int rows, cudaStream_t st);

// ---------------------------------------------------------------------------- state-space mixer (Mamba-2 form)
// Between the projections: causal convolution and silu on x | B | C, recurrence per head, gate, grouped norm.
struct SsmShape {
    int H, P, N, G, taps, parts;            // heads, value size, state size, groups of B and C, convolution taps, parts of the norm
    int P8, N8, Np;                         // sizes padded to 8 (per head / group: columns of the projection) and to 4 (state rows)
    int inner, ch;                          // H * P8; channels of the convolution: inner + 2 G N8, in the order x | B | C
    int x_off, dt_off;                      // columns of the fused projection: z 0.., x | B | C x_off.., dt dt_off..
    long ld;                                // its row length
};
struct SsmCall {
    SsmShape s;
    const void* proj;                       // T [rows][s.ld]
    const float *conv_w, *conv_b;           // [taps][ch] (last row: the current token), [ch]; 0 in the padding
    const float *dt_bias, *A, *D;           // [H]; A = -exp(A_log)
    const float* gain; float eps;           // [inner], 0 in the padding
    float* state;                           // [slot][H][P][Np], zero in the padding
    void* conv_state;                       // T [slot][taps][ch]: inputs of the convolution, position p in row p % taps
    const int32_t* ctx;                     // position of the first of the call's Sc tokens per sequence (0: the state starts at zero)
    int B, Sc;
    void* xbc;                              // scratch T [rows][ch]
    void* y;                                // scratch T [rows][inner]: gated outputs before the norm
    void* out;                              // T [rows][inner]
};
// Convolution, then the recurrence and the gate (bf16 prompts: in chunks on the tensor cores; otherwise token by token), then the
// norm. States and histories of the call's sequences are advanced.
template <class T> int ssm_mixer(const SsmCall& c, cudaStream_t st);
void ssm_layout(SsmShape* s);               // fills in the derived members
bool ssm_supported(const SsmShape& s);
inline size_t ssm_state_floats(const SsmShape& s) { return (size_t)s.H * s.P * s.Np; }

// ---------------------------------------------------------------------------- windowed attention
constexpr int kBiasPad = 192;               // masked (-inf) distances on either side of the window in the bias tables
struct AttnShape {
    int H, G, dk, dv, dkp;                  // heads, key/value heads, sizes; dkp = dk rounded up to 8 (rows of Q and of the K pages)
    int window;                             // i sees j with 0 <= i - j < window ...
    int keep;                               // ... and every j < keep (0 <= j <= i)
    float scale, softcap;                   // softcap 0: none
    int sink;                               // an extra score without a value in the denominator: 0 none, 1 a score of 0, 2 one per head
    int q_off, k_off, v_off, g_off;         // columns of the fused projection; g_off < 0: no output gate; k_off < 0: no keys and
                                            // values of its own (the pools are another layer's, nothing is appended)
    long ld;                                // its row length
};
struct AttnCall {
    AttnShape s;
    const void* proj;                       // fused projection, T [rows][s.ld]
    const float *q_gain, *k_gain; float eps;   // norm over the whole q (k) projection before the split into heads; nullptr: none
    const float* bias;                      // [G][kBiasPad + window + kBiasPad][H / G]: bias by distance, -inf outside the window;
    float bias_max_abs;                     // nullptr: none
    const float* sinks;                     // [H], sink == 2
    void *k_pool, *v_pool;                  // T pages of this layer: K [page][G][64][dkp], V^T [page][G][dv][64]
    long n_pages;
    const int32_t* page_table; int max_pages;
    const int32_t* ctx; int max_pos;        // position of the first of the call's Sc tokens per sequence (device)
    int B, Sc;
    void* q;                                // scratch T [rows][H][dkp] (unused by the decode form)
    void* out; long ldo;                    // T [rows][ldo]: gated head outputs
    float* ws; int* counters;               // split-key partial results (decode form)
    size_t ws_floats; int n_counters;
};
// Norms, appends to the cache and attends. Sc == 1: one fused kernel; else preparation, then the prompt kernel (tcgen05 for
// bf16 shapes it covers, row by row otherwise).
template <class T> int attn_window(const AttnCall& c, cudaStream_t st);
size_t attn_window_ws_floats(int max_batch, int G, int R, int dv);
// Pages of a sequence that the first `keep` positions occupy (they stay where they are when the other pages form a ring).
inline int attn_keep_pages(int keep) { return (keep + 63) / 64; }
// Fills in the derived members: dkp, the columns of the fused projection (parts padded to multiples of 8) and its row length.
void attn_layout(AttnShape* s, bool gate, bool own_kv = true);
// The bias table of AttnCall::bias on the host, from a table [rows][H] of learned biases by bucketed distance.
void attn_bias_table(const AttnShape& s, const float* table, int rows, int bias_max, float* out);
inline size_t attn_bias_floats(const AttnShape& s) { return (size_t)s.H * (2 * kBiasPad + s.window); }

}  // namespace flexllm
