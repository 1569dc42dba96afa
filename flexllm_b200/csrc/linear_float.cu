// Linear layers of the floating-point model path apart from the tcgen05 GEMMs (gemm_bf16.cu), and the choice between the
// forms: a weight-streaming GEMV for one or two tokens (T = bf16 or float activations, bf16 weights), its warp-MMA form for
// more, and a tiled fp32 GEMM for the 32-bit mode.
#include "float_common.cuh"

namespace flexllm {

namespace {

__device__ __forceinline__ uint4 ldg_stream16(const bf16* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0,%1,%2,%3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// Weight row of slot r of the warp whose first output is n0 (GLU: slots 2 i and 2 i + 1 are gate and up row of output n0 + i).
// Slots past the last output repeat it: no row past the matrix is read.
template <bool GLU> __device__ __forceinline__ long weight_row(int n0, int r, int n_out) {
    const int n = min(n0 + (GLU ? r >> 1 : r), n_out - 1);
    return GLU ? (long)(n >> 4) * 32 + (n & 15) + (r & 1) * 16 : (long)n;
}

// The structure of the int8 GEMV (gemv.cu). KS = 1: each of the CTA's four warps owns R weight rows over the whole K;
// KS = 4: the four warps share R rows, a quarter of K each.
template <class T, int BT, int R, int KS, bool GLU>
__global__ void __launch_bounds__(128) gemv_float_kernel(const T* __restrict__ a, long lda, const bf16* __restrict__ w, long ldw,
                                                         const float* __restrict__ bias, int M, int n_out, int kv, int relu2, float* y32, T* yt,
                                                         long ldy) {
    extern __shared__ __align__(16) uint8_t a_raw[];
    T* a_sm = reinterpret_cast<T*>(a_raw);               // [BT][kv * 8]
    constexpr int OUT = GLU ? R / 2 : R;                 // outputs per warp (KS = 1) or CTA (KS = 4)
    constexpr bool FAST = sizeof(T) == 2;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int n0 = KS == 1 ? (blockIdx.x * 4 + warp) * OUT : blockIdx.x * OUT;
    const int kbeg = KS == 1 ? 0 : (int)((long)warp * kv / KS), kend = KS == 1 ? kv : (int)((long)(warp + 1) * kv / KS);
    const bool active = n0 < n_out;
    const bf16* wr[R];
#pragma unroll
    for (int r = 0; r < R; r++) wr[r] = w + weight_row<GLU>(n0, r, n_out) * ldw;
    uint4 nx[R][2];
    const uint4 zero = make_uint4(0, 0, 0, 0);
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
        for (int u = 0; u < 2; u++) { const int c = kbeg + lane + 32 * u; nx[r][u] = (active && c < kend) ? ldg_stream16(wr[r] + (long)c * 8) : zero; }
    pdl_sync();
    for (int i = threadIdx.x; i < BT * kv; i += 128) {
        const int b = i / kv, c = i - b * kv;
        float f[8] = {0, 0, 0, 0, 0, 0, 0, 0};
        if (b < M) load8(a + (long)b * lda + (long)c * 8, f);
        store4(a_sm + (long)i * 8, make_float4(f[0], f[1], f[2], f[3]));
        store4(a_sm + (long)i * 8 + 4, make_float4(f[4], f[5], f[6], f[7]));
    }
    __syncthreads();
    float acc[R][BT];
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
        for (int b = 0; b < BT; b++) acc[r][b] = 0.0f;
    if (active) {
        for (int c0 = kbeg + lane; c0 < kend; c0 += 64) {
            uint4 wv[R][2];
#pragma unroll
            for (int r = 0; r < R; r++)
#pragma unroll
                for (int u = 0; u < 2; u++) {
                    wv[r][u] = nx[r][u];
                    const int d = c0 + 64 + 32 * u;
                    nx[r][u] = d < kend ? ldg_stream16(wr[r] + (long)d * 8) : zero;
                }
#pragma unroll
            for (int u = 0; u < 2; u++) {
                const int c = c0 + 32 * u;
                if (c < kend) {
                    float wf[R][8];
#pragma unroll
                    for (int r = 0; r < R; r++) unpack8(wv[r][u], wf[r]);
#pragma unroll
                    for (int b = 0; b < BT; b++) {
                        float f[8];
                        load8(a_sm + ((long)b * kv + c) * 8, f);
#pragma unroll
                        for (int r = 0; r < R; r++)
#pragma unroll
                            for (int e = 0; e < 8; e++) acc[r][b] = __fmaf_rn(wf[r][e], f[e], acc[r][b]);
                    }
                }
            }
        }
    }
#pragma unroll
    for (int r = 0; r < R; r++)
#pragma unroll
        for (int b = 0; b < BT; b++) acc[r][b] = warp_sum(acc[r][b]);
    if (KS > 1) {
        __shared__ float part[KS > 1 ? KS : 1][R][BT];
        if (lane == 0)
#pragma unroll
            for (int r = 0; r < R; r++)
#pragma unroll
                for (int b = 0; b < BT; b++) part[warp][r][b] = acc[r][b];
        __syncthreads();
        if (warp != 0) return;
#pragma unroll
        for (int r = 0; r < R; r++)
#pragma unroll
            for (int b = 0; b < BT; b++) {
                float s = 0.0f;
#pragma unroll
                for (int k = 0; k < KS; k++) s += part[k][r][b];
                acc[r][b] = s;
            }
    }
    if (!active || lane != 0) return;
#pragma unroll
    for (int o = 0; o < OUT; o++) {
        const int n = n0 + o;
        if (n >= n_out) continue;
#pragma unroll
        for (int b = 0; b < BT; b++) {
            if (b >= M) continue;
            float v;
            if (GLU) {
                const long rg = weight_row<true>(n, 0, n_out), ru = weight_row<true>(n, 1, n_out);
                const float gt = acc[2 * o < R ? 2 * o : 0][b] + (bias ? bias[rg] : 0.0f), up = acc[2 * o + 1 < R ? 2 * o + 1 : 0][b] + (bias ? bias[ru] : 0.0f);
                v = gelu_tanh_f<FAST>(gt) * up;
            } else {
                v = acc[o][b] + (bias ? bias[n] : 0.0f);
                if (relu2) v = relu2_f(v);
            }
            if (y32) y32[(long)b * ldy + n] = v;
            else yt[(long)b * ldy + n] = from_f<T>(v);
        }
    }
}

// A few tokens, bf16: weight streaming with warp-level bf16 MMAs. A CTA takes RT blocks of 16 weight rows (the MMA's row side;
// GLU: one gate and one up block), its eight warps share K; the tokens are the column side, NT blocks of 8. Rows of both
// operands are read straight from memory with 16-byte loads: lane % 4 holds elements 8 c .. 8 c + 7 of every 32, i.e. the inner
// index is permuted, the same way on both sides. The warps' partial sums are added in warp order.
template <int NT, int RT, bool GLU>
__global__ void __launch_bounds__(256) skinny_mma_kernel(const bf16* __restrict__ a, long lda, const bf16* __restrict__ w, long ldw,
                                                         const float* __restrict__ bias, int M, int N, int kv, int relu2, float* y32, bf16* y16, long ldy) {
    constexpr int G = NT * RT >= 4 ? 2 : 4;                 // 32-element chunks per step
    __shared__ float part[8][RT * 16][NT * 8 + 1];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, lr = lane >> 2, lc = lane & 3;
    const int row0 = blockIdx.x * RT * 16;
    const int n_ch = (kv + 3) >> 2;                         // kv: 8-element vectors per row
    const int c_beg = (int)((long)warp * n_ch / 8), c_end = (int)((long)(warp + 1) * n_ch / 8);
    const uint4 zero = make_uint4(0, 0, 0, 0);
    const bf16* wr[RT][2];
#pragma unroll
    for (int r = 0; r < RT; r++)
#pragma unroll
        for (int h = 0; h < 2; h++) wr[r][h] = w + (long)min(row0 + r * 16 + h * 8 + lr, N - 1) * ldw + lc * 8;
    uint4 wv[G][RT][2], nx[G][RT][2];
    auto load_w = [&](uint4 (&v)[G][RT][2], int c) {
#pragma unroll
        for (int g = 0; g < G; g++)
#pragma unroll
            for (int r = 0; r < RT; r++)
#pragma unroll
                for (int h = 0; h < 2; h++)
                    v[g][r][h] = (c + g < c_end && (c + g) * 4 + lc < kv) ? ldg_stream16(wr[r][h] + (long)(c + g) * 32) : zero;
    };
    load_w(nx, c_beg);
    pdl_sync();
    float acc[RT][NT][4] = {};
    for (int c = c_beg; c < c_end; c += G) {
#pragma unroll
        for (int g = 0; g < G; g++)
#pragma unroll
            for (int r = 0; r < RT; r++)
#pragma unroll
                for (int h = 0; h < 2; h++) wv[g][r][h] = nx[g][r][h];
        uint4 av[G][NT];
#pragma unroll
        for (int g = 0; g < G; g++)
#pragma unroll
            for (int t = 0; t < NT; t++)
                av[g][t] = (t * 8 + lr < M && c + g < c_end && (c + g) * 4 + lc < kv)
                               ? *reinterpret_cast<const uint4*>(a + (long)(t * 8 + lr) * lda + (long)(c + g) * 32 + lc * 8) : zero;
        load_w(nx, c + G);
#pragma unroll
        for (int g = 0; g < G; g++)
#pragma unroll
            for (int r = 0; r < RT; r++)
#pragma unroll
                for (int t = 0; t < NT; t++) {
                    mma_bf16(acc[r][t], wv[g][r][0].x, wv[g][r][1].x, wv[g][r][0].y, wv[g][r][1].y, av[g][t].x, av[g][t].y);
                    mma_bf16(acc[r][t], wv[g][r][0].z, wv[g][r][1].z, wv[g][r][0].w, wv[g][r][1].w, av[g][t].z, av[g][t].w);
                }
    }
#pragma unroll
    for (int r = 0; r < RT; r++)
#pragma unroll
        for (int t = 0; t < NT; t++)
#pragma unroll
            for (int i = 0; i < 4; i++) part[warp][r * 16 + lr + 8 * (i >> 1)][t * 8 + lc * 2 + (i & 1)] = acc[r][t][i];
    __syncthreads();
    auto total = [&](int row, int tok) {
        float v = part[0][row][tok];
#pragma unroll
        for (int k = 1; k < 8; k++) v += part[k][row][tok];
        const int n = row0 + row;
        return v + (bias && n < N ? bias[n] : 0.0f);
    };
    constexpr int OUT = GLU ? 16 : RT * 16;                 // output columns of the CTA
    const int n0 = GLU ? row0 >> 1 : row0, n_out = GLU ? N >> 1 : N;
    for (int i = threadIdx.x; i < OUT * M; i += 256) {
        const int tok = i / OUT, o = i - tok * OUT;
        if (n0 + o >= n_out) continue;
        float v = GLU ? gelu_tanh_f<true>(total(o, tok)) * total(RT * 16 - 16 + o, tok) : total(o, tok);
        if (!GLU && relu2) v = relu2_f(v);
        if (y32) y32[(long)tok * ldy + n0 + o] = v;
        else y16[(long)tok * ldy + n0 + o] = __float2bfloat16_rn(v);
    }
}

template <int NT>
int skinny_nt(const bf16* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y, cudaStream_t st) {
    const int kv = (K + 7) / 8, r2 = act == kActRelu2;
    if (act == kActGeluGate) launch_k(skinny_mma_kernel<NT, 2, true>, dim3((N + 31) / 32), dim3(256), 0, st, a, lda, w, ldw, bias, M, N, kv, r2, y.f32, (bf16*)y.t, y.ld);
    else if (N >= 148 * 4 * 16) launch_k(skinny_mma_kernel<NT, 2, false>, dim3((N + 31) / 32), dim3(256), 0, st, a, lda, w, ldw, bias, M, N, kv, r2, y.f32, (bf16*)y.t, y.ld);
    else launch_k(skinny_mma_kernel<NT, 1, false>, dim3((N + 15) / 16), dim3(256), 0, st, a, lda, w, ldw, bias, M, N, kv, r2, y.f32, (bf16*)y.t, y.ld);
    return launch_status();
}
int skinny_mma(const bf16* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y, cudaStream_t st) {
    if (M <= 8) return skinny_nt<1>(a, lda, w, ldw, bias, M, N, K, act, y, st);
    if (M <= 16) return skinny_nt<2>(a, lda, w, ldw, bias, M, N, K, act, y, st);
    return skinny_nt<4>(a, lda, w, ldw, bias, M, N, K, act, y, st);
}

template <class T, int BT, int R, int KS, bool GLU>
int launch_gemv(const T* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int relu2, LinearOut y, cudaStream_t st) {
    const int kv = (K + 7) / 8;
    const size_t smem = (size_t)BT * kv * 8 * sizeof(T);
    auto kern = gemv_float_kernel<T, BT, R, KS, GLU>;
    if (smem > 220 * 1024) return FLEXLLM_ENOTSUP;
    if (smem > 48 * 1024) FLEXLLM_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    const int n_out = GLU ? N / 2 : N, out = GLU ? R / 2 : R;
    const int per_cta = KS == 1 ? 4 * out : out;
    launch_k(kern, dim3((n_out + per_cta - 1) / per_cta), dim3(128), smem, st, a, lda, w, ldw, bias, M, n_out, kv, relu2, y.f32, (T*)y.t, y.ld);
    return launch_status();
}

template <class T, int BT, bool GLU>
int gemv_bt(const T* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int relu2, LinearOut y, cudaStream_t st) {
    if (N >= 148 * 4 * 4 * 4) return launch_gemv<T, BT, 4, 1, GLU>(a, lda, w, ldw, bias, M, N, K, relu2, y, st);
    if (N / 2 < 148 * 16 && K >= 1024) return launch_gemv<T, BT, 2, 4, GLU>(a, lda, w, ldw, bias, M, N, K, relu2, y, st);
    return launch_gemv<T, BT, 2, 1, GLU>(a, lda, w, ldw, bias, M, N, K, relu2, y, st);
}

template <class T>               // M <= 4 (bf16: M <= 2, more goes to the MMA forms)
int gemv_any(const T* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y, cudaStream_t st) {
#define FLEXLLM_GEMV(BT_) return act == kActGeluGate ? gemv_bt<T, BT_, true>(a, lda, w, ldw, bias, M, N, K, 0, y, st) \
                                                     : gemv_bt<T, BT_, false>(a, lda, w, ldw, bias, M, N, K, act == kActRelu2, y, st)
    if (M <= 1) FLEXLLM_GEMV(1);
    if (sizeof(T) == 2 || M <= 2) FLEXLLM_GEMV(2);
    FLEXLLM_GEMV(sizeof(T) == 2 ? 2 : 4);
#undef FLEXLLM_GEMV
}

// 32-bit mode, any M: 64 x 64 tile, 4 x 4 values per thread (columns 16 apart, so a thread of a gated layer holds the gate and
// up values of its outputs), fp32 fused multiply-adds in increasing k.
__global__ void __launch_bounds__(256) gemm_f32_kernel(const float* __restrict__ a, long lda, const bf16* __restrict__ w, long ldw,
                                                       const float* __restrict__ bias, int M, int N, int K, int act, float* __restrict__ y,
                                                       long ldy) {
    __shared__ float as[16][65], ws[16][65];
    pdl_sync();
    const int m0 = blockIdx.y * 64, n0 = blockIdx.x * 64;
    const int tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += 16) {
        for (int i = threadIdx.x; i < 64 * 16; i += 256) {
            const int r = i >> 4, k = i & 15;
            as[k][r] = (m0 + r < M && k0 + k < K) ? a[(long)(m0 + r) * lda + k0 + k] : 0.0f;
            ws[k][r] = (n0 + r < N && k0 + k < K) ? to_f(w[(long)(n0 + r) * ldw + k0 + k]) : 0.0f;
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; k++) {
            float av[4], wv[4];
#pragma unroll
            for (int i = 0; i < 4; i++) { av[i] = as[k][ty + 16 * i]; wv[i] = ws[k][tx + 16 * i]; }
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = __fmaf_rn(av[i], wv[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; i++) {
        const int m = m0 + ty + 16 * i;
        if (m >= M) continue;
        if (act == kActGeluGate) {
#pragma unroll
            for (int j = 0; j < 4; j += 2) {
                const int rg = n0 + tx + 16 * j, ru = rg + 16;
                if (ru < N) {
                    const float gt = acc[i][j] + (bias ? bias[rg] : 0.0f), up = acc[i][j + 1] + (bias ? bias[ru] : 0.0f);
                    y[(long)m * ldy + (n0 >> 1) + tx + 8 * j] = gelu_tanh_f<false>(gt) * up;
                }
            }
        } else {
#pragma unroll
            for (int j = 0; j < 4; j++) {
                const int n = n0 + tx + 16 * j;
                if (n < N) {
                    const float v = acc[i][j] + (bias ? bias[n] : 0.0f);
                    y[(long)m * ldy + n] = act == kActRelu2 ? relu2_f(v) : v;
                }
            }
        }
    }
}

int check(const void* a, long lda, const void* w, long ldw, int M, int N, int K, int act, const LinearOut& y) {
    const bool glu = act == kActGeluGate;
    FLEXLLM_REQUIRE(act >= kActNone && act <= kActRelu2);
    FLEXLLM_REQUIRE(a && w && (y.f32 || y.t) && M >= 0 && N > 0 && K > 0);
    FLEXLLM_REQUIRE(lda % 8 == 0 && ldw % 8 == 0 && lda >= up_to(K, 8) && ldw >= up_to(K, 8) && aligned(a, 16) && aligned(w, 16));
    FLEXLLM_REQUIRE(!glu || N % 32 == 0);
    FLEXLLM_REQUIRE(y.ld >= (glu ? N / 2 : N));
    return FLEXLLM_OK;
}

}  // namespace

int linear_bf16(const bf16* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y, cudaStream_t st) {
    TRY_RC(check(a, lda, w, ldw, M, N, K, act, y));
    if (M == 0) return FLEXLLM_OK;
    // Measured on the layer shapes of 1B to 8B models: the scalar GEMV wins for one token (two for wide matrices), the
    // tensor-core form where its 128-row tiles alone fill most SMs, the warp-MMA form for the narrow rest.
    const bool wide = (N + 127) / 128 >= 100;
    if ((M == 1 && K <= 12288) || (M == 2 && wide)) {
        const int rc = gemv_any<bf16>(a, lda, w, ldw, bias, M, N, K, act, y, st);
        if (rc != FLEXLLM_ENOTSUP) return rc;
    }
    if (M <= 16 ? !wide : M <= 32 && !wide && (long)N * K <= (17L << 20)) return skinny_mma(a, lda, w, ldw, bias, M, N, K, act, y, st);
    if (M <= 64) return gemm_bf16_decode(a, lda, w, ldw, bias, M, N, K, act, y, st);
    return gemm_bf16_prefill(a, lda, w, ldw, bias, M, N, K, act, y, st);
}

int linear_f32(const float* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y, cudaStream_t st) {
    TRY_RC(check(a, lda, w, ldw, M, N, K, act, y));
    if (M == 0) return FLEXLLM_OK;
    if (M <= 4) {
        const int rc = gemv_any<float>(a, lda, w, ldw, bias, M, N, K, act, y, st);
        if (rc != FLEXLLM_ENOTSUP) return rc;
    }
    float* out = y.f32 ? y.f32 : (float*)y.t;
    launch_k(gemm_f32_kernel, dim3((N + 63) / 64, (M + 63) / 64), dim3(256), 0, st, a, lda, w, ldw, bias, M, N, K, act, out, y.ld);
    return launch_status();
}

}  // namespace flexllm

using namespace flexllm;

// See include/flexllm_b200.h.
extern "C" int flexllm_linear_float(int dtype, const void* a, long lda, const void* w, long ldw, const float* bias, int M, int N, int K,
                                    int act, void* y, long ldy, int y_f32, void* stream) {
    FLEXLLM_REQUIRE(dtype == FLEXLLM_F32 || dtype == FLEXLLM_BF16);
    LinearOut o = {y_f32 || dtype == FLEXLLM_F32 ? (float*)y : nullptr, y_f32 || dtype == FLEXLLM_F32 ? nullptr : y, ldy};
    if (dtype == FLEXLLM_BF16)
        return linear_bf16((const bf16*)a, lda, (const bf16*)w, ldw, bias, M, N, K, act, o, (cudaStream_t)stream);
    return linear_f32((const float*)a, lda, (const bf16*)w, ldw, bias, M, N, K, act, o, (cudaStream_t)stream);
}
