// bf16 linear layers on the 5th-generation tensor cores (tcgen05, kind::f16, fp32 accumulation).
//
// The pipeline of the int8 GEMM (gemm_tcgen05.cu) for 16-bit operands: one persistent CTA per SM, a TMA
// producer warp (128-byte-swizzled K-major tiles), one MMA-issuing thread, four epilogue warps on a
// double-buffered TMEM accumulator.
//   prompts: A = activations (128-row side), B = weights (BN rows)
//   decode : A = weights, B = activations (M <= 64), split over K within a thread-block cluster: each CTA leaves its
//            fp32 partial tile in shared memory and the cluster's CTAs add them, a share of the tokens each, over
//            distributed shared memory and in rank order, so the result does not depend on timing
// Epilogue: optional bias, optional gated GELU (weight rows alternating in blocks of 16 gate / 16 up rows) or squared ReLU,
// fp32 or bf16 output.
#include <atomic>

#include "float_common.cuh"
#include "tc_common.cuh"

namespace flexllm {

using namespace tc;

namespace {

struct GemmBfArgs {
    int rowsA, rowsB, num_kb;          // rows of the two sides, K in 128-byte blocks
    int tilesA, tilesB, ksplit;
    long ldo;
    float* y32; bf16* y16;
    const float* bias;                 // per output channel (row of the weights)
    int glu, relu2, vec;               // vec: rows of the output are 16-byte aligned
    int* error_flag;
};

template <int BN, int KCH> struct GemmBfCfg {
    static constexpr int A_TILE = 128 * 128;
    static constexpr int B_TILE = BN * 128;
    static constexpr int A_BYTES = KCH * A_TILE;
    static constexpr int B_BYTES = KCH * B_TILE;
    static constexpr int STAGE_BYTES = A_BYTES + B_BYTES;
    static constexpr int STAGES_MAX = (196 * 1024) / STAGE_BYTES;
    static constexpr int STAGES = STAGES_MAX > 8 ? 8 : STAGES_MAX;
    static constexpr int TMEM_COLS = 2 * BN < 32 ? 32 : 2 * BN;
    static constexpr int STG_WARP_FLOATS = 32 * 32 + 256;      // one 32 x 32 chunk + the tile's biases
    static constexpr int STG_BYTES = 4 * STG_WARP_FLOATS * 4;
    static constexpr int SMEM_BYTES = STAGES * STAGE_BYTES + 1024 + 256 + STG_BYTES;
};

template <int BN, bool SWAP, int KCH>
__global__ void __launch_bounds__(192, 1) gemm_bf16_tcgen05_kernel(const __grid_constant__ CUtensorMap tmapA,
                                                                   const __grid_constant__ CUtensorMap tmapB, const GemmBfArgs args) {
    using Cfg = GemmBfCfg<BN, KCH>;
    constexpr int STAGES = Cfg::STAGES;
    extern __shared__ uint8_t smem_raw[];
    const uint32_t raw = smem_u32(smem_raw);
    const uint32_t ring = (raw + 1023u) & ~1023u;
    uint8_t* ring_ptr = smem_raw + (ring - raw);
    uint64_t* bars = reinterpret_cast<uint64_t*>(ring_ptr + STAGES * Cfg::STAGE_BYTES);
    const uint32_t bar_full = smem_u32(bars);
    const uint32_t bar_empty = bar_full + 8 * STAGES;
    const uint32_t bar_tfull = bar_empty + 8 * STAGES;
    const uint32_t bar_tempty = bar_tfull + 16;
    uint32_t* tmem_base_slot = reinterpret_cast<uint32_t*>(bars + 2 * STAGES + 4);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_base_slot + 1);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int num_kb = args.num_kb / KCH;
    const int total_tiles = args.tilesA * args.tilesB * args.ksplit;

    if (threadIdx.x == 0) {
        for (int s = 0; s < STAGES; s++) { mbar_init(bar_full + 8 * s, 1); mbar_init(bar_empty + 8 * s, 1); }
        for (int s = 0; s < 2; s++) { mbar_init(bar_tfull + 8 * s, 1); mbar_init(bar_tempty + 8 * s, 4); }
        *abort_flag = 0;
        fence_barrier_init();
    }
    if (warp == 1) { tmem_alloc(smem_u32(tmem_base_slot), Cfg::TMEM_COLS); tmem_relinquish(); }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_base_slot;
    pdl_sync();

    // decode form: one value of token `tok`, weight row rowA (this lane's; row0: the warp's first); a warp store covers 32 channels
    auto emit = [&](float v, int tok, int rowA, int row0, float bA) {
        v += bA;
        if (args.glu) {
            const float up = __shfl_xor_sync(0xffffffffu, v, 16);
            if (lane < 16 && rowA < args.rowsA) {
                const float r = gelu_tanh_f<true>(v) * up;
                const long o = (long)tok * args.ldo + (row0 >> 1) + lane;
                if (args.y16) args.y16[o] = __float2bfloat16_rn(r); else args.y32[o] = r;
            }
        } else if (rowA < args.rowsA) {
            if (args.relu2) v = relu2_f(v);
            const long o = (long)tok * args.ldo + rowA;
            if (args.y16) args.y16[o] = __float2bfloat16_rn(v); else args.y32[o] = v;
        }
    };

    if (warp == 0) {
        if (lane == 0) {
            tma_prefetch_desc(&tmapA);
            tma_prefetch_desc(&tmapB);
            int stage = 0; uint32_t phase = 0;
            bool ok = true;
            for (int t = blockIdx.x; ok && t < total_tiles; t += gridDim.x) {
                const int split = t % args.ksplit;
                const int tb = (t / args.ksplit) % args.tilesB;
                const int ta = t / (args.ksplit * args.tilesB);
                const int kb0 = (int)((long)split * num_kb / args.ksplit), kb1 = (int)((long)(split + 1) * num_kb / args.ksplit);
                for (int kb = kb0; kb < kb1; kb++) {
                    if (!mbar_wait(bar_empty + 8 * stage, phase ^ 1u, abort_flag)) { ok = false; break; }
                    const uint32_t full = bar_full + 8 * stage;
                    mbar_expect_tx(full, Cfg::STAGE_BYTES);
                    const uint32_t dstA = ring + stage * Cfg::STAGE_BYTES;
                    if (KCH == 1) {
                        tma_load_2d(dstA, &tmapA, full, kb * 128, ta * 128);
                        tma_load_2d(dstA + Cfg::A_BYTES, &tmapB, full, kb * 128, tb * BN);
                    } else {
                        tma_load_3d(dstA, &tmapA, full, 0, ta * 128, kb * KCH);
                        tma_load_3d(dstA + Cfg::A_BYTES, &tmapB, full, 0, tb * BN, kb * KCH);
                    }
                    if (++stage == STAGES) { stage = 0; phase ^= 1u; }
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = umma_idesc_bf16(128, BN);
            int stage = 0; uint32_t phase = 0;
            int it = 0;
            bool ok = true;
            for (int t = blockIdx.x; ok && t < total_tiles; t += gridDim.x, it++) {
                const int split = t % args.ksplit;
                const int kb0 = (int)((long)split * num_kb / args.ksplit), kb1 = (int)((long)(split + 1) * num_kb / args.ksplit);
                const int as = it & 1;
                const uint32_t aphase = (it >> 1) & 1;
                if (!mbar_wait(bar_tempty + 8 * as, aphase ^ 1u, abort_flag)) { ok = false; break; }
                tc_fence_after();
                const uint32_t tmem_d = tmem_base + as * BN;
                for (int kb = kb0; kb < kb1; kb++) {
                    if (!mbar_wait(bar_full + 8 * stage, phase, abort_flag)) { ok = false; break; }
                    tc_fence_after();
                    const uint32_t sa = ring + stage * Cfg::STAGE_BYTES;
#pragma unroll
                    for (int c = 0; c < KCH; c++) {
                        const uint64_t adesc = umma_desc_k_sw128(sa + c * Cfg::A_TILE);
                        const uint64_t bdesc = umma_desc_k_sw128(sa + Cfg::A_BYTES + c * Cfg::B_TILE);
#pragma unroll
                        for (int k = 0; k < 4; k++)   // 16 bf16 = 32 bytes = 2 descriptor address units per step
                            umma_bf16(tmem_d, adesc + 2 * k, bdesc + 2 * k, idesc, (kb > kb0 || c > 0 || k > 0) ? 1u : 0u);
                    }
                    umma_commit(bar_empty + 8 * stage);
                    if (++stage == STAGES) { stage = 0; phase ^= 1u; }
                }
                if (ok) umma_commit(bar_tfull + 8 * as);
            }
        }
    } else {
        const int q = warp & 3;
        int it = 0;
        bool ok = true;
        float* stg = reinterpret_cast<float*>(ring_ptr + STAGES * Cfg::STAGE_BYTES + 256) + q * Cfg::STG_WARP_FLOATS;
        for (int t = blockIdx.x; ok && t < total_tiles; t += gridDim.x, it++) {
            const int split = t % args.ksplit;
            const int tb = (t / args.ksplit) % args.tilesB;
            const int ta = t / (args.ksplit * args.tilesB);
            const int as = it & 1;
            const uint32_t aphase = (it >> 1) & 1;
            const int row0 = ta * 128 + q * 32;           // this warp's rows of the A side
            const int rowA = row0 + lane;
            const bool rowA_ok = rowA < args.rowsA;
            float* bw = stg + 1024;
            if (!SWAP)
                for (int i = lane; i < BN; i += 32) bw[i] = (args.bias && tb * BN + i < args.rowsB) ? args.bias[tb * BN + i] : 0.0f;
            const float bA = (SWAP && args.bias && rowA_ok) ? args.bias[rowA] : 0.0f;
            int got = (lane == 0) ? (mbar_wait(bar_tfull + 8 * as, aphase, abort_flag) ? 1 : 0) : 1;
            got = __shfl_sync(0xffffffffu, got, 0);
            if (!got) { ok = false; break; }
            tc_fence_after();
            const uint32_t tsrc = tmem_base + ((uint32_t)(q * 32) << 16) + as * BN;
            if constexpr (!SWAP) {
                __syncwarp();
                // 32 columns at a time go through this warp's staging buffer (16-byte granules XOR-swizzled by the
                // row), so that the global stores of a warp cover whole sectors of few rows
                auto process = [&](const uint32_t (&v)[32], const int c) {
                    const int col0 = tb * BN + c * 32;
                    if (col0 >= args.rowsB) return;
                    const int s7 = lane & 7;
                    if (args.glu) {
#pragma unroll
                        for (int g = 0; g < 4; g++) {
                            float r[4];
#pragma unroll
                            for (int i = 0; i < 4; i++) {
                                const float gt = __uint_as_float(v[4 * g + i]) + bw[c * 32 + 4 * g + i];
                                const float up = __uint_as_float(v[16 + 4 * g + i]) + bw[c * 32 + 16 + 4 * g + i];
                                r[i] = gelu_tanh_f<true>(gt) * up;
                            }
                            *reinterpret_cast<float4*>(stg + lane * 32 + ((g ^ s7) << 2)) = make_float4(r[0], r[1], r[2], r[3]);
                        }
                    } else {
#pragma unroll
                        for (int g = 0; g < 8; g++) {
                            const float4 b4 = *reinterpret_cast<const float4*>(bw + c * 32 + 4 * g);
                            float4 o4 = make_float4(__uint_as_float(v[4 * g]) + b4.x, __uint_as_float(v[4 * g + 1]) + b4.y,
                                                    __uint_as_float(v[4 * g + 2]) + b4.z, __uint_as_float(v[4 * g + 3]) + b4.w);
                            if (args.relu2) o4 = make_float4(relu2_f(o4.x), relu2_f(o4.y), relu2_f(o4.z), relu2_f(o4.w));
                            *reinterpret_cast<float4*>(stg + lane * 32 + ((g ^ s7) << 2)) = o4;
                        }
                    }
                    __syncwarp();
                    const int ocol0 = args.glu ? col0 >> 1 : col0;            // first output column of the chunk
                    const int n_out = args.glu ? args.rowsB >> 1 : args.rowsB;
                    const int width = args.glu ? 16 : 32;
                    if (args.vec && args.y16) {
                        const int lpr = width >> 3;                            // lanes per row, 8 columns each
                        const int rstep = 32 / lpr, g2 = (lane % lpr) * 2, r0 = lane / lpr;
                        for (int rr = r0; rr < 32; rr += rstep) {
                            const int row = row0 + rr, col = ocol0 + g2 * 4;
                            if (row < args.rowsA && col < n_out) {
                                const float4 x = *reinterpret_cast<const float4*>(stg + rr * 32 + ((g2 ^ (rr & 7)) << 2));
                                const float4 z = *reinterpret_cast<const float4*>(stg + rr * 32 + (((g2 + 1) ^ (rr & 7)) << 2));
                                *reinterpret_cast<uint4*>(args.y16 + (long)row * args.ldo + col) =
                                    make_uint4(bf_pack(x.x, x.y), bf_pack(x.z, x.w), bf_pack(z.x, z.y), bf_pack(z.z, z.w));
                            }
                        }
                    } else if (args.vec) {
                        const int lpr = width >> 2, rstep = 32 / lpr, g1 = lane % lpr, r0 = lane / lpr;
                        for (int rr = r0; rr < 32; rr += rstep) {
                            const int row = row0 + rr, col = ocol0 + g1 * 4;
                            if (row < args.rowsA && col < n_out)
                                *reinterpret_cast<float4*>(args.y32 + (long)row * args.ldo + col) =
                                    *reinterpret_cast<const float4*>(stg + rr * 32 + ((g1 ^ (rr & 7)) << 2));
                        }
                    } else {
                        for (int i = lane; i < 32 * width; i += 32) {
                            const int rr = i / width, cc = i - rr * width;
                            const int row = row0 + rr, col = ocol0 + cc;
                            if (row < args.rowsA && col < n_out) {
                                const float x = stg[rr * 32 + (((cc >> 2) ^ (rr & 7)) << 2) + (cc & 3)];
                                if (args.y16) args.y16[(long)row * args.ldo + col] = __float2bfloat16_rn(x);
                                else args.y32[(long)row * args.ldo + col] = x;
                            }
                        }
                    }
                    __syncwarp();
                };
                constexpr int NCH = BN / 32;
                uint32_t va[32], vb[32];
                tmem_ld_32x32(tsrc, va);
#pragma unroll 1
                for (int c = 0; c < NCH; c += 2) {
                    tmem_ld_wait();
                    if (c + 1 < NCH) tmem_ld_32x32(tsrc + (c + 1) * 32, vb);
                    process(va, c);
                    if (c + 1 < NCH) {
                        tmem_ld_wait();
                        if (c + 2 < NCH) tmem_ld_32x32(tsrc + (c + 2) * 32, va);
                        process(vb, c + 1);
                    }
                }
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(bar_tempty + 8 * as);
            } else {
                // lane = weight row, columns = tokens
                float* part = reinterpret_cast<float*>(ring_ptr);
#pragma unroll
                for (int c = 0; c < BN / 16; c++) {
                    uint32_t v[16];
                    tmem_ld_32x16(tsrc + c * 16, v);
                    tmem_ld_wait();
#pragma unroll
                    for (int j = 0; j < 16; j++) {
                        const int tok = tb * BN + c * 16 + j;
                        if (args.ksplit > 1) part[(c * 16 + j) * 128 + q * 32 + lane] = __uint_as_float(v[j]);
                        else if (tok < args.rowsB) emit(__uint_as_float(v[j]), tok, rowA, row0, bA);
                    }
                }
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(bar_tempty + 8 * as);
            }
        }
    }

    if (SWAP && args.ksplit > 1) {
        // every CTA of the cluster has one tile, the same for all of them: the partial tiles are in the rings (their MMAs
        // have finished reading), and CTA r adds up tokens r, r + ksplit, ...
        tc_fence_before();
        cluster_sync();
        if (warp >= 2 && !*abort_flag) {
            const int q = warp & 3, ta = blockIdx.x / args.ksplit, r = blockIdx.x % args.ksplit;
            const int row0 = ta * 128 + q * 32, rowA = row0 + lane;
            const float bA = (args.bias && rowA < args.rowsA) ? args.bias[rowA] : 0.0f;
            for (int tok = r; tok < args.rowsB; tok += args.ksplit) {
                float p[8];
#pragma unroll
                for (int k = 0; k < 8; k++)
                    p[k] = k < args.ksplit ? ld_cluster_f32(cluster_addr(ring + (uint32_t)(tok * 128 + q * 32 + lane) * 4u, k)) : 0.0f;
                float s = p[0];
#pragma unroll
                for (int k = 1; k < 8; k++) s += p[k];
                emit(s, tok, rowA, row0, bA);
            }
        }
        cluster_sync();                      // nobody leaves while its partial tile may still be read
    }
    tc_fence_before();
    __syncthreads();
    if (*abort_flag) {
        // a wait ran out: give copies still in flight time to land before shared memory is released
        const unsigned long long t0 = globaltimer_ns();
        while (globaltimer_ns() - t0 < 200000ull) { __nanosleep(1000); }
        if (threadIdx.x == 0 && args.error_flag) atomicOr(args.error_flag, 1);
        __syncthreads();
    }
    if (warp == 1) { tc_fence_after(); tmem_dealloc(tmem_base, Cfg::TMEM_COLS); }
}

template <int BN, bool SWAP, int KCH>
int launch(const bf16* A, int rowsA, long ldA, const bf16* B, int rowsB, long ldB, int K, GemmBfArgs g, cudaStream_t st) {
    using Cfg = GemmBfCfg<BN, KCH>;
    CUtensorMap ta, tb;
    TRY_RC(cached_tmap_u8(&ta, A, (uint64_t)rowsA, (uint64_t)ldA * 2, 128, KCH > 1 ? KCH : 0));
    TRY_RC(cached_tmap_u8(&tb, B, (uint64_t)rowsB, (uint64_t)ldB * 2, BN, KCH > 1 ? KCH : 0));
    g.rowsA = rowsA; g.rowsB = rowsB; g.num_kb = (K + 63) / 64;
    g.tilesA = (rowsA + 127) / 128; g.tilesB = (rowsB + BN - 1) / BN;
    g.error_flag = device_error_flag();
    auto kern = gemm_bf16_tcgen05_kernel<BN, SWAP, KCH>;
    static std::atomic<bool> attr_set[kMaxDevices];
    const int dev = current_device();
    if (dev < 0) return FLEXLLM_ECUDA;
    if (!attr_set[dev].load(std::memory_order_acquire)) {
        FLEXLLM_CHECK_CUDA(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, Cfg::SMEM_BYTES));
        attr_set[dev].store(true, std::memory_order_release);
    }
    const int total = g.tilesA * g.tilesB * g.ksplit;
    if (SWAP && g.ksplit > 1) {
        // one tile per CTA, the splits of a tile form a cluster
        launch_cluster(kern, dim3(total), dim3(192), g.ksplit, (size_t)Cfg::SMEM_BYTES, st, ta, tb, g);
        return launch_status();
    }
    const int grid = total < gemm_sm_count() ? total : gemm_sm_count();
    launch_k(kern, dim3(grid), dim3(192), (size_t)Cfg::SMEM_BYTES, st, ta, tb, g);
    return launch_status();
}

GemmBfArgs base_args(const float* bias, int act, const LinearOut& y) {
    GemmBfArgs g = {};
    g.ksplit = 1; g.ldo = y.ld; g.y32 = y.f32; g.y16 = (bf16*)y.t; g.bias = bias;
    g.glu = act == kActGeluGate; g.relu2 = act == kActRelu2;
    return g;
}

}  // namespace

int gemm_bf16_prefill(const bf16* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y,
                      cudaStream_t st) {
    GemmBfArgs g = base_args(bias, act, y);
    const int n_out = g.glu ? N / 2 : N;
    g.vec = y.t ? (y.ld % 8 == 0 && n_out % 8 == 0 && aligned(y.t, 16)) : (y.ld % 4 == 0 && n_out % 4 == 0 && aligned(y.f32, 16));
    // the widest tile that still gives every SM work
    const long tiles256 = (long)((M + 127) / 128) * ((N + 255) / 256);
    if (N > 128 && tiles256 >= gemm_sm_count()) return launch<256, false, 1>(a, M, lda, w, N, ldw, K, g, st);
    if (N > 64 && tiles256 * 2 >= gemm_sm_count()) return launch<128, false, 1>(a, M, lda, w, N, ldw, K, g, st);
    return launch<64, false, 1>(a, M, lda, w, N, ldw, K, g, st);
}

int gemm_bf16_decode(const bf16* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut y,
                     cudaStream_t st) {
    if (M > 64) return FLEXLLM_ENOTSUP;
    GemmBfArgs g = base_args(bias, act, y);
    // K blocks per pipeline stage: longer contiguous runs per weight row and TMA request
    // ... as long as the splits that give every SM work keep two steps each
    const int kb = (K + 63) / 64, tiles = (N + 127) / 128;
    int ks = 1;
    while (ks < 8 && tiles * ks * 2 <= gemm_sm_count() && kb >= 4 * ks) ks *= 2;
    int kch = 1;
    if (lda % 64 == 0 && ldw % 64 == 0) {
        if (kb % 4 == 0 && kb / 4 >= 2 * ks) kch = 4;
        else if (kb % 2 == 0 && kb / 2 >= 2 * ks) kch = 2;
    }
    g.ksplit = ks;
#define FLEXLLM_DEC(BN_, KCH_) return launch<BN_, true, KCH_>(w, N, ldw, a, M, lda, K, g, st)
    if (M > 32) { if (kch == 4) FLEXLLM_DEC(64, 4); if (kch == 2) FLEXLLM_DEC(64, 2); FLEXLLM_DEC(64, 1); }
    if (M > 16) { if (kch == 4) FLEXLLM_DEC(32, 4); if (kch == 2) FLEXLLM_DEC(32, 2); FLEXLLM_DEC(32, 1); }
    if (kch == 4) FLEXLLM_DEC(16, 4);
    if (kch == 2) FLEXLLM_DEC(16, 2);
    FLEXLLM_DEC(16, 1);
#undef FLEXLLM_DEC
}

}  // namespace flexllm
