// The model runner's state, and what a model family plugs into it. The runner (model.cu) owns the page table, context
// lengths, token table, CUDA graph, sampling and the generation loop of every family; the W8A8 Llama's operator graph is
// built in, other families supply their weights and one step of the network (model_decoder.cu).
#pragma once
#include <vector>

#include "common.cuh"
#include "decode_mega.h"
#include "kv_cache.h"

struct flexllm_tp;
struct flexllm_model;

namespace flexllm {
struct ModelFamily {
    virtual ~ModelFamily() {}
    // One weight tensor by its name in the checkpoint (host or device memory). Unknown names: FLEXLLM_EINVAL.
    virtual int load_tensor(flexllm_model* m, const char* name, int dtype, int ndim, const int64_t* shape, const void* data, cudaStream_t st) = 0;
    virtual bool knows(const char* name) = 0;
    virtual int check_loaded() = 0;                            // FLEXLLM_EINVAL while a tensor is missing
    // Tokens (b, t), t < Sc, = tok[b * S + c0 + t] at positions ctx[b] + t through all layers: keys and values go to the
    // cache, the rows b * Sc + t of the residual stream stay in the runner's x. Does not advance ctx.
    virtual int forward(flexllm_model* m, const int32_t* tok, int B, int S, int c0, int Sc, cudaStream_t st) = 0;
    // Logits [n][vocab] of rows rows[0 .. n) of the last forward (device indices; nullptr: rows 0 .. n-1).
    virtual int logits(flexllm_model* m, const int32_t* rows, int n, float* out, cudaStream_t st) = 0;
    virtual int set_trace(float*, size_t) { return FLEXLLM_ENOTSUP; }
};
// Takes over fam and cache (also on failure). seq_pages: pages per sequence, of which the first keep_pages stay outside the ring;
// x_floats: residual stream of the largest chunk.
int runner_create(flexllm_model** out, const flexllm_model_config& cfg, ModelFamily* fam, flexllm_kv_cache* cache, int seq_pages, int keep_pages,
                  size_t x_floats);
}  // namespace flexllm

struct LayerW {
    int8_t *wqkv, *wo, *wgu, *wd;
    float *sqkv, *so, *sgu, *sd, *g0, *g1, *a_s;
};

struct flexllm_model {
    flexllm_model_config cfg;
    std::vector<LayerW> L;
    int8_t* lm_w = nullptr; float* lm_s = nullptr; float* g_final = nullptr;
    float *cos_t = nullptr, *sin_t = nullptr; int table_len = 0;
    flexllm_kv_cache* cache = nullptr;
    int max_pages = 0;
    int32_t *page_table = nullptr, *ctx = nullptr, *next = nullptr, *state = nullptr, *tokens = nullptr, *out_tokens = nullptr;
    size_t out_capacity = 0;
    // activations (sized for max_batch * max_prefill rows)
    float *x = nullptr, *qkv = nullptr, *att = nullptr, *tmp = nullptr, *gu = nullptr, *xs = nullptr, *logits = nullptr, *xlast = nullptr;
    int8_t *xq = nullptr, *hq = nullptr;
    void *attn_ws = nullptr, *dec_ws = nullptr;
    size_t attn_ws_bytes = 0, dec_ws_bytes = 0;
    // decode state
    int B = 0, S = 0;
    int last_chunk = 0;                         // rows per sequence the residual stream x holds after the last prefill
    int n_new = 0;                              // columns of the token table of the running generation
    int pos = 0;                                // context length of the batch = position the next decode step writes
    cudaGraphExec_t graph = nullptr; int graph_B = 0; int graph_kernels = 0;
    int mega_variant = 0, graph_variant = 0;   // attention variant of the persistent kernel for the current decode call / in the captured step
    std::vector<void*> owned;
    // tensor parallelism: g ranks, this one is r; *l = local (per-rank) sizes
    flexllm_tp* tp = nullptr;
    int g = 1, r = 0, HQl = 0, HKVl = 0, Fl = 0, Dl = 0, Vl = 0;
    float *gath = nullptr, *hloc = nullptr;     // all-gather target / local silu(gate)*up slice
    // token-row partition of the prefill + batch-parallel decode (see flexllm_model_prefill)
    flexllm_model* dm = nullptr;                // single-GPU model of this rank's sequences: full weights, all KV heads
    float *amax = nullptr, *xs2 = nullptr;      // per-token largest magnitudes / scales of the row-parallel inputs
    int8_t* aq = nullptr;                       // quantised attention output, this rank's columns
    uint8_t *kv_stage = nullptr, *kvs_stage = nullptr;   // KV hand-over: pages / scale rows as received
    bool rows_mode = false;                     // the last prefill used the token-row partition
    int32_t* acc32 = nullptr;                   // row-parallel partial sums
    void *pairs_l = nullptr, *pairs_g = nullptr;
    // persistent decode-step kernel: -1 not tried yet, 0 not usable for this model, 1 ready
    flexllm::MegaPlan* mega = nullptr; int mega_state = -1;
    // token choice: greedy (sample_k == 0) or the reference's top-k sampling with uniform numbers rnd [n_new][B]
    int sample_lanes = 0, sample_k = 0; const float* sample_rnd = nullptr;
    float* own_rnd = nullptr; size_t own_rnd_floats = 0;      // numbers copied in by flexllm_model_set_sampling_host
    // a family other than the W8A8 Llama (nullptr: that one), and what its steps need
    flexllm::ModelFamily* fam = nullptr;
    int32_t* rows = nullptr; int logits_rows = 0;              // rows whose logits are asked for; rows the logits buffer holds
};

template <class T> inline int dmalloc(flexllm_model* m, T** p, size_t n) {
    void* q = nullptr;
    cudaError_t e = cudaMalloc(&q, n * sizeof(T) + 256);
    if (e != cudaSuccess) { flexllm::g_last_cuda_error = (int)e; return e == cudaErrorMemoryAllocation ? FLEXLLM_ENOMEM : FLEXLLM_ECUDA; }
    m->owned.push_back(q);
    *p = (T*)q;
    return FLEXLLM_OK;
}
#define TRY(expr) do { int _rc = (expr); if (_rc != FLEXLLM_OK) return _rc; } while (0)
