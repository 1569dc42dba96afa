// Decoder family with floating-point weights. bf16 weights; activations bf16 (residual stream, norms, scores, recurrent states
// fp32), or everything fp32. Two designs are composed from the same parts:
//   Pibidra  sandwich norms around every sublayer, windowed grouped-query attention with query/key norms over the whole projection,
//            softcapped scores, a learned distance bias, a softmax sink and an output gate (attention_window.cu), a gated-GELU
//            feed-forward, and an optional block of layers that runs several times with the same weights
//   Sabisun  several residual streams mixed around every sublayer (norm_float.cu), state-space mixers (ssm.cu) and windowed
//            attention with kept first tokens, per-head sinks and keys and values shared between layers, a squared-ReLU
//            feed-forward, tied embeddings
//
// A step is, per layer run: fused input projection (q|k|v|gate, or z|x|B|C|dt) -> mixer -> output projection -> [residual, norm]
// -> fused gate|up (or up) projection with the activation in its epilogue -> down projection -> [residual, norm]. The same step
// serves prompts, portions of prompts and decoding; row counts choose the kernels.
#include <cmath>
#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <new>
#include <string>

#include "float_common.cuh"
#include "model.h"

namespace flexllm {

namespace {

struct DecLayer {
    flexllm_decoder_layer c;
    AttnShape s;                                // attention
    SsmShape m;                                 // state-space mixer
    bool ssm;
    long ld_mix;                                // row length of the mixer's outputs
    int n_mix;                                  // ... of which the output projection reads this many
    int proj_n, ffp;                            // rows of the fused projection; ff rounded up to 16
    bf16 *w_proj, *w_o, *w_gu, *w_down;
    float *b_proj;                              // biases of the fused projection (zero where it has none)
    float *n1, *n1b, *n2, *n2b;                 // norm gains (1 + stored weight)
    float *q_gain, *k_gain, *bias;
    float bias_max = 0.0f;
    float *sinks;
    float *conv_w, *conv_b, *dt_bias, *A, *D, *m_gain;
    float *hc1, *hc2;                           // stream coefficients of a sublayer: mix [n][n], out [n] (times residual_mult), in [n]
};

float bf16_to_float(uint16_t v) { uint32_t u = (uint32_t)v << 16; float f; memcpy(&f, &u, 4); return f; }

struct Want { std::string name; std::vector<int64_t> shape; bool loaded; };

class DecoderFamily : public ModelFamily {
  public:
    flexllm_decoder_config cfg;
    std::vector<flexllm_decoder_layer> specs;
    std::vector<DecLayer> L;
    struct Run { int layer; int pass; int cache; };   // pass >= 0 on the first layer of a pass of the loop; cache: its pools or states
    std::vector<Run> runs;
    std::vector<Want> wants;
    std::vector<void*> owned;
    int D = 0, ldD = 0;
    bf16 *embed = nullptr, *head = nullptr;
    float *final_gain = nullptr, *loop_step = nullptr, *ones = nullptr;
    // activations (T = bf16 or float by cfg.dtype)
    void *h = nullptr, *proj = nullptr, *q = nullptr, *att = nullptr, *act = nullptr, *xbc = nullptr, *gated = nullptr;
    float* y = nullptr;
    float* attn_ws = nullptr; size_t attn_ws_floats = 0;
    int* attn_counters = nullptr; int n_counters = 0;
    float* trace = nullptr; size_t trace_floats = 0;

    ~DecoderFamily() override { for (void* p : owned) cudaFree(p); }

    template <class P> int alloc(P** p, size_t bytes) {            // zeroed
        void* v = nullptr;
        cudaError_t e = cudaMalloc(&v, bytes + 256);
        if (e != cudaSuccess) { g_last_cuda_error = (int)e; return e == cudaErrorMemoryAllocation ? FLEXLLM_ENOMEM : FLEXLLM_ECUDA; }
        owned.push_back(v);
        *p = (P*)v;
        return cuda_status(cudaMemset(v, 0, bytes + 256));
    }

    void want(const std::string& name, std::vector<int64_t> shape) { wants.push_back({name, std::move(shape), false}); }

    int create(flexllm_model** out, const flexllm_decoder_config* c) {
        cfg = *c;
        specs.assign(c->layer, c->layer + c->layers);
        cfg.layer = specs.data();
        D = cfg.width; ldD = (int)up_to(D, 8);
        const int NL = cfg.layers;
        const size_t es = cfg.dtype == FLEXLLM_BF16 ? 2 : 4;
        const long Mmax = (long)cfg.max_batch * (cfg.max_prefill > 1 ? cfg.max_prefill : 1);
        for (int i = 0; i < NL; i++) {
            if (i == cfg.loop_start && cfg.loop_times > 0) {
                for (int t = 0; t < cfg.loop_times; t++)
                    for (int k = cfg.loop_start; k < cfg.loop_stop; k++) runs.push_back({k, k == cfg.loop_start ? t : -1, 0});
                i = cfg.loop_stop - 1;
            } else {
                runs.push_back({i, -1, 0});
            }
        }
        want("embed", {cfg.vocab, D});
        want("final.norm", {D});
        TRY(alloc(&embed, (size_t)cfg.vocab * ldD * 2));
        if (cfg.streams > 0) {
            head = embed;
            TRY(alloc(&ones, (size_t)cfg.streams * 4));
            const std::vector<float> one((size_t)cfg.streams, 1.0f);
            FLEXLLM_CHECK_CUDA(cudaMemcpy(ones, one.data(), one.size() * 4, cudaMemcpyHostToDevice));
        } else {
            want("head", {cfg.vocab, D});
            TRY(alloc(&head, (size_t)cfg.vocab * ldD * 2));
        }
        TRY(alloc(&final_gain, (size_t)ldD * 4));
        if (cfg.loop_times > 0) {
            want("loop.step", {cfg.loop_times, D});
            TRY(alloc(&loop_step, (size_t)cfg.loop_times * ldD * 4));
        }
        L.resize(NL);
        long max_proj = 8, max_q = 8, max_att = 8, max_act = 8, max_xbc = 8, max_inner = 8;
        int max_window = 1, max_keep = 0;
        for (int i = 0; i < NL; i++) {
            DecLayer& l = L[i];
            l = DecLayer();
            l.c = specs[i];
            const flexllm_decoder_layer& a = l.c;
            l.ssm = a.mixer == FLEXLLM_MIXER_SSM;
            l.ffp = (int)up_to(a.ff, 16);
            max_act = l.ffp > max_act ? l.ffp : max_act;
            const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.";
            if (l.ssm) {
                SsmShape& s = l.m;
                s.H = a.heads; s.P = a.vdim; s.N = a.state; s.G = a.groups; s.taps = a.conv; s.parts = a.norm_groups;
                ssm_layout(&s);
                if (!ssm_supported(s)) return FLEXLLM_ENOTSUP;
                l.proj_n = (int)s.ld; l.ld_mix = l.n_mix = s.inner;
                max_xbc = s.ch > max_xbc ? s.ch : max_xbc;
                max_inner = s.inner > max_inner ? s.inner : max_inner;
                const int64_t inner = (int64_t)s.H * s.P, gn = (int64_t)s.G * s.N;
                TRY(alloc(&l.conv_w, (size_t)s.taps * s.ch * 4));
                TRY(alloc(&l.conv_b, (size_t)s.ch * 4));
                TRY(alloc(&l.dt_bias, (size_t)s.H * 4));
                TRY(alloc(&l.A, (size_t)s.H * 4));
                TRY(alloc(&l.D, (size_t)s.H * 4));
                TRY(alloc(&l.m_gain, (size_t)s.inner * 4));
                want(m + "in", {2 * inner + 2 * gn + s.H, D});
                want(m + "conv", {inner + 2 * gn, s.taps});
                want(m + "conv.b", {inner + 2 * gn});
                want(m + "dt_bias", {s.H}); want(m + "A_log", {s.H}); want(m + "D", {s.H});
                want(m + "norm", {inner});
                want(m + "o", {D, inner});
            } else {
                AttnShape& s = l.s;
                s.H = a.heads; s.G = a.kv_heads; s.dk = a.dim; s.dv = a.vdim;
                s.window = a.window < cfg.max_ctx + 1 ? a.window : cfg.max_ctx + 1;      // nothing is further away than that
                s.keep = a.keep_first < cfg.max_ctx + 1 ? a.keep_first : cfg.max_ctx + 1;
                s.scale = a.scale; s.softcap = a.softcap;
                s.sink = has(a, FLEXLLM_ATTN_HEAD_SINKS) ? 2 : has(a, FLEXLLM_ATTN_UNIT_SINK) ? 1 : 0;
                attn_layout(&s, has(a, FLEXLLM_ATTN_GATE), a.kv_from < 0);
                l.proj_n = (int)s.ld;
                l.n_mix = s.H * s.dv;
                l.ld_mix = up_to(l.n_mix, 8);
                max_window = s.window > max_window ? s.window : max_window;
                max_keep = s.keep > max_keep ? s.keep : max_keep;
                const long nq = (long)s.H * s.dkp;
                max_q = nq > max_q ? nq : max_q;
                want(m + "q", {(int64_t)s.H * s.dk, D});
                if (a.kv_from < 0) { want(m + "k", {(int64_t)s.G * s.dk, D}); want(m + "v", {(int64_t)s.G * s.dv, D}); }
                if (has(a, FLEXLLM_ATTN_PROJ_BIAS)) {
                    TRY(alloc(&l.b_proj, (size_t)l.proj_n * 4));
                    want(m + "q.b", {(int64_t)s.H * s.dk}); want(m + "k.b", {(int64_t)s.G * s.dk}); want(m + "v.b", {(int64_t)s.G * s.dv});
                }
                if (has(a, FLEXLLM_ATTN_QK_NORM)) {
                    TRY(alloc(&l.q_gain, (size_t)s.H * s.dk * 4));
                    TRY(alloc(&l.k_gain, (size_t)s.G * s.dk * 4));
                    want(m + "q.norm", {(int64_t)s.H * s.dk});
                    want(m + "k.norm", {(int64_t)s.G * s.dk});
                }
                if (has(a, FLEXLLM_ATTN_DISTANCE_BIAS)) {
                    TRY(alloc(&l.bias, attn_bias_floats(s) * 4));
                    want(m + "rel", {-1, s.H});
                }
                if (s.sink == 2) {
                    TRY(alloc(&l.sinks, (size_t)s.H * 4));
                    want(m + "sink", {s.H});
                }
                if (has(a, FLEXLLM_ATTN_GATE)) want(m + "g", {(int64_t)s.H * s.dv, D});
                want(m + "o", {D, (int64_t)s.H * s.dv});
                const size_t ws = attn_window_ws_floats(cfg.max_batch, s.G, s.H / s.G, s.dv);
                attn_ws_floats = ws > attn_ws_floats ? ws : attn_ws_floats;
                n_counters = cfg.max_batch * s.G > n_counters ? cfg.max_batch * s.G : n_counters;
            }
            max_proj = l.proj_n > max_proj ? l.proj_n : max_proj;
            max_att = l.ld_mix > max_att ? l.ld_mix : max_att;
            TRY(alloc(&l.w_proj, (size_t)l.proj_n * ldD * 2));
            TRY(alloc(&l.w_o, (size_t)D * l.ld_mix * 2));
            TRY(alloc(&l.n1, (size_t)ldD * 4));
            want(p + "norm1", {D});
            if (a.ff > 0) {
                const int parts = a.act == FLEXLLM_FF_GELU_GATE ? 2 : 1;
                TRY(alloc(&l.w_gu, (size_t)parts * l.ffp * ldD * 2));
                TRY(alloc(&l.w_down, (size_t)D * l.ffp * 2));
                TRY(alloc(&l.n2, (size_t)ldD * 4));
                want(p + "norm2", {D});
                if (parts == 2) want(p + "mlp.gate", {a.ff, D});
                want(p + "mlp.up", {a.ff, D});
                want(p + "mlp.down", {D, a.ff});
            }
            if (cfg.streams > 0) {
                const int64_t n = cfg.streams;
                TRY(alloc(&l.hc1, (size_t)(n * n + 2 * n) * 4));
                want(p + "hc1.in", {n}); want(p + "hc1.out", {n}); want(p + "hc1.mix", {n, n});
                if (a.ff > 0) {
                    TRY(alloc(&l.hc2, (size_t)(n * n + 2 * n) * 4));
                    want(p + "hc2.in", {n}); want(p + "hc2.out", {n}); want(p + "hc2.mix", {n, n});
                }
            } else {
                TRY(alloc(&l.n1b, (size_t)ldD * 4));
                want(p + "norm1b", {D});
                if (a.ff > 0) {
                    TRY(alloc(&l.n2b, (size_t)ldD * 4));
                    want(p + "norm2b", {D});
                }
            }
        }
        const size_t rows = (size_t)(Mmax > 64 ? Mmax : 64);           // the head normalises up to 64 gathered rows
        TRY(alloc(&h, rows * ldD * es));
        TRY(alloc(&proj, (size_t)Mmax * max_proj * es));
        TRY(alloc(&q, (size_t)Mmax * max_q * es));
        TRY(alloc(&att, (size_t)Mmax * max_att * es));
        TRY(alloc(&act, (size_t)Mmax * max_act * es));
        TRY(alloc(&y, (size_t)Mmax * ldD * 4));
        TRY(alloc(&attn_ws, attn_ws_floats * 4));
        TRY(alloc(&attn_counters, (size_t)n_counters * 4));
        if (max_xbc > 8) {
            TRY(alloc(&xbc, (size_t)Mmax * max_xbc * es));
            TRY(alloc(&gated, (size_t)Mmax * max_inner * es));
        }
        // one cache layer per layer RUN (every pass of the loop has its own) that has keys and values of its own, two states per run
        // of a state-space layer; the pages of a sequence are those of the kept first tokens and a ring that holds the widest
        // window and one chunk
        std::vector<flexllm_kv_shape> shapes;
        std::vector<size_t> states;
        std::vector<int> cache_of(NL, -1);
        for (Run& r : runs) {
            const DecLayer& l = L[r.layer];
            if (l.ssm) {
                r.cache = (int)states.size();
                states.push_back(ssm_state_floats(l.m) * 4);
                states.push_back((size_t)l.m.taps * l.m.ch * es);
            } else if (l.c.kv_from >= 0) {
                r.cache = cache_of[l.c.kv_from];
            } else {
                r.cache = cache_of[r.layer] = (int)shapes.size();
                shapes.push_back({l.s.G, l.s.dkp, l.s.dv});
            }
        }
        const int max_pages = (cfg.max_ctx + 64) / 64;
        long ring = ((long)max_window + cfg.max_prefill + 63) / 64 + 2;
        long keep = attn_keep_pages(max_keep);
        if (ring + keep > max_pages) { ring = max_pages; keep = 0; }
        n_pages = (ring + keep) * cfg.max_batch;
        flexllm_kv_cache* cache = nullptr;
        TRY(flexllm_kv_cache_create_float(&cache, (int)shapes.size(), (int)n_pages, shapes.data(), 64, (int)es));
        const int rc_states = kv_cache_add_states(cache, cfg.max_batch, states);
        if (rc_states != FLEXLLM_OK) { flexllm_kv_cache_destroy(cache); return rc_states; }
        flexllm_model_config rc = {};
        rc.layers = NL; rc.hidden = D; rc.vocab = cfg.vocab; rc.eps = cfg.eps;
        rc.max_batch = cfg.max_batch; rc.max_prefill = cfg.max_prefill; rc.max_ctx = cfg.max_ctx;
        handed_over = true;                                            // from here on the runner owns this object
        return runner_create(out, rc, this, cache, (int)(ring + keep), (int)keep, (size_t)Mmax * ldD * (cfg.streams > 1 ? cfg.streams : 1));
    }
    static bool has(const flexllm_decoder_layer& a, int feature) { return (a.features & feature) != 0; }
    bool handed_over = false;
    long n_pages = 0;

    // ------------------------------------------------------------------------------------------ weights
    bool knows(const char* name) override {
        for (const Want& w : wants) if (w.name == name) return true;
        return false;
    }
    int check_loaded() override {
        for (const Want& w : wants) if (!w.loaded) return FLEXLLM_EINVAL;
        return FLEXLLM_OK;
    }
    // matrix [n][k] -> rows r0.. of dst (row length ld); block 16: rows go to alternating blocks of 16 (gated layers)
    int put_matrix(bf16* dst, long ld, const void* src, long n, long k, cudaStream_t st, bool alternate = false) {
        if (!alternate) return cuda_status(cudaMemcpy2DAsync(dst, ld * 2, src, k * 2, k * 2, n, cudaMemcpyDefault, st));
        if (n % 16 == 0 && ld == k)
            return cuda_status(cudaMemcpy2DAsync(dst, 32 * ld * 2, src, 16 * k * 2, 16 * k * 2, n / 16, cudaMemcpyDefault, st));
        for (long r = 0; r < n; r += 16) {
            const long c = n - r < 16 ? n - r : 16;
            FLEXLLM_CHECK_CUDA(cudaMemcpy2DAsync(dst + 2 * r * ld, ld * 2, (const bf16*)src + r * k, k * 2, k * 2, c, cudaMemcpyDefault, st));
        }
        return FLEXLLM_OK;
    }
    // n values as floats on the host (+ add)
    int get_floats(const void* src, long n, float add, std::vector<float>* out, cudaStream_t st) {
        std::vector<uint16_t> raw(n);
        FLEXLLM_CHECK_CUDA(cudaMemcpyAsync(raw.data(), src, (size_t)n * 2, cudaMemcpyDefault, st));
        FLEXLLM_CHECK_CUDA(cudaStreamSynchronize(st));
        out->resize(n);
        for (long i = 0; i < n; i++) (*out)[i] = bf16_to_float(raw[i]) + add;
        return FLEXLLM_OK;
    }
    int put_floats(float* dst, const std::vector<float>& v, cudaStream_t st) {
        FLEXLLM_CHECK_CUDA(cudaMemcpyAsync(dst, v.data(), v.size() * 4, cudaMemcpyHostToDevice, st));
        return cuda_status(cudaStreamSynchronize(st));
    }
    int put_vector(float* dst, const void* src, long n, float add, cudaStream_t st, float mult = 1.0f) {
        std::vector<float> v;
        TRY(get_floats(src, n, add, &v, st));
        for (float& x : v) x *= mult;
        return put_floats(dst, v, st);
    }
    int put_distance_bias(DecLayer& l, const void* src, int rows, cudaStream_t st) {
        std::vector<float> t;
        TRY(get_floats(src, (long)rows * l.s.H, 0.0f, &t, st));
        l.bias_max = 0.0f;
        for (float v : t) l.bias_max = std::fmax(l.bias_max, std::fabs(v));
        std::vector<float> out(attn_bias_floats(l.s));
        attn_bias_table(l.s, t.data(), rows, l.c.bias_max, out.data());
        return put_floats(l.bias, out, st);
    }

    // `blocks` blocks of n rows at src -> rows r0 + i * n8 of dst (row length ld)
    int put_blocks(bf16* dst, long ld, const bf16* src, int blocks, int n, int n8, long k, cudaStream_t st) {
        for (int i = 0; i < blocks; i++) TRY(put_matrix(dst + (long)i * n8 * ld, ld, src + (long)i * n * k, n, k, st));
        return FLEXLLM_OK;
    }
    // Tensors of a state-space mixer; z, x, B, C and what belongs to them are padded per head or group.
    int place_ssm(DecLayer& l, const std::string& k, const void* src, cudaStream_t st) {
        const SsmShape& s = l.m;
        const long inner = (long)s.H * s.P, gn = (long)s.G * s.N;
        if (k == "in") {
            const bf16* w = (const bf16*)src;
            TRY(put_blocks(l.w_proj, ldD, w, s.H, s.P, s.P8, D, st));
            TRY(put_blocks(l.w_proj + (long)s.x_off * ldD, ldD, w + inner * D, s.H, s.P, s.P8, D, st));
            const long b = s.x_off + s.inner;
            TRY(put_blocks(l.w_proj + b * ldD, ldD, w + 2 * inner * D, 2 * s.G, s.N, s.N8, D, st));           // B, then C
            return put_matrix(l.w_proj + (long)s.dt_off * ldD, ldD, w + (2 * inner + 2 * gn) * D, s.H, D, st);
        }
        // padded channel of the convolution for true channel c
        auto channel = [&](long c) { return c < inner ? c / s.P * s.P8 + c % s.P : s.inner + (c - inner) / s.N * s.N8 + (c - inner) % s.N; };
        if (k == "o") {
            for (int h = 0; h < s.H; h++)
                TRY(cuda_status(cudaMemcpy2DAsync(l.w_o + (long)h * s.P8, l.ld_mix * 2, (const bf16*)src + (long)h * s.P, inner * 2, (size_t)s.P * 2, D,
                                                  cudaMemcpyDefault, st)));
            return FLEXLLM_OK;
        }
        const long n = k == "conv" ? (inner + 2 * gn) * s.taps : k == "conv.b" ? inner + 2 * gn : k == "norm" ? inner : s.H;
        std::vector<float> v;
        TRY(get_floats(src, n, 0.0f, &v, st));
        if (k == "conv") {
            std::vector<float> o((size_t)s.taps * s.ch, 0.0f);
            for (long c = 0; c < inner + 2 * gn; c++)
                for (int j = 0; j < s.taps; j++) o[(size_t)j * s.ch + channel(c)] = v[c * s.taps + j];
            return put_floats(l.conv_w, o, st);
        }
        if (k == "conv.b" || k == "norm") {
            std::vector<float> o((size_t)(k == "norm" ? s.inner : s.ch), 0.0f);
            for (long c = 0; c < n; c++) o[channel(c)] = v[c];
            return put_floats(k == "norm" ? l.m_gain : l.conv_b, o, st);
        }
        if (k == "A_log") {
            for (float& x : v) x = -std::exp(x);
            return put_floats(l.A, v, st);
        }
        return put_floats(k == "D" ? l.D : l.dt_bias, v, st);
    }

    int load_tensor(flexllm_model*, const char* name, int dtype, int ndim, const int64_t* shape, const void* data, cudaStream_t st) override {
        Want* w = nullptr;
        for (Want& x : wants) if (x.name == name) w = &x;
        if (!w) return FLEXLLM_EINVAL;
        if (dtype != FLEXLLM_BF16) return FLEXLLM_ENOTSUP;
        if (ndim != (int)w->shape.size()) return FLEXLLM_EINVAL;
        for (int i = 0; i < ndim; i++)
            if (w->shape[i] >= 0 ? shape[i] != w->shape[i] : shape[i] < 1) return FLEXLLM_EINVAL;
        const int rc = place(w->name, shape, data, st);
        if (rc == FLEXLLM_OK) w->loaded = true;
        return rc;
    }
    int place(const std::string& n, const int64_t* shape, const void* d, cudaStream_t st) {
        if (n == "embed") return put_matrix(embed, ldD, d, cfg.vocab, D, st);
        if (n == "head") return put_matrix(head, ldD, d, cfg.vocab, D, st);
        if (n == "final.norm")
            return cfg.streams > 0 ? put_vector(final_gain, d, D, 0.0f, st, cfg.logit_scale) : put_vector(final_gain, d, D, 1.0f, st);
        if (n == "loop.step") {
            for (int t = 0; t < cfg.loop_times; t++) TRY(put_vector(loop_step + (size_t)t * ldD, (const bf16*)d + (size_t)t * D, D, 0.0f, st));
            return FLEXLLM_OK;
        }
        const size_t dot = n.find('.');
        DecLayer& l = L[atoi(n.c_str() + 1)];
        const AttnShape& s = l.s;
        const std::string k = n.substr(dot + 1);
        if (cfg.streams > 0 && (k == "norm1" || k == "norm2")) return put_vector(k == "norm1" ? l.n1 : l.n2, d, D, 0.0f, st);
        if (k.compare(0, 2, "hc") == 0) {
            float* c = k[2] == '1' ? l.hc1 : l.hc2;
            const long ns = cfg.streams;
            const std::string part = k.substr(4);
            if (part == "mix") return put_vector(c, d, ns * ns, 0.0f, st);
            if (part == "out") return put_vector(c + ns * ns, d, ns, 0.0f, st, cfg.residual_mult);
            return put_vector(c + ns * ns + ns, d, ns, 0.0f, st);
        }
        if (k == "mix.sink") return put_vector(l.sinks, d, s.H, 0.0f, st);
        if (l.ssm && k.compare(0, 4, "mix.") == 0) return place_ssm(l, k.substr(4), d, st);
        if (k == "norm1") return put_vector(l.n1, d, D, 1.0f, st);
        if (k == "norm1b") return put_vector(l.n1b, d, D, 1.0f, st);
        if (k == "norm2") return put_vector(l.n2, d, D, 1.0f, st);
        if (k == "norm2b") return put_vector(l.n2b, d, D, 1.0f, st);
        if (k == "mix.q") return put_matrix(l.w_proj + (long)s.q_off * ldD, ldD, d, shape[0], D, st);
        if (k == "mix.k") return put_matrix(l.w_proj + (long)s.k_off * ldD, ldD, d, shape[0], D, st);
        if (k == "mix.v") return put_matrix(l.w_proj + (long)s.v_off * ldD, ldD, d, shape[0], D, st);
        if (k == "mix.g") return put_matrix(l.w_proj + (long)s.g_off * ldD, ldD, d, shape[0], D, st);
        if (k == "mix.q.b") return put_vector(l.b_proj + s.q_off, d, shape[0], 0.0f, st);
        if (k == "mix.k.b") return put_vector(l.b_proj + s.k_off, d, shape[0], 0.0f, st);
        if (k == "mix.v.b") return put_vector(l.b_proj + s.v_off, d, shape[0], 0.0f, st);
        if (k == "mix.q.norm") return put_vector(l.q_gain, d, shape[0], 0.0f, st);
        if (k == "mix.k.norm") return put_vector(l.k_gain, d, shape[0], 0.0f, st);
        if (k == "mix.rel") return put_distance_bias(l, d, (int)shape[0], st);
        if (k == "mix.o") return put_matrix(l.w_o, up_to((long)s.H * s.dv, 8), d, D, (long)s.H * s.dv, st);
        if (k == "mlp.gate") return put_matrix(l.w_gu, ldD, d, l.c.ff, D, st, true);
        if (k == "mlp.up" && l.c.act == FLEXLLM_FF_RELU2) return put_matrix(l.w_gu, ldD, d, l.c.ff, D, st);
        if (k == "mlp.up") return put_matrix(l.w_gu + 16 * (long)ldD, ldD, d, l.c.ff, D, st, true);
        if (k == "mlp.down") return put_matrix(l.w_down, l.ffp, d, D, l.c.ff, st);
        return FLEXLLM_EINVAL;
    }

    // ------------------------------------------------------------------------------------------ a step
    template <class T> int linear(const void* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act, LinearOut o,
                                  cudaStream_t st);
    // the mixer of run i between its projections: proj -> att
    template <class T> int mix(flexllm_model* m, int i, int B, int Sc, cudaStream_t st) {
        const Run& r = runs[i];
        const DecLayer& l = L[r.layer];
        const flexllm_kv_cache* kv = m->cache;
        if (l.ssm) {
            SsmCall c = {};
            c.s = l.m; c.proj = proj; c.conv_w = l.conv_w; c.conv_b = l.conv_b; c.dt_bias = l.dt_bias; c.A = l.A; c.D = l.D;
            c.gain = l.m_gain; c.eps = cfg.eps;
            c.state = (float*)(kv->states + kv->s_off[r.cache]); c.conv_state = kv->states + kv->s_off[r.cache + 1];
            c.ctx = m->ctx; c.B = B; c.Sc = Sc; c.xbc = xbc; c.y = gated; c.out = att;
            return ssm_mixer<T>(c, st);
        }
        AttnCall c = {};
        c.s = l.s; c.proj = proj; c.q_gain = l.q_gain; c.k_gain = l.k_gain; c.eps = cfg.eps;
        c.bias = l.bias; c.bias_max_abs = l.bias_max; c.sinks = l.sinks;
        c.k_pool = kv->k + kv->k_off[r.cache]; c.v_pool = kv->v + kv->v_off[r.cache]; c.n_pages = n_pages;
        c.page_table = m->page_table; c.max_pages = m->max_pages; c.ctx = m->ctx; c.max_pos = m->cfg.max_ctx;
        c.B = B; c.Sc = Sc; c.q = q; c.out = att; c.ldo = l.ld_mix;
        c.ws = attn_ws; c.counters = attn_counters; c.ws_floats = attn_ws_floats; c.n_counters = n_counters;
        return attn_window<T>(c, st);
    }
    // The rows' residual between sublayers. Sublayer q of run i is about to follow what is in y (q = 0: the mixer, 1: the
    // feed-forward; i == runs: the head); `after` adds the sublayer before it to the residual and forms its input h.
    struct Sub { int run, ff; };
    Sub before(int i, int q) const {
        if (q == 1) return {i, 0};
        return {i - 1, i > 0 && L[runs[i - 1].layer].c.ff > 0 ? 1 : 0};
    }
    template <class T> int after(flexllm_model* m, int i, int q, const int32_t* tok, int B, int S, int c0, int Sc, cudaStream_t st) {
        const int M = B * Sc, nr = (int)runs.size();
        const Sub p = before(i, q);                                    // p.run < 0: the start of the step
        const DecLayer* l = i < nr ? &L[runs[i].layer] : nullptr;
        const DecLayer* pl = p.run >= 0 ? &L[runs[p.run].layer] : nullptr;
        float* tr = nullptr;
        if (trace && q == 0 && i > 0) {
            if ((size_t)i * M * D > trace_floats) return FLEXLLM_ETOOBIG;
            tr = trace + (size_t)(i - 1) * M * D;
        }
        if (cfg.streams > 0) {
            const long n = cfg.streams;
            HyperNormArgs a = {};
            a.x = m->x; a.lds = ldD; a.n = cfg.streams; a.D = D; a.eps = cfg.eps; a.trace = tr;
            if (!pl) {
                a.tok = tok; a.S = S; a.c0 = c0; a.Sc = Sc;
                a.emb = embed; a.lde = ldD; a.emb_scale = cfg.embed_scale; a.V = cfg.vocab; a.error_flag = device_error_flag();
            } else {
                a.y = y; a.ldy = ldD; a.mix = p.ff ? pl->hc2 : pl->hc1; a.out = a.mix + n * n;
            }
            if (l) { a.in = (q ? l->hc2 : l->hc1) + n * n + n; a.gain = q ? l->n2 : l->n1; a.h = h; a.ldh = ldD; }
            return hyper_norm<T>(a, M, st);
        }
        ResNormArgs a = {};
        a.x = m->x; a.ldx = ldD; a.D = D; a.eps = cfg.eps;
        a.tok = tok; a.S = S; a.c0 = c0; a.Sc = Sc;
        a.emb = embed; a.lde = ldD; a.emb_scale = cfg.embed_scale; a.V = cfg.vocab; a.error_flag = device_error_flag();
        a.h = h; a.ldh = ldD; a.trace = tr;
        if (pl) { a.y = y; a.ldy = ldD; a.gain_post = p.ff ? pl->n2b : pl->n1b; }
        else a.emb_mode = 1;
        if (l && q == 0) {                                             // a pass of the loop begins with its additions
            const Run& r = runs[i];
            if (r.pass > 0) a.emb_mode = 2;
            if (r.pass >= 0) a.add_vec = loop_step + (size_t)r.pass * ldD;
        }
        if (l) a.gain_pre = q ? l->n2 : l->n1;
        return res_norm<T>(a, M, st);
    }
    template <class T> int step(flexllm_model* m, const int32_t* tok, int B, int S, int c0, int Sc, cudaStream_t st) {
        const int M = B * Sc, nr = (int)runs.size();
        for (int i = 0; i < nr; i++) {
            const DecLayer& l = L[runs[i].layer];
            TRY(after<T>(m, i, 0, tok, B, S, c0, Sc, st));
            TRY(linear<T>(h, ldD, l.w_proj, ldD, l.b_proj, M, l.proj_n, D, kActNone, {nullptr, proj, l.proj_n}, st));
            TRY(mix<T>(m, i, B, Sc, st));
            TRY(linear<T>(att, l.ld_mix, l.w_o, l.ld_mix, nullptr, M, D, l.n_mix, kActNone, {y, nullptr, ldD}, st));
            if (l.c.ff > 0) {
                const bool gated_ff = l.c.act == FLEXLLM_FF_GELU_GATE;
                TRY(after<T>(m, i, 1, tok, B, S, c0, Sc, st));
                TRY(linear<T>(h, ldD, l.w_gu, ldD, nullptr, M, gated_ff ? 2 * l.ffp : l.ffp, D, gated_ff ? kActGeluGate : kActRelu2,
                              {nullptr, act, (long)l.ffp}, st));
                TRY(linear<T>(act, l.ffp, l.w_down, l.ffp, nullptr, M, D, l.c.ff, kActNone, {y, nullptr, ldD}, st));
            }
        }
        return after<T>(m, nr, 0, tok, B, S, c0, Sc, st);
    }
    template <class T> int head_rows(flexllm_model* m, const int32_t* rows, int n, float* out, cudaStream_t st) {
        if (cfg.streams > 0) {
            HyperNormArgs a = {};
            a.x = m->x; a.lds = ldD; a.n = cfg.streams; a.D = D; a.eps = cfg.eps; a.rows = rows;
            a.in = ones; a.gain = final_gain; a.h = h; a.ldh = ldD;
            TRY(hyper_norm<T>(a, n, st));
        } else {
            ResNormArgs a = {};
            a.x = m->x; a.ldx = ldD; a.D = D; a.eps = cfg.eps; a.Sc = 1; a.rows = rows; a.keep_x = 1;
            a.gain_pre = final_gain; a.h = h; a.ldh = ldD;
            TRY(res_norm<T>(a, n, st));
        }
        return linear<T>(h, ldD, head, ldD, nullptr, n, cfg.vocab, D, kActNone, {out, nullptr, cfg.vocab}, st);
    }
    int forward(flexllm_model* m, const int32_t* tok, int B, int S, int c0, int Sc, cudaStream_t st) override {
        return cfg.dtype == FLEXLLM_BF16 ? step<bf16>(m, tok, B, S, c0, Sc, st) : step<float>(m, tok, B, S, c0, Sc, st);
    }
    int logits(flexllm_model* m, const int32_t* rows, int n, float* out, cudaStream_t st) override {
        return cfg.dtype == FLEXLLM_BF16 ? head_rows<bf16>(m, rows, n, out, st) : head_rows<float>(m, rows, n, out, st);
    }
    int set_trace(float* t, size_t floats) override { trace = t; trace_floats = floats; return FLEXLLM_OK; }
};

template <> int DecoderFamily::linear<bf16>(const void* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act,
                                            LinearOut o, cudaStream_t st) {
    return linear_bf16((const bf16*)a, lda, w, ldw, bias, M, N, K, act, o, st);
}
template <> int DecoderFamily::linear<float>(const void* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, int act,
                                             LinearOut o, cudaStream_t st) {
    return linear_f32((const float*)a, lda, w, ldw, bias, M, N, K, act, o, st);
}

}  // namespace

}  // namespace flexllm

using namespace flexllm;

// See include/flexllm_b200.h.
extern "C" int flexllm_model_create_decoder(flexllm_model** out, const flexllm_decoder_config* c) {
    FLEXLLM_REQUIRE(out && c && c->layers > 0 && c->layer && c->width > 0 && c->vocab > 0);
    FLEXLLM_REQUIRE(c->dtype == FLEXLLM_BF16 || c->dtype == FLEXLLM_F32);
    FLEXLLM_REQUIRE(c->max_batch > 0 && c->max_batch <= 64 && c->max_prefill > 0 && c->max_ctx >= c->max_prefill);
    FLEXLLM_REQUIRE(c->loop_times >= 0 && (c->loop_times == 0 || (c->loop_start >= 0 && c->loop_start < c->loop_stop && c->loop_stop <= c->layers)));
    FLEXLLM_REQUIRE(c->streams >= 0);
    if (c->streams > kMaxStreams) return FLEXLLM_ENOTSUP;
    for (int i = 0; i < c->layers; i++) {
        const flexllm_decoder_layer& a = c->layer[i];
        FLEXLLM_REQUIRE(a.heads > 0 && a.vdim > 0 && a.ff >= 0);
        FLEXLLM_REQUIRE(a.ff == 0 || a.act == FLEXLLM_FF_GELU_GATE || a.act == FLEXLLM_FF_RELU2);
        if (a.mixer == FLEXLLM_MIXER_SSM) {
            FLEXLLM_REQUIRE(a.state > 0 && a.groups > 0 && a.heads % a.groups == 0 && a.conv > 0);
            FLEXLLM_REQUIRE(a.norm_groups > 0 && (long)a.heads * a.vdim % a.norm_groups == 0);
            continue;
        }
        FLEXLLM_REQUIRE(a.mixer == FLEXLLM_MIXER_ATTENTION && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.window > 0 && a.keep_first >= 0);
        FLEXLLM_REQUIRE(!(a.features & FLEXLLM_ATTN_DISTANCE_BIAS) || a.keep_first == 0);
        if (a.kv_from < 0) continue;
        // another layer's keys and values: an earlier layer that has its own, of the same sizes
        FLEXLLM_REQUIRE(a.kv_from < i && c->loop_times == 0 && !(a.features & (FLEXLLM_ATTN_QK_NORM | FLEXLLM_ATTN_PROJ_BIAS)));
        const flexllm_decoder_layer& o = c->layer[a.kv_from];
        FLEXLLM_REQUIRE(o.mixer == FLEXLLM_MIXER_ATTENTION && o.kv_from < 0 && o.kv_heads == a.kv_heads && o.dim == a.dim && o.vdim == a.vdim);
    }
    DecoderFamily* f = new (std::nothrow) DecoderFamily();
    if (!f) return FLEXLLM_ENOMEM;
    const int rc = f->create(out, c);
    if (rc != FLEXLLM_OK && !f->handed_over) delete f;
    return rc;
}
