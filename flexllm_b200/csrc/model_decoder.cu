// Decoder family with floating-point weights (the Pibidra design): sandwich norms around every sublayer, windowed
// grouped-query attention with query/key norms over the whole projection, softcapped scores, a learned distance bias, a
// softmax sink and an output gate (attention_window.cu), a gated-GELU feed-forward, and an optional block of layers that
// runs several times with the same weights. bf16 weights; activations bf16 (residual stream, norms, scores fp32), or
// everything fp32.
//
// A step is, per layer run: fused q|k|v|gate projection -> attention -> output projection -> [norm, residual, norm]
// -> fused gate|up projection with the gated GELU in its epilogue -> down projection -> [norm, residual, loop additions,
// norm]. The same step serves prompts, portions of prompts and decoding; row counts choose the kernels.
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
    AttnShape s;
    int proj_n, ffp;                            // rows of the fused projection; ff rounded up to 16
    bf16 *w_proj, *w_o, *w_gu, *w_down;
    float *b_proj;                              // biases of the fused projection (zero where it has none)
    float *n1, *n1b, *n2, *n2b;                 // norm gains (1 + stored weight)
    float *q_gain, *k_gain, *bias;
    float bias_max = 0.0f;
};

float bf16_to_float(uint16_t v) { uint32_t u = (uint32_t)v << 16; float f; memcpy(&f, &u, 4); return f; }

struct Want { std::string name; std::vector<int64_t> shape; bool loaded; };

class DecoderFamily : public ModelFamily {
  public:
    flexllm_decoder_config cfg;
    std::vector<flexllm_decoder_layer> specs;
    std::vector<DecLayer> L;
    struct Run { int layer; int pass; };        // pass >= 0 on the first layer of a pass of the loop
    std::vector<Run> runs;
    std::vector<Want> wants;
    std::vector<void*> owned;
    int D = 0, ldD = 0;
    bf16 *embed = nullptr, *head = nullptr;
    float *final_gain = nullptr, *loop_step = nullptr;
    // activations (T = bf16 or float by cfg.dtype)
    void *h = nullptr, *proj = nullptr, *q = nullptr, *att = nullptr, *act = nullptr;
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
                    for (int k = cfg.loop_start; k < cfg.loop_stop; k++) runs.push_back({k, k == cfg.loop_start ? t : -1});
                i = cfg.loop_stop - 1;
            } else {
                runs.push_back({i, -1});
            }
        }
        want("embed", {cfg.vocab, D});
        want("head", {cfg.vocab, D});
        want("final.norm", {D});
        TRY(alloc(&embed, (size_t)cfg.vocab * ldD * 2));
        TRY(alloc(&head, (size_t)cfg.vocab * ldD * 2));
        TRY(alloc(&final_gain, (size_t)ldD * 4));
        if (cfg.loop_times > 0) {
            want("loop.step", {cfg.loop_times, D});
            TRY(alloc(&loop_step, (size_t)cfg.loop_times * ldD * 4));
        }
        L.resize(NL);
        long max_proj = 8, max_q = 8, max_att = 8, max_act = 8;
        int max_window = 1;
        for (int i = 0; i < NL; i++) {
            DecLayer& l = L[i];
            l = DecLayer();
            l.c = specs[i];
            const flexllm_decoder_layer& a = l.c;
            AttnShape& s = l.s;
            s.H = a.heads; s.G = a.kv_heads; s.dk = a.dim; s.dv = a.vdim;
            s.window = a.window < cfg.max_ctx + 1 ? a.window : cfg.max_ctx + 1;      // nothing is further away than that
            s.scale = a.scale; s.softcap = a.softcap; s.sink = 1;
            attn_layout(&s, true);
            l.proj_n = (int)s.ld;
            l.ffp = (int)up_to(a.ff, 16);
            max_window = s.window > max_window ? s.window : max_window;
            max_proj = l.proj_n > max_proj ? l.proj_n : max_proj;
            const long nq = (long)s.H * s.dkp, na = up_to((long)s.H * s.dv, 8);
            max_q = nq > max_q ? nq : max_q;
            max_att = na > max_att ? na : max_att;
            max_act = l.ffp > max_act ? l.ffp : max_act;
            TRY(alloc(&l.w_proj, (size_t)l.proj_n * ldD * 2));
            TRY(alloc(&l.b_proj, (size_t)l.proj_n * 4));
            TRY(alloc(&l.w_o, (size_t)D * na * 2));
            TRY(alloc(&l.n1, (size_t)ldD * 4));
            TRY(alloc(&l.n1b, (size_t)ldD * 4));
            TRY(alloc(&l.q_gain, (size_t)s.H * s.dk * 4));
            TRY(alloc(&l.k_gain, (size_t)s.G * s.dk * 4));
            TRY(alloc(&l.bias, attn_bias_floats(s) * 4));
            const std::string p = "l" + std::to_string(i) + ".", m = p + "mix.";
            want(p + "norm1", {D});
            want(p + "norm1b", {D});
            want(m + "q", {(int64_t)s.H * s.dk, D}); want(m + "q.b", {(int64_t)s.H * s.dk});
            want(m + "k", {(int64_t)s.G * s.dk, D}); want(m + "k.b", {(int64_t)s.G * s.dk});
            want(m + "v", {(int64_t)s.G * s.dv, D}); want(m + "v.b", {(int64_t)s.G * s.dv});
            want(m + "q.norm", {(int64_t)s.H * s.dk});
            want(m + "k.norm", {(int64_t)s.G * s.dk});
            want(m + "rel", {-1, s.H});
            want(m + "g", {(int64_t)s.H * s.dv, D});
            want(m + "o", {D, (int64_t)s.H * s.dv});
            if (a.ff > 0) {
                TRY(alloc(&l.w_gu, (size_t)2 * l.ffp * ldD * 2));
                TRY(alloc(&l.w_down, (size_t)D * l.ffp * 2));
                TRY(alloc(&l.n2, (size_t)ldD * 4));
                TRY(alloc(&l.n2b, (size_t)ldD * 4));
                want(p + "norm2", {D});
                want(p + "norm2b", {D});
                want(p + "mlp.gate", {a.ff, D});
                want(p + "mlp.up", {a.ff, D});
                want(p + "mlp.down", {D, a.ff});
            }
            const size_t ws = attn_window_ws_floats(cfg.max_batch, s.G, s.H / s.G, s.dv);
            attn_ws_floats = ws > attn_ws_floats ? ws : attn_ws_floats;
            n_counters = cfg.max_batch * s.G > n_counters ? cfg.max_batch * s.G : n_counters;
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
        // one cache layer per layer RUN (every pass of the loop has its own); the pages of a sequence form a ring that
        // holds the widest window and one chunk
        std::vector<flexllm_kv_shape> shapes;
        for (const Run& r : runs) shapes.push_back({L[r.layer].s.G, L[r.layer].s.dkp, L[r.layer].s.dv});
        const int max_pages = (cfg.max_ctx + 64) / 64;
        long ring = ((long)max_window + cfg.max_prefill + 63) / 64 + 2;
        if (ring > max_pages) ring = max_pages;
        n_pages = ring * cfg.max_batch;
        flexllm_kv_cache* cache = nullptr;
        TRY(flexllm_kv_cache_create_float(&cache, (int)runs.size(), (int)n_pages, shapes.data(), 64, (int)es));
        flexllm_model_config rc = {};
        rc.layers = NL; rc.hidden = D; rc.vocab = cfg.vocab; rc.eps = cfg.eps;
        rc.max_batch = cfg.max_batch; rc.max_prefill = cfg.max_prefill; rc.max_ctx = cfg.max_ctx;
        handed_over = true;                                            // from here on the runner owns this object
        return runner_create(out, rc, this, cache, (int)ring, (size_t)Mmax * ldD);
    }
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
    int put_vector(float* dst, const void* src, long n, float add, cudaStream_t st) {
        std::vector<float> v;
        TRY(get_floats(src, n, add, &v, st));
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
        if (n == "final.norm") return put_vector(final_gain, d, D, 1.0f, st);
        if (n == "loop.step") {
            for (int t = 0; t < cfg.loop_times; t++) TRY(put_vector(loop_step + (size_t)t * ldD, (const bf16*)d + (size_t)t * D, D, 0.0f, st));
            return FLEXLLM_OK;
        }
        const size_t dot = n.find('.');
        DecLayer& l = L[atoi(n.c_str() + 1)];
        const AttnShape& s = l.s;
        const std::string k = n.substr(dot + 1);
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
        if (k == "mlp.up") return put_matrix(l.w_gu + 16 * (long)ldD, ldD, d, l.c.ff, D, st, true);
        if (k == "mlp.down") return put_matrix(l.w_down, l.ffp, d, D, l.c.ff, st);
        return FLEXLLM_EINVAL;
    }

    // ------------------------------------------------------------------------------------------ a step
    template <class T> int linear(const void* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, bool glu, LinearOut o,
                                  cudaStream_t st);
    template <class T> int step(flexllm_model* m, const int32_t* tok, int B, int S, int c0, int Sc, cudaStream_t st) {
        const int M = B * Sc, nr = (int)runs.size();
        ResNormArgs base = {};
        base.x = m->x; base.ldx = ldD; base.D = D; base.eps = cfg.eps;
        base.tok = tok; base.S = S; base.c0 = c0; base.Sc = Sc;
        base.emb = embed; base.lde = ldD; base.emb_scale = cfg.embed_scale; base.V = cfg.vocab; base.error_flag = device_error_flag();
        base.ldy = ldD; base.h = h; base.ldh = ldD;
        // what precedes run i: the pass's additions, then its first norm
        auto lead_in = [&](ResNormArgs& a, int i) {
            if (i >= nr) return;
            const Run& r = runs[i];
            if (r.pass > 0) a.emb_mode = 2;
            if (r.pass >= 0) a.add_vec = loop_step + (size_t)r.pass * ldD;
            a.gain_pre = L[r.layer].n1;
        };
        ResNormArgs a = base;
        lead_in(a, 0);
        a.emb_mode = 1;
        TRY(res_norm<T>(a, M, st));
        for (int i = 0; i < nr; i++) {
            const DecLayer& l = L[runs[i].layer];
            const long ld_att = up_to((long)l.s.H * l.s.dv, 8);
            TRY(linear<T>(h, ldD, l.w_proj, ldD, l.b_proj, M, l.proj_n, D, false, {nullptr, proj, l.s.ld}, st));
            AttnCall c = {};
            c.s = l.s; c.proj = proj; c.q_gain = l.q_gain; c.k_gain = l.k_gain; c.eps = cfg.eps;
            c.bias = l.bias; c.bias_max_abs = l.bias_max;
            c.k_pool = m->cache->k + m->cache->k_off[i]; c.v_pool = m->cache->v + m->cache->v_off[i]; c.n_pages = n_pages;
            c.page_table = m->page_table; c.max_pages = m->max_pages; c.ctx = m->ctx; c.max_pos = m->cfg.max_ctx;
            c.B = B; c.Sc = Sc; c.q = q; c.out = att; c.ldo = ld_att;
            c.ws = attn_ws; c.counters = attn_counters; c.ws_floats = attn_ws_floats; c.n_counters = n_counters;
            TRY(attn_window<T>(c, st));
            TRY(linear<T>(att, ld_att, l.w_o, ld_att, nullptr, M, D, l.s.H * l.s.dv, false, {y, nullptr, ldD}, st));
            a = base;
            a.y = y; a.gain_post = l.n1b;
            if (l.c.ff > 0) {
                a.gain_pre = l.n2;
                TRY(res_norm<T>(a, M, st));
                TRY(linear<T>(h, ldD, l.w_gu, ldD, nullptr, M, 2 * l.ffp, D, true, {nullptr, act, (long)l.ffp}, st));
                TRY(linear<T>(act, l.ffp, l.w_down, l.ffp, nullptr, M, D, l.c.ff, false, {y, nullptr, ldD}, st));
                a = base;
                a.y = y; a.gain_post = l.n2b;
            }
            if (trace) {
                if ((size_t)(i + 1) * M * D > trace_floats) return FLEXLLM_ETOOBIG;
                a.trace = trace + (size_t)i * M * D;
            }
            lead_in(a, i + 1);
            TRY(res_norm<T>(a, M, st));
        }
        return FLEXLLM_OK;
    }
    template <class T> int head_rows(flexllm_model* m, const int32_t* rows, int n, float* out, cudaStream_t st) {
        ResNormArgs a = {};
        a.x = m->x; a.ldx = ldD; a.D = D; a.eps = cfg.eps; a.Sc = 1; a.rows = rows; a.keep_x = 1;
        a.gain_pre = final_gain; a.h = h; a.ldh = ldD;
        TRY(res_norm<T>(a, n, st));
        return linear<T>(h, ldD, head, ldD, nullptr, n, cfg.vocab, D, false, {out, nullptr, cfg.vocab}, st);
    }
    int forward(flexllm_model* m, const int32_t* tok, int B, int S, int c0, int Sc, cudaStream_t st) override {
        return cfg.dtype == FLEXLLM_BF16 ? step<bf16>(m, tok, B, S, c0, Sc, st) : step<float>(m, tok, B, S, c0, Sc, st);
    }
    int logits(flexllm_model* m, const int32_t* rows, int n, float* out, cudaStream_t st) override {
        return cfg.dtype == FLEXLLM_BF16 ? head_rows<bf16>(m, rows, n, out, st) : head_rows<float>(m, rows, n, out, st);
    }
    int set_trace(float* t, size_t floats) override { trace = t; trace_floats = floats; return FLEXLLM_OK; }
};

template <> int DecoderFamily::linear<bf16>(const void* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, bool glu,
                                            LinearOut o, cudaStream_t st) {
    return linear_bf16((const bf16*)a, lda, w, ldw, bias, M, N, K, glu, o, st);
}
template <> int DecoderFamily::linear<float>(const void* a, long lda, const bf16* w, long ldw, const float* bias, int M, int N, int K, bool glu,
                                             LinearOut o, cudaStream_t st) {
    return linear_f32((const float*)a, lda, w, ldw, bias, M, N, K, glu, o, st);
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
    for (int i = 0; i < c->layers; i++) {
        const flexllm_decoder_layer& a = c->layer[i];
        FLEXLLM_REQUIRE(a.heads > 0 && a.kv_heads > 0 && a.heads % a.kv_heads == 0 && a.dim > 0 && a.vdim > 0 && a.window > 0 && a.ff >= 0);
    }
    DecoderFamily* f = new (std::nothrow) DecoderFamily();
    if (!f) return FLEXLLM_ENOMEM;
    const int rc = f->create(out, c);
    if (rc != FLEXLLM_OK && !f->handed_over) delete f;
    return rc;
}
