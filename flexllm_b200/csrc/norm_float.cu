// Norms of the floating-point model path: everything between two sublayers in one pass over the residual
// stream's rows (norm after a sublayer, residual sum, embedding and vector additions, norm before the next one; or the
// mixing of several residual streams and the norm before the next sublayer).
#include "float_common.cuh"

namespace flexllm {

namespace {

// One CTA of NT threads per row, VPT float4 of the row per thread. All sums and the residual are fp32. The columns from D
// up to the next multiple of 4 are zero in x, the gains, y and the embedding table.
template <class T, int NT, int VPT>
__global__ void __launch_bounds__(NT) res_norm_kernel(const ResNormArgs a) {
    __shared__ float red[2 * NT / 32];
    pdl_sync();
    const int r = blockIdx.x, tid = threadIdx.x;
    const int nv = (a.D + 3) >> 2;
    const long row = a.rows ? a.rows[r] : r;
    float* xr = a.x + row * a.ldx;
    const bf16* er = nullptr;
    if (a.emb_mode) {
        int id = a.tok[(long)(r / a.Sc) * a.S + a.c0 + r % a.Sc];
        if (id < 0 || id >= a.V) {                        // device data the host has not seen: clamp and report
            if (tid == 0 && a.error_flag) atomicOr(a.error_flag, 2);
            id = id < 0 ? 0 : a.V - 1;
        }
        er = a.emb + (long)id * a.lde;
    }
    auto emb4 = [&](int c) {
        const float4 e = load4(er + 4 * c);
        return make_float4(e.x * a.emb_scale, e.y * a.emb_scale, e.z * a.emb_scale, e.w * a.emb_scale);
    };
    float4 v[VPT];
#pragma unroll
    for (int i = 0; i < VPT; i++) {
        const int c = tid + i * NT;
        v[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (c < nv) v[i] = a.emb_mode == 1 ? emb4(c) : load4(xr + 4 * c);
    }
    if (a.y) {
        const float* yr = a.y + (long)r * a.ldy;
        float4 y[VPT];
        float ss = 0.0f;
#pragma unroll
        for (int i = 0; i < VPT; i++) {
            const int c = tid + i * NT;
            y[i] = c < nv ? load4(yr + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
            ss += (y[i].x * y[i].x + y[i].y * y[i].y) + (y[i].z * y[i].z + y[i].w * y[i].w);
        }
        ss = block_sum2<NT>(ss, 0.0f, red).x;
        const float rinv = 1.0f / sqrtf(ss / (float)a.D + a.eps);
#pragma unroll
        for (int i = 0; i < VPT; i++) {
            const int c = tid + i * NT;
            if (c < nv) {
                const float4 g = load4(a.gain_post + 4 * c);
                v[i].x += (y[i].x * rinv) * g.x; v[i].y += (y[i].y * rinv) * g.y;
                v[i].z += (y[i].z * rinv) * g.z; v[i].w += (y[i].w * rinv) * g.w;
            }
        }
    }
    if (a.trace) {
        float* t = a.trace + (long)r * a.D;
#pragma unroll
        for (int i = 0; i < VPT; i++) {
            const int e = 4 * (tid + i * NT);
            const float x4[4] = {v[i].x, v[i].y, v[i].z, v[i].w};
            for (int k = 0; k < 4; k++)
                if (e + k < a.D) t[e + k] = x4[k];
        }
    }
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < VPT; i++) {
        const int c = tid + i * NT;
        if (c < nv) {
            if (a.emb_mode == 2) { const float4 e = emb4(c); v[i].x += e.x; v[i].y += e.y; v[i].z += e.z; v[i].w += e.w; }
            if (a.add_vec) { const float4 e = load4(a.add_vec + 4 * c); v[i].x += e.x; v[i].y += e.y; v[i].z += e.z; v[i].w += e.w; }
            if (!a.keep_x) store4(xr + 4 * c, v[i]);
            ss += (v[i].x * v[i].x + v[i].y * v[i].y) + (v[i].z * v[i].z + v[i].w * v[i].w);
        }
    }
    if (!a.gain_pre) return;
    ss = block_sum2<NT>(ss, 0.0f, red).x;
    const float rinv = 1.0f / sqrtf(ss / (float)a.D + a.eps);
    T* hr = (T*)a.h + (long)r * a.ldh;
#pragma unroll
    for (int i = 0; i < VPT; i++) {
        const int c = tid + i * NT;
        if (c < nv) {
            const float4 g = load4(a.gain_pre + 4 * c);
            store4(hr + 4 * c, make_float4((v[i].x * rinv) * g.x, (v[i].y * rinv) * g.y, (v[i].z * rinv) * g.z, (v[i].w * rinv) * g.w));
        }
    }
}

// One CTA per row, all streams of VPT float4 per thread in registers.
template <class T, int NS, int NT, int VPT>
__global__ void __launch_bounds__(NT) hyper_norm_kernel(const HyperNormArgs a) {
    __shared__ float red[2 * NT / 32];
    pdl_sync();
    const int r = blockIdx.x, tid = threadIdx.x, n = a.n;
    const int nv = (a.D + 3) >> 2;
    const long row = a.rows ? a.rows[r] : r;
    float* xr = a.x + row * n * a.lds;
    float4 v[NS][VPT];
    if (a.emb) {
        int id = a.tok[(long)(r / a.Sc) * a.S + a.c0 + r % a.Sc];
        if (id < 0 || id >= a.V) {                        // device data the host has not seen: clamp and report
            if (tid == 0 && a.error_flag) atomicOr(a.error_flag, 2);
            id = id < 0 ? 0 : a.V - 1;
        }
        const bf16* er = a.emb + (long)id * a.lde;
#pragma unroll
        for (int i = 0; i < VPT; i++) {
            const int c = tid + i * NT;
            float4 e = make_float4(0.f, 0.f, 0.f, 0.f);
            if (c < nv) e = load4(er + 4 * c);
            e.x *= a.emb_scale; e.y *= a.emb_scale; e.z *= a.emb_scale; e.w *= a.emb_scale;
#pragma unroll
            for (int s = 0; s < NS; s++) v[s][i] = e;
        }
    } else {
#pragma unroll
        for (int s = 0; s < NS; s++)
#pragma unroll
            for (int i = 0; i < VPT; i++) {
                const int c = tid + i * NT;
                v[s][i] = s < n && c < nv ? load4(xr + s * a.lds + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
            }
    }
    if (a.y) {
        const float* yr = a.y + (long)r * a.ldy;
#pragma unroll
        for (int i = 0; i < VPT; i++) {
            const int c = tid + i * NT;
            const float4 y = c < nv ? load4(yr + 4 * c) : make_float4(0.f, 0.f, 0.f, 0.f);
            float4 w[NS];
#pragma unroll
            for (int t = 0; t < NS; t++) {
                w[t] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (t >= n) continue;
                const float o = a.out[t];
                w[t] = make_float4(o * y.x, o * y.y, o * y.z, o * y.w);
#pragma unroll
                for (int s = 0; s < NS; s++) {
                    if (s >= n) continue;
                    const float k = a.mix[s * n + t];
                    w[t].x = __fmaf_rn(k, v[s][i].x, w[t].x); w[t].y = __fmaf_rn(k, v[s][i].y, w[t].y);
                    w[t].z = __fmaf_rn(k, v[s][i].z, w[t].z); w[t].w = __fmaf_rn(k, v[s][i].w, w[t].w);
                }
            }
#pragma unroll
            for (int t = 0; t < NS; t++) v[t][i] = w[t];
        }
    }
    if (a.trace) {
        float* t = a.trace + (long)r * a.D;
#pragma unroll
        for (int i = 0; i < VPT; i++) {
            const int e = 4 * (tid + i * NT);
            float x4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int s = 0; s < NS; s++)
                if (s < n) { x4[0] += v[s][i].x; x4[1] += v[s][i].y; x4[2] += v[s][i].z; x4[3] += v[s][i].w; }
            for (int k = 0; k < 4; k++)
                if (e + k < a.D) t[e + k] = x4[k];
        }
    }
    if (a.emb || a.y)
#pragma unroll
        for (int s = 0; s < NS; s++)
#pragma unroll
            for (int i = 0; i < VPT; i++) {
                const int c = tid + i * NT;
                if (s < n && c < nv) store4(xr + s * a.lds + 4 * c, v[s][i]);
            }
    if (!a.gain) return;
    float4 u[VPT];
    float ss = 0.0f;
#pragma unroll
    for (int i = 0; i < VPT; i++) {
        u[i] = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int s = 0; s < NS; s++) {
            if (s >= n) continue;
            const float k = a.in[s];
            u[i].x = __fmaf_rn(k, v[s][i].x, u[i].x); u[i].y = __fmaf_rn(k, v[s][i].y, u[i].y);
            u[i].z = __fmaf_rn(k, v[s][i].z, u[i].z); u[i].w = __fmaf_rn(k, v[s][i].w, u[i].w);
        }
        if (tid + i * NT < nv) ss += (u[i].x * u[i].x + u[i].y * u[i].y) + (u[i].z * u[i].z + u[i].w * u[i].w);
    }
    ss = block_sum2<NT>(ss, 0.0f, red).x;
    const float rinv = 1.0f / sqrtf(ss / (float)a.D + a.eps);
    T* hr = (T*)a.h + (long)r * a.ldh;
#pragma unroll
    for (int i = 0; i < VPT; i++) {
        const int c = tid + i * NT;
        if (c < nv) {
            const float4 g = load4(a.gain + 4 * c);
            store4(hr + 4 * c, make_float4((u[i].x * rinv) * g.x, (u[i].y * rinv) * g.y, (u[i].z * rinv) * g.z, (u[i].w * rinv) * g.w));
        }
    }
}

template <class T, int NS> int launch_hyper(const HyperNormArgs& a, int rows, cudaStream_t st) {
    const int nv = (a.D + 3) / 4;
    if (nv <= 128) launch_k(hyper_norm_kernel<T, NS, 128, 1>, dim3(rows), dim3(128), 0, st, a);
    else if (nv <= 256) launch_k(hyper_norm_kernel<T, NS, 256, 1>, dim3(rows), dim3(256), 0, st, a);
    else if (nv <= 512) launch_k(hyper_norm_kernel<T, NS, 256, 2>, dim3(rows), dim3(256), 0, st, a);
    else if (nv <= 1024) launch_k(hyper_norm_kernel<T, NS, 256, 4>, dim3(rows), dim3(256), 0, st, a);
    else if (nv <= 4096) launch_k(hyper_norm_kernel<T, NS, 512, 8>, dim3(rows), dim3(512), 0, st, a);
    else return FLEXLLM_ENOTSUP;
    return launch_status();
}

}  // namespace

template <class T> int hyper_norm(const HyperNormArgs& a, int rows, cudaStream_t st) {
    FLEXLLM_REQUIRE(a.D > 0 && rows >= 0 && a.lds % 4 == 0 && a.lds >= up_to(a.D, 4) && a.n > 0);
    FLEXLLM_REQUIRE((!a.y || (a.mix && a.out && a.ldy % 4 == 0)) && (!a.gain || (a.in && a.h && a.ldh % 4 == 0)));
    if (a.n > kMaxStreams) return FLEXLLM_ENOTSUP;
    if (rows == 0) return FLEXLLM_OK;
    if (a.n == 1) return launch_hyper<T, 1>(a, rows, st);
    if (a.n == 2) return launch_hyper<T, 2>(a, rows, st);
    if (a.n <= 4) return launch_hyper<T, 4>(a, rows, st);
    return launch_hyper<T, 8>(a, rows, st);
}
template int hyper_norm<float>(const HyperNormArgs&, int, cudaStream_t);
template int hyper_norm<bf16>(const HyperNormArgs&, int, cudaStream_t);

template <class T> int res_norm(const ResNormArgs& a, int rows, cudaStream_t st) {
    FLEXLLM_REQUIRE(a.D > 0 && rows >= 0 && a.ldx % 4 == 0 && a.ldx >= up_to(a.D, 4));
    if (rows == 0) return FLEXLLM_OK;
    const int nv = (a.D + 3) / 4;
    if (nv <= 128) launch_k(res_norm_kernel<T, 128, 1>, dim3(rows), dim3(128), 0, st, a);
    else if (nv <= 256) launch_k(res_norm_kernel<T, 256, 1>, dim3(rows), dim3(256), 0, st, a);
    else if (nv <= 512) launch_k(res_norm_kernel<T, 256, 2>, dim3(rows), dim3(256), 0, st, a);
    else if (nv <= 1024) launch_k(res_norm_kernel<T, 256, 4>, dim3(rows), dim3(256), 0, st, a);
    else if (nv <= 4096) launch_k(res_norm_kernel<T, 1024, 4>, dim3(rows), dim3(1024), 0, st, a);
    else return FLEXLLM_ENOTSUP;
    return launch_status();
}
template int res_norm<float>(const ResNormArgs&, int, cudaStream_t);
template int res_norm<bf16>(const ResNormArgs&, int, cudaStream_t);

}  // namespace flexllm

using namespace flexllm;

// See include/flexllm_b200.h.
extern "C" int flexllm_sandwich_norm(int dtype, float* x, long ldx, int M, int D, float eps, const float* y, long ldy, const float* gain_post,
                                     const float* add_vec, const float* gain_pre, void* h, long ldh, void* stream) {
    FLEXLLM_REQUIRE(dtype == FLEXLLM_F32 || dtype == FLEXLLM_BF16);
    FLEXLLM_REQUIRE(x && (!y || (gain_post && ldy % 4 == 0)) && (!gain_pre || (h && ldh % 4 == 0)));
    FLEXLLM_REQUIRE(aligned(x, 16) && aligned(y, 16) && aligned(gain_post, 16) && aligned(add_vec, 16) && aligned(gain_pre, 16) && aligned(h, 16));
    ResNormArgs a = {};
    a.x = x; a.ldx = ldx; a.D = D; a.eps = eps; a.Sc = 1; a.y = y; a.ldy = ldy; a.gain_post = gain_post; a.add_vec = add_vec;
    a.gain_pre = gain_pre; a.h = h; a.ldh = ldh;
    return dtype == FLEXLLM_BF16 ? res_norm<bf16>(a, M, (cudaStream_t)stream) : res_norm<float>(a, M, (cudaStream_t)stream);
}

extern "C" int flexllm_hyper_norm(int dtype, float* x, long lds, int streams, int M, int D, float eps, const float* y, long ldy, const float* mix,
                                  const float* out, const float* in, const float* gain, void* h, long ldh, void* stream) {
    FLEXLLM_REQUIRE(dtype == FLEXLLM_F32 || dtype == FLEXLLM_BF16);
    FLEXLLM_REQUIRE(x && aligned(x, 16) && aligned(y, 16) && aligned(gain, 16) && aligned(h, 16));
    HyperNormArgs a = {};
    a.x = x; a.lds = lds; a.n = streams; a.D = D; a.eps = eps; a.Sc = 1; a.y = y; a.ldy = ldy; a.mix = mix; a.out = out;
    a.in = in; a.gain = gain; a.h = h; a.ldh = ldh;
    return dtype == FLEXLLM_BF16 ? hyper_norm<bf16>(a, M, (cudaStream_t)stream) : hyper_norm<float>(a, M, (cudaStream_t)stream);
}
