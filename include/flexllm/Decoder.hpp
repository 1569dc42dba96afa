// Decoder family with floating-point weights (the Pibidra and Sabisun designs) on the common model runner: create, load, then the same
// prefill / decode / generate calls as every model, plus steps of any length with logits at chosen places.
#pragma once
#include "common.hpp"
namespace flexllm {
class DecoderModel {
  public:
    DecoderModel() = default;
    DecoderModel(const DecoderModel&) = delete;
    DecoderModel& operator=(const DecoderModel&) = delete;
    ~DecoderModel() { flexllm_model_destroy(h_); }
    int create(const flexllm_decoder_config& cfg) { return flexllm_model_create_decoder(&h_, &cfg); }
    int load_safetensors(const char* path, stream_t st = nullptr) { return flexllm_model_load_safetensors(h_, path, st); }
    int load_tensor(const char* name, int ndim, const int64_t* shape, const void* bf16_data, stream_t st = nullptr) {
        return flexllm_model_load_tensor(h_, name, FLEXLLM_BF16, ndim, shape, bf16_data, st);
    }
    int reset(stream_t st = nullptr) { return flexllm_model_reset(h_, st); }
    // the next n tokens of each of B sequences (host buffers)
    int step(const int32_t* tokens, int B, int n, const int32_t* want, int n_want, float* logits, int32_t* next = nullptr,
             stream_t st = nullptr) {
        return flexllm_model_extend_host(h_, tokens, B, n, want, n_want, logits, next, st);
    }
    int generate(const int32_t* tokens_host, int B, int S, int n_new, int32_t* out_host, bool use_graph = true, stream_t st = nullptr) {
        return flexllm_model_generate_host(h_, tokens_host, B, S, n_new, out_host, use_graph ? 1 : 0, st);
    }
    flexllm_model* handle() const { return h_; }

  private:
    flexllm_model* h_ = nullptr;
};
}  // namespace flexllm
