// Paged KV cache, all layers: pages of 64 tokens addressed through a page table, V transposed inside the page.
// Two flavours in one object:
//   int8  every layer alike, K [page][hkv][token][64], V [page][hkv][64][token], per-token scales beside them
//   float (elem_bytes 2 = bf16 or 4 = fp32) every layer with its own head count and sizes,
//         K [page][hkv][token][kdim], V [page][hkv][vdim][token], no scales
#pragma once
#include <stddef.h>
#include <stdint.h>

#include <vector>

#include "../../include/flexllm_b200.h"

struct flexllm_kv_cache {
    int layers, n_pages, hkv, page;
    int8_t* k; float* ks; int8_t* v; float* vs;   // [layers][...]
    size_t page_bytes, scale_bytes;               // per layer (int8)
    int elem_bytes;                               // 1: int8 with scales; 2 / 4: floating point
    size_t k_bytes, v_bytes;                      // whole pools (floating point)
    std::vector<flexllm_kv_shape> shape;          // per layer (floating point) ...
    std::vector<size_t> k_off, v_off;             // ... and byte offsets of its pools
};
