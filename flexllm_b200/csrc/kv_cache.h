// Paged KV cache, all layers: pages of 64 tokens addressed through a page table, V transposed inside the page.
// Two flavours in one object:
//   int8  every layer alike, K [page][hkv][token][64], V [page][hkv][64][token], per-token scales beside them
//   float (elem_bytes 2 = bf16 or 4 = fp32) every layer with its own head count and sizes,
//         K [page][hkv][token][kdim], V [page][hkv][vdim][token], no scales
// The floating-point flavour may also hold states of fixed size (recurrent mixers): per state layer one slot per sequence,
// [state layer][slot][bytes]. A sequence that starts over ignores what its slot holds.
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
    uint8_t* states; size_t states_bytes;         // all states ...
    std::vector<size_t> s_off, s_slot;            // ... byte offset and slot size per state layer
};

namespace flexllm {
// Adds states to a cache that has none: slot_bytes[i] per sequence for state layer i, zeroed.
int kv_cache_add_states(flexllm_kv_cache* c, int slots, const std::vector<size_t>& slot_bytes);
}
