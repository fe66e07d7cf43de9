// Arguments shared by the latent-attention kernels (mma.sync and tcgen05).
#pragma once
#include "common.cuh"

namespace pie {

struct LatentMmaArgs {
    const void* q;                 // [n, heads, row]
    const void* cache;             // [pages, page_size, cache_row]
    const int* page_indices;
    const int* kv_page_indptr;
    const int* item_req;           // request of an item
    const int* item_start;         // decode: first key; prefill: first query token (within the request)
    const int* item_end;           // decode: one past the last key; null: prefill
    const int* req_item_indptr;    // decode: items of a request
    const int* cta_items;          // decode: CTA b runs items [cta_items[b], cta_items[b + 1])
    const int* qo_indptr;
    const int* kv_lens;
    const uint32_t* mask_bits;     // prefill: custom mask words, or null
    const long* mask_word_indptr;
    void* out;                     // [n, heads, rank_pad]
    float* scratch;                // decode: [max_items, heads, rank_pad] partial outputs, then [max_items, heads] log2 sums
    int items, max_items, heads, row, rank_pad, cache_row, page_size, window_left, stages, reqs;
    int page_shift;                // log2(page_size)
    int cache_rows;                // rows of `cache` in all
    float scale_log2;
};

}  // namespace pie
