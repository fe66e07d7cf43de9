// Paged attention over inferlet-owned page tables: launchers of the mma.sync kernels in attention_mma.cuh.
#include "attention_mma.cuh"

using namespace pie;

extern "C" int* pie_status_word_current();      // elementwise.cu

// Merge pass of split-KV decode on its own (used by the fp8-KV decode kernel of attention_kv8.cu).
PIE_API int pie_decode_merge(const float* o_part, const float* lse_part, const int* req_item_indptr, void* out,
                             int num_reqs, int hq, int hkv, int head_dim, const float* sinks_log2, int max_items,
                             cudaStream_t st) {
    if (num_reqs <= 0) return 0;
    dim3 grid(num_reqs, hq);
    const int group = hq / hkv;
    if (head_dim == 128)
        launch_pdl(paged_decode_merge_kernel<128>, grid, dim3(128), 0, st, o_part, lse_part, req_item_indptr,
                   (bf16*)out, hq, hkv, group, sinks_log2, max_items);
    else if (head_dim == 256)
        launch_pdl(paged_decode_merge_kernel<256>, grid, dim3(256), 0, st, o_part, lse_part, req_item_indptr,
                   (bf16*)out, hq, hkv, group, sinks_log2, max_items);
    else if (head_dim == 64)
        launch_pdl(paged_decode_merge_kernel<64>, grid, dim3(64), 0, st, o_part, lse_part, req_item_indptr,
                   (bf16*)out, hq, hkv, group, sinks_log2, max_items);
    else
        return (int)cudaErrorInvalidValue;
    return (int)cudaGetLastError();
}

// Scratch sizes (in floats) a caller must provide for `max_items` work items.
PIE_API long pie_decode_attn_scratch_floats(int max_items, int hq, int head_dim) {
    return (long)max_items * hq * head_dim + (long)max_items * hq;
}

static int launch_decode(const void* q, const void* kv_layer, const int* page_indices,
                         const int* kv_page_indptr, const int* item_req, const int* item_start,
                         const int* item_end, const int* req_item_indptr, const int* num_items_ptr,
                         void* out, float* scratch, int max_items, int num_reqs, int hq, int hkv,
                         int head_dim, int page_size, float sm_scale, int num_ctas, int run_merge,
                         int window_left, const float* sinks_log2, const int* item_slot,
                         const int* item_tile, const int* tile_members, cudaStream_t st, float softcap = 0.f,
                         int keep_first = 0) {
    if (num_reqs <= 0) return 0;
    if (hkv <= 0 || hq % hkv || page_size % 16) return (int)cudaErrorInvalidValue;
    if (keep_first < 0) return (int)cudaErrorInvalidValue;
    const bool cascade = item_tile != nullptr;
    if (cascade && (!item_slot || !tile_members || window_left >= 0 || softcap > 0.f)) return (int)cudaErrorInvalidValue;
    const int group = hq / hkv;
    float* o_part = scratch;
    float* lse_part = scratch + (size_t)max_items * hq * head_dim;
    const float scale_log2 = softcap > 0.f ? sm_scale / softcap : sm_scale * 1.4426950408889634f;
    const float cap_log2 = softcap * 1.4426950408889634f;
    DISPATCH_DG(head_dim, group, {
        constexpr int SM = decode_smem_bytes<D>();
        if (softcap > 0.f) {
            auto kern = paged_decode_attn_kernel<D, G, false, MODE_CAP>;
            cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM);
            launch_pdl(kern, dim3(num_ctas), dim3(DEC_WARPS * 32), SM, st,
                (const bf16*)q, (const bf16*)kv_layer, page_indices, kv_page_indptr, item_req,
                item_start, item_end, req_item_indptr, num_items_ptr, (bf16*)out, o_part, lse_part, hq,
                hkv, page_size, scale_log2, window_left, sinks_log2, max_items, num_reqs, pie_status_word_current(),
                (const int*)nullptr, (const int*)nullptr, (const int*)nullptr, cap_log2, (const float*)nullptr, 0, keep_first, KeyLayout());
        } else if (cascade) {
            auto kern = paged_decode_attn_kernel<D, G, true>;
            cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM);
            launch_pdl(kern, dim3(num_ctas), dim3(DEC_WARPS * 32), SM, st,
                (const bf16*)q, (const bf16*)kv_layer, page_indices, kv_page_indptr, item_req,
                item_start, item_end, req_item_indptr, num_items_ptr, (bf16*)out, o_part, lse_part, hq,
                hkv, page_size, scale_log2, window_left, sinks_log2, max_items, num_reqs, pie_status_word_current(),
                item_slot, item_tile, tile_members, 0.f, (const float*)nullptr, 0, 0, KeyLayout());
        } else {
            auto kern = paged_decode_attn_kernel<D, G, false>;
            cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM);
            launch_pdl(kern, dim3(num_ctas), dim3(DEC_WARPS * 32), SM, st,
                (const bf16*)q, (const bf16*)kv_layer, page_indices, kv_page_indptr, item_req,
                item_start, item_end, req_item_indptr, num_items_ptr, (bf16*)out, o_part, lse_part, hq,
                hkv, page_size, scale_log2, window_left, sinks_log2, max_items, num_reqs, pie_status_word_current(),
                (const int*)nullptr, (const int*)nullptr, (const int*)nullptr, 0.f, (const float*)nullptr, 0, keep_first, KeyLayout());
        }
    });
    int err = (int)cudaGetLastError();
    if (err || !run_merge) return err;
    dim3 grid(num_reqs, hq);
    if (head_dim == 128)
        launch_pdl(paged_decode_merge_kernel<128>, grid, dim3(128), 0, st, (const float*)o_part,
                   (const float*)lse_part, req_item_indptr, (bf16*)out, hq, hkv, group, sinks_log2, max_items);
    else if (head_dim == 256)
        launch_pdl(paged_decode_merge_kernel<256>, grid, dim3(256), 0, st, (const float*)o_part,
                   (const float*)lse_part, req_item_indptr, (bf16*)out, hq, hkv, group, sinks_log2, max_items);
    else
        launch_pdl(paged_decode_merge_kernel<64>, grid, dim3(64), 0, st, (const float*)o_part,
                   (const float*)lse_part, req_item_indptr, (bf16*)out, hq, hkv, group, sinks_log2, max_items);
    return (int)cudaGetLastError();
}

// window_left >= 0: each request's single query token sees only the last window_left + 1 keys; the
// caller's items then start at the 16-token boundary at or below the first visible key (items that
// start lower are masked). sinks_log2 (optional, [hq], logit * log2(e)): per-head attention sinks.
PIE_API int pie_paged_decode_attn_window(const void* q, const void* kv_layer, const int* page_indices,
                                         const int* kv_page_indptr, const int* item_req,
                                         const int* item_start, const int* item_end,
                                         const int* req_item_indptr, const int* num_items_ptr,
                                         void* out, float* scratch, int max_items, int num_reqs, int hq,
                                         int hkv, int head_dim, int page_size, float sm_scale,
                                         int num_ctas, int run_merge, int window_left,
                                         const float* sinks_log2, cudaStream_t st) {
    return launch_decode(q, kv_layer, page_indices, kv_page_indptr, item_req, item_start, item_end, req_item_indptr,
                         num_items_ptr, out, scratch, max_items, num_reqs, hq, hkv, head_dim, page_size, sm_scale,
                         num_ctas, run_merge, window_left, sinks_log2, nullptr, nullptr, nullptr, st);
}

// The same with soft-capped scores (softcap > 0): softmax over softcap * tanh(q.k * sm_scale / softcap).
PIE_API int pie_paged_decode_attn_softcap(const void* q, const void* kv_layer, const int* page_indices,
                                          const int* kv_page_indptr, const int* item_req,
                                          const int* item_start, const int* item_end,
                                          const int* req_item_indptr, const int* num_items_ptr,
                                          void* out, float* scratch, int max_items, int num_reqs, int hq,
                                          int hkv, int head_dim, int page_size, float sm_scale,
                                          int num_ctas, int run_merge, int window_left,
                                          const float* sinks_log2, float softcap, cudaStream_t st) {
    return launch_decode(q, kv_layer, page_indices, kv_page_indptr, item_req, item_start, item_end, req_item_indptr,
                         num_items_ptr, out, scratch, max_items, num_reqs, hq, hkv, head_dim, page_size, sm_scale,
                         num_ctas, run_merge, window_left, sinks_log2, nullptr, nullptr, nullptr, st, softcap);
}

// The window form with the first `keep_first` keys visible beside the window; the items must cover them.
PIE_API int pie_paged_decode_attn_kept(const void* q, const void* kv_layer, const int* page_indices,
                                       const int* kv_page_indptr, const int* item_req,
                                       const int* item_start, const int* item_end,
                                       const int* req_item_indptr, const int* num_items_ptr,
                                       void* out, float* scratch, int max_items, int num_reqs, int hq,
                                       int hkv, int head_dim, int page_size, float sm_scale,
                                       int num_ctas, int window_left, int keep_first,
                                       const float* sinks_log2, cudaStream_t st) {
    return launch_decode(q, kv_layer, page_indices, kv_page_indptr, item_req, item_start, item_end, req_item_indptr,
                         num_items_ptr, out, scratch, max_items, num_reqs, hq, hkv, head_dim, page_size, sm_scale,
                         num_ctas, 1, window_left, sinks_log2, nullptr, nullptr, nullptr, st, 0.f, keep_first);
}

// Decode attention over a plan with shared-prefix items (see the kernel): requests that were forked
// from one context read their common pages once. item_req of a shared item names the member whose
// page table addresses the range. req_item_indptr counts partial-result slots, all below max_items.
PIE_API int pie_paged_decode_attn_cascade(const void* q, const void* kv_layer, const int* page_indices,
                                          const int* kv_page_indptr, const int* item_req,
                                          const int* item_start, const int* item_end,
                                          const int* req_item_indptr, const int* num_items_ptr,
                                          void* out, float* scratch, int max_items, int num_reqs, int hq,
                                          int hkv, int head_dim, int page_size, float sm_scale,
                                          int num_ctas, const float* sinks_log2, const int* item_slot,
                                          const int* item_tile, const int* tile_members, cudaStream_t st) {
    if (!item_tile) return (int)cudaErrorInvalidValue;
    return launch_decode(q, kv_layer, page_indices, kv_page_indptr, item_req, item_start, item_end, req_item_indptr,
                         num_items_ptr, out, scratch, max_items, num_reqs, hq, hkv, head_dim, page_size, sm_scale,
                         num_ctas, 1, -1, sinks_log2, item_slot, item_tile, tile_members, st);
}

PIE_API int pie_paged_decode_attn(const void* q, const void* kv_layer, const int* page_indices,
                                  const int* kv_page_indptr, const int* item_req,
                                  const int* item_start, const int* item_end,
                                  const int* req_item_indptr, const int* num_items_ptr,
                                  void* out, float* scratch, int max_items, int num_reqs, int hq,
                                  int hkv, int head_dim, int page_size, float sm_scale,
                                  int num_ctas, int run_merge, cudaStream_t st) {
    return pie_paged_decode_attn_window(q, kv_layer, page_indices, kv_page_indptr, item_req, item_start, item_end,
                                        req_item_indptr, num_items_ptr, out, scratch, max_items, num_reqs, hq, hkv,
                                        head_dim, page_size, sm_scale, num_ctas, run_merge, -1, nullptr, st);
}

PIE_API int pie_paged_prefill_attn_kept(const void*, const void*, const int*, const int*, const int*, const int*, const int*, const int*, int,
                                        const uint32_t*, const long*, void*, float*, int, int, int, int, float, int, const float*, float,
                                        int, cudaStream_t);

// softcap > 0: softmax over softcap * tanh(q.k * sm_scale / softcap) (Gemma-2).
PIE_API int pie_paged_prefill_attn_softcap(const void* q, const void* kv_layer, const int* page_indices,
                                           const int* kv_page_indptr, const int* qo_indptr,
                                           const int* kv_lens, const int* tile_req, const int* tile_qstart,
                                           int num_tiles, const uint32_t* mask_bits,
                                           const long* mask_word_indptr, void* out, float* lse_out, int hq,
                                           int hkv, int head_dim, int page_size, float sm_scale,
                                           int window_left, const float* sinks_log2, float softcap,
                                           cudaStream_t st) {
    return pie_paged_prefill_attn_kept(q, kv_layer, page_indices, kv_page_indptr, qo_indptr, kv_lens, tile_req, tile_qstart,
                                       num_tiles, mask_bits, mask_word_indptr, out, lse_out, hq, hkv, head_dim, page_size,
                                       sm_scale, window_left, sinks_log2, softcap, 0, st);
}

// The same with the first `keep_first` keys visible beside the window.
PIE_API int pie_paged_prefill_attn_kept(const void* q, const void* kv_layer, const int* page_indices,
                                        const int* kv_page_indptr, const int* qo_indptr,
                                        const int* kv_lens, const int* tile_req, const int* tile_qstart,
                                        int num_tiles, const uint32_t* mask_bits,
                                        const long* mask_word_indptr, void* out, float* lse_out, int hq,
                                        int hkv, int head_dim, int page_size, float sm_scale,
                                        int window_left, const float* sinks_log2, float softcap, int keep_first,
                                        cudaStream_t st) {
    if (num_tiles <= 0) return 0;
    if (keep_first < 0) return (int)cudaErrorInvalidValue;
    if (hkv <= 0 || hq % hkv || page_size % 16) return (int)cudaErrorInvalidValue;
    const int group = hq / hkv;
    const float scale_log2 = softcap > 0.f ? sm_scale / softcap : sm_scale * 1.4426950408889634f;
    const float cap_log2 = softcap * 1.4426950408889634f;
    dim3 grid(num_tiles, hkv);
    DISPATCH_DG(head_dim, group, {
        constexpr int SM = prefill_smem_bytes<D>();
        if (softcap > 0.f) {
            auto kern = paged_prefill_attn_kernel<D, G, MODE_CAP>;
            cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM);
            kern<<<grid, PF_WARPS * 32, SM, st>>>(
                (const bf16*)q, (const bf16*)kv_layer, page_indices, kv_page_indptr, qo_indptr, kv_lens,
                tile_req, tile_qstart, mask_bits, mask_word_indptr, (bf16*)out, lse_out, sinks_log2, hq, hkv,
                page_size, scale_log2, window_left, cap_log2, nullptr, 0, keep_first, KeyLayout());
        } else {
            auto kern = paged_prefill_attn_kernel<D, G>;
            cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM);
            kern<<<grid, PF_WARPS * 32, SM, st>>>(
                (const bf16*)q, (const bf16*)kv_layer, page_indices, kv_page_indptr, qo_indptr, kv_lens,
                tile_req, tile_qstart, mask_bits, mask_word_indptr, (bf16*)out, lse_out, sinks_log2, hq, hkv,
                page_size, scale_log2, window_left, 0.f, nullptr, 0, keep_first, KeyLayout());
        }
    });
    return (int)cudaGetLastError();
}

PIE_API int pie_paged_prefill_attn(const void* q, const void* kv_layer, const int* page_indices,
                                   const int* kv_page_indptr, const int* qo_indptr,
                                   const int* kv_lens, const int* tile_req, const int* tile_qstart,
                                   int num_tiles, const uint32_t* mask_bits,
                                   const long* mask_word_indptr, void* out, float* lse_out, int hq,
                                   int hkv, int head_dim, int page_size, float sm_scale,
                                   int window_left, const float* sinks_log2, cudaStream_t st) {
    return pie_paged_prefill_attn_softcap(q, kv_layer, page_indices, kv_page_indptr, qo_indptr, kv_lens, tile_req,
                                          tile_qstart, num_tiles, mask_bits, mask_word_indptr, out, lse_out, hq, hkv,
                                          head_dim, page_size, sm_scale, window_left, sinks_log2, 0.f, st);
}

// Query tokens covered by one prefill tile for a given GQA group size.
PIE_API int pie_prefill_tile_tokens(int group) { return PF_ROWS / group; }

// ------------------------------------------------- allocation-free variant
// See pie_noalloc.h: split-KV decode attention whose scratch lives in this
// library instead of being passed in, for callers that cannot allocate.
#include <stdio.h>
#include <mutex>
#include "pie_noalloc.h"

// Split-KV partial outputs and log-sum-exps of the allocation-free entry point.
// Host code must not use this name as an address: it is a host-side stand-in;
// the device address comes from cudaGetSymbolAddress below.
static __device__ __align__(256) float pie_noalloc_scratch[PIE_NOALLOC_SCRATCH_FLOATS];

namespace {
constexpr int kMaxDevices = 64;
float* g_noalloc_ptr[kMaxDevices] = {};
std::mutex g_noalloc_mutex;

// Device address of the scratch array on the current device (looked up once per device).
int noalloc_scratch_for_current_device(float** out) {
    int dev = -1;
    cudaError_t e = cudaGetDevice(&dev);
    if (e != cudaSuccess) return (int)e;
    if (dev < 0 || dev >= kMaxDevices) return PIE_NOALLOC_ERR_SETUP;
    std::lock_guard<std::mutex> lock(g_noalloc_mutex);
    if (!g_noalloc_ptr[dev]) {
        float* p = nullptr;
        e = cudaGetSymbolAddress((void**)&p, pie_noalloc_scratch);
        if (e != cudaSuccess) return (int)e;
        if (!p) return PIE_NOALLOC_ERR_SETUP;
        g_noalloc_ptr[dev] = p;
    }
    *out = g_noalloc_ptr[dev];
    return 0;
}
}  // namespace

PIE_API int pie_paged_decode_attn_noalloc(const void* q, const void* kv_layer,
                                          const int* page_indices, const int* kv_page_indptr,
                                          const int* item_req, const int* item_start,
                                          const int* item_end, const int* req_item_indptr,
                                          const int* num_items_ptr, void* out, int max_items,
                                          int num_reqs, int hq, int hkv, int head_dim,
                                          int page_size, float sm_scale, int num_ctas,
                                          cudaStream_t stream) {
    if (max_items < 0 || hq <= 0 || head_dim <= 0) return (int)cudaErrorInvalidValue;
    const long need = pie_decode_attn_scratch_floats(max_items, hq, head_dim);
    if (need > (long)PIE_NOALLOC_SCRATCH_FLOATS) {
        fprintf(stderr,
                "pie_paged_decode_attn_noalloc: max_items=%d, hq=%d, head_dim=%d need %ld floats of "
                "scratch; the built-in array holds %u. Use fewer work items or pie_paged_decode_attn "
                "with your own buffer.\n",
                max_items, hq, head_dim, need, (unsigned)PIE_NOALLOC_SCRATCH_FLOATS);
        return PIE_NOALLOC_ERR_TOO_LARGE;
    }
    float* scratch = nullptr;
    const int rc = noalloc_scratch_for_current_device(&scratch);
    if (rc != 0) return rc;
    return pie_paged_decode_attn(q, kv_layer, page_indices, kv_page_indptr, item_req, item_start,
                                 item_end, req_item_indptr, num_items_ptr, out, scratch, max_items,
                                 num_reqs, hq, hkv, head_dim, page_size, sm_scale, num_ctas, 1, stream);
}
