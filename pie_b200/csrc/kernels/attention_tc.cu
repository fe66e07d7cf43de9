// Paged prefill attention on tcgen05: launchers of the kernel in attention_tc.cuh.
#include "attention_tc.cuh"

using namespace pie;

// 1 when the tensor-core kernel covers the shape (head_dim 64 or 128, 16-token pages, group size dividing 128).
PIE_API int pie_prefill_attn_tc_supported(int hq, int hkv, int head_dim, int page_size) {
    if (hkv <= 0 || hq % hkv) return 0;
    const int g = hq / hkv;
    return (head_dim == 128 || head_dim == 64) && page_size == 16 && (g == 1 || g == 2 || g == 4 || g == 8 || g == 16) ? 1 : 0;
}

PIE_API int pie_paged_prefill_attn_tc_kept(const void*, const void*, const int*, const int*, const int*, const int*, const int*, const int*,
                                           int, const uint32_t*, const long*, void*, float*, int, int, int, int, int, float, int, int,
                                           const float*, int*, float, int, cudaStream_t);

// Same contract as pie_paged_prefill_attn, with tiles of tile_rows / group query tokens (tile_rows = 128 or
// 256: one or two MMA tiles per CTA) and `total_pages` = pages of kv_layer including the pad page (last).
// softcap > 0 (tile_rows 256 only): softmax over softcap * tanh(q.k * sm_scale / softcap).
PIE_API int pie_paged_prefill_attn_tc_softcap(const void* q, const void* kv_layer, const int* page_indices,
                                              const int* kv_page_indptr, const int* qo_indptr, const int* kv_lens,
                                              const int* tile_req, const int* tile_qstart, int num_tiles,
                                              const uint32_t* mask_bits, const long* mask_word_indptr, void* out,
                                              float* lse_out, int n_tokens, int hq, int hkv, int head_dim, int total_pages,
                                              float sm_scale, int window_left, int tile_rows, const float* sinks_log2,
                                              int* status, float softcap, cudaStream_t st) {
    return pie_paged_prefill_attn_tc_kept(q, kv_layer, page_indices, kv_page_indptr, qo_indptr, kv_lens, tile_req, tile_qstart,
                                          num_tiles, mask_bits, mask_word_indptr, out, lse_out, n_tokens, hq, hkv, head_dim,
                                          total_pages, sm_scale, window_left, tile_rows, sinks_log2, status, softcap, 0, st);
}

// The same with the first `keep_first` keys visible beside the window.
PIE_API int pie_paged_prefill_attn_tc_kept(const void* q, const void* kv_layer, const int* page_indices,
                                           const int* kv_page_indptr, const int* qo_indptr, const int* kv_lens,
                                           const int* tile_req, const int* tile_qstart, int num_tiles,
                                           const uint32_t* mask_bits, const long* mask_word_indptr, void* out,
                                           float* lse_out, int n_tokens, int hq, int hkv, int head_dim, int total_pages,
                                           float sm_scale, int window_left, int tile_rows, const float* sinks_log2,
                                           int* status, float softcap, int keep_first, cudaStream_t st) {
    if (num_tiles <= 0) return 0;
    if (keep_first < 0) return (int)cudaErrorInvalidValue;
    const int D_ = head_dim;
    if (!pie_prefill_attn_tc_supported(hq, hkv, head_dim, 16) || (tile_rows != 128 && tile_rows != 256) || !status)
        return (int)cudaErrorInvalidValue;
    if (softcap > 0.f && tile_rows != 256) return (int)cudaErrorInvalidValue;
    EncodeTiledFnA enc = at_encoder();
    if (!enc) return (int)cudaErrorNotSupported;
    const int G = hq / hkv;
    CUtensorMap tq, tkv;
    {
        cuuint64_t dims[3] = {(cuuint64_t)D_, (cuuint64_t)hq, (cuuint64_t)n_tokens};
        cuuint64_t strides[2] = {(cuuint64_t)D_ * 2, (cuuint64_t)hq * D_ * 2};
        cuuint32_t box[3] = {64, (cuuint32_t)G, (cuuint32_t)(AT_ROWS / G)};
        cuuint32_t estr[3] = {1, 1, 1};
        if (enc(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(q), dims, strides, box, estr,
                CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
            return (int)cudaErrorInvalidValue;
    }
    {
        cuuint64_t dims[2] = {(cuuint64_t)D_, (cuuint64_t)total_pages * 2 * hkv * 16};
        cuuint64_t strides[1] = {(cuuint64_t)D_ * 2};
        cuuint32_t box[2] = {64, 16};
        cuuint32_t estr[2] = {1, 1};
        if (enc(&tkv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(kv_layer), dims, strides, box, estr,
                CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B,
                CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
            return (int)cudaErrorInvalidValue;
    }
    const float scale_log2 = sm_scale * 1.4426950408889634f;
    dim3 grid(num_tiles, hkv);
    const float cap_pre = softcap > 0.f ? sm_scale / softcap : 0.f, cap_post = softcap > 0.f ? softcap / sm_scale : 0.f;
#define GO4(G_, NT_, D__, CAP_)                                                                                       \
    {                                                                                                                 \
        auto kern = paged_prefill_attn_tc_kernel<G_, NT_, D__, CAP_>;                                                 \
        using Cfg = AtCfg<NT_, D__>;                                                                                  \
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Cfg::SMEM);      \
        if (e != cudaSuccess) return (int)e;                                                                          \
        kern<<<grid, Cfg::THREADS, Cfg::SMEM, st>>>(                                                                  \
            tq, tkv, tkv, TcMeans(), 2, page_indices, kv_page_indptr, qo_indptr, kv_lens, tile_req, tile_qstart, mask_bits,              \
            mask_word_indptr, (bf16*)out, lse_out, sinks_log2, hq, hkv, total_pages - 1, scale_log2, window_left,     \
            status, cap_pre, cap_post, hq * D_, D_, nullptr, 0, 0, keep_first);                                                                 \
        return (int)cudaGetLastError();                                                                               \
    }
#define GO2(G_, NT_)           \
    if (D_ == 128) GO4(G_, NT_, 128, false) else GO4(G_, NT_, 64, false)
#define GO(G_)                 \
    if (softcap > 0.f) { if (D_ == 128) GO4(G_, 2, 128, true) else GO4(G_, 2, 64, true) } \
    else if (tile_rows == 128) GO2(G_, 1) else GO2(G_, 2)
    switch (G) {
        case 1: GO(1)
        case 2: GO(2)
        case 4: GO(4)
        case 8: GO(8)
        case 16: GO(16)
    }
#undef GO
#undef GO2
#undef GO4
    return (int)cudaErrorInvalidValue;
}

PIE_API int pie_paged_prefill_attn_tc(const void* q, const void* kv_layer, const int* page_indices,
                                      const int* kv_page_indptr, const int* qo_indptr, const int* kv_lens,
                                      const int* tile_req, const int* tile_qstart, int num_tiles,
                                      const uint32_t* mask_bits, const long* mask_word_indptr, void* out,
                                      float* lse_out, int n_tokens, int hq, int hkv, int head_dim, int total_pages,
                                      float sm_scale,
                                      int window_left, int tile_rows, const float* sinks_log2, int* status,
                                      cudaStream_t st) {
    return pie_paged_prefill_attn_tc_softcap(q, kv_layer, page_indices, kv_page_indptr, qo_indptr, kv_lens, tile_req,
                                             tile_qstart, num_tiles, mask_bits, mask_word_indptr, out, lse_out, n_tokens,
                                             hq, hkv, head_dim, total_pages, sm_scale, window_left, tile_rows, sinks_log2,
                                             status, 0.f, st);
}


// Prefill attention over keys and values that were projected from latents for this pass: kv [total_tokens][heads][2][D],
// "page" p of page_indices = tokens 16 p .. 16 p + 15 (page ids from total_tokens / 16 on read zeros). q [n_tokens][heads][D]
// with zeros past the query's width; out row of a token at out_ld elements, vdim (a multiple of 8) per head. Tiles of 256.
PIE_API int pie_projected_prefill_attn_tc(const void* q, const void* kv, const int* page_indices, const int* kv_page_indptr,
                                          const int* qo_indptr, const int* kv_lens, const int* tile_req, const int* tile_qstart,
                                          int num_tiles, const uint32_t* mask_bits, const long* mask_word_indptr, void* out,
                                          int n_tokens, int heads, int head_dim, int total_tokens, int vdim, int out_ld,
                                          float sm_scale, int window_left, int* status, cudaStream_t st) {
    if (num_tiles <= 0) return 0;
    const int D_ = head_dim;
    if ((D_ != 64 && D_ != 128) || vdim > D_ || vdim % 8 || out_ld % 8 || total_tokens % 16 || !status) return (int)cudaErrorInvalidValue;
    EncodeTiledFnA enc = at_encoder();
    if (!enc) return (int)cudaErrorNotSupported;
    CUtensorMap tq, tkv;
    cuuint32_t estr[3] = {1, 1, 1};
    cuuint64_t qd[3] = {(cuuint64_t)D_, (cuuint64_t)heads, (cuuint64_t)n_tokens};
    cuuint64_t qs[2] = {(cuuint64_t)D_ * 2, (cuuint64_t)heads * D_ * 2};
    cuuint32_t qb[3] = {64, 1, (cuuint32_t)AT_ROWS};
    cuuint64_t kd[3] = {(cuuint64_t)D_, (cuuint64_t)heads * 2, (cuuint64_t)total_tokens};
    cuuint64_t ks[2] = {(cuuint64_t)D_ * 2, (cuuint64_t)heads * 2 * D_ * 2};
    cuuint32_t kb[3] = {64, 1, 16};
    if (enc(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(q), qd, qs, qb, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS ||
        enc(&tkv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(kv), kd, ks, kb, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
        return (int)cudaErrorInvalidValue;
    const float scale_log2 = sm_scale * 1.4426950408889634f;
    const dim3 grid(num_tiles, heads);
#define GO(D__)                                                                                                       \
    {                                                                                                                 \
        auto kern = paged_prefill_attn_tc_kernel<1, 2, D__, false, true>;                                             \
        using Cfg = AtCfg<2, D__>;                                                                                    \
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Cfg::SMEM);      \
        if (e != cudaSuccess) return (int)e;                                                                          \
        kern<<<grid, Cfg::THREADS, Cfg::SMEM, st>>>(tq, tkv, tkv, TcMeans(), 2, page_indices, kv_page_indptr, qo_indptr, kv_lens, tile_req,  \
                                                    tile_qstart, mask_bits, mask_word_indptr, (bf16*)out, nullptr,    \
                                                    nullptr, heads, heads, total_tokens / 16, scale_log2, window_left, status,  \
                                                    0.f, 0.f, out_ld, vdim, nullptr, 0, 0, 0);                                         \
        return (int)cudaGetLastError();                                                                               \
    }
    if (D_ == 128) GO(128) else GO(64)
#undef GO
}
