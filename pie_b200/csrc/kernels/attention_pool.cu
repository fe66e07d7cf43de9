// Attention over keys that a layer lays out in its own way: pages that hold keys only, the values being the keys, or pages with
// means of key and value blocks beside them, which a query sees ahead of its sliding window. Launchers of the kernels in
// attention_mma.cuh and attention_tc.cuh, and the passes around the means:
//
//   pie_pool_rows      means of the blocks that a fire's tokens complete, into the pages
//   pie_pool_gather    a fire's means in 16-row pages, for prefill
//   pie_laid_decode    split-KV decode
//   pie_laid_prefill   prompts on tcgen05, or mma.sync for other shapes
#include "attention_mma.cuh"
#include "attention_tc.cuh"
#include "typed.cuh"

namespace pie {

struct PoolArgs {
    const void* cache;              // this layer's pages [pages][2][hkv][page][D]
    void* means;                    // [pages][2][hkv][per_page][D]
    const int *page_indices, *kv_page_indptr, *kv_lens, *qo_indptr, *tok_req, *slots;
    void* gathered;                 // gather: [total][2][hkv][16][D], the last page zeros
    const int *first, *seen;        // gather: first page and means of every request
    const int* page_req;            // gather: request of every page
    int n, hkv, D, page_size, pool, per_page, total;
};

// One block per token; it works where the token ends a block of `pool` tokens.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) pool_rows_kernel(const PoolArgs a) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    if (a.slots[t] < 0) return;
    const int r = a.tok_req[t], pos = a.kv_lens[r] - a.qo_indptr[r + 1] + t;
    if ((pos + 1) % a.pool) return;
    const int* pages = a.page_indices + a.kv_page_indptr[r];
    int page_at;
    const int row = mean_row(pos / a.pool, a.pool, a.page_size, page_at);
    const T* cache = static_cast<const T*>(a.cache);
    T* dst = static_cast<T*>(a.means) + (size_t)pages[page_at] * 2 * a.hkv * a.per_page * a.D;
    const int vecs = 2 * a.hkv * (a.D / VEC);
    for (int i = threadIdx.x; i < vecs; i += 256) {
        const int head = i / (a.D / VEC), d = (i - head * (a.D / VEC)) * VEC;       // head: keys, then values
        float s[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) s[e] = 0.f;
        for (int j0 = pos + 1 - a.pool; j0 <= pos; j0 += 8) {
            float f[8][VEC];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int j = min(j0 + u, pos);
                load_vec<VEC>(cache + (((size_t)pages[j / a.page_size] * 2 * a.hkv + head) * a.page_size + j % a.page_size) * a.D + d, f[u]);
            }
#pragma unroll
            for (int u = 0; u < 8; ++u)
#pragma unroll
                for (int e = 0; e < VEC; ++e) s[e] += j0 + u <= pos ? f[u][e] : 0.f;
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) s[e] /= (float)a.pool;
        store_vec<VEC>(dst + ((size_t)head * a.per_page + row) * a.D + d, s);
    }
}

// One block per page of sixteen means and head (keys, then values); rows past a request's last are zeros, and so is the last page.
__global__ void __launch_bounds__(128) pool_gather_kernel(const PoolArgs a) {
    const int p = blockIdx.x, head = blockIdx.y, r = p < a.total - 1 ? a.page_req[p] : -1, ch = a.D / 8;
    const int b0 = r >= 0 ? (p - a.first[r]) * 16 : 0, seen = r >= 0 ? a.seen[r] : 0;
    const int* pages = r >= 0 ? a.page_indices + a.kv_page_indptr[r] : nullptr;
    const bf16* means = static_cast<const bf16*>(a.means);
    uint4* dst = static_cast<uint4*>(a.gathered) + ((size_t)p * 2 * a.hkv + head) * 16 * ch;
    for (int i = threadIdx.x; i < 16 * ch; i += 128) {
        const int row = i / ch, c = i % ch, b = b0 + row;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (b < seen) {
            int page_at;
            const int m = mean_row(b, a.pool, a.page_size, page_at);
            v = *reinterpret_cast<const uint4*>(means + (((size_t)pages[page_at] * 2 * a.hkv + head) * a.per_page + m) * a.D + c * 8);
        }
        dst[i] = v;
    }
}

struct LaidAttnArgs {
    const void *q, *kv, *means;     // [n][hq][D], this layer's pages, means (decode: with the pages; prefill: gathered)
    void* out;                      // [n][hq][D]
    const float* sinks_log2;        // [hq], or null
    const int *page_indices, *kv_page_indptr, *kv_lens, *qo_indptr, *tile_req, *tile_qstart;
    const uint32_t* mask_bits;
    const long* mask_word_indptr;
    const int* first;               // prefill: first page of means of every request
    const int *item_req, *item_start, *item_end, *req_item_indptr, *num_items;
    float* scratch;
    int n, hq, hkv, D, page_size, window_left, planes, pool, per_page, num_tiles, total_pages, means_pages, max_items, num_reqs, num_ctas;
    float scale;
};

static bool laid_ok(const LaidAttnArgs& a) {
    return a.hkv > 0 && a.hq % a.hkv == 0 && a.page_size % 16 == 0 && (a.planes == 1 || a.planes == 2) &&
           (!a.pool || (a.pool > 0 && a.planes == 2 && a.means && a.window_left >= 0 && !a.mask_bits));
}

}  // namespace pie

using namespace pie;

extern "C" int* pie_status_word_current();      // elementwise.cu

PIE_API int pie_pool_rows(const PoolArgs* args, int f32, cudaStream_t st) {
    const PoolArgs& a = *args;
    if (a.n <= 0) return 0;
    if (a.pool <= 0 || a.page_size <= 0 || a.per_page != (a.page_size + a.pool - 1) / a.pool) return (int)cudaErrorInvalidValue;
    const bool vec = a.D % 4 == 0;
    auto kern = f32 ? (vec ? pool_rows_kernel<float, 4> : pool_rows_kernel<float, 1>)
                    : (vec ? pool_rows_kernel<bf16, 4> : pool_rows_kernel<bf16, 1>);
    return (int)launch_pdl(kern, dim3(a.n), dim3(256), 0, st, a);
}

PIE_API int pie_pool_gather(const PoolArgs* args, cudaStream_t st) {
    const PoolArgs& a = *args;
    if (a.total <= 0 || a.D % 8 || a.pool <= 0) return (int)cudaErrorInvalidValue;
    pool_gather_kernel<<<dim3(a.total, 2 * a.hkv), 128, 0, st>>>(a);
    return (int)cudaGetLastError();
}

PIE_API int pie_laid_decode(const LaidAttnArgs* args, cudaStream_t st) {
    const LaidAttnArgs& a = *args;
    if (a.num_reqs <= 0) return 0;
    if (!laid_ok(a)) return (int)cudaErrorInvalidValue;
    const int group = a.hq / a.hkv;
    float* lse = a.scratch + (size_t)a.max_items * a.hq * a.D;
    const KeyLayout kl{a.planes, a.pool, a.per_page, (const bf16*)a.means, nullptr};
    DISPATCH_DG(a.D, group, {
        const int SM = a.planes == 1 ? decode_smem_bytes<D, true>() : decode_smem_bytes<D>();
        const int ctas = a.planes == 1 && D <= 128 ? a.num_ctas * 3 / 2 : a.num_ctas;
        auto kern = a.pool ? paged_decode_attn_kernel<D, G, false, MODE_PLAIN, true>
                  : a.planes == 1 ? paged_decode_attn_kernel<D, G, false, MODE_PLAIN, false, true> : paged_decode_attn_kernel<D, G, false>;
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM);
        if (e == cudaSuccess)
            e = launch_pdl(kern, dim3(ctas), dim3(DEC_WARPS * 32), SM, st, (const bf16*)a.q, (const bf16*)a.kv, a.page_indices,
                           a.kv_page_indptr, a.item_req, a.item_start, a.item_end, a.req_item_indptr, a.num_items, (bf16*)a.out, a.scratch,
                           lse, a.hq, a.hkv, a.page_size, a.scale * 1.4426950408889634f, a.window_left, a.sinks_log2, a.max_items,
                           a.num_reqs, pie_status_word_current(), (const int*)nullptr, (const int*)nullptr, (const int*)nullptr, 0.f,
                           (const float*)nullptr, 0, 0, kl);
        if (e == cudaSuccess)
            e = launch_pdl(paged_decode_merge_kernel<D>, dim3(a.num_reqs, a.hq), dim3(D), 0, st, (const float*)a.scratch, (const float*)lse,
                           a.req_item_indptr, (bf16*)a.out, a.hq, a.hkv, group, a.sinks_log2, a.max_items);
        return (int)(e != cudaSuccess ? e : cudaGetLastError());
    });
    return (int)cudaErrorInvalidValue;
}

// tile_rows 256: the tcgen05 kernel (head_dim 64 / 128, 16-token pages, total_pages with the pad page last); 64: mma.sync.
PIE_API int pie_laid_prefill(const LaidAttnArgs* args, int tile_rows, int* status, cudaStream_t st) {
    const LaidAttnArgs& a = *args;
    if (a.num_tiles <= 0) return 0;
    if (!laid_ok(a) || !status || (a.pool && !a.first)) return (int)cudaErrorInvalidValue;
    const int group = a.hq / a.hkv;
    const float scale_log2 = a.scale * 1.4426950408889634f;
    const dim3 grid(a.num_tiles, a.hkv);
    if (tile_rows == 64) {
        const KeyLayout kl{a.planes, a.pool, 0, (const bf16*)a.means, a.first};
        DISPATCH_DG(a.D, group, {
            constexpr int SM = prefill_smem_bytes<D>();
            auto kern = a.pool ? paged_prefill_attn_kernel<D, G, MODE_PLAIN, true> : paged_prefill_attn_kernel<D, G>;
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM);
            if (e != cudaSuccess) return (int)e;
            kern<<<grid, PF_WARPS * 32, SM, st>>>((const bf16*)a.q, (const bf16*)a.kv, a.page_indices, a.kv_page_indptr, a.qo_indptr,
                                                  a.kv_lens, a.tile_req, a.tile_qstart, a.mask_bits, a.mask_word_indptr, (bf16*)a.out,
                                                  nullptr, a.sinks_log2, a.hq, a.hkv, a.page_size, scale_log2, a.window_left, 0.f,
                                                  nullptr, 0, 0, kl);
            return (int)cudaGetLastError();
        });
        return (int)cudaErrorInvalidValue;
    }
    if (tile_rows != 256 || a.page_size != 16) return (int)cudaErrorInvalidValue;
    EncodeTiledFnA enc = at_encoder();
    if (!enc) return (int)cudaErrorNotSupported;
    CUtensorMap tq, tkv, tm;
    cuuint32_t estr[3] = {1, 1, 1};
    cuuint64_t qd[3] = {(cuuint64_t)a.D, (cuuint64_t)a.hq, (cuuint64_t)a.n};
    cuuint64_t qs[2] = {(cuuint64_t)a.D * 2, (cuuint64_t)a.hq * a.D * 2};
    cuuint32_t qb[3] = {64, (cuuint32_t)group, (cuuint32_t)(AT_ROWS / group)};
    auto pages = [&](CUtensorMap* m, const void* p, int count, int planes) {
        cuuint64_t kd[2] = {(cuuint64_t)a.D, (cuuint64_t)count * planes * a.hkv * 16};
        cuuint64_t ks[1] = {(cuuint64_t)a.D * 2};
        cuuint32_t kb[2] = {64, 16};
        return enc(m, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(p), kd, ks, kb, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
                   CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    };
    if (enc(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(a.q), qd, qs, qb, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS ||
        pages(&tkv, a.kv, a.total_pages, a.planes) != CUDA_SUCCESS || (a.pool && pages(&tm, a.means, a.means_pages, 2) != CUDA_SUCCESS))
        return (int)cudaErrorInvalidValue;
    if (!a.pool) tm = tkv;
    TcMeans ml;
    ml.first = a.first;
    ml.pool = a.pool;
    ml.pad_page = a.means_pages - 1;
#define GO2(G_, D_)                                                                                                              \
    {                                                                                                                            \
        auto kern = a.pool ? paged_prefill_attn_tc_kernel<G_, 2, D_, false, false, false, true>                                  \
                           : paged_prefill_attn_tc_kernel<G_, 2, D_>;                                                            \
        using Cfg = AtCfg<2, D_>;                                                                                                \
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)Cfg::SMEM);           \
        if (e != cudaSuccess) return (int)e;                                                                                     \
        kern<<<grid, Cfg::THREADS, Cfg::SMEM, st>>>(tq, tkv, tm, ml, a.planes, a.page_indices, a.kv_page_indptr, a.qo_indptr,    \
                                                    a.kv_lens, a.tile_req, a.tile_qstart, a.mask_bits, a.mask_word_indptr,       \
                                                    (bf16*)a.out, nullptr, a.sinks_log2, a.hq, a.hkv, a.total_pages - 1,         \
                                                    scale_log2, a.window_left, status, 0.f, 0.f, a.hq * D_, D_, nullptr, 0, 0, 0); \
        return (int)cudaGetLastError();                                                                                          \
    }
#define GO(G_) if (a.D == 128) GO2(G_, 128) else if (a.D == 64) GO2(G_, 64) break;
    switch (group) {
        case 1: GO(1)
        case 2: GO(2)
        case 4: GO(4)
        case 8: GO(8)
        case 16: GO(16)
    }
#undef GO
#undef GO2
    return (int)cudaErrorInvalidValue;
}
