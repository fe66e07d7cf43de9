// Attention with soft-capped scores and a learned bias per distance: softmax over cap * tanh(q.k * scale / cap) + bias[n],
// n = query position - key position, in a sliding window. Keys and values live in the ordinary KV pages
// ([pages][2][hkv][page][D], zeros past a head's own sizes) without rotation.
//
//   pie_biased_rows     q / k RMS norm over the whole projection, padded query rows, page writes
//   pie_biased_decode   split-KV decode on the kernels of attention_mma.cuh
//   pie_biased_prefill  prompts on tcgen05 (attention_tc.cuh) or, for other shapes, attention_mma.cuh
//   pie_biased_any      one warp per (token, head), any sizes, bf16 or true 32-bit
//
// The bias table is [kv heads * padded group][pitch] in units of log2: 64 entries that repeat the bias of distance 0 (a custom
// mask may show later keys), the `pitch` - 128 distances 0 .. window - 1, 64 unused entries.
#include "attention_mma.cuh"
#include "attention_tc.cuh"
#include "typed.cuh"

namespace pie {

static_assert(BIAS_GUARD == AT_BIAS_GUARD, "one table for both kernels");

struct BiasedRowsArgs {
    const void *q, *k, *v;          // row t at t * ld: heads x dim, kv_heads x dim, kv_heads x vdim
    const void *q_norm, *k_norm;    // [heads * dim], [kv_heads * dim]
    const int* slots;               // KV slot of every token (< 0: no write)
    void* q_out;                    // [n][kv_heads * group_pad][D]
    void* cache;                    // this layer's pages
    int n, ld, heads, kv_heads, group, group_pad, dim, vdim, D, page_size;
    float eps;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(256) biased_rows_kernel(const BiasedRowsArgs a) {
    __shared__ float red[32];
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    const T* q = static_cast<const T*>(a.q) + (size_t)t * a.ld;
    const T* k = static_cast<const T*>(a.k) + (size_t)t * a.ld;
    const T* v = static_cast<const T*>(a.v) + (size_t)t * a.ld;
    const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim;
    auto squares = [&](const T* x, int n) {
        float s = 0.f;
        for (int i = threadIdx.x * VEC; i < n; i += 256 * VEC) {
            float f[VEC];
            load_vec<VEC>(x + i, f);
#pragma unroll
            for (int e = 0; e < VEC; ++e) s += f[e] * f[e];
        }
        return s;
    };
    const float sq = squares(q, nq), sk = squares(k, nk);
    const float iq = 1.f / sqrtf(block_sum(sq, red) / (float)nq + a.eps);
    const float ik = 1.f / sqrtf(block_sum(sk, red) / (float)nk + a.eps);
    const T* wq = static_cast<const T*>(a.q_norm);
    const T* wk = static_cast<const T*>(a.k_norm);
    // columns past a head's size and rows past a group's are zeros
    auto emit = [&](T* dst, const T* src, const T* w, float inv, bool ok) {
        float f[VEC], g[VEC];
#pragma unroll
        for (int e = 0; e < VEC; ++e) f[e] = 0.f;
        if (ok) {
            load_vec<VEC>(src, f);
            if (w) {
                load_vec<VEC>(w, g);
#pragma unroll
                for (int e = 0; e < VEC; ++e) f[e] *= inv * g[e];
            }
        }
        store_vec<VEC>(dst, f);
    };
    T* qo = static_cast<T*>(a.q_out) + (size_t)t * a.kv_heads * a.group_pad * a.D;
    for (int i = threadIdx.x * VEC; i < a.kv_heads * a.group_pad * a.D; i += 256 * VEC) {
        const int hp = i / a.D, d = i - hp * a.D, kv = hp / a.group_pad, g = hp - kv * a.group_pad;
        const int src = (kv * a.group + g) * a.dim + d;
        emit(qo + i, q + src, wq + src, iq, g < a.group && d < a.dim);
    }
    const int slot = a.slots[t];
    if (slot < 0) return;
    const int page = slot / a.page_size, off = slot % a.page_size;
    T* base = static_cast<T*>(a.cache) + (size_t)page * 2 * a.kv_heads * a.page_size * a.D;
    for (int i = threadIdx.x * VEC; i < 2 * a.kv_heads * a.D; i += 256 * VEC) {
        const int hv = i / a.D, d = i - hv * a.D, h = hv % a.kv_heads;
        T* dst = base + ((size_t)hv * a.page_size + off) * a.D + d;
        if (hv < a.kv_heads) emit(dst, k + h * a.dim + d, wk + h * a.dim + d, ik, d < a.dim);
        else emit(dst, v + h * a.vdim + d, nullptr, 1.f, d < a.vdim);
    }
}

struct BiasedAttnArgs {
    const void *q, *kv;             // [n][hq][D], this layer's pages
    void* out;                      // [n][hq][D]
    const float* bias;              // [hq][bias_pitch]
    const int *page_indices, *kv_page_indptr, *kv_lens;
    // any: rows of the batch; prefill: tiles
    const int *qo_indptr, *tok_req, *slots, *tile_req, *tile_qstart;
    const uint32_t* mask_bits;
    const long* mask_word_indptr;
    // decode: split-KV work items
    const int *item_req, *item_start, *item_end, *req_item_indptr, *num_items;
    float* scratch;
    int n, hq, hkv, D, page_size, bias_pitch, window_left, num_tiles, total_pages, max_items, num_reqs, num_ctas;
    float scale, softcap;
};

template <typename T, int ME>
__global__ void __launch_bounds__(128) biased_attn_any_kernel(const BiasedAttnArgs a) {
    pdl_trigger();
    pdl_wait();
    const long w = (blockIdx.x * 128L + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (w >= (long)a.n * a.hq) return;
    const int t = (int)(w / a.hq), h = (int)(w - (long)t * a.hq), kvh = h / (a.hq / a.hkv);
    float q[ME], acc[ME], m = -INFINITY, l = 0.f;
    const T* qr = static_cast<const T*>(a.q) + w * a.D;
    const float pre = a.scale / a.softcap, post = a.softcap * 1.4426950408889634f;
#pragma unroll
    for (int i = 0; i < ME; ++i) {
        const int e = lane + 32 * i;
        q[i] = e < a.D ? to_f(qr[e]) * pre : 0.f;
        acc[i] = 0.f;
    }
    if (a.slots[t] >= 0) {
        const int r = a.tok_req[t], q0 = a.qo_indptr[r], qlen = a.qo_indptr[r + 1] - q0, kv_len = a.kv_lens[r];
        const int pos = kv_len - qlen + (t - q0), last = a.bias_pitch - 2 * BIAS_GUARD - 1;
        const uint32_t* bits = nullptr;
        if (a.mask_bits) bits = a.mask_bits + a.mask_word_indptr[r] + (long)(t - q0) * ((kv_len + 31) / 32);
        const int* pages = a.page_indices + a.kv_page_indptr[r];
        const float* tab = a.bias + (size_t)h * a.bias_pitch + BIAS_GUARD;
        const int hi = bits ? kv_len : pos + 1;
        for (int j = max(0, pos - a.window_left); j < hi; ++j) {
            if (bits && !(bits[j >> 5] >> (j & 31) & 1u)) continue;
            const T* kr = static_cast<const T*>(a.kv) +
                          (((size_t)pages[j / a.page_size] * 2 * a.hkv + kvh) * a.page_size + j % a.page_size) * a.D;
            const T* vr = kr + (size_t)a.hkv * a.page_size * a.D;
            float s = 0.f, v[ME];
#pragma unroll
            for (int i = 0; i < ME; ++i) {
                const int e = lane + 32 * i;
                s += q[i] * (e < a.D ? to_f(kr[e]) : 0.f);
                v[i] = e < a.D ? to_f(vr[e]) : 0.f;
            }
            s = post * tanhf(warp_sum(s)) + tab[min(max(pos - j, 0), last)];
            const float mn = fmaxf(m, s), c = exp2f(m - mn), p = exp2f(s - mn);
            m = mn;
            l = l * c + p;
#pragma unroll
            for (int i = 0; i < ME; ++i) acc[i] = acc[i] * c + p * v[i];
        }
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    T* dst = static_cast<T*>(a.out) + w * a.D;
#pragma unroll
    for (int i = 0; i < ME; ++i) {
        const int e = lane + 32 * i;
        if (e < a.D) dst[e] = from_f<T>(acc[i] * inv);
    }
}

static bool bias_ok(const BiasedAttnArgs& a) {
    return a.hkv > 0 && a.hq % a.hkv == 0 && a.page_size % 16 == 0 && a.softcap > 0.f && a.window_left >= 0 && a.bias &&
           a.bias_pitch % 4 == 0 && a.bias_pitch - 2 * BIAS_GUARD > a.window_left;
}

}  // namespace pie

using namespace pie;

extern "C" int* pie_status_word_current();      // elementwise.cu

PIE_API int pie_biased_rows(const BiasedRowsArgs* args, int f32, cudaStream_t st) {
    const BiasedRowsArgs& a = *args;
    if (a.n <= 0) return 0;
    if (a.group > a.group_pad || a.heads != a.kv_heads * a.group || a.dim > a.D || a.vdim > a.D) return (int)cudaErrorInvalidValue;
    auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.ld % 4 == 0 && aligned(a.q) && aligned(a.k) && aligned(a.v) &&
                     aligned(a.q_norm) && aligned(a.k_norm) && aligned(a.q_out) && aligned(a.cache);
    auto kern = f32 ? (vec ? biased_rows_kernel<float, 4> : biased_rows_kernel<float, 1>)
                    : (vec ? biased_rows_kernel<bf16, 4> : biased_rows_kernel<bf16, 1>);
    return (int)launch_pdl(kern, dim3(a.n), dim3(256), 0, st, a);
}

PIE_API int pie_biased_any(const BiasedAttnArgs* args, int f32, cudaStream_t st) {
    const BiasedAttnArgs& a = *args;
    if (a.n <= 0) return 0;
    if (!bias_ok(a) || a.D > 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid((unsigned)(((long)a.n * a.hq + 3) / 4));
#define GO(T_, M_) return (int)launch_pdl(biased_attn_any_kernel<T_, M_>, grid, dim3(128), 0, st, a)
#define GO_M(T_) \
    if (a.D <= 64) GO(T_, 2); if (a.D <= 128) GO(T_, 4); if (a.D <= 256) GO(T_, 8); if (a.D <= 512) GO(T_, 16); GO(T_, 32)
    if (f32) { GO_M(float); }
    GO_M(bf16);
#undef GO_M
#undef GO
}

// 1 when decode and prefill attention have tensor-core kernels for the shape.
PIE_API int pie_biased_mma_supported(int group, int head_dim) {
    const bool g = group == 1 || group == 2 || group == 4 || group == 8 || group == 16;
    return g && (head_dim == 64 || head_dim == 128 || (head_dim == 256 && group <= 8)) ? 1 : 0;
}

PIE_API int pie_biased_decode(const BiasedAttnArgs* args, cudaStream_t st) {
    const BiasedAttnArgs& a = *args;
    if (a.num_reqs <= 0) return 0;
    if (!bias_ok(a)) return (int)cudaErrorInvalidValue;
    const int group = a.hq / a.hkv;
    float* lse = a.scratch + (size_t)a.max_items * a.hq * a.D;
    DISPATCH_DG(a.D, group, {
        constexpr int SM = decode_smem_bytes<D>();
        auto kern = paged_decode_attn_kernel<D, G, false, MODE_BIAS>;
        cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM);
        if (e == cudaSuccess)
            e = launch_pdl(kern, dim3(a.num_ctas), dim3(DEC_WARPS * 32), SM, st, (const bf16*)a.q, (const bf16*)a.kv, a.page_indices,
                           a.kv_page_indptr, a.item_req, a.item_start, a.item_end, a.req_item_indptr, a.num_items, (bf16*)a.out, a.scratch,
                           lse, a.hq, a.hkv, a.page_size, a.scale / a.softcap, a.window_left, (const float*)nullptr, a.max_items,
                           a.num_reqs, pie_status_word_current(), (const int*)nullptr, (const int*)nullptr, (const int*)nullptr,
                           a.softcap * 1.4426950408889634f, a.bias, a.bias_pitch, 0, KeyLayout());
        if (e == cudaSuccess)
            e = launch_pdl(paged_decode_merge_kernel<D>, dim3(a.num_reqs, a.hq), dim3(D), 0, st, (const float*)a.scratch, (const float*)lse,
                           a.req_item_indptr, (bf16*)a.out, a.hq, a.hkv, group, (const float*)nullptr, a.max_items);
        return (int)(e != cudaSuccess ? e : cudaGetLastError());
    });
    return (int)cudaErrorInvalidValue;
}

// tile_rows 256: the tcgen05 kernel (head_dim 64 / 128, 16-token pages, total_pages with the pad page last); 64: mma.sync.
PIE_API int pie_biased_prefill(const BiasedAttnArgs* args, int tile_rows, int* status, cudaStream_t st) {
    const BiasedAttnArgs& a = *args;
    if (a.num_tiles <= 0) return 0;
    if (!bias_ok(a) || !status) return (int)cudaErrorInvalidValue;
    const int group = a.hq / a.hkv;
    const float pre = a.scale / a.softcap, post = a.softcap * 1.4426950408889634f;
    const dim3 grid(a.num_tiles, a.hkv);
    if (tile_rows == 64) {
        DISPATCH_DG(a.D, group, {
            constexpr int SM = prefill_smem_bytes<D>();
            auto kern = paged_prefill_attn_kernel<D, G, MODE_BIAS>;
            const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, SM);
            if (e != cudaSuccess) return (int)e;
            kern<<<grid, PF_WARPS * 32, SM, st>>>((const bf16*)a.q, (const bf16*)a.kv, a.page_indices, a.kv_page_indptr, a.qo_indptr,
                                                  a.kv_lens, a.tile_req, a.tile_qstart, a.mask_bits, a.mask_word_indptr, (bf16*)a.out,
                                                  nullptr, nullptr, a.hq, a.hkv, a.page_size, pre, a.window_left, post, a.bias, a.bias_pitch, 0,
                                                  KeyLayout());
            return (int)cudaGetLastError();
        });
        return (int)cudaErrorInvalidValue;
    }
    if (tile_rows != 256 || a.page_size != 16) return (int)cudaErrorInvalidValue;
    EncodeTiledFnA enc = at_encoder();
    if (!enc) return (int)cudaErrorNotSupported;
    CUtensorMap tq, tkv;
    cuuint32_t estr[3] = {1, 1, 1};
    cuuint64_t qd[3] = {(cuuint64_t)a.D, (cuuint64_t)a.hq, (cuuint64_t)a.n};
    cuuint64_t qs[2] = {(cuuint64_t)a.D * 2, (cuuint64_t)a.hq * a.D * 2};
    cuuint32_t qb[3] = {64, (cuuint32_t)group, (cuuint32_t)(AT_ROWS / group)};
    cuuint64_t kd[2] = {(cuuint64_t)a.D, (cuuint64_t)a.total_pages * 2 * a.hkv * 16};
    cuuint64_t ks[1] = {(cuuint64_t)a.D * 2};
    cuuint32_t kb[2] = {64, 16};
    if (enc(&tq, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 3, const_cast<void*>(a.q), qd, qs, qb, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS ||
        enc(&tkv, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<void*>(a.kv), kd, ks, kb, estr, CU_TENSOR_MAP_INTERLEAVE_NONE,
            CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) != CUDA_SUCCESS)
        return (int)cudaErrorInvalidValue;
#define GO2(G_, D_)                                                                                                              \
    {                                                                                                                            \
        auto kern = paged_prefill_attn_tc_kernel<G_, 2, D_, false, false, true>;                                                 \
        using Cfg = AtCfg<2, D_, D_ == 128 ? 2 : AT_STAGES>;                                                                     \
        const size_t table = (size_t)G_ * a.bias_pitch * 4;                                                                      \
        const int in_smem = Cfg::SMEM + table <= 227 * 1024 ? 1 : 0;                                                             \
        const size_t smem = Cfg::SMEM + (in_smem ? table : 0);                                                                   \
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);                \
        if (e != cudaSuccess) return (int)e;                                                                                     \
        kern<<<grid, Cfg::THREADS, smem, st>>>(tq, tkv, tkv, TcMeans(), 2, a.page_indices, a.kv_page_indptr, a.qo_indptr, a.kv_lens, a.tile_req,    \
                                               a.tile_qstart, a.mask_bits, a.mask_word_indptr, (bf16*)a.out, nullptr, nullptr,   \
                                               a.hq, a.hkv, a.total_pages - 1, 1.f, a.window_left, status, pre, post,            \
                                               a.hq * D_, D_, a.bias, a.bias_pitch, in_smem, 0);                                  \
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
