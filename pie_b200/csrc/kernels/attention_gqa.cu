// Around grouped-query attention whose projections carry biases, whose queries and keys are normed over all heads together
// and rotated in part:
//
//   pie_gqa_rows   bias, RMS norm over the whole projection, rotation, value mixing, padded query rows, page writes
//   pie_head_rows  the same without biases, with a norm per head or none, half-apart pairs, a factor on the query by position
//   pie_gqa_any    attention, one warp per (token, head): any sizes, bf16 or true 32-bit
//
// Keys and values live in the ordinary KV pages ([pages][2][hkv][page][D], zeros past a head's own sizes); attention on
// tensor cores runs on the kernels of attention_mma.cuh and attention_tc.cuh.
#include "typed.cuh"

namespace pie {

struct GqaRowsArgs {
    const void *q, *k, *v;          // row t at t * ld: heads x dim, kv_heads x dim, kv_heads x vdim
    const void *q_b, *k_b, *v_b;    // biases, or all null
    const void *q_norm, *k_norm;    // [heads * dim], [kv_heads * dim]
    const int *positions, *slots;   // KV slot of every token (< 0: no write)
    const float* inv_freq;          // [rot_dims / 2]
    const float* v_first;           // [n, kv_heads * vdim] values to mix in: v <- v + mix (v_first - v); null: none
    float* v_keep;                  // [n, kv_heads * vdim] copy of the values in 32-bit; null: none
    void* q_out;                    // [n][kv_heads * group_pad][D]
    void* cache;                    // this layer's pages
    int n, ld, heads, kv_heads, group, group_pad, dim, vdim, D, page_size, rot_dims, adjacent;
    float eps, mix;
};

// One block per token. Biased and normed queries and keys are staged in shared memory, where the partner of a rotated
// element is at hand; then rows are written VEC elements at a time.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) gqa_rows_kernel(const GqaRowsArgs a) {
    extern __shared__ __align__(16) float sm[];
    pdl_trigger();
    const int t = blockIdx.x, half = a.rot_dims / 2;
    const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
    float* red = sm;                    // [32]
    float* cs = red + 32;               // [half] cos, [half] sin
    float* sq = cs + (a.rot_dims + 3) / 4 * 4;
    float* sk = sq + (nq + 3) / 4 * 4;
    pdl_wait();
    for (int i = threadIdx.x; i < half; i += 256) sincosf((float)a.positions[t] * a.inv_freq[i], cs + half + i, cs + i);
    auto stage = [&](const void* x, const void* bias, int n, float* dst) {
        const T* src = static_cast<const T*>(x) + (size_t)t * a.ld;
        const T* b = static_cast<const T*>(bias);
        float s = 0.f;
        for (int i = threadIdx.x * VEC; i < n; i += 256 * VEC) {
            float f[VEC], g[VEC];
            load_vec<VEC>(src + i, f);
            if (b) load_vec<VEC>(b + i, g);
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                if (b) f[e] += g[e];
                s += f[e] * f[e];
            }
            store_vec<VEC>(dst + i, f);
        }
        return s;
    };
    const float ssq = stage(a.q, a.q_b, nq, sq), ssk = stage(a.k, a.k_b, nk, sk);
    const float iq = 1.f / sqrtf(block_sum(ssq, red) / (float)nq + a.eps);
    const float ik = 1.f / sqrtf(block_sum(ssk, red) / (float)nk + a.eps);
    auto scale = [&](const void* norm, float inv, int n, float* x) {
        const T* w = static_cast<const T*>(norm);
        for (int i = threadIdx.x * VEC; i < n; i += 256 * VEC) {
            float f[VEC], g[VEC];
            load_vec<VEC>(x + i, f);
            load_vec<VEC>(w + i, g);
#pragma unroll
            for (int e = 0; e < VEC; ++e) f[e] *= inv * g[e];
            store_vec<VEC>(x + i, f);
        }
    };
    scale(a.q_norm, iq, nq, sq);
    scale(a.k_norm, ik, nk, sk);
    __syncthreads();
    // VEC elements of a head from d on: rotated, or as they are. A vector's partners are neighbours or another vector where
    // pairs and halves fall on vectors.
    const bool whole = VEC == 4 && a.rot_dims % 4 == 0 && (a.adjacent || half % 4 == 0);
    auto head_vec = [&](const float* x, int d, float (&f)[VEC]) {
        if (VEC == 4 && (whole || d >= a.rot_dims)) {
            load_vec<VEC>(x + d, f);
            if (d >= a.rot_dims) return;
            if (a.adjacent) {
#pragma unroll
                for (int e = 0; e + 1 < VEC; e += 2) {
                    const float c = cs[(d + e) >> 1], sn = cs[half + ((d + e) >> 1)], u = f[e], v = f[e + 1];
                    f[e] = u * c - v * sn;
                    f[e + 1] = v * c + u * sn;
                }
            } else {
                const bool lower = d < half;
                const int p = lower ? d : d - half;
                float o[VEC], c[VEC], sn[VEC];
                load_vec<VEC>(x + (lower ? d + half : p), o);
                load_vec<VEC>(cs + p, c);
                load_vec<VEC>(cs + half + p, sn);
#pragma unroll
                for (int e = 0; e < VEC; ++e) f[e] = f[e] * c[e] + (lower ? -o[e] : o[e]) * sn[e];
            }
            return;
        }
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const int i = d + e;
            f[e] = x[i];
            if (i >= a.rot_dims) continue;
            const int p = a.adjacent ? i >> 1 : (i < half ? i : i - half);
            const bool lower = a.adjacent ? (i & 1) == 0 : i < half;
            const float o = x[a.adjacent ? i ^ 1 : (lower ? i + half : i - half)];
            f[e] = f[e] * cs[p] + (lower ? -o : o) * cs[half + p];
        }
    };
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    auto emit = [&](T* dst, const float* head) {         // one warp per row of D; null: zeros
        for (int d = lane * VEC; d < a.D; d += 32 * VEC) {
            float f[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) f[e] = 0.f;
            if (head && d < a.dim) head_vec(head, d, f);
            store_vec<VEC>(dst + d, f);
        }
    };
    T* qo = static_cast<T*>(a.q_out) + (size_t)t * a.kv_heads * a.group_pad * a.D;
    for (int hp = warp; hp < a.kv_heads * a.group_pad; hp += 8) {
        const int kv = hp / a.group_pad, g = hp - kv * a.group_pad;
        emit(qo + (size_t)hp * a.D, g < a.group ? sq + (kv * a.group + g) * a.dim : nullptr);
    }
    const int slot = a.slots[t];
    T* base = nullptr;
    int off = 0;
    if (slot >= 0) {
        off = slot % a.page_size;
        base = static_cast<T*>(a.cache) + (size_t)(slot / a.page_size) * 2 * a.kv_heads * a.page_size * a.D;
        for (int h = warp; h < a.kv_heads; h += 8) emit(base + ((size_t)h * a.page_size + off) * a.D, sk + h * a.dim);
    }
    if (!base && !a.v_keep) return;
    const T* vr = static_cast<const T*>(a.v) + (size_t)t * a.ld;
    const T* vb = static_cast<const T*>(a.v_b);
    for (int h = warp; h < a.kv_heads; h += 8)
        for (int d = lane * VEC; d < a.D; d += 32 * VEC) {
            float f[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) f[e] = 0.f;
            if (d < a.vdim) {
                const int at = h * a.vdim + d;
                float g[VEC];
                load_vec<VEC>(vr + at, f);
                if (vb) {
                    load_vec<VEC>(vb + at, g);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) f[e] += g[e];
                }
                if (a.v_keep) store_vec<VEC>(a.v_keep + (size_t)t * nv + at, f);
                if (a.v_first) {
                    load_vec<VEC>(a.v_first + (size_t)t * nv + at, g);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) f[e] = (1.f - a.mix) * f[e] + a.mix * g[e];
                }
            }
            if (base) store_vec<VEC>(base + ((size_t)(a.kv_heads + h) * a.page_size + off) * a.D + d, f);
        }
}

struct HeadRowsArgs {
    const void *q, *k, *v;          // row t at t * ld: heads x dim, kv_heads x dim, kv_heads x vdim; v null: the values are the keys
    const float *q_norm, *k_norm;   // [dim], or null
    const int *positions, *slots;   // KV slot of every token (< 0: no write)
    const float* inv_freq;          // [rot_dims / 2]
    void* q_out;                    // [n][kv_heads * group_pad][D]
    void* cache;                    // this layer's pages, two planes or (v null) one
    int n, ld, heads, kv_heads, group, group_pad, dim, vdim, D, page_size, rot_dims, temp_every;   // temp_every 0: no factor
    float eps, rot_factor, temp_coef;
};

// One block per token; a warp takes a head at a time through its row in shared memory, where a rotated element finds its
// partner. The factor on the query at position p is 1 + temp_coef * ln(floor((p + 1) / temp_every) + 1).
template <typename T, int VEC>
__global__ void __launch_bounds__(256) head_rows_kernel(const HeadRowsArgs a) {
    extern __shared__ __align__(16) float sm[];
    pdl_trigger();
    const int t = blockIdx.x, half = a.rot_dims / 2, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    float* cs = sm;                     // [half] cos, [half] sin
    float* row = cs + (a.rot_dims + 3) / 4 * 4 + warp * ((a.dim + 3) / 4 * 4);
    pdl_wait();
    const int pos = a.positions[t];
    for (int i = threadIdx.x; i < half; i += 256) {
        float s, c;
        sincosf((float)pos * a.inv_freq[i], &s, &c);
        cs[i] = c * a.rot_factor;
        cs[half + i] = s * a.rot_factor;
    }
    __syncthreads();
    const float temp = a.temp_every ? 1.f + a.temp_coef * logf((float)((pos + 1) / a.temp_every) + 1.f) : 1.f;
    const bool pairs_of_vecs = VEC == 4 && half % 4 == 0;
    auto emit = [&](T* dst, const T* src, int n, const float* norm, bool turn, float scale) {       // src null: zeros
        float ss = 0.f;
        turn = turn && half > 0;
        if (src && (norm || turn)) {
            __syncwarp();
            for (int d = lane * VEC; d < n; d += 32 * VEC) {
                float f[VEC], g[VEC];
                load_vec<VEC>(src + d, f);
                if (norm) load_vec<VEC>(norm + d, g);
#pragma unroll
                for (int e = 0; e < VEC; ++e) {
                    ss += f[e] * f[e];
                    if (norm) f[e] *= g[e];
                }
                store_vec<VEC>(row + d, f);
            }
            if (norm) scale *= 1.f / sqrtf(warp_sum(ss) / (float)n + a.eps);
            __syncwarp();
        }
        for (int d = lane * VEC; d < a.D; d += 32 * VEC) {
            float f[VEC];
#pragma unroll
            for (int e = 0; e < VEC; ++e) f[e] = 0.f;
            if (src && d < n) {
                if (!norm && !turn) load_vec<VEC>(src + d, f);
                else load_vec<VEC>(row + d, f);
                if (turn && d < a.rot_dims && pairs_of_vecs) {
                    const bool lower = d < half;
                    const int p = lower ? d : d - half;
                    float o[VEC], c[VEC], sn[VEC];
                    load_vec<VEC>(row + (lower ? d + half : p), o);
                    load_vec<VEC>(cs + p, c);
                    load_vec<VEC>(cs + half + p, sn);
#pragma unroll
                    for (int e = 0; e < VEC; ++e) f[e] = f[e] * c[e] + (lower ? -o[e] : o[e]) * sn[e];
                } else if (turn) {
#pragma unroll
                    for (int e = 0; e < VEC; ++e) {
                        const int i = d + e, p = i < half ? i : i - half;
                        if (i < a.rot_dims) f[e] = f[e] * cs[p] + (i < half ? -row[i + half] : row[p]) * cs[half + p];
                    }
                }
#pragma unroll
                for (int e = 0; e < VEC; ++e) f[e] *= scale;
            }
            store_vec<VEC>(dst + d, f);
        }
    };
    const T* q = static_cast<const T*>(a.q) + (size_t)t * a.ld;
    T* qo = static_cast<T*>(a.q_out) + (size_t)t * a.kv_heads * a.group_pad * a.D;
    const int nq = a.kv_heads * a.group_pad, slot = a.slots[t], planes = a.v ? 2 : 1;
    T* base = slot < 0 ? nullptr : static_cast<T*>(a.cache) + (size_t)(slot / a.page_size) * planes * a.kv_heads * a.page_size * a.D;
    for (int u = warp; u < nq + (base ? planes * a.kv_heads : 0); u += 8) {
        if (u < nq) {
            const int kv = u / a.group_pad, g = u - kv * a.group_pad;
            emit(qo + (size_t)u * a.D, g < a.group ? q + (kv * a.group + g) * a.dim : nullptr, a.dim, a.q_norm, true, temp);
            continue;
        }
        T* dst = base + ((size_t)(u - nq) * a.page_size + slot % a.page_size) * a.D;
        const int h = (u - nq) % a.kv_heads;
        if (u - nq < a.kv_heads) emit(dst, static_cast<const T*>(a.k) + (size_t)t * a.ld + h * a.dim, a.dim, a.k_norm, true, 1.f);
        else emit(dst, static_cast<const T*>(a.v) + (size_t)t * a.ld + h * a.vdim, a.vdim, nullptr, false, 1.f);
    }
}

struct GqaAnyArgs {
    const void *q, *kv;             // [n][hq][D], this layer's pages
    void* out;                      // [n][hq][D]
    const float* sink_scores;       // [hq] natural logarithms, or null
    const void* means;              // with pool: means of key and value blocks, see KeyLayout in attention_mma.cuh
    const int *page_indices, *kv_page_indptr, *kv_lens, *qo_indptr, *tok_req, *slots;
    const uint32_t* mask_bits;      // custom mask words, or null (causal)
    const long* mask_word_indptr;
    int n, hq, hkv, D, page_size, window_left, keep_first, sink, planes, pool, per_page;   // window_left < 0: no window; sink: a score of 0
    float scale;
};

template <typename T, int ME>
__global__ void __launch_bounds__(128) gqa_any_kernel(const GqaAnyArgs a) {
    pdl_trigger();
    pdl_wait();
    const long w = (blockIdx.x * 128L + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (w >= (long)a.n * a.hq) return;
    const int t = (int)(w / a.hq), h = (int)(w - (long)t * a.hq), kvh = h / (a.hq / a.hkv);
    float q[ME], acc[ME], m = -INFINITY, l = 0.f;
    const T* qr = static_cast<const T*>(a.q) + w * a.D;
#pragma unroll
    for (int i = 0; i < ME; ++i) {
        const int e = lane + 32 * i;
        q[i] = e < a.D ? to_f(qr[e]) * a.scale : 0.f;
        acc[i] = 0.f;
    }
    if (a.slots[t] >= 0) {
        const int r = a.tok_req[t], q0 = a.qo_indptr[r], qlen = a.qo_indptr[r + 1] - q0, kv_len = a.kv_lens[r];
        const int pos = kv_len - qlen + (t - q0);
        const uint32_t* bits = nullptr;
        if (a.mask_bits) bits = a.mask_bits + a.mask_word_indptr[r] + (long)(t - q0) * ((kv_len + 31) / 32);
        const int* pages = a.page_indices + a.kv_page_indptr[r];
        const int hi = bits ? kv_len : pos + 1, lo = a.window_left >= 0 ? max(0, pos - a.window_left) : 0;
        if (a.sink) { m = 0.f; l = 1.f; }
        if (a.sink_scores) { m = a.sink_scores[h]; l = 1.f; }
        auto attend = [&](const T* kr, const T* vr) {
            float s = 0.f, v[ME];
#pragma unroll
            for (int i = 0; i < ME; ++i) {
                const int e = lane + 32 * i;
                s += q[i] * (e < a.D ? to_f(kr[e]) : 0.f);
                v[i] = e < a.D ? to_f(vr[e]) : 0.f;
            }
            s = warp_sum(s);
            const float mn = fmaxf(m, s), c = expf(m - mn), p = expf(s - mn);
            m = mn;
            l = l * c + p;
#pragma unroll
            for (int i = 0; i < ME; ++i) acc[i] = acc[i] * c + p * v[i];
        };
        auto hidden = [&](int j) { return bits && !(bits[j >> 5] >> (j & 31) & 1u); };
        // the mean of a block counts once the block lies before the window, and under a mask if that shows all its tokens
        for (int b = 0; a.pool && b < lo / a.pool; ++b) {
            bool whole = true;
            for (int j = b * a.pool; bits && j < (b + 1) * a.pool; ++j) whole = whole && !hidden(j);
            if (!whole) continue;
            const int page_at = ((b + 1) * a.pool - 1) / a.page_size, row = b - page_at * a.page_size / a.pool;
            const T* kr = static_cast<const T*>(a.means) + (((size_t)pages[page_at] * 2 * a.hkv + kvh) * a.per_page + row) * a.D;
            attend(kr, kr + (size_t)a.hkv * a.per_page * a.D);
        }
        for (int j = 0; j < hi; ++j) {
            if (j >= a.keep_first && j < lo) { j = lo - 1; continue; }
            if (hidden(j)) continue;
            const T* kr = static_cast<const T*>(a.kv) +
                          (((size_t)pages[j / a.page_size] * a.planes * a.hkv + kvh) * a.page_size + j % a.page_size) * a.D;
            attend(kr, kr + (size_t)(a.planes - 1) * a.hkv * a.page_size * a.D);
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

}  // namespace pie

using namespace pie;

PIE_API int pie_gqa_rows(const GqaRowsArgs* args, int f32, cudaStream_t st) {
    const GqaRowsArgs& a = *args;
    if (a.n <= 0) return 0;
    if (a.group > a.group_pad || a.heads != a.kv_heads * a.group || a.dim > a.D || a.vdim > a.D || a.rot_dims % 2 || a.rot_dims > a.dim ||
        a.page_size <= 0 || (!a.q_b) != (!a.k_b) || (!a.q_b) != (!a.v_b))
        return (int)cudaErrorInvalidValue;
    auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.D % 4 == 0 && a.ld % 4 == 0 && aligned(a.q) && aligned(a.k) && aligned(a.v) &&
                     aligned(a.q_b) && aligned(a.k_b) && aligned(a.v_b) && aligned(a.q_norm) && aligned(a.k_norm) && aligned(a.q_out) &&
                     aligned(a.cache) && aligned(a.v_first) && aligned(a.v_keep);
    const int sm = (32 + (a.rot_dims + 3) / 4 * 4 + (a.heads * a.dim + 3) / 4 * 4 + (a.kv_heads * a.dim + 3) / 4 * 4) * 4;
    if (sm > 227 * 1024) return (int)cudaErrorInvalidValue;
    auto kern = f32 ? (vec ? gqa_rows_kernel<float, 4> : gqa_rows_kernel<float, 1>)
                    : (vec ? gqa_rows_kernel<bf16, 4> : gqa_rows_kernel<bf16, 1>);
    if (sm > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, sm);
        if (e != cudaSuccess) return (int)e;
    }
    return (int)launch_pdl(kern, dim3(a.n), dim3(256), sm, st, a);
}

PIE_API int pie_head_rows(const HeadRowsArgs* args, int f32, cudaStream_t st) {
    const HeadRowsArgs& a = *args;
    if (a.n <= 0) return 0;
    if (a.group > a.group_pad || a.heads != a.kv_heads * a.group || a.dim > a.D || a.vdim > a.D || a.rot_dims % 2 || a.rot_dims > a.dim ||
        a.page_size <= 0 || a.temp_every < 0 || (!a.q_norm) != (!a.k_norm))
        return (int)cudaErrorInvalidValue;
    auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.D % 4 == 0 && a.ld % 4 == 0 && aligned(a.q) && aligned(a.k) && aligned(a.v) &&
                     aligned(a.q_norm) && aligned(a.k_norm) && aligned(a.q_out) && aligned(a.cache);
    const int sm = ((a.rot_dims + 3) / 4 * 4 + 8 * ((a.dim + 3) / 4 * 4)) * 4;
    if (sm > 48 * 1024) return (int)cudaErrorInvalidValue;
    auto kern = f32 ? (vec ? head_rows_kernel<float, 4> : head_rows_kernel<float, 1>)
                    : (vec ? head_rows_kernel<bf16, 4> : head_rows_kernel<bf16, 1>);
    return (int)launch_pdl(kern, dim3(a.n), dim3(256), sm, st, a);
}

PIE_API int pie_gqa_any(const GqaAnyArgs* args, int f32, cudaStream_t st) {
    const GqaAnyArgs& a = *args;
    if (a.n <= 0) return 0;
    if (a.hkv <= 0 || a.hq % a.hkv || a.D > 1024 || a.page_size <= 0 || a.keep_first < 0 || (a.planes != 1 && a.planes != 2) ||
        (a.pool && (a.pool < 0 || !a.means || a.window_left < 0)))
        return (int)cudaErrorInvalidValue;
    const dim3 grid((unsigned)(((long)a.n * a.hq + 3) / 4));
#define GO(T_, M_) return (int)launch_pdl(gqa_any_kernel<T_, M_>, grid, dim3(128), 0, st, a)
#define GO_M(T_) \
    if (a.D <= 64) GO(T_, 2); if (a.D <= 128) GO(T_, 4); if (a.D <= 256) GO(T_, 8); if (a.D <= 512) GO(T_, 16); GO(T_, 32)
    if (f32) { GO_M(float); }
    GO_M(bf16);
#undef GO_M
#undef GO
}

// 1 when decode (and 64-row prefill) attention have a tensor-core kernel for the shape.
PIE_API int pie_gqa_mma_supported(int group, int head_dim, int page_size) {
    const bool g = group == 1 || group == 2 || group == 4 || group == 8 || group == 16;
    return g && page_size % 16 == 0 && (head_dim == 64 || head_dim == 128 || (head_dim == 256 && group <= 8)) ? 1 : 0;
}
