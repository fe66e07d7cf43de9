// Latent attention in the absorbed form on the tensor cores (mma.sync, bf16): keys and values of every head are the
// cached rows themselves, so a tile of cache rows is read once into shared memory and serves all heads as K and as V.
//
// One CTA takes a work item - a span of one request's keys for its single decoded token (split-KV), or a few query tokens
// of a prefill - and packs (token, head) into 16 * MT rows. Per 64 keys: S = Q K^T with the rows split over MT warps and
// the keys over the other warps, softmax over shared memory with several threads per row, O += P V with the latent's
// columns split over the eight warps. The cache rows arrive by cp.async in a ring of stages.
// Also here: the merge of split spans, and the small products around the attention.
#include "latent_args.cuh"

namespace pie {

__device__ __forceinline__ uint32_t la_smem(const void* p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void la_cp16(uint32_t dst, const void* src, bool ok) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(dst), "l"(src), "r"(ok ? 16 : 0) : "memory");
}
__device__ __forceinline__ void la_commit() { asm volatile("cp.async.commit_group;\n" ::: "memory"); }
template <int N> __device__ __forceinline__ void la_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N) : "memory"); }
__device__ __forceinline__ void la_ldm4(uint32_t (&r)[4], uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void la_ldm2(uint32_t& r0, uint32_t& r1, uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x2.shared.b16 {%0,%1}, [%2];\n" : "=r"(r0), "=r"(r1) : "r"(a));
}
__device__ __forceinline__ void la_ldm4t(uint32_t (&r)[4], uint32_t a) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void la_mma(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ float la_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

constexpr int LA_BK = 64;          // keys per tile
constexpr int LA_MAX_STAGES = 4;

// Bytes of the parts of shared memory in front of the ring, and of one stage.
__host__ __device__ constexpr int la_rows(int mt) { return 16 * mt; }
__host__ __device__ inline int la_ldk(int row) { return row + 8; }          // odd multiple of 16 bytes mod 128: no bank conflicts
__host__ __device__ inline int la_lds(int mt) { return LA_BK + 256 / la_rows(mt); }
__host__ __device__ inline int la_fixed_bytes(int mt, int row) {
    return la_rows(mt) * (la_ldk(row) * 2 + la_lds(mt) * 4 + (LA_BK + 8) * 2 + 5 * 4);
}
__host__ __device__ inline int la_stage_bytes(int row) { return LA_BK * la_ldk(row) * 2; }

// MT: 16-row tiles of packed (token, head) rows. NTW: 8-column tiles of the latent per warp (8 warps).
template <int MT, int NTW>
__global__ void __launch_bounds__(256, (MT * NTW <= 8) ? 2 : 1) latent_attn_mma_kernel(const LatentMmaArgs a) {
    constexpr int ROWS = la_rows(MT), WN = 8 / MT, TPR = 256 / ROWS, VPT = LA_BK / TPR, LDS = LA_BK + TPR, LDP = LA_BK + 8;
    extern __shared__ __align__(16) uint8_t la_raw[];
    const int ldk = la_ldk(a.row);
    bf16* q_s = reinterpret_cast<bf16*>(la_raw);
    bf16* p_s = q_s + ROWS * ldk;
    float* s_s = reinterpret_cast<float*>(p_s + ROWS * LDP);
    float* alpha_s = s_s + ROWS * LDS;
    float* m_s = alpha_s + ROWS;
    float* l_s = m_s + ROWS;
    int* lo_s = reinterpret_cast<int*>(l_s + ROWS);
    int* lim_s = lo_s + ROWS;
    bf16* ring = reinterpret_cast<bf16*>(la_raw + la_fixed_bytes(MT, a.row));
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int chunks = a.row >> 3, stage_elems = LA_BK * ldk, lrow = warp * 8 + (lane >> 2);
    const bool prefill = a.item_end == nullptr;
    const int hg = min(a.heads, ROWS), h0 = blockIdx.y * hg, hn = min(hg, a.heads - h0);
    const int tq = prefill ? ROWS / hg : 1;
    pdl_trigger();
    pdl_wait();
    const int item1 = prefill ? a.items : min(a.cta_items[blockIdx.x + 1], a.max_items), step = prefill ? gridDim.x : 1;

    for (int item = prefill ? blockIdx.x : a.cta_items[blockIdx.x]; item < item1; item += step) {
        const int r = a.item_req[item];
        if (r < 0 || r >= a.reqs) continue;
        const int q_base = a.qo_indptr[r], qlen = a.qo_indptr[r + 1] - q_base;
        const int qs = prefill ? a.item_start[item] : 0;
        const int kv_len = a.kv_lens[r], past = kv_len - qlen;
        const int tn = min(tq, qlen - qs), used = tn * hn;        // packed rows: token i, head h at i * hn + h
        const uint32_t* bits = a.mask_bits ? a.mask_bits + a.mask_word_indptr[r] : nullptr;
        const int words = (kv_len + 31) >> 5;
        // keys of this item that some row can see
        int k_lo = max(0, past + qs - a.window_left), k_hi = bits ? kv_len : past + qs + tn;
        if (!prefill) {
            k_lo = max(k_lo, a.item_start[item]);
            k_hi = min(k_hi, a.item_end[item]);
        }
        const int tiles = k_hi > k_lo ? (k_hi - k_lo + LA_BK - 1) / LA_BK : 0;
        const int* pages = a.page_indices + a.kv_page_indptr[r];

        // a warp brings eight rows, four lanes to a row; the page of a thread's next row is looked up one tile ahead
        auto page_of = [&](int t) { return t < tiles ? pages[min(k_lo + t * LA_BK + lrow, k_hi - 1) >> a.page_shift] : 0; };
        int next_page = page_of(0);
        auto load_tile = [&](int t) {
            if (t < tiles) {
                const int key = k_lo + t * LA_BK + lrow, kk = min(key, k_hi - 1);
                const bf16* src = static_cast<const bf16*>(a.cache) +
                                  (((size_t)next_page << a.page_shift) + (kk & (a.page_size - 1))) * a.cache_row;
                const uint32_t dst = la_smem(ring + (t % a.stages) * stage_elems + lrow * ldk);
                const bool ok = key < k_hi;
                next_page = page_of(t + 1);
#pragma unroll 3
                for (int c = lane & 3; c < chunks; c += 4) la_cp16(dst + c * 16, src + c * 8, ok);
            }
            la_commit();
        };
        __syncthreads();                                          // the previous item is done with shared memory
        for (int row = lrow; row < ROWS; row += 64) {
            const bool ok = row < used;
            const int tok = ok ? row / hn : 0, h = ok ? row - tok * hn : 0;
            const bf16* src = static_cast<const bf16*>(a.q) + ((size_t)(q_base + qs + tok) * a.heads + h0 + h) * a.row;
            for (int c = lane & 3; c < chunks; c += 4) la_cp16(la_smem(q_s + row * ldk) + c * 16, src + c * 8, ok);
        }
        if (tid < ROWS) {
            const int pos = past + qs + tid / hn;
            lo_s[tid] = max(pos - a.window_left, prefill ? 0 : a.item_start[item]);
            lim_s[tid] = tid < used ? (bits ? k_hi : min(pos + 1, k_hi)) : 0;
        }
        for (int s = 0; s < a.stages - 1; ++s) load_tile(s);      // the first group also holds Q

        float o[MT][NTW][4];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int n = 0; n < NTW; ++n) o[m][n][0] = o[m][n][1] = o[m][n][2] = o[m][n][3] = 0.f;
        float row_m = -INFINITY, row_l = 0.f;                     // of softmax row tid / TPR
        const int wm = warp % MT, wn = warp / MT;

        for (int t = 0; t < tiles; ++t) {
            if (a.stages == 4) la_wait<2>(); else if (a.stages == 3) la_wait<1>(); else la_wait<0>();
            __syncthreads();
            load_tile(t + a.stages - 1);
            const bf16* k_s = ring + (t % a.stages) * stage_elems;
            // ---- S: rows [16 wm, +16), keys [wn * 8 MT, +8 MT)
            float s[MT][4], s2[MT][4];                            // two chains: even and odd k steps
#pragma unroll
            for (int n = 0; n < MT; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[n][e] = s2[n][e] = 0.f;
            const uint32_t qa = la_smem(q_s + (wm * 16 + (lane & 15)) * ldk + (lane >> 4) * 8);
            const int key0 = wn * 8 * MT;
            const uint32_t kb = MT == 1 ? la_smem(k_s + (key0 + (lane & 7)) * ldk + ((lane >> 3) & 1) * 8)
                                        : la_smem(k_s + (key0 + (lane & 7) + ((lane >> 4) << 3)) * ldk + ((lane >> 3) & 1) * 8);
            // KB k steps at a time: their fragments are all on the way before the first product needs one
            constexpr int KB = MT == 4 ? 2 : 3;
            const int ksteps = a.row >> 4;
            for (int k0 = 0; k0 < ksteps; k0 += KB) {
                uint32_t fa[KB][4], fb[KB][MT == 1 ? 1 : MT / 2][4];
#pragma unroll
                for (int i = 0; i < KB; ++i) {
                    if (k0 + i < ksteps) {
                        la_ldm4(fa[i], qa + (k0 + i) * 32);
                        if constexpr (MT == 1) {
                            la_ldm2(fb[i][0][0], fb[i][0][1], kb + (k0 + i) * 32);
                        } else {
#pragma unroll
                            for (int n = 0; n < MT / 2; ++n) la_ldm4(fb[i][n], kb + n * 16 * ldk * 2 + (k0 + i) * 32);
                        }
                    }
                }
#pragma unroll
                for (int i = 0; i < KB; ++i) {
                    if (k0 + i < ksteps) {
                        float(&acc)[MT][4] = (i & 1) ? s2 : s;
                        if constexpr (MT == 1) {
                            la_mma(acc[0], fa[i], fb[i][0][0], fb[i][0][1]);
                        } else {
#pragma unroll
                            for (int n = 0; n < MT / 2; ++n) {
                                la_mma(acc[2 * n], fa[i], fb[i][n][0], fb[i][n][1]);
                                la_mma(acc[2 * n + 1], fa[i], fb[i][n][2], fb[i][n][3]);
                            }
                        }
                    }
                }
            }
#pragma unroll
            for (int n = 0; n < MT; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[n][e] += s2[n][e];
#pragma unroll
            for (int n = 0; n < MT; ++n) {
                float* d = s_s + (wm * 16 + (lane >> 2)) * LDS + key0 + n * 8 + (lane & 3) * 2;
                *reinterpret_cast<float2*>(d) = make_float2(s[n][0], s[n][1]);
                *reinterpret_cast<float2*>(d + 8 * LDS) = make_float2(s[n][2], s[n][3]);
            }
            __syncthreads();
            // ---- softmax: TPR threads per row
            {
                // a thread has VPT / 2 pairs of neighbouring keys, 2 TPR apart; scores stay unscaled, the maximum too
                const int row = tid / TPR, sub = tid % TPR, kbase = k_lo + t * LA_BK;
                const int lo = lo_s[row] - kbase, lim = lim_s[row] - kbase;
                const uint32_t* rb = bits ? bits + (size_t)(qs + min(row / hn, tn - 1)) * words : nullptr;
                float v[VPT], mx = -INFINITY;
#pragma unroll
                for (int i = 0; i < VPT; i += 2) {
                    const float2 x = *reinterpret_cast<const float2*>(s_s + row * LDS + sub * 2 + i * TPR);
                    v[i] = x.x;
                    v[i + 1] = x.y;
                }
                if (!__all_sync(0xffffffffu, lo <= 0 && lim >= LA_BK && !rb)) {
#pragma unroll
                    for (int i = 0; i < VPT; ++i) {
                        const int c = sub * 2 + (i & 1) + (i & ~1) * TPR;
                        bool see = c >= lo && c < lim;
                        if (rb && see) see = rb[(kbase + c) >> 5] >> ((kbase + c) & 31) & 1u;
                        if (!see) v[i] = -INFINITY;
                    }
                }
#pragma unroll
                for (int i = 0; i < VPT; ++i) mx = fmaxf(mx, v[i]);
#pragma unroll
                for (int d = TPR / 2; d > 0; d >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
                const float mn = fmaxf(row_m, mx), base = mn == -INFINITY ? 0.f : mn * a.scale_log2;
                const float al = la_exp2(fmaf(row_m, a.scale_log2, -base));      // 0 while nothing was seen
                float sum = 0.f;
#pragma unroll
                for (int i = 0; i < VPT; i += 2) {
                    const float p0 = la_exp2(fmaf(v[i], a.scale_log2, -base)), p1 = la_exp2(fmaf(v[i + 1], a.scale_log2, -base));
                    sum += p0 + p1;
                    *reinterpret_cast<bf162*>(p_s + row * LDP + sub * 2 + i * TPR) = __floats2bfloat162_rn(p0, p1);
                }
#pragma unroll
                for (int d = TPR / 2; d > 0; d >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, d);
                row_m = mn;
                row_l = row_l * al + sum;
                if (sub == 0) alpha_s[row] = al;
            }
            __syncthreads();
            // ---- O += P V: latent columns [warp * 8 NTW, +8 NTW)
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                const float a0 = alpha_s[m * 16 + (lane >> 2)], a1 = alpha_s[m * 16 + 8 + (lane >> 2)];
                if (__all_sync(0xffffffffu, a0 == 1.f && a1 == 1.f)) continue;      // no row's maximum moved
#pragma unroll
                for (int n = 0; n < NTW; ++n) {
                    o[m][n][0] *= a0;
                    o[m][n][1] *= a0;
                    o[m][n][2] *= a1;
                    o[m][n][3] *= a1;
                }
            }
            const int col0 = warp * 8 * NTW;
            if (col0 < a.rank_pad) {
#pragma unroll
                for (int k = 0; k < LA_BK / 16; ++k) {
                    uint32_t fp[MT][4];
#pragma unroll
                    for (int m = 0; m < MT; ++m)
                        la_ldm4(fp[m], la_smem(p_s + (m * 16 + (lane & 15)) * LDP + k * 16 + (lane >> 4) * 8));
                    const uint32_t va = la_smem(k_s + (k * 16 + (lane & 15)) * ldk + col0 + (lane >> 4) * 8);
#pragma unroll
                    for (int n = 0; n < NTW; n += 2) {
                        if (col0 + n * 8 < a.rank_pad) {
                            uint32_t fv[4];
                            la_ldm4t(fv, va + n * 16);
#pragma unroll
                            for (int m = 0; m < MT; ++m) {
                                la_mma(o[m][n], fp[m], fv[0], fv[1]);
                                la_mma(o[m][n + 1], fp[m], fv[2], fv[3]);
                            }
                        }
                    }
                }
            }
        }
        la_wait<0>();
        if (tid % TPR == 0) {
            m_s[tid / TPR] = row_m * a.scale_log2;
            l_s[tid / TPR] = row_l;
        }
        __syncthreads();
        const bool whole = prefill || a.req_item_indptr[r + 1] - a.req_item_indptr[r] == 1;
        float* lse = a.scratch + (size_t)a.max_items * a.heads * a.rank_pad;
        if (!whole && tid < used)
            lse[(size_t)item * a.heads + h0 + tid] = l_s[tid] > 0.f ? m_s[tid] + log2f(l_s[tid]) : -INFINITY;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int row = m * 16 + half * 8 + (lane >> 2);
                if (row >= used) continue;
                const float inv = l_s[row] > 0.f ? 1.f / l_s[row] : 0.f;
                const int tok = row / hn, h = h0 + row - tok * hn;
#pragma unroll
                for (int n = 0; n < NTW; ++n) {
                    const int col = warp * 8 * NTW + n * 8 + (lane & 3) * 2;
                    if (col >= a.rank_pad) continue;
                    const float x = o[m][n][half * 2] * inv, y = o[m][n][half * 2 + 1] * inv;
                    if (whole)
                        *reinterpret_cast<bf162*>(static_cast<bf16*>(a.out) + ((size_t)(q_base + qs + tok) * a.heads + h) * a.rank_pad + col) =
                            __floats2bfloat162_rn(x, y);
                    else
                        *reinterpret_cast<float2*>(a.scratch + ((size_t)item * a.heads + h) * a.rank_pad + col) = make_float2(x, y);
                }
            }
    }
}

// Decode: combine the spans of requests that were split. One warp per (request, head).
__global__ void __launch_bounds__(256) latent_merge_kernel(const float* __restrict__ scratch, const int* __restrict__ req_item_indptr,
                                                           bf16* __restrict__ out, int heads, int rank_pad, int max_items, int reqs) {
    pdl_trigger();
    pdl_wait();
    const int w = (blockIdx.x * 256 + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    if (w >= reqs * heads) return;
    const int r = w / heads, h = w - r * heads;
    const int i0 = req_item_indptr[r], i1 = min(req_item_indptr[r + 1], max_items);
    if (i1 - i0 < 2) return;
    const float* lse = scratch + (size_t)max_items * heads * rank_pad;
    float mx = -INFINITY, sum = 0.f;
    for (int i = i0; i < i1; ++i) mx = fmaxf(mx, lse[(size_t)i * heads + h]);
    const float base = mx == -INFINITY ? 0.f : mx;
    for (int i = i0; i < i1; ++i) sum += exp2f(lse[(size_t)i * heads + h] - base);
    const float inv = sum > 0.f ? 1.f / sum : 0.f;
    for (int c = lane * 4; c < rank_pad; c += 128) {
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
        for (int i = i0; i < i1; ++i) {
            const float f = exp2f(lse[(size_t)i * heads + h] - base) * inv;
            const float4 v = *reinterpret_cast<const float4*>(scratch + ((size_t)i * heads + h) * rank_pad + c);
            acc.x += f * v.x; acc.y += f * v.y; acc.z += f * v.z; acc.w += f * v.w;
        }
        bf162* d = reinterpret_cast<bf162*>(out + ((size_t)r * heads + h) * rank_pad + c);
        d[0] = __floats2bfloat162_rn(acc.x, acc.y);
        d[1] = __floats2bfloat162_rn(acc.z, acc.w);
    }
}

// ----------------------------------------------- small products around them
// out[t, h, :] = W_h x[t, h, :]: per-head factors, or a product split along K (a "head" then is a K range of length k, and
// out collects 32-bit partial sums).
struct SmallProductArgs {
    const void* x;                 // x[t, h, k] at t * x_tok + h * x_head + k
    const void* w;                 // w[h, m, k] at h * w_head + m * w_row + k
    void* out;                     // out[t, h, m] at t * out_tok + h * out_head + m
    long x_tok, x_head, w_head, w_row, out_tok, out_head;
    int n, heads, m, k, k_total;   // k_total > 0: the last head's range ends there
    int out_f32;
};

constexpr int PH_T = 64, PH_K = 64, PH_LD = PH_K + 8;

// One CTA per (64 tokens, 64 outputs, head); four warps of 16 tokens, K in double-buffered chunks of 64. VEC: every row
// starts on a 16-byte boundary and the K ranges are multiples of 8, else the tiles are filled element by element.
template <bool VEC>
__global__ void __launch_bounds__(128) small_product_kernel(const SmallProductArgs a) {
    __shared__ __align__(16) bf16 x_s[2][PH_T * PH_LD];
    __shared__ __align__(16) bf16 w_s[2][PH_T * PH_LD];
    const int t0 = blockIdx.x * PH_T, m0 = blockIdx.y * PH_T, h = blockIdx.z;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int kn = a.k_total > 0 ? min(a.k, a.k_total - h * a.k) : a.k;
    const bf16* x = static_cast<const bf16*>(a.x) + (size_t)h * a.x_head;
    const bf16* w = static_cast<const bf16*>(a.w) + (size_t)h * a.w_head;
    auto load_w = [&](int k0, int b) {
        if constexpr (VEC) {
            for (int i = tid; i < PH_T * (PH_K / 8); i += 128) {
                const int r = i >> 3, c = (i & 7) * 8;
                const bool ok = k0 + c < kn && m0 + r < a.m;
                la_cp16(la_smem(w_s[b] + r * PH_LD + c), w + (size_t)(ok ? m0 + r : 0) * a.w_row + (ok ? k0 + c : 0), ok);
            }
        } else {
            for (int i = tid; i < PH_T * PH_K; i += 128) {
                const int r = i / PH_K, c = i - r * PH_K;
                w_s[b][r * PH_LD + c] = k0 + c < kn && m0 + r < a.m ? w[(size_t)(m0 + r) * a.w_row + k0 + c] : __float2bfloat16(0.f);
            }
        }
    };
    auto load_x = [&](int k0, int b) {
        if constexpr (VEC) {
            for (int i = tid; i < PH_T * (PH_K / 8); i += 128) {
                const int r = i >> 3, c = (i & 7) * 8;
                const bool ok = k0 + c < kn && t0 + r < a.n;
                la_cp16(la_smem(x_s[b] + r * PH_LD + c), x + (size_t)(ok ? t0 + r : 0) * a.x_tok + (ok ? k0 + c : 0), ok);
            }
        } else {
            for (int i = tid; i < PH_T * PH_K; i += 128) {
                const int r = i / PH_K, c = i - r * PH_K;
                x_s[b][r * PH_LD + c] = k0 + c < kn && t0 + r < a.n ? x[(size_t)(t0 + r) * a.x_tok + k0 + c] : __float2bfloat16(0.f);
            }
        }
    };
    float acc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
    pdl_trigger();
    load_w(0, 0);                  // weights depend on nothing
    pdl_wait();
    load_x(0, 0);
    la_commit();
    const int chunks = (kn + PH_K - 1) / PH_K;
    for (int j = 0; j < chunks; ++j) {
        const int b = j & 1;
        if (j + 1 < chunks) {
            load_w((j + 1) * PH_K, b ^ 1);
            load_x((j + 1) * PH_K, b ^ 1);
            la_commit();
            la_wait<1>();
        } else {
            la_wait<0>();
        }
        __syncthreads();
        const uint32_t xa = la_smem(x_s[b] + (warp * 16 + (lane & 15)) * PH_LD + (lane >> 4) * 8);
        const uint32_t wb = la_smem(w_s[b] + ((lane & 7) + ((lane >> 4) << 3)) * PH_LD + ((lane >> 3) & 1) * 8);
#pragma unroll
        for (int k = 0; k < PH_K / 16; ++k) {
            uint32_t fa[4];
            la_ldm4(fa, xa + k * 32);
#pragma unroll
            for (int n = 0; n < 8; n += 2) {
                uint32_t fb[4];
                la_ldm4(fb, wb + n * 8 * PH_LD * 2 + k * 32);
                la_mma(acc[n], fa, fb[0], fb[1]);
                la_mma(acc[n + 1], fa, fb[2], fb[3]);
            }
        }
        __syncthreads();
    }
    const bool pair = ((a.out_tok | a.out_head | a.m) & 1) == 0 && ((uintptr_t)a.out & 7) == 0;
#pragma unroll
    for (int n = 0; n < 8; ++n)
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const int t = t0 + warp * 16 + (lane >> 2) + half * 8, m = m0 + n * 8 + (lane & 3) * 2;
            if (t >= a.n || m >= a.m) continue;
            const size_t at = (size_t)t * a.out_tok + (size_t)h * a.out_head + m;
            const float p = acc[n][half * 2], q = acc[n][half * 2 + 1];
            if (a.out_f32) {
                float* d = static_cast<float*>(a.out) + at;
                if (pair) *reinterpret_cast<float2*>(d) = make_float2(p, q);
                else { d[0] = p; if (m + 1 < a.m) d[1] = q; }
            } else {
                bf16* d = static_cast<bf16*>(a.out) + at;
                if (pair) *reinterpret_cast<bf162*>(d) = __floats2bfloat162_rn(p, q);
                else { d[0] = __float2bfloat16(p); if (m + 1 < a.m) d[1] = __float2bfloat16(q); }
            }
        }
}

}  // namespace pie

using namespace pie;

// 16-row tiles of packed rows per CTA for a head count and latent width; 0: the kernel does not cover the shape.
PIE_API int pie_latent_attn_mma_tiles(int heads, int row, int rank_pad) {
    if (heads < 1 || rank_pad > 512 || rank_pad % 16 || row % 16) return 0;
    int mt = heads <= 16 ? 1 : (heads <= 32 ? 2 : 4);
    while (mt > 1 && (rank_pad > 256 ? mt > 2 : false)) mt >>= 1;
    while (mt > 1 && la_fixed_bytes(mt, row) + 2 * la_stage_bytes(row) > 227 * 1024) mt >>= 1;
    return la_fixed_bytes(mt, row) + 2 * la_stage_bytes(row) <= 227 * 1024 ? mt : 0;
}

// The merge of a decode launch's split requests (also for the tcgen05 kernel).
int pie_latent_merge(const LatentMmaArgs& a, cudaStream_t st) {
    const cudaError_t e = launch_pdl(latent_merge_kernel, dim3((a.reqs * a.heads + 7) / 8), dim3(256), 0, st, (const float*)a.scratch,
                                     a.req_item_indptr, (bf16*)a.out, a.heads, a.rank_pad, a.max_items, a.reqs);
    return (int)(e != cudaSuccess ? e : cudaGetLastError());
}

PIE_API int pie_latent_attn_mma(const LatentMmaArgs* args, int num_ctas, cudaStream_t st) {
    LatentMmaArgs a = *args;
    const int mt = pie_latent_attn_mma_tiles(a.heads, a.row, a.rank_pad);
    if (!mt || a.rank_pad > a.row || a.page_size != 1 << a.page_shift || a.row > a.cache_row || a.cache_row % 8 ||
        num_ctas <= 0)
        return (int)cudaErrorInvalidValue;
    if (a.item_end && (!a.scratch || !a.req_item_indptr || !a.cta_items)) return (int)cudaErrorInvalidValue;
    if (!a.item_end && a.items <= 0) return 0;
    const int fixed = la_fixed_bytes(mt, a.row), stage = la_stage_bytes(a.row);
    const int ntw = a.rank_pad <= 128 ? 2 : (a.rank_pad <= 256 ? 4 : 8);
    // two CTAs per SM where the registers allow it: half of the shared memory each
    const int budget = (mt * ntw <= 8 ? 113 : 227) * 1024;
    int stages = (budget - fixed) / stage;
    if (stages < 2) stages = 2;
    a.stages = stages > LA_MAX_STAGES ? LA_MAX_STAGES : stages;
    const int smem = fixed + a.stages * stage;
    const int hg = a.heads < la_rows(mt) ? a.heads : la_rows(mt);
    const int gx = a.item_end ? num_ctas : (a.items < num_ctas ? a.items : num_ctas);
    const dim3 grid(gx, (a.heads + hg - 1) / hg);
#define GO(M_, N_)                                                                                                        \
    {                                                                                                                     \
        cudaError_t e = cudaFuncSetAttribute(latent_attn_mma_kernel<M_, N_>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem); \
        if (e != cudaSuccess) return (int)e;                                                                              \
        e = launch_pdl(latent_attn_mma_kernel<M_, N_>, grid, dim3(256), (size_t)smem, st, a);                             \
        if (e != cudaSuccess) return (int)e;                                                                              \
    }
    if (mt == 1) { if (ntw == 2) GO(1, 2) else if (ntw == 4) GO(1, 4) else GO(1, 8) }
    else if (mt == 2) { if (ntw == 2) GO(2, 2) else if (ntw == 4) GO(2, 4) else GO(2, 8) }
    else { if (ntw == 2) GO(4, 2) else if (ntw == 4) GO(4, 4) else return (int)cudaErrorInvalidValue; }
#undef GO
    if (a.item_end) return pie_latent_merge(a, st);
    return (int)cudaGetLastError();
}

PIE_API int pie_small_product(const SmallProductArgs* args, cudaStream_t st) {
    const SmallProductArgs& a = *args;
    if (a.n <= 0 || a.m <= 0 || a.heads <= 0) return 0;
    if (a.k <= 0 || (a.k_total > 0 && (long)(a.heads - 1) * a.k >= a.k_total)) return (int)cudaErrorInvalidValue;
    const bool vec = a.k % 8 == 0 && a.k_total % 8 == 0 && a.w_row % 8 == 0 && a.w_head % 8 == 0 && ((uintptr_t)a.w & 15) == 0 &&
                     a.x_tok % 8 == 0 && a.x_head % 8 == 0 && ((uintptr_t)a.x & 15) == 0;
    const dim3 grid((a.n + PH_T - 1) / PH_T, (a.m + PH_T - 1) / PH_T, a.heads);
    const cudaError_t e = vec ? launch_pdl(small_product_kernel<true>, grid, dim3(128), 0, st, a)
                              : launch_pdl(small_product_kernel<false>, grid, dim3(128), 0, st, a);
    return (int)(e != cudaSuccess ? e : cudaGetLastError());
}
