// Paged attention kernels on mma.sync m16n8k16 tiles, shared by the launchers of attention.cu and attention_bias.cu.
//
//  * paged_decode_attn: one query token per request, GQA heads of one KV head
//    packed as the rows of a 16-row tensor-core tile, split-KV over a host-built
//    list of (request, kv range) work items walked by a persistent grid (graph
//    safe: the item count is read from device memory), partial results merged
//    by a second kernel when a request has more than one item.
//  * paged_prefill_attn: ragged query lengths, causal or custom bit-mask,
//    optional sliding window, 64-row tiles of (query token, head-in-group).
//  Beside a sliding window the first `keep_first` keys stay visible; 16-key (prefill: 64-key) blocks without a visible key
//  are skipped.
//
// KV layer layout: [pages][2][Hkv][page_size][D] bf16 (K then V per page), so a
// (page, head) K or V block is one contiguous page_size*D*2-byte run.
// page_size must be a multiple of 16.
//
// Reference behaviour: driver/cuda/src/ops/attention_flashinfer.cu:301-312,714
// (decode, split-KV plan), :612,848,1075 (prefill, custom mask, window).
#pragma once
#include "common.cuh"

namespace pie {

__device__ __forceinline__ uint32_t smem_u32(const void* p) {
    return (uint32_t)__cvta_generic_to_shared(p);
}
__device__ __forceinline__ void ldsm_x4(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2,
                                        uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void ldsm_x4_t(uint32_t addr, uint32_t& r0, uint32_t& r1, uint32_t& r2,
                                          uint32_t& r3) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r0), "=r"(r1), "=r"(r2), "=r"(r3) : "r"(addr));
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0,
                                         uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, "
        "{%8,%9}, {%0,%1,%2,%3};\n"
        : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void cp_async16(uint32_t dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(dst), "l"(src));
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n"); }
template <int N>
__device__ __forceinline__ void cp_async_wait() {
    asm volatile("cp.async.wait_group %0;\n" ::"n"(N));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) {
    bf162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<uint32_t*>(&v);
}

// Byte offset of 16-byte chunk `chunk` of row `row` in a [rows][D] bf16 tile
// whose chunks are XOR-swizzled with the row index (bank-conflict-free ldmatrix).
template <int D>
__device__ __forceinline__ uint32_t swz(int row, int chunk) {
    return (uint32_t)(row * (D * 2) + ((chunk ^ (row & 7)) << 4));
}

template <int D>
struct AttnState {
    float o[D / 8][4];
    float m[2];
    float l[2];
    __device__ __forceinline__ void init() {
#pragma unroll
        for (int i = 0; i < D / 8; ++i) { o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f; }
        m[0] = m[1] = -INFINITY;
        l[0] = l[1] = 0.f;
    }
};

// One warp: S = Q(16 x D) K(16 tokens)^T, online softmax, O += P V.
// allow0/allow1: bit c set when token c of the block is visible to row g /
// row g+8 of the warp's tile (g = lane/4).
// CAP (Gemma-2's soft-capped scores): the scores pass through cap * tanh(s * sm_scale / cap) before the softmax;
// scale_log2 then carries sm_scale / cap and cap_log2 = cap * log2(e).
__device__ __forceinline__ float tanh_approx(float x) {
    float y;
    asm("tanh.approx.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// Soft cap without the short-cut of tanh.approx: (e^2x - 1) / (e^2x + 1), absolute error of a few 2^-24.
__device__ __forceinline__ float tanh_exp(float x) { return 1.f - __fdividef(2.f, 1.f + exp2f(2.8853900817779268f * x)); }

// Learned bias per distance (MODE_BIAS): entry n of a head's table is added to the capped score of the key n tokens back,
// in units of log2. p0 / p1: tables of the heads of rows g and g + 8; n0 / n1: their distances to token 0 of the block.
struct DistanceBias {
    const float *p0, *p1;
    int n0, n1, last;
};
enum AttnMode : int { MODE_PLAIN = 0, MODE_CAP = 1, MODE_BIAS = 2 };

template <int D, int MODE = MODE_PLAIN>
__device__ __forceinline__ void attn_block16(const uint32_t (&qf)[D / 16][4], uint32_t k_smem,
                                             uint32_t v_smem, float scale_log2, uint32_t allow0,
                                             uint32_t allow1, AttnState<D>& st, float cap_log2 = 0.f,
                                             const DistanceBias& db = DistanceBias{}) {
    const int lane = threadIdx.x & 31;
    const int mi = lane >> 3, r = lane & 7;
    float s[2][2][4];
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
        for (int b = 0; b < 2; ++b) s[a][b][0] = s[a][b][1] = s[a][b][2] = s[a][b][3] = 0.f;
    {
        const int token = r + (mi >> 1) * 8;
#pragma unroll
        for (int ks = 0; ks < D / 16; ++ks) {
            uint32_t b00, b01, b10, b11;
            ldsm_x4(k_smem + swz<D>(token, ks * 2 + (mi & 1)), b00, b01, b10, b11);
            mma_bf16(s[0][ks & 1], qf[ks], b00, b01);
            mma_bf16(s[1][ks & 1], qf[ks], b10, b11);
        }
    }
    const int t = lane & 3;
    float p[2][4];
    float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int tok = j * 8 + 2 * t + (e & 1);
            const uint32_t allow = (e >> 1) ? allow1 : allow0;
            float v = (s[j][0][e] + s[j][1][e]) * scale_log2;
            if (MODE == MODE_CAP) v = cap_log2 * tanh_approx(v);
            if (MODE == MODE_BIAS) {
                const int n = ((e >> 1) ? db.n1 : db.n0) - tok;
                v = fmaf(cap_log2, tanh_exp(v), __ldg(((e >> 1) ? db.p1 : db.p0) + min(max(n, 0), db.last)));
            }
            v = ((allow >> tok) & 1u) ? v : -INFINITY;
            p[j][e] = v;
            mx[e >> 1] = fmaxf(mx[e >> 1], v);
        }
    float alpha[2], mref[2];
#pragma unroll
    for (int h = 0; h < 2; ++h) {
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 1));
        mx[h] = fmaxf(mx[h], __shfl_xor_sync(0xffffffffu, mx[h], 2));
        const float mnew = fmaxf(st.m[h], mx[h]);
        mref[h] = (mnew == -INFINITY) ? 0.f : mnew;
        alpha[h] = exp2f(st.m[h] - mref[h]);
        st.m[h] = mnew;
    }
    float rs[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < 2; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            p[j][e] = exp2f(p[j][e] - mref[e >> 1]);
            rs[e >> 1] += p[j][e];
        }
    st.l[0] = st.l[0] * alpha[0] + rs[0];
    st.l[1] = st.l[1] * alpha[1] + rs[1];
#pragma unroll
    for (int n = 0; n < D / 8; ++n) {
        st.o[n][0] *= alpha[0];
        st.o[n][1] *= alpha[0];
        st.o[n][2] *= alpha[1];
        st.o[n][3] *= alpha[1];
    }
    uint32_t pa[4];
    pa[0] = pack_bf16(p[0][0], p[0][1]);
    pa[1] = pack_bf16(p[0][2], p[0][3]);
    pa[2] = pack_bf16(p[1][0], p[1][1]);
    pa[3] = pack_bf16(p[1][2], p[1][3]);
    {
        const int token = r + (mi & 1) * 8;
#pragma unroll
        for (int np = 0; np < D / 16; ++np) {
            uint32_t v0, v1, v2, v3;
            ldsm_x4_t(v_smem + swz<D>(token, np * 2 + (mi >> 1)), v0, v1, v2, v3);
            mma_bf16(st.o[2 * np], pa, v0, v1);
            mma_bf16(st.o[2 * np + 1], pa, v2, v3);
        }
    }
}

// Load the warp's 16 x D query tile fragments from a swizzled smem tile.
template <int D>
__device__ __forceinline__ void load_q_frags(uint32_t q_smem, int row0, uint32_t (&qf)[D / 16][4]) {
    const int lane = threadIdx.x & 31;
    const int mi = lane >> 3, r = lane & 7;
    const int row = row0 + r + (mi & 1) * 8;
#pragma unroll
    for (int ks = 0; ks < D / 16; ++ks)
        ldsm_x4(q_smem + swz<D>(row, ks * 2 + (mi >> 1)), qf[ks][0], qf[ks][1], qf[ks][2],
                qf[ks][3]);
}

// ------------------------------------------------------------------ decode
constexpr int DEC_WARPS = 4;
constexpr int DEC_STAGES = 3;

constexpr int DEC_OWN_STAGES = 4;      // of one tile each, see OWN below

template <int D, bool OWN = false>
constexpr int decode_smem_bytes() {
    return 16 * D * 2 + DEC_WARPS * (OWN ? DEC_OWN_STAGES : 2 * DEC_STAGES) * 16 * D * 2;
}

// CASCADE: shared-prefix items. A work item may then cover a KV range that up to 16 / G requests
// (the "members" of a tile: forks of one context, whose leading pages are the same physical pages)
// have in common: the Q tile holds the heads of all members (row = member * G + head), the keys and
// values of the range are read ONCE, and every member gets its own partial result. Partial results go
// to slots: a request's slots are [req_item_indptr[r], req_item_indptr[r + 1]) and a shared item with
// chunk index c fills slot req_item_indptr[member] + c of every member; an unshared item names its
// slot directly. The merge pass combines a request's slots as before.
//   item_slot  [items]  : chunk index (shared item) or slot (unshared item)
//   item_tile  [items]  : row of tile_members for a shared item, -1 otherwise
//   tile_members [tiles][16] : request of each member, -1 for unused rows
// Without CASCADE the three arrays are unused and slot == item index.
// MODE_BIAS: `bias` [hq][bias_pitch] holds BIAS_GUARD guard entries, the bias of every distance the window shows, and a
// guard again.
constexpr int BIAS_GUARD = 64;

// Where a layer's keys and values lie. planes 1: the values are the keys, pages hold them once ([pages][hkv][page][D]).
// POOL kernels: beside the window a query sees the mean key and value of every block of `pool` tokens wholly before it. A mean
// lies with the page of its block's last token, [pages][2][hkv][per_page][D], `per_page` = ceil(page / pool); prefill reads
// them gathered into 16-row pages, [pages][2][hkv][16][D], `first`[r] the first of request r.
struct KeyLayout {
    int planes = 2, pool = 0, per_page = 0;
    const bf16* means = nullptr;
    const int* first = nullptr;
};
// Means that a query at `pos` sees beside the window_left tokens before it.
__device__ __forceinline__ int means_seen(int pos, int window_left, int pool) { return max(0, pos - window_left) / pool; }
// Row of block b among the means of its page, and that page's place in the request's table.
__device__ __forceinline__ int mean_row(int b, int pool, int page_size, int& page_at) {
    page_at = ((b + 1) * pool - 1) / page_size;
    return b - page_at * page_size / pool;
}

// POOL: an item of a request takes its share of the 16-key tiles (means, then the window's tokens) whatever range the plan
// gave it, so that any plan spreads the work evenly.
// OWN: the values are the keys (planes 1); a stage then holds one tile, which leaves room for a third block per SM.
template <int D, int G, bool CASCADE, int MODE = MODE_PLAIN, bool POOL = false, bool OWN = false>
__global__ void __launch_bounds__(DEC_WARPS * 32, OWN && D <= 128 ? 3 : 1)
paged_decode_attn_kernel(const bf16* __restrict__ q, const bf16* __restrict__ kv_layer,
                         const int* __restrict__ page_indices,
                         const int* __restrict__ kv_page_indptr, const int* __restrict__ item_req,
                         const int* __restrict__ item_start, const int* __restrict__ item_end,
                         const int* __restrict__ req_item_indptr,
                         const int* __restrict__ num_items_ptr, bf16* __restrict__ out,
                         float* __restrict__ o_part, float* __restrict__ lse_part, int hq, int hkv,
                         int page_size, float scale_log2, int window_left,
                         const float* __restrict__ sinks_log2, int max_items, int num_reqs,
                         int* __restrict__ status, const int* __restrict__ item_slot,
                         const int* __restrict__ item_tile, const int* __restrict__ tile_members,
                         float cap_log2, const float* __restrict__ bias, int bias_pitch, int keep_first, const KeyLayout kl) {
    static_assert(G <= 16, "at most 16 query heads per KV head");
    constexpr int ROWS = CASCADE ? (16 / G) * G : G;      // rows of the Q tile in use
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr int CH = D / 8;              // 16-byte chunks per row
    constexpr int TILE_BYTES = 16 * D * 2; // one 16-token K or V tile
    constexpr int STAGES = OWN ? DEC_OWN_STAGES : DEC_STAGES, STAGE_BYTES = (OWN ? 1 : 2) * TILE_BYTES;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t q_smem = smem_u32(smem);
    const uint32_t warp_smem = q_smem + TILE_BYTES + warp * STAGES * STAGE_BYTES;
    pdl_trigger();
    pdl_wait();
    // The work count lives in device memory (graph replays refresh it): never trust it past the
    // size of the scratch the launcher was given. Work beyond that is dropped and reported.
    int n_items = *num_items_ptr;
    if (n_items > max_items || n_items < 0) {
        if (threadIdx.x == 0 && blockIdx.x == 0 && status) atomicCAS(status, 0, PIE_ERR_BOUNDS);
        n_items = n_items < 0 ? 0 : max_items;
    }
    const long total = (long)n_items * hkv;

    for (long w = blockIdx.x; w < total; w += gridDim.x) {
        const int it = (int)(w / hkv), h = (int)(w - (long)it * hkv);
        const int req = item_req[it];
        if (req < 0 || req >= num_reqs) {      // block-uniform: a corrupt item is skipped, not followed
            if (threadIdx.x == 0 && status) atomicCAS(status, 0, PIE_ERR_BOUNDS);
            continue;
        }
        const int kv_start = POOL ? 0 : item_start[it], kv_end = item_end[POOL ? req_item_indptr[req + 1] - 1 : it];
        const int tile = CASCADE ? item_tile[it] : -1;
        const int* members = (CASCADE && tile >= 0) ? tile_members + (size_t)tile * 16 : nullptr;
        // sliding window: the query sits at position kv_len - 1 (kv_len = end of the request's last
        // item) and sees keys >= kv_len - 1 - window_left; items start on a 16-token boundary below that
        // (plans with shared items carry no window)
        const int kv_lo = (!CASCADE && window_left >= 0)
                              ? max(0, item_end[req_item_indptr[req + 1] - 1] - 1 - window_left) : 0;
        __syncthreads();  // previous item's merge reads are done
        // Q tile: rows < G are the heads of this KV head (of member row / G in a shared item), the rest zeros
        for (int c = threadIdx.x; c < 16 * CH; c += blockDim.x) {
            const int row = c / CH, col = c - row * CH;
            uint4 v = make_uint4(0, 0, 0, 0);
            if (row < ROWS) {
                int rq = req;
                if (CASCADE) {
                    const int mem = row / G;
                    rq = members ? members[mem] : (mem == 0 ? req : -1);
                    if (rq >= num_reqs) rq = -1;
                }
                if (rq >= 0)
                    v = *reinterpret_cast<const uint4*>(q + ((size_t)rq * hq + h * G + (row % G)) * D + col * 8);
            }
            *reinterpret_cast<uint4*>(smem + swz<D>(row, col)) = v;
        }
        __syncthreads();
        uint32_t qf[D / 16][4];
        load_q_frags<D>(q_smem, 0, qf);

        AttnState<D> st;
        st.init();
        // blocks [hidden, hidden + gap) of the item lie between the kept first keys and the window
        const int nb_item = (kv_end - kv_start + 15) >> 4;
        const int hidden = min(nb_item, max(0, (keep_first - kv_start + 15) >> 4));
        const int gap = max(0, min(nb_item, (kv_lo - kv_start) >> 4) - hidden);
        // POOL: this item's tiles are first_tile .. first_tile + nb_total - 1, tile t < mean_tiles being sixteen means
        const int n_means = POOL ? means_seen(kv_end - 1, window_left, kl.pool) : 0, mean_tiles = (n_means + 15) >> 4;
        int first_tile = 0, nb_total = nb_item - gap;
        if (POOL) {
            const long all = mean_tiles + nb_total;
            const int i0 = req_item_indptr[req], parts = req_item_indptr[req + 1] - i0;
            first_tile = (int)(all * (it - i0) / parts);
            nb_total = (int)(all * (it - i0 + 1) / parts) - first_tile;
        }
        auto block_start = [&](int b) {
            if (POOL) return (first_tile + b - mean_tiles + gap) * 16;
            return kv_start + (b < hidden ? b : b + gap) * 16;
        };
        const int my_count = nb_total > warp ? (nb_total - warp + DEC_WARPS - 1) / DEC_WARPS : 0;
        const int* pages = page_indices + kv_page_indptr[req];

        auto issue = [&](int j) {
            if (POOL && first_tile + warp + DEC_WARPS * j < mean_tiles) {
                // lane r knows where mean r of the tile lies
                const int b = (first_tile + warp + DEC_WARPS * j) * 16 + (lane & 15);
                long at = -1;
                if (b < n_means) {
                    int pg;
                    const int row = mean_row(b, kl.pool, page_size, pg);
                    at = ((((long)pages[pg] * 2) * hkv + h) * kl.per_page + row) * D;
                }
                const uint32_t kdst = warp_smem + (j % STAGES) * STAGE_BYTES;
#pragma unroll
                for (int i = 0; i < (16 * CH) / 32; ++i) {
                    const int c = lane + 32 * i, row = c / CH, col = c - row * CH;
                    const long src = __shfl_sync(0xffffffffu, at, row);
                    if (src >= 0) {
                        cp_async16(kdst + swz<D>(row, col), kl.means + src + col * 8);
                        cp_async16(kdst + TILE_BYTES + swz<D>(row, col), kl.means + src + (long)hkv * kl.per_page * D + col * 8);
                    } else {           // multiplied by p == 0: must be finite
                        uint8_t* z = smem + (kdst - q_smem) + swz<D>(row, col);
                        *reinterpret_cast<uint4*>(z) = *reinterpret_cast<uint4*>(z + TILE_BYTES) = make_uint4(0, 0, 0, 0);
                    }
                }
                return;
            }
            const int tok0 = block_start(warp + DEC_WARPS * j);
            const int page = pages[tok0 / page_size];
            const int off = tok0 % page_size;
            const bf16* ksrc = kv_layer + ((((size_t)page * (OWN ? 1 : 2)) * hkv + h) * page_size + off) * D;
            const bf16* vsrc = ksrc + (size_t)hkv * page_size * D;
            const uint32_t kdst = warp_smem + (j % STAGES) * STAGE_BYTES;
            const uint32_t vdst = kdst + TILE_BYTES;
#pragma unroll
            for (int i = 0; i < (16 * CH) / 32; ++i) {
                const int c = lane + 32 * i;
                const int row = c / CH, col = c - row * CH;
                cp_async16(kdst + swz<D>(row, col), ksrc + (size_t)c * 8);
                if (!OWN) cp_async16(vdst + swz<D>(row, col), vsrc + (size_t)c * 8);
            }
        };
#pragma unroll
        for (int s = 0; s < STAGES - 1; ++s) {
            if (s < my_count) issue(s);
            cp_async_commit();
        }
        for (int i = 0; i < my_count; ++i) {
            if (i + STAGES - 1 < my_count) issue(i + STAGES - 1);
            cp_async_commit();
            cp_async_wait<STAGES - 1>();
            __syncwarp();
            const bool means = POOL && first_tile + warp + DEC_WARPS * i < mean_tiles;
            const int tok0 = means ? (first_tile + warp + DEC_WARPS * i) * 16 : block_start(warp + DEC_WARPS * i);
            const int nvalid = (means ? n_means : kv_end) - tok0;
            uint32_t allow = nvalid >= 16 ? 0xffffu : ((1u << nvalid) - 1u);
            if (!means && kv_lo > tok0) {
                uint32_t see = kv_lo - tok0 >= 16 ? 0u : ~((1u << (kv_lo - tok0)) - 1u);
                if (keep_first > tok0) see |= keep_first - tok0 >= 16 ? 0xffffu : (1u << (keep_first - tok0)) - 1u;
                allow &= see;
            }
            const uint32_t kt = warp_smem + (i % STAGES) * STAGE_BYTES;
            DistanceBias db{};
            if (MODE == MODE_BIAS) {
                const int g = lane >> 2, n = item_end[req_item_indptr[req + 1] - 1] - 1 - tok0;
                const float* tab = bias + (size_t)h * G * bias_pitch + BIAS_GUARD;
                db = DistanceBias{tab + (g < G ? g : 0) * bias_pitch, tab + (g + 8 < G ? g + 8 : 0) * bias_pitch, n, n,
                                  bias_pitch - 2 * BIAS_GUARD - 1};
            }
            attn_block16<D, MODE>(qf, kt, OWN ? kt : kt + TILE_BYTES, scale_log2, allow, allow, st, cap_log2, db);
            __syncwarp();
        }
        cp_async_wait<0>();
        // row sums across the 4 lanes that share a row
#pragma unroll
        for (int hh = 0; hh < 2; ++hh) {
            st.l[hh] += __shfl_xor_sync(0xffffffffu, st.l[hh], 1);
            st.l[hh] += __shfl_xor_sync(0xffffffffu, st.l[hh], 2);
        }
        __syncthreads();  // every warp is done with its K/V stages: reuse as merge space
        float* sm_m = reinterpret_cast<float*>(smem + TILE_BYTES);  // [W][16]
        float* sm_l = sm_m + DEC_WARPS * 16;                         // [W][16]
        float* sm_o = sm_l + DEC_WARPS * 16;                         // [W][ROWS][D]
        {
            const int g = lane >> 2, t = lane & 3;
            if (t == 0) {
                sm_m[warp * 16 + g] = st.m[0];
                sm_l[warp * 16 + g] = st.l[0];
                sm_m[warp * 16 + g + 8] = st.m[1];
                sm_l[warp * 16 + g + 8] = st.l[1];
            }
#pragma unroll
            for (int n = 0; n < D / 8; ++n) {
                if (g < ROWS) {
                    sm_o[(warp * ROWS + g) * D + n * 8 + 2 * t] = st.o[n][0];
                    sm_o[(warp * ROWS + g) * D + n * 8 + 2 * t + 1] = st.o[n][1];
                }
                if (ROWS > 8 && g + 8 < ROWS) {
                    sm_o[(warp * ROWS + g + 8) * D + n * 8 + 2 * t] = st.o[n][2];
                    sm_o[(warp * ROWS + g + 8) * D + n * 8 + 2 * t + 1] = st.o[n][3];
                }
            }
        }
        __syncthreads();
        const bool single = !(CASCADE && members) && (req_item_indptr[req + 1] - req_item_indptr[req]) == 1;
        const int my_slot = CASCADE ? item_slot[it] : it;
        for (int idx = threadIdx.x; idx < ROWS * D; idx += blockDim.x) {
            const int row = idx / D, dim = idx - row * D;
            int rq = req, slot = my_slot, hrow = row;
            if (CASCADE) {
                const int mem = row / G;
                hrow = row - mem * G;
                if (members) {
                    rq = members[mem];
                    if (rq < 0 || rq >= num_reqs) continue;
                    slot = req_item_indptr[rq] + my_slot;
                } else if (mem != 0) {
                    continue;
                }
                if (slot < 0 || slot >= max_items) {          // a plan that outgrew the scratch: drop, report
                    if (status) atomicCAS(status, 0, PIE_ERR_BOUNDS);
                    continue;
                }
            }
            float M = -INFINITY;
#pragma unroll
            for (int ww = 0; ww < DEC_WARPS; ++ww) M = fmaxf(M, sm_m[ww * 16 + row]);
            float L = 0.f, O = 0.f;
            if (M != -INFINITY) {
#pragma unroll
                for (int ww = 0; ww < DEC_WARPS; ++ww) {
                    const float sc = exp2f(sm_m[ww * 16 + row] - M);
                    L += sm_l[ww * 16 + row] * sc;
                    O += sm_o[(ww * ROWS + row) * D + dim] * sc;
                }
            }
            float val = L > 0.f ? O / L : 0.f;
            if (single) {
                // attention sink: a per-head logit that takes probability mass but has no value row
                if (sinks_log2 && L > 0.f) val = O / (L + exp2f(sinks_log2[h * G + hrow] - M));
                out[((size_t)rq * hq + h * G + hrow) * D + dim] = __float2bfloat16(val);
            } else {
                o_part[(((size_t)slot * hkv + h) * G + hrow) * D + dim] = val;
                if (dim == 0)
                    lse_part[((size_t)slot * hkv + h) * G + hrow] = L > 0.f ? M + log2f(L) : -INFINITY;
            }
        }
    }
}

// Merge the partial results of requests that were split into several items.
template <int D>
__global__ void paged_decode_merge_kernel(const float* __restrict__ o_part,
                                          const float* __restrict__ lse_part,
                                          const int* __restrict__ req_item_indptr,
                                          bf16* __restrict__ out, int hq, int hkv, int group,
                                          const float* __restrict__ sinks_log2, int max_items) {
    const int req = blockIdx.x, qh = blockIdx.y;
    pdl_trigger();
    pdl_wait();
    const int a = req_item_indptr[req], b = min(req_item_indptr[req + 1], max_items);
    if (b - a <= 1) return;
    const int kvh = qh / group, row = qh - kvh * group;
    float M = -INFINITY;
    for (int i = a; i < b; ++i) M = fmaxf(M, lse_part[((size_t)i * hkv + kvh) * group + row]);
    for (int dim = threadIdx.x; dim < D; dim += blockDim.x) {
        float L = 0.f, O = 0.f;
        if (M != -INFINITY) {
            for (int i = a; i < b; ++i) {
                const size_t base = ((size_t)i * hkv + kvh) * group + row;
                const float sc = exp2f(lse_part[base] - M);
                L += sc;
                O += o_part[base * D + dim] * sc;
            }
            if (sinks_log2) L += exp2f(sinks_log2[qh] - M);
        }
        out[((size_t)req * hq + qh) * D + dim] = __float2bfloat16(L > 0.f ? O / L : 0.f);
    }
}

// ----------------------------------------------------------------- prefill
constexpr int PF_WARPS = 4;
constexpr int PF_ROWS = 64;  // packed (token, head-in-group) rows per tile
constexpr int PF_KV = 64;    // KV tokens per pipeline stage

template <int D>
constexpr int prefill_smem_bytes() {
    return PF_ROWS * D * 2 + 2 * 2 * PF_KV * D * 2;
}

template <int D, int G, int MODE = MODE_PLAIN, bool POOL = false>
__global__ void __launch_bounds__(PF_WARPS * 32)
paged_prefill_attn_kernel(const bf16* __restrict__ q, const bf16* __restrict__ kv_layer,
                          const int* __restrict__ page_indices,
                          const int* __restrict__ kv_page_indptr,
                          const int* __restrict__ qo_indptr, const int* __restrict__ kv_lens,
                          const int* __restrict__ tile_req, const int* __restrict__ tile_qstart,
                          const uint32_t* __restrict__ mask_bits,
                          const long* __restrict__ mask_word_indptr, bf16* __restrict__ out,
                          float* __restrict__ lse_out, const float* __restrict__ sinks_log2, int hq, int hkv, int page_size,
                          float scale_log2, int window_left, float cap_log2, const float* __restrict__ bias,
                          int bias_pitch, int keep_first, const KeyLayout kl) {
    extern __shared__ __align__(1024) uint8_t smem[];
    constexpr int CH = D / 8;
    constexpr int TQ = PF_ROWS / G;  // query tokens per tile
    constexpr int Q_BYTES = PF_ROWS * D * 2;
    constexpr int KV_TILE = PF_KV * D * 2;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int tile = blockIdx.x, h = blockIdx.y;
    const int req = tile_req[tile], qstart = tile_qstart[tile];
    const int q_base = qo_indptr[req];
    const int qo_len = qo_indptr[req + 1] - q_base;
    const int kv_len = kv_lens[req];
    const int* pages = page_indices + kv_page_indptr[req];
    const bool custom = mask_bits != nullptr;
    const int mask_words = (kv_len + 31) >> 5;
    const uint32_t* req_mask = custom ? mask_bits + mask_word_indptr[req] : nullptr;

    const uint32_t q_smem = smem_u32(smem);
    const uint32_t kv_smem = q_smem + Q_BYTES;
    for (int c = threadIdx.x; c < PF_ROWS * CH; c += blockDim.x) {
        const int row = c / CH, col = c - row * CH;
        const int qt = qstart + row / G;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (qt < qo_len)
            v = *reinterpret_cast<const uint4*>(
                q + ((size_t)(q_base + qt) * hq + h * G + row % G) * D + col * 8);
        *reinterpret_cast<uint4*>(smem + swz<D>(row, col)) = v;
    }
    __syncthreads();
    uint32_t qf[D / 16][4];
    load_q_frags<D>(q_smem, warp * 16, qf);

    // per-thread rows g and g+8 of the warp tile
    const int g = lane >> 2;
    int qtok[2], lim[2], lo[2];
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        const int row = warp * 16 + g + hh * 8;
        qtok[hh] = qstart + row / G;
        const bool valid = qtok[hh] < qo_len;
        // causal: query token i of qo_len sees kv positions < kv_len - qo_len + i + 1
        lim[hh] = valid ? (custom ? kv_len : kv_len - qo_len + qtok[hh] + 1) : 0;
        lo[hh] = (window_left >= 0 && valid) ? max(0, kv_len - qo_len + qtok[hh] - window_left) : 0;
    }
    const int last_q = min(qstart + TQ, qo_len) - 1;
    const int kv_hi = custom ? kv_len : max(0, min(kv_len, kv_len - qo_len + last_q + 1));
    // the warp's last row has the largest causal limit of the warp
    const int warp_last_q = min(qstart + (warp * 16 + 15) / G, qo_len - 1);
    const int warp_hi = custom ? kv_len : kv_len - qo_len + warp_last_q + 1;
    // key blocks [hidden, hidden + gap) lie between the kept first keys and the window of the tile's first query
    const int nkb_all = (kv_hi + PF_KV - 1) / PF_KV;
    const int hidden = min(nkb_all, (keep_first + PF_KV - 1) / PF_KV);
    const int gap = window_left >= 0 ? max(0, min(nkb_all, max(0, kv_len - qo_len + qstart - window_left) / PF_KV) - hidden) : 0;
    // POOL: blocks of means come first, as many as the tile's last query sees
    const int n_means = POOL ? means_seen(kv_len - qo_len + last_q, window_left, kl.pool) : 0, mean_blocks = (n_means + PF_KV - 1) / PF_KV;
    const int nkb = nkb_all - gap + mean_blocks;
    auto key_block = [&](int i) { return POOL ? i - mean_blocks + gap : (i < hidden ? i : i + gap); };

    auto load_stage = [&](int i_kb) {
        const bool means = POOL && i_kb < mean_blocks;
        const int kb = means ? i_kb : key_block(i_kb);
        const uint32_t kdst = kv_smem + (i_kb & 1) * 2 * KV_TILE;
        const uint32_t vdst = kdst + KV_TILE;
#pragma unroll
        for (int i = 0; i < (PF_KV * CH) / (PF_WARPS * 32); ++i) {
            const int c = threadIdx.x + PF_WARPS * 32 * i;
            const int row = c / CH, col = c - row * CH;
            const int tok = kb * PF_KV + row;
            if (means && tok < n_means) {
                const bf16* ksrc = kl.means + ((((size_t)kl.first[req] + tok / 16) * 2 * hkv + h) * 16 + tok % 16) * D + col * 8;
                cp_async16(kdst + swz<D>(row, col), ksrc);
                cp_async16(vdst + swz<D>(row, col), ksrc + (size_t)hkv * 16 * D);
            } else if (!means && tok < kv_hi) {
                const int page = pages[tok / page_size];
                const int off = tok % page_size;
                const bf16* ksrc =
                    kv_layer + ((((size_t)page * kl.planes) * hkv + h) * page_size + off) * D + col * 8;
                const bf16* vsrc = ksrc + (size_t)(kl.planes - 1) * hkv * page_size * D;
                cp_async16(kdst + swz<D>(row, col), ksrc);
                cp_async16(vdst + swz<D>(row, col), vsrc);
            } else {
                // rows past the end are multiplied by p == 0: they must be finite
                *reinterpret_cast<uint4*>(smem + (vdst - q_smem) + swz<D>(row, col)) =
                    make_uint4(0, 0, 0, 0);
                *reinterpret_cast<uint4*>(smem + (kdst - q_smem) + swz<D>(row, col)) =
                    make_uint4(0, 0, 0, 0);
            }
        }
    };

    AttnState<D> st;
    st.init();
    if (nkb > 0) load_stage(0);
    cp_async_commit();
    for (int i_kb = 0; i_kb < nkb; ++i_kb) {
        if (i_kb + 1 < nkb) load_stage(i_kb + 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const bool means = POOL && i_kb < mean_blocks;
        const int kb = means ? i_kb : key_block(i_kb);
        const uint32_t kt = kv_smem + (i_kb & 1) * 2 * KV_TILE;
#pragma unroll
        for (int sb = 0; sb < PF_KV / 16; ++sb) {
            const int tb = kb * PF_KV + sb * 16;
            if (means ? tb >= n_means : (tb >= warp_hi || tb >= kv_hi)) break;
            uint32_t allow[2];
#pragma unroll
            for (int hh = 0; hh < 2; ++hh) {
                const int n = (means ? lo[hh] / kl.pool : lim[hh]) - tb;
                uint32_t a = n >= 16 ? 0xffffu : (n <= 0 ? 0u : ((1u << n) - 1u));
                const int nl = means ? 0 : lo[hh] - tb;
                if (nl > 0) {
                    uint32_t see = nl >= 16 ? 0u : ~((1u << nl) - 1u);
                    if (keep_first > tb) see |= keep_first - tb >= 16 ? 0xffffu : (1u << (keep_first - tb)) - 1u;
                    a &= see;
                }
                if (custom && a) {
                    const uint32_t wv = req_mask[(size_t)qtok[hh] * mask_words + (tb >> 5)];
                    a &= (wv >> (tb & 31)) & 0xffffu;
                }
                allow[hh] = a;
            }
            DistanceBias db{};
            if (MODE == MODE_BIAS) {
                const float* tab = bias + (size_t)h * G * bias_pitch + BIAS_GUARD;
                const int pos0 = kv_len - qo_len - tb;
                db = DistanceBias{tab + (warp * 16 + g) % G * bias_pitch, tab + (warp * 16 + g + 8) % G * bias_pitch, pos0 + qtok[0],
                                  pos0 + qtok[1], bias_pitch - 2 * BIAS_GUARD - 1};
            }
            attn_block16<D, MODE>(qf, kt + sb * 16 * D * 2, kt + KV_TILE + sb * 16 * D * 2, scale_log2,
                                  allow[0], allow[1], st, cap_log2, db);
        }
        __syncthreads();
    }
    cp_async_wait<0>();
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        st.l[hh] += __shfl_xor_sync(0xffffffffu, st.l[hh], 1);
        st.l[hh] += __shfl_xor_sync(0xffffffffu, st.l[hh], 2);
    }
    const int t = lane & 3;
#pragma unroll
    for (int hh = 0; hh < 2; ++hh) {
        if (qtok[hh] >= qo_len) continue;
        const int row = warp * 16 + g + hh * 8;
        const int head = h * G + row % G;
        if (sinks_log2 && st.l[hh] > 0.f) st.l[hh] += exp2f(sinks_log2[head] - st.m[hh]);
        const float inv = st.l[hh] > 0.f ? 1.f / st.l[hh] : 0.f;
        bf16* dst = out + ((size_t)(q_base + qtok[hh]) * hq + head) * D;
#pragma unroll
        for (int n = 0; n < D / 8; ++n) {
            bf162 v = __floats2bfloat162_rn(st.o[n][2 * hh] * inv, st.o[n][2 * hh + 1] * inv);
            *reinterpret_cast<bf162*>(dst + n * 8 + 2 * t) = v;
        }
        if (lse_out && t == 0)
            lse_out[(size_t)(q_base + qtok[hh]) * hq + head] =
                st.l[hh] > 0.f ? (st.m[hh] + log2f(st.l[hh])) * 0.6931471805599453f : -INFINITY;
    }
}

}  // namespace pie

#define DISPATCH_DG(D_, G_, ...)                                      \
    do {                                                               \
        bool ok_ = true;                                               \
        if (D_ == 128) {                                               \
            constexpr int D = 128;                                     \
            switch (G_) {                                              \
                case 1: { constexpr int G = 1; __VA_ARGS__; } break;          \
                case 2: { constexpr int G = 2; __VA_ARGS__; } break;          \
                case 4: { constexpr int G = 4; __VA_ARGS__; } break;          \
                case 8: { constexpr int G = 8; __VA_ARGS__; } break;          \
                case 16: { constexpr int G = 16; __VA_ARGS__; } break;        \
                default: ok_ = false;                                  \
            }                                                          \
        } else if (D_ == 256) {                                        \
            constexpr int D = 256;                                     \
            switch (G_) {                                              \
                case 1: { constexpr int G = 1; __VA_ARGS__; } break;          \
                case 2: { constexpr int G = 2; __VA_ARGS__; } break;          \
                case 4: { constexpr int G = 4; __VA_ARGS__; } break;          \
                case 8: { constexpr int G = 8; __VA_ARGS__; } break;          \
                default: ok_ = false;                                  \
            }                                                          \
        } else if (D_ == 64) {                                         \
            constexpr int D = 64;                                      \
            switch (G_) {                                              \
                case 1: { constexpr int G = 1; __VA_ARGS__; } break;          \
                case 2: { constexpr int G = 2; __VA_ARGS__; } break;          \
                case 4: { constexpr int G = 4; __VA_ARGS__; } break;          \
                case 8: { constexpr int G = 8; __VA_ARGS__; } break;          \
                case 16: { constexpr int G = 16; __VA_ARGS__; } break;        \
                default: ok_ = false;                                  \
            }                                                          \
        } else {                                                       \
            ok_ = false;                                               \
        }                                                              \
        if (!ok_) return (int)cudaErrorInvalidValue;                   \
    } while (0)

