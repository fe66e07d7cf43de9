// Latent decode attention on the 5th-generation tensor cores, with keys on the rows of the accumulators.
//
// The few query rows of a decode step (one token, up to 32 heads) would leave most of a 128-row MMA empty, so both
// products are turned around: S^T = K Q^T has 128 keys as rows and the heads as columns, O^T += V^T P^T has 128 latent
// columns as rows. The tile of cache rows in shared memory serves as K (K-major) and as V^T (MN-major) as it stands, and
// every byte of it is read twice by the tensor cores and by nobody else.
//   warp 0      TMA producer: the item's query rows; per tile the 128 keys' pages, as boxes of 16 rows x 64 columns with the
//               128-byte swizzle, into a ring of two stages (all lanes look pages up and issue)
//   warp 1      tcgen05.mma issuer: S^T of a tile into one of two TMEM buffers, a tile ahead where the keys have arrived, and
//               O^T into its own TMEM columns once the softmax warps have handed over P
//   warps 2-9   softmax, two groups of four warps with 16 heads each, one key per thread: a column of S^T is a head, so its
//               maximum is a warp reduction per head and an exchange between the group's four warps; exponentials
//               against a reference maximum that follows the true one lazily (O^T is rescaled in TMEM only when a head's
//               maximum outgrows it by 2^8); P as bf16 into a swizzled tile [heads][keys]. At the end of an item the sums are
//               reduced and O^T leaves, normalised, for `out` (a request that was not split) or the split-KV scratch.
// A CTA runs a contiguous range of work items: the keys of all requests are cut evenly over the CTAs.
// Every wait is bounded; on a time-out the kernel records a status word and leaves.
#include "latent_args.cuh"
#include "tcgen05.cuh"

namespace pie {
using namespace sm100;

constexpr int LT_HEADS = 32;                 // heads per CTA (columns of S^T and O^T)
constexpr int LT_KEYS = 128;                 // keys per tile (rows of S^T)
constexpr int LT_STAGES = 2;
constexpr int LT_HALF = LT_HEADS / 2;        // heads per softmax group
constexpr int LT_THREADS = 64 + 256;
constexpr uint32_t LT_BLOCK = LT_KEYS * 128;           // 64 columns of a tile: 128 rows of 128 bytes
constexpr uint32_t LT_QBLOCK = LT_HEADS * 128;
constexpr uint32_t LT_P_BYTES = LT_HEADS * LT_KEYS * 2;
constexpr float LT_RESCALE_LOG2 = 8.f;

__host__ __device__ inline int lt_mtiles(int rank_pad) { return (rank_pad + 127) / 128; }
__host__ __device__ inline int lt_blocks(int row, int rank_pad) {        // 64-column blocks: all of the row, and whole V^T tiles
    const int k = (row + 63) / 64, v = 2 * lt_mtiles(rank_pad);
    return k > v ? k : v;
}
__host__ __device__ inline uint32_t lt_smem(int row, int rank_pad) {
    const uint32_t nb = lt_blocks(row, rank_pad);
    return LT_STAGES * nb * LT_BLOCK + nb * LT_QBLOCK + 2 * LT_P_BYTES + 1024 /*align*/ + 256 /*barriers*/ + 8 * LT_HEADS * 4 /*exchanges*/ + 128 + 8;
}

// MN-major SW128 operand: 64 elements of the contiguous dimension per 128-byte row, 8-row groups of the other dimension
// 1024 bytes apart, the next 64 elements `lbo` bytes further.
__device__ __forceinline__ uint64_t lt_desc_mn(uint32_t saddr, uint32_t lbo) {
    uint64_t d = 0;
    d |= (uint64_t)((saddr & 0x3FFFFu) >> 4);
    d |= (uint64_t)(lbo >> 4) << 16;
    d |= (uint64_t)(1024 >> 4) << 32;
    d |= (uint64_t)1 << 46;
    d |= (uint64_t)2 << 61;
    return d;
}
__device__ __forceinline__ float lt_exp2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float lt_warp_max(float x) {
    float y;
    asm volatile("redux.sync.max.f32 %0, %1, 0xffffffff;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void lt_group_sync(int group) { asm volatile("bar.sync %0, 128;" ::"r"(group + 1) : "memory"); }
// Barrier of a group that also tells whether any of its threads passed `flag`.
__device__ __forceinline__ bool lt_group_any(int group, bool flag) {
    uint32_t r;
    asm volatile(
        "{\n"
        ".reg .pred p, q;\n"
        "setp.ne.b32 q, %1, 0;\n"
        "bar.red.or.pred p, %2, 128, q;\n"
        "selp.u32 %0, 1, 0, p;\n"
        "}\n"
        : "=r"(r) : "r"((uint32_t)flag), "r"(group + 1) : "memory");
    return r != 0;
}
// 32 lanes x 16 columns of 32-bit accumulators
__device__ __forceinline__ void lt_tmem_ld(uint32_t taddr, uint32_t (&v)[16]) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];\n"
        : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]), "=r"(v[8]), "=r"(v[9]),
          "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
        : "r"(taddr)
        : "memory");
}
__device__ __forceinline__ void lt_tmem_st(uint32_t taddr, const uint32_t (&v)[16]) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x16.b32 [%0], {%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15,%16};\n" ::"r"(taddr),
        "r"(v[0]), "r"(v[1]), "r"(v[2]), "r"(v[3]), "r"(v[4]), "r"(v[5]), "r"(v[6]), "r"(v[7]), "r"(v[8]), "r"(v[9]), "r"(v[10]),
        "r"(v[11]), "r"(v[12]), "r"(v[13]), "r"(v[14]), "r"(v[15])
        : "memory");
}

// What every role derives from an item of the work list. A warp looks 32 items up at once, one per lane.
struct LtItem {
    int tok, k0, lo, hi, tiles;    // query token; first key loaded (a multiple of 16); visible keys [lo, hi); tiles of keys
    int pages;                     // offset of the request's page table
    int whole;                     // the request's only item: normalised output instead of a partial one
    __device__ __forceinline__ LtItem of_lane(int src) const {
        const unsigned all = 0xffffffffu;
        return LtItem{__shfl_sync(all, tok, src),   __shfl_sync(all, k0, src),    __shfl_sync(all, lo, src),   __shfl_sync(all, hi, src),
                      __shfl_sync(all, tiles, src), __shfl_sync(all, pages, src), __shfl_sync(all, whole, src)};
    }
};
__device__ __forceinline__ LtItem lt_item(const LatentMmaArgs& a, int item, int item1) {
    LtItem t{0, 0, 0, 0, 0, 0, 1};
    const int r = item < item1 ? a.item_req[item] : -1;
    if (r < 0 || r >= a.reqs) return t;
    const int kv_len = a.kv_lens[r];
    t.tok = a.qo_indptr[r];
    t.pages = a.kv_page_indptr[r];
    t.lo = max(max(0, kv_len - 1 - a.window_left), a.item_start[item]);
    t.hi = min(kv_len, a.item_end[item]);
    t.k0 = t.lo & ~15;
    t.tiles = t.hi > t.lo ? (t.hi - t.k0 + LT_KEYS - 1) / LT_KEYS : 0;
    t.whole = a.req_item_indptr[r + 1] - a.req_item_indptr[r] == 1;
    return t;
}

// MT: 128-column tiles of the latent (rows of O^T).
template <int MT>
__global__ void __launch_bounds__(LT_THREADS, 1)
latent_attn_tc_kernel(const __grid_constant__ CUtensorMap tma_q, const __grid_constant__ CUtensorMap tma_c, const LatentMmaArgs a,
                      int* status) {
    constexpr uint32_t TMEM_COLS = 128;                        // two S^T, then MT x O^T, 32 columns each
    static_assert(MT <= 2, "TMEM columns");
    extern __shared__ uint8_t lt_raw[];
    const uint32_t raw = smem_addr(lt_raw), base = (raw + 1023u) & ~1023u;
    uint8_t* base_ptr = lt_raw + (base - raw);
    const int nb = lt_blocks(a.row, a.rank_pad);
    const uint32_t stage_bytes = nb * LT_BLOCK;
    const uint32_t k_s = base, q_s = k_s + LT_STAGES * stage_bytes, p_s = q_s + nb * LT_QBLOCK, bar0 = p_s + 2 * LT_P_BYTES;
    auto k_full = [&](int s) { return bar0 + 8u * s; };
    auto k_empty = [&](int s) { return bar0 + 16u + 8u * s; };
    const uint32_t q_full = bar0 + 32, q_empty = bar0 + 40, o_final = bar0 + 48, o_free = bar0 + 56, pv_done = bar0 + 64;
    // one per buffer: two tiles may be under way, and a parity wait tells apart neighbouring phases only
    auto s_full = [&](uint32_t n) { return bar0 + 72u + 8u * (n & 1u); };
    auto p_full = [&](uint32_t n) { return bar0 + 88u + 8u * (n & 1u); };
    volatile uint32_t* tmem_slot = reinterpret_cast<volatile uint32_t*>(base_ptr + (bar0 - base) + 104);
    float* mx_s = reinterpret_cast<float*>(base_ptr + (bar0 - base) + 256);      // [2 groups][4 warps][heads]
    float* l_s = mx_s + 4 * LT_HEADS;                                           // [2 groups][4 warps][heads]
    int* tiles_s = reinterpret_cast<int*>(l_s + 4 * LT_HEADS);                  // tiles of the MMA warp's next 32 items
    volatile int* failed = tiles_s + 32;                                        // [2 groups] a warp of the group gave up on a wait

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h0 = blockIdx.y * LT_HEADS, hn = min(LT_HEADS, a.heads - h0);
    if (threadIdx.x == 0) {
        for (int s = 0; s < LT_STAGES; ++s) {
            mbar_init(k_full(s), 1);
            mbar_init(k_empty(s), 1);
        }
        mbar_init(q_full, 1);
        mbar_init(q_empty, 1);
        for (int b = 0; b < 2; ++b) {
            mbar_init(s_full(b), 1);
            mbar_init(p_full(b), 8);
        }
        mbar_init(o_final, 1);
        mbar_init(o_free, 8);
        mbar_init(pv_done, 1);
        failed[0] = failed[1] = 0;
        fence_barrier_init();
        fence_proxy_async();
    }
    if (warp == 1) {
        tmem_alloc(smem_addr(const_cast<uint32_t*>(tmem_slot)), TMEM_COLS);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_s = *tmem_slot, tmem_o = tmem_s + 2 * LT_HEADS;
    pdl_trigger();
    pdl_wait();
    const int item0 = a.cta_items[blockIdx.x], item1 = min(a.cta_items[blockIdx.x + 1], a.max_items);

    if (warp == 0) {
        // ------------------------------------------------------ TMA producer
        uint32_t g = 0, ni = 0;
        bool ok = true;
        LtItem mine{};
        for (int item = item0; item < item1 && ok; ++item) {
            if (((item - item0) & 31) == 0) mine = lt_item(a, item + lane, item1);
            const LtItem t = mine.of_lane((item - item0) & 31);
            if (t.tiles == 0) continue;
            bool w = true;
            if (lane == 0) {
                w = mbar_wait(q_empty, (ni & 1u) ^ 1u, status, PIE_ERR_WAIT_TMA);
                if (w) mbar_arrive_expect_tx(q_full, nb * LT_QBLOCK);
            }
            ok = __shfl_sync(0xffffffffu, (int)w, 0) != 0;
            if (!ok) break;
            ++ni;
            for (int b = lane; b < nb; b += 32) tma_load_2d(q_s + b * LT_QBLOCK, &tma_q, q_full, b * 64, t.tok * a.heads + h0);
            for (int j = 0; j < t.tiles && ok; ++j, ++g) {
                const int s = g % LT_STAGES;
                // a lane's boxes are all of one 16-key piece; a piece past the end reads zeros (rows outside the tensor)
                const int key = t.k0 + j * LT_KEYS + (lane & 7) * 16;
                const int row = key < t.hi ? (a.page_indices[t.pages + (key >> a.page_shift)] << a.page_shift) + (key & (a.page_size - 1))
                                           : a.cache_rows;
                if (lane == 0) {
                    w = mbar_wait(k_empty(s), ((g / LT_STAGES) & 1u) ^ 1u, status, PIE_ERR_WAIT_TMA);
                    if (w) mbar_arrive_expect_tx(k_full(s), stage_bytes);
                }
                ok = __shfl_sync(0xffffffffu, (int)w, 0) != 0;
                if (!ok) break;
                for (int i = lane; i < 8 * nb; i += 32)
                    tma_load_2d(k_s + s * stage_bytes + (i >> 3) * LT_BLOCK + (i & 7) * 2048, &tma_c, k_full(s), (i >> 3) * 64, row);
            }
        }
        // no copy of this CTA may still be in flight when it exits
        if (lane == 0) {
            const uint32_t first = g > (uint32_t)LT_STAGES ? g - LT_STAGES : 0u;
            for (uint32_t j = first; j < g; ++j)
                mbar_wait(k_full(j % LT_STAGES), (j / LT_STAGES) & 1u, status, PIE_ERR_WAIT_TMA, 200000000ll);
            if (ni > 0) mbar_wait(q_full, (ni - 1) & 1u, status, PIE_ERR_WAIT_TMA, 200000000ll);
        }
    } else if (warp == 1) {
        // -------------------------------------------------------- MMA issuer
        constexpr uint32_t idesc_s = make_idesc_bf16(LT_KEYS, LT_HEADS);
        constexpr uint32_t idesc_o = make_idesc_bf16(128, LT_HEADS) | (1u << 15);      // A is MN-major
        uint32_t g = 0, ni = 0;
        bool ok = true;
        for (int chunk = item0; chunk < item1; chunk += 32) {
            __syncwarp();
            tiles_s[lane] = lt_item(a, chunk + lane, item1).tiles;
            __syncwarp();
            if (lane != 0) continue;
            for (int i = 0; i < min(32, item1 - chunk) && ok; ++i) {
                const int tiles = tiles_s[i];
                if (tiles == 0) continue;
                if (!mbar_wait(q_full, ni & 1u, status, PIE_ERR_WAIT_TMA)) { ok = false; break; }
                // S^T of tile n (counted over all items) into TMEM buffer n & 1
                auto issue_s = [&](uint32_t n, bool last) {
                    const uint32_t tile = k_s + (n % LT_STAGES) * stage_bytes;
                    tc_fence_after();
                    for (int k = 0; k < (a.row >> 4); ++k)
                        umma_bf16(tmem_s + (n & 1u) * LT_HEADS, make_smem_desc_sw128(tile + (k >> 2) * LT_BLOCK) + 2u * (k & 3),
                                  make_smem_desc_sw128(q_s + (k >> 2) * LT_QBLOCK) + 2u * (k & 3), idesc_s, k != 0);
                    // arrives when all products issued so far are complete, O^T of the tile before the last included
                    umma_commit(s_full(n));
                    if (last) umma_commit(q_empty);
                };
                auto keys_ready = [&](uint32_t n) {
                    return mbar_wait(k_full(n % LT_STAGES), (n / LT_STAGES) & 1u, status, PIE_ERR_WAIT_TMA);
                };
                if (!keys_ready(g)) { ok = false; break; }
                issue_s(g, tiles == 1);
                for (int j = 0; j < tiles; ++j, ++g) {
                    const int s = g % LT_STAGES;
                    const uint32_t tile = k_s + s * stage_bytes;
                    const bool more = j + 1 < tiles;
                    // the next tile's scores go first where its keys are there: the softmax then finds them finished
                    const bool ahead = more && mbar_try_wait(k_full((g + 1) % LT_STAGES), ((g + 1) / LT_STAGES) & 1u);
                    if (ahead) issue_s(g + 1, j + 2 == tiles);
                    if (!mbar_wait(p_full(g), (g >> 1) & 1u, status, PIE_ERR_WAIT_EPILOGUE)) { ok = false; break; }
                    if (j == 0 && !mbar_wait(o_free, (ni & 1u) ^ 1u, status, PIE_ERR_WAIT_EPILOGUE)) { ok = false; break; }
                    tc_fence_after();
                    const uint32_t p_tile = p_s + (g & 1u) * LT_P_BYTES;
#pragma unroll
                    for (int m = 0; m < MT; ++m)
#pragma unroll
                        for (int k = 0; k < LT_KEYS / 16; ++k)
                            umma_bf16(tmem_o + m * LT_HEADS, lt_desc_mn(tile + 2 * m * LT_BLOCK + k * 2048, LT_BLOCK),
                                      make_smem_desc_sw128(p_tile + (k >> 2) * (LT_HEADS * 128)) + 2u * (k & 3), idesc_o, (j | k) != 0);
                    umma_commit(k_empty(s));
                    umma_commit(pv_done);
                    if (!more) umma_commit(o_final);
                    if (more && !ahead) {
                        if (!keys_ready(g + 1)) { ok = false; break; }
                        issue_s(g + 1, j + 2 == tiles);
                    }
                }
                ++ni;
            }
        }
    } else {
        // ------------------- softmax: thread = key of the tile, lane = head of the group in the exchanges
        const int q4 = warp & 3, group = (warp - 2) >> 2, hb = group * LT_HALF;      // q4: the TMEM lane quarter of this warp
        const uint32_t quarter = (uint32_t)(q4 * 32) << 16;
        const int kin = (q4 & 1) * 32 + lane;            // key within the 64-key half of P
        uint8_t* p_row = base_ptr + (p_s - base) + (q4 >> 1) * (LT_HEADS * 128) + hb * 128 + (kin & 7) * 2;
        float* lx = l_s + group * 4 * LT_HALF;
        const int hl = lane & (LT_HALF - 1), head = h0 + hb + hl;       // of this lane in the exchanges
        const bool owner = q4 == 0 && lane < LT_HALF && hb + hl < hn;
        float* lse = a.scratch + (size_t)a.max_items * a.heads * a.rank_pad;
        uint32_t g = 0, ni = 0;
        bool ok = true;
        LtItem own{};
        for (int item = item0; item < item1 && ok; ++item) {
            if (((item - item0) & 31) == 0) own = lt_item(a, item + lane, item1);
            const LtItem t = own.of_lane((item - item0) & 31);
            if (t.tiles == 0) {
                if (!t.whole) {                          // a span that a narrower layer sees nothing of: no weight in the merge
                    if (owner) lse[(size_t)item * a.heads + head] = -INFINITY;
                    for (int i = threadIdx.x - 64; i < hn * a.rank_pad; i += 256)
                        a.scratch[((size_t)item * a.heads + h0) * a.rank_pad + i] = 0.f;
                }
                continue;
            }
            float m_ref = -INFINITY, neg[LT_HALF], l[LT_HALF];
#pragma unroll
            for (int h = 0; h < LT_HALF; ++h) neg[h] = l[h] = 0.f;
            for (int j = 0; j < t.tiles; ++j, ++g) {
                // a wait that ran out is told to the group at its next barrier, which every warp reaches: all leave together
                if (!mbar_wait(s_full(g), (g >> 1) & 1u, status, PIE_ERR_WAIT_MMA)) failed[group] = 1;
                __syncwarp();
                tc_fence_after();
                uint32_t v[LT_HALF];
                lt_tmem_ld(tmem_s + quarter + (g & 1u) * LT_HEADS + hb, v);
                tmem_ld_wait();
                const int key = t.k0 + j * LT_KEYS + q4 * 32 + lane;
                const bool see = key >= t.lo && key < t.hi;
                float e[LT_HALF], top = -INFINITY;        // exponents against the reference
#pragma unroll
                for (int h = 0; h < LT_HALF; ++h) {
                    e[h] = see ? fmaf(__uint_as_float(v[h]), a.scale_log2, neg[h]) : -INFINITY;
                    top = fmaxf(top, e[h]);
                }
                // while no head's score outgrows its reference by 2^8 (the first tile sets it), nobody needs a maximum
                const bool outgrown = lt_group_any(group, j == 0 || top > LT_RESCALE_LOG2);
                if (failed[group]) { ok = false; break; }
                if (outgrown) {
                    float mine = -INFINITY;
#pragma unroll
                    for (int h = 0; h < LT_HALF; ++h) {
                        const float m = lt_warp_max(see ? __uint_as_float(v[h]) : -INFINITY);
                        if (hl == h) mine = m;
                    }
                    float* mx = mx_s + group * 4 * LT_HALF;
                    if (lane < LT_HALF) mx[q4 * LT_HALF + hl] = mine;
                    lt_group_sync(group);
                    const float tmax = fmaxf(fmaxf(mx[hl], mx[LT_HALF + hl]), fmaxf(mx[2 * LT_HALF + hl], mx[3 * LT_HALF + hl]));
                    const float m_new = fmaxf(m_ref, tmax);
                    const float alpha = m_new == -INFINITY ? 1.f : lt_exp2((m_ref - m_new) * a.scale_log2);
                    const float nl = m_new == -INFINITY ? 0.f : -m_new * a.scale_log2;
                    m_ref = m_new;
#pragma unroll
                    for (int h = 0; h < LT_HALF; ++h) {
                        neg[h] = __shfl_sync(0xffffffffu, nl, h);
                        l[h] *= __shfl_sync(0xffffffffu, alpha, h);
                        e[h] = see ? fmaf(__uint_as_float(v[h]), a.scale_log2, neg[h]) : -INFINITY;
                    }
                    if (j > 0) {
                        if (!mbar_wait(pv_done, (g - 1) & 1u, status, PIE_ERR_WAIT_MMA)) failed[group] = 1;
                        __syncwarp();
                        tc_fence_after();
#pragma unroll
                        for (int m = 0; m < MT; ++m) {
                            uint32_t o[LT_HALF];
                            lt_tmem_ld(tmem_o + quarter + m * LT_HEADS + hb, o);
                            tmem_ld_wait();
#pragma unroll
                            for (int h = 0; h < LT_HALF; ++h)
                                o[h] = __float_as_uint(__uint_as_float(o[h]) * __shfl_sync(0xffffffffu, alpha, h));
                            lt_tmem_st(tmem_o + quarter + m * LT_HEADS + hb, o);
                        }
                        tmem_st_wait();
                    }
                }
                uint8_t* prow = p_row + (g & 1u) * LT_P_BYTES;
#pragma unroll
                for (int h = 0; h < LT_HALF; ++h) {
                    const float p = lt_exp2(e[h]);
                    l[h] += p;
                    *reinterpret_cast<bf16*>(prow + h * 128 + (((kin >> 3) ^ (h & 7)) << 4)) = __float2bfloat16(p);
                }
                fence_proxy_async();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(p_full(g));
            }
            if (!ok) break;
            if (!mbar_wait(o_final, ni & 1u, status, PIE_ERR_WAIT_MMA)) failed[group] = 1;
            __syncwarp();
            ++ni;
            tc_fence_after();
            float mine = 0.f;
#pragma unroll
            for (int d = 16; d > 0; d >>= 1)              // sixteen independent chains at a time
#pragma unroll
                for (int h = 0; h < LT_HALF; ++h) l[h] += __shfl_xor_sync(0xffffffffu, l[h], d);
#pragma unroll
            for (int h = 0; h < LT_HALF; ++h) mine = hl == h ? l[h] : mine;
            if (lane < LT_HALF) lx[q4 * LT_HALF + hl] = mine;
            lt_group_sync(group);
            if (failed[group]) break;
            const float lt = lx[hl] + lx[LT_HALF + hl] + lx[2 * LT_HALF + hl] + lx[3 * LT_HALF + hl];
            const float inv = lt > 0.f ? 1.f / lt : 0.f;
            if (!t.whole && owner) lse[(size_t)item * a.heads + head] = lt > 0.f ? m_ref * a.scale_log2 + log2f(lt) : -INFINITY;
#pragma unroll
            for (int h = 0; h < LT_HALF; ++h) l[h] = __shfl_sync(0xffffffffu, inv, h);
            const int heads_here = min(LT_HALF, hn - hb);
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                uint32_t o[LT_HALF];
                lt_tmem_ld(tmem_o + quarter + m * LT_HEADS + hb, o);
                tmem_ld_wait();
                const int col = m * 128 + q4 * 32 + lane;
                if (col >= a.rank_pad) continue;
                if (t.whole) {
                    bf16* dst = static_cast<bf16*>(a.out) + ((size_t)t.tok * a.heads + h0 + hb) * a.rank_pad + col;
#pragma unroll
                    for (int h = 0; h < LT_HALF; ++h)
                        if (h < heads_here) dst[h * a.rank_pad] = __float2bfloat16(__uint_as_float(o[h]) * l[h]);
                } else {
                    float* dst = a.scratch + ((size_t)item * a.heads + h0 + hb) * a.rank_pad + col;
#pragma unroll
                    for (int h = 0; h < LT_HALF; ++h)
                        if (h < heads_here) dst[h * a.rank_pad] = __uint_as_float(o[h]) * l[h];
                }
            }
            __syncwarp();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(o_free);
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) {
        __syncwarp();
        tc_fence_after();
        tmem_dealloc(tmem_s, TMEM_COLS);
    }
}

}  // namespace pie

using namespace pie;

extern "C" int pie_make_tma_2d_bf16(CUtensorMap* map, const void* ptr, long rows, long cols, long ld, int box_rows);
int pie_latent_merge(const LatentMmaArgs& a, cudaStream_t st);

PIE_API int pie_latent_attn_tc_supported(int row, int rank_pad, int page_size) {
    return row > 0 && row % 16 == 0 && rank_pad % 16 == 0 && rank_pad <= row && rank_pad <= 256 && page_size >= 16 &&
           (page_size & (page_size - 1)) == 0 && lt_smem(row, rank_pad) <= 227 * 1024 ? 1 : 0;
}

// Decode only: one query token per request, work items cut over `num_ctas` CTAs (cta_items).
PIE_API int pie_latent_attn_tc(const LatentMmaArgs* args, int num_ctas, int* status, cudaStream_t st) {
    const LatentMmaArgs& a = *args;
    if (!pie_latent_attn_tc_supported(a.row, a.rank_pad, a.page_size) || a.page_size != 1 << a.page_shift || a.row > a.cache_row ||
        a.cache_row % 16 || !a.item_end || !a.scratch || !a.req_item_indptr || !a.cta_items || a.reqs <= 0 || num_ctas <= 0 || !status)
        return (int)cudaErrorInvalidValue;
    CUtensorMap tq, tc;
    if (pie_make_tma_2d_bf16(&tq, a.q, (long)a.reqs * a.heads, a.row, a.row, LT_HEADS) != 0 ||
        pie_make_tma_2d_bf16(&tc, a.cache, a.cache_rows, a.row, a.cache_row, 16) != 0)
        return (int)cudaErrorInvalidValue;
    const uint32_t smem = lt_smem(a.row, a.rank_pad);
    const dim3 grid(num_ctas, (a.heads + LT_HEADS - 1) / LT_HEADS);
#define GO(M_)                                                                                                                       \
    {                                                                                                                                \
        cudaError_t e = cudaFuncSetAttribute(latent_attn_tc_kernel<M_>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);     \
        if (e != cudaSuccess) return (int)e;                                                                                         \
        e = launch_pdl(latent_attn_tc_kernel<M_>, grid, dim3(LT_THREADS), (size_t)smem, st, tq, tc, a, status);                      \
        if (e != cudaSuccess) return (int)e;                                                                                         \
    }
    if (lt_mtiles(a.rank_pad) == 1) GO(1) else GO(2)
#undef GO
    return pie_latent_merge(a, st);
}
