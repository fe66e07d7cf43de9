// Blocks that read their 32-bit residual stream through a layer norm and a short causal convolution over time:
//
//   pie_pair_embed   token rows plus rows for the pair (token before, token), as a 32-bit stream
//   pie_conv_norm    [normed sublayer outputs join the stream] + layer norm + convolution, in one pass
//
// T is the activation type (bf16 when serving, float on the 32-bit path); stream, norms, history and weights are 32-bit. What a
// sequence carries from fire to fire lies in its state slot: the token before, and the last taps - 1 norm outputs of every
// convolution.
#include "typed.cuh"

namespace pie {

struct PairEmbedArgs {
    const int* tokens;
    const void *table, *pairs;      // [vocab, width], [buckets + 1, width]
    float* x;                       // [n, ldx]
    const int *tok_req, *qo_indptr, *slots, *reset;
    int* state;                     // the token before, of slot 0
    long slot_stride, buckets, mul_prev, mul_cur;
    int n, reqs, width, ldx, vocab;
};

template <typename T>
__global__ void __launch_bounds__(256) pair_embed_kernel(const PairEmbedArgs a) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x, id = a.tokens[t], r = a.tok_req[t], q0 = a.qo_indptr[r], slot = a.slots[r];
    long row = a.buckets;
    if (t > q0) row = ((long)a.tokens[t - 1] * a.mul_prev + (long)id * a.mul_cur) % a.buckets;
    else if (slot >= 0 && !a.reset[r]) row = ((long)a.state[slot * a.slot_stride] * a.mul_prev + (long)id * a.mul_cur) % a.buckets;
    row = row < 0 ? a.buckets : row;
    const bool ok = id >= 0 && id < a.vocab;
    const T* e = static_cast<const T*>(a.table) + (size_t)(ok ? id : 0) * a.width;
    const T* p = static_cast<const T*>(a.pairs) + (size_t)row * a.width;
    float* dst = a.x + (size_t)t * a.ldx;
    for (int i = threadIdx.x; i < a.ldx; i += 256) dst[i] = i < a.width ? (ok ? to_f(e[i]) : 0.f) + to_f(p[i]) : 0.f;
    if (a.qo_indptr[r + 1] - q0 > 1 || slot < 0) return;       // longer portions: pair_commit_kernel
    __syncthreads();
    if (threadIdx.x == 0) a.state[slot * a.slot_stride] = id;
}

__global__ void pair_commit_kernel(const PairEmbedArgs a) {
    const int r = blockIdx.x * blockDim.x + threadIdx.x;
    if (r >= a.reqs) return;
    const int q0 = a.qo_indptr[r], q1 = a.qo_indptr[r + 1], slot = a.slots[r];
    if (q1 - q0 > 1 && slot >= 0) a.state[slot * a.slot_stride] = a.tokens[q1 - 1];
}

// ------------------------------------------------ layer norm + convolution
struct ConvNormArgs {
    const float* x;                 // [n, ldx] residual stream
    float* x_out;                   // with y: x + sum of y / rms(y) * y_norm; never aliases x
    const void *y0, *y1;            // [n, ldy] pending outputs, or null (y1 only with y0)
    const float *y0_norm, *y1_norm; // [width]
    const float *w, *b;             // [width] layer norm; w null: only the pending outputs
    const float* conv;              // [taps][width], the current token's factor last; null: no convolution
    void* h;                        // [n, ldh]
    const int *tok_req, *qo_indptr, *slots, *reset;
    float* state;                   // slot 0: [taps - 1][width], oldest first
    float* stage;                   // [requests][taps - 1][width]: the new state of portions that several blocks walk
    float2* stats;                  // [n], or null: the form for few rows
    long slot_stride;
    int n, width, ldx, ldy, ldh, taps, rows_per_block;
    float eps;
};

// Two block-wide sums at once; red: 64 floats.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    a = warp_sum(a);
    b = warp_sum(b);
    __syncthreads();
    if (lane == 0) { red[warp] = a; red[32 + warp] = b; }
    __syncthreads();
    return make_float2(warp_sum(lane < nw ? red[lane] : 0.f), warp_sum(lane < nw ? red[32 + lane] : 0.f));
}

// A portion is walked by one block alone where all its rows fall into the block's rows: the state is then updated in place.
__device__ __forceinline__ bool one_block(int q0, int q1, int rows) { return q0 / rows == (q1 - 1) / rows; }

// Mean and 1 / deviation of row t, by the whole block (WIDE) or by a warp; pending outputs join the stream on the way.
template <typename T, int VEC, bool WIDE>
__device__ __forceinline__ float2 row_stats(const ConvNormArgs& a, int t, float* red) {
    const int nvec = a.width / VEC, i0 = WIDE ? threadIdx.x : threadIdx.x & 31, di = WIDE ? 256 : 32;
    auto sum2 = [&](float x, float y) {
        if constexpr (WIDE) return block_sum2(x, y, red);
        else return make_float2(warp_sum(x), warp_sum(y));
    };
    const float* xr = a.x + (size_t)t * a.ldx;
    const T* pr = static_cast<const T*>(a.y0) + (size_t)t * a.ldy;
    const T* qr = static_cast<const T*>(a.y1) + (size_t)t * a.ldy;
    float ip = 0.f, iq = 0.f;
    if (a.y0) {
        float sp = 0.f, sq = 0.f;
#pragma unroll 4
        for (int i = i0; i < nvec; i += di) {
            float f[VEC];
            load_vec<VEC>(pr + i * VEC, f);
#pragma unroll
            for (int k = 0; k < VEC; ++k) sp += f[k] * f[k];
            if (!a.y1) continue;
            load_vec<VEC>(qr + i * VEC, f);
#pragma unroll
            for (int k = 0; k < VEC; ++k) sq += f[k] * f[k];
        }
        const float2 s = sum2(sp, sq);
        ip = 1.f / sqrtf(s.x / (float)a.width + a.eps);
        iq = 1.f / sqrtf(s.y / (float)a.width + a.eps);
    }
    auto value = [&](int i, float (&v)[VEC]) {
        load_vec<VEC>(xr + i * VEC, v);
        if (!a.y0) return;
        float f[VEC], g[VEC];
        load_vec<VEC>(pr + i * VEC, f);
        load_vec<VEC>(a.y0_norm + i * VEC, g);
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[k] += f[k] * ip * g[k];
        if (!a.y1) return;
        load_vec<VEC>(qr + i * VEC, f);
        load_vec<VEC>(a.y1_norm + i * VEC, g);
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[k] += f[k] * iq * g[k];
    };
    // deviations are taken from the mean of the row's first columns: no digits lost where the mean is large
    float first[VEC], s0 = 0.f, n0 = 0.f, m = 0.f, d = 0.f;
    if (i0 < nvec) {
        value(i0, first);
#pragma unroll
        for (int k = 0; k < VEC; ++k) s0 += first[k];
        n0 = VEC;
    }
    const float2 lead = sum2(s0, n0);
    const float shift = lead.x / lead.y;
    float* xo = a.x_out ? a.x_out + (size_t)t * a.ldx : nullptr;
#pragma unroll 8
    for (int i = i0; i < nvec; i += di) {
        float v[VEC];
        value(i, v);
        if (xo) store_vec<VEC>(xo + i * VEC, v);
#pragma unroll
        for (int k = 0; k < VEC; ++k) {
            const float e = v[k] - shift;
            m += e;
            d += e * e;
        }
    }
    if (xo)
        for (int i = a.width + i0; i < a.ldx; i += di) xo[i] = 0.f;
    if (!a.w) return make_float2(0.f, 0.f);
    const float2 s = sum2(m, d);
    const float off = s.x / (float)a.width, var = fmaxf(s.y / (float)a.width - off * off, 0.f);
    return make_float2(shift + off, 1.f / sqrtf(var + a.eps));
}

// Columns [c, c + VEC) of the rows t0 .. t1 - 1, four rows' loads ahead; stats[t] of a row t, also of the rows ahead that belong to
// the first one's portion. BACK > 0: the convolution reaches back so far, and the norm outputs it reaches stay in registers; -1:
// any reach, they are formed again.
template <typename T, int VEC, int BACK>
__device__ __forceinline__ void conv_columns(const ConvNormArgs& a, int c, int t0, int t1, const float2* stats) {
    const int back = a.conv ? a.taps - 1 : 0;
    const float* x = a.x_out ? a.x_out : a.x;
    float w[VEC], bias[VEC];
    load_vec<VEC>(a.w + c, w);
    load_vec<VEC>(a.b + c, bias);
    int r = -1, q0 = 0, q1 = 0;
    const float* st = nullptr;
    bool fresh = false;
    auto norm = [&](int t, float (&v)[VEC]) {
        const float2 s = stats[t];
#pragma unroll
        for (int k = 0; k < VEC; ++k) v[k] = (v[k] - s.x) * s.y * w[k] + bias[k];
    };
    auto normed = [&](int t, float (&v)[VEC]) {      // of a row from `start` on, or of one ahead of the portion
        if (t >= q0) {
            load_vec<VEC>(x + (size_t)t * a.ldx + c, v);
            norm(t, v);
        } else if (fresh) {
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[k] = 0.f;
        } else {
            load_vec<VEC>(st + (size_t)(back + t - q0) * a.width + c, v);
        }
    };
    constexpr int KEEP = BACK > 0 ? BACK : 1;
    float past[KEEP][VEC], tap[KEEP + 1][VEC], ahead[4][VEC];
    if (BACK > 0) {
#pragma unroll
        for (int s = 0; s <= BACK; ++s) load_vec<VEC>(a.conv + (size_t)s * a.width + c, tap[s]);
    }
    for (int tb = t0; tb < t1; tb += 4) {
#pragma unroll
        for (int u = 0; u < 4; ++u)
            if (tb + u < t1) load_vec<VEC>(x + (size_t)(tb + u) * a.ldx + c, ahead[u]);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int t = tb + u;
            if (t >= t1) break;
            if (back && (r < 0 || t >= q1)) {
                r = a.tok_req[t];
                q0 = a.qo_indptr[r];
                q1 = a.qo_indptr[r + 1];
                const int slot = a.slots[r];
                fresh = slot < 0 || a.reset[r] != 0;
                st = a.state + (size_t)max(slot, 0) * a.slot_stride;
                if (BACK > 0) {
#pragma unroll
                    for (int s = 0; s < BACK; ++s) normed(t - BACK + s, past[s]);
                }
            }
            float o[VEC], v[VEC], g[VEC];
            norm(t, ahead[u]);
            if (BACK > 0) {
#pragma unroll
                for (int k = 0; k < VEC; ++k) {
                    o[k] = tap[BACK][k] * ahead[u][k];
#pragma unroll
                    for (int s = 0; s < BACK; ++s) o[k] += tap[s][k] * past[s][k];
#pragma unroll
                    for (int s = 0; s + 1 < BACK; ++s) past[s][k] = past[s + 1][k];
                    past[KEEP - 1][k] = ahead[u][k];
                }
            } else {
#pragma unroll
                for (int k = 0; k < VEC; ++k) o[k] = ahead[u][k];
                if (a.conv) {
                    load_vec<VEC>(a.conv + (size_t)back * a.width + c, g);
#pragma unroll
                    for (int k = 0; k < VEC; ++k) o[k] *= g[k];
                    for (int s = 0; s < back; ++s) {
                        normed(t - back + s, v);
                        load_vec<VEC>(a.conv + (size_t)s * a.width + c, g);
#pragma unroll
                        for (int k = 0; k < VEC; ++k) o[k] += g[k] * v[k];
                    }
                }
            }
            store_vec<VEC>(static_cast<T*>(a.h) + (size_t)t * a.ldh + c, o);
            if (!back || t != q1 - 1 || a.slots[r] < 0) continue;
            // the new history, oldest first: an old row is read before its place is written
            float* keep = one_block(q0, q1, a.rows_per_block) ? const_cast<float*>(st) : a.stage + (size_t)r * back * a.width;
            if (BACK > 0) {
#pragma unroll
                for (int s = 0; s < BACK; ++s) store_vec<VEC>(keep + (size_t)s * a.width + c, past[s]);
            } else {
                for (int s = 0; s < back; ++s) {
                    normed(t - back + 1 + s, v);
                    store_vec<VEC>(keep + (size_t)s * a.width + c, v);
                }
            }
        }
    }
}

// Zeros past the width of the rows t0 .. t1 - 1.
template <typename T>
__device__ __forceinline__ void pad_rows(const ConvNormArgs& a, int t0, int t1) {
    for (int t = t0 + (threadIdx.x >> 5); t < t1; t += 8)
        for (int i = a.width + (threadIdx.x & 31); i < a.ldh; i += 32) static_cast<T*>(a.h)[(size_t)t * a.ldh + i] = from_f<T>(0.f);
}

// Few rows: a block takes rows_per_block of them, whole; for the rows ahead of its first it forms the value that their own block
// writes too.
template <typename T, int VEC, int BACK>
__global__ void __launch_bounds__(256) conv_norm_kernel(const ConvNormArgs a) {
    extern __shared__ float2 stats[];                   // [taps - 1 + rows_per_block]
    __shared__ float red[64];
    pdl_trigger();
    // on their way to the L2 while the kernel ahead drains: what the norm and the convolution multiply with, then the history
    auto ahead = [](const float* p, long n) {
        for (long i = threadIdx.x * 32L; p && i < n; i += 256 * 32) asm volatile("prefetch.global.L2 [%0];" ::"l"(p + i));
    };
    ahead(a.y0_norm, a.width);
    ahead(a.y1_norm, a.width);
    ahead(a.w, a.width);
    ahead(a.b, a.width);
    ahead(a.conv, (long)a.taps * a.width);
    pdl_wait();
    const int back = a.conv ? a.taps - 1 : 0, t0 = blockIdx.x * a.rows_per_block, t1 = min(a.n, t0 + a.rows_per_block);
    int start = t0;
    if (back) {
        const int r = a.tok_req[t0], slot = a.slots[r];
        start = max(a.qo_indptr[r], t0 - back);
        if (slot >= 0) ahead(a.state + (size_t)slot * a.slot_stride, (long)back * a.width);
    }
    for (int t = start; t < t1; ++t) {
        const float2 s = row_stats<T, VEC, true>(a, t, red);
        if (threadIdx.x == 0) stats[t - t0 + back] = s;
    }
    if (!a.w) return;
    __syncthreads();
    for (int c = threadIdx.x * VEC; c + VEC <= a.width; c += 256 * VEC) conv_columns<T, VEC, BACK>(a, c, t0, t1, stats + back - t0);
    pad_rows<T>(a, t0, t1);
}

// Many rows, in two launches: statistics by a warp per row, then a block per rows_per_block rows and 256 vectors of columns.
template <typename T, int VEC>
__global__ void __launch_bounds__(256) conv_stats_kernel(const ConvNormArgs a) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (t >= a.n) return;
    const float2 s = row_stats<T, VEC, false>(a, t, nullptr);
    if ((threadIdx.x & 31) == 0) a.stats[t] = s;
}
template <typename T, int VEC, int BACK>
__global__ void __launch_bounds__(256) conv_apply_kernel(const ConvNormArgs a) {
    pdl_trigger();
    pdl_wait();
    const int t0 = blockIdx.y * a.rows_per_block, t1 = min(a.n, t0 + a.rows_per_block), c = (blockIdx.x * 256 + threadIdx.x) * VEC;
    if (c + VEC <= a.width) conv_columns<T, VEC, BACK>(a, c, t0, t1, a.stats);
    if (blockIdx.x == 0) pad_rows<T>(a, t0, t1);
}

__global__ void __launch_bounds__(256) conv_commit_kernel(const float* __restrict__ stage, float* __restrict__ state,
                                                          const int* __restrict__ qo_indptr, const int* __restrict__ slots,
                                                          long slot_stride, int elems, int rows_per_block) {
    const int r = blockIdx.x, slot = slots[r], q0 = qo_indptr[r], q1 = qo_indptr[r + 1];
    if (slot < 0 || q1 <= q0 || one_block(q0, q1, rows_per_block)) return;
    const int i = blockIdx.y * 256 + threadIdx.x;
    if (i < elems) state[(size_t)slot * slot_stride + i] = stage[(size_t)r * elems + i];
}

}  // namespace pie

using namespace pie;

// portions: some request brings more than one token
PIE_API int pie_pair_embed(const PairEmbedArgs* args, int f32, int portions, cudaStream_t st) {
    const PairEmbedArgs& a = *args;
    if (a.n <= 0) return 0;
    if (a.buckets <= 0 || a.width <= 0 || a.ldx < a.width) return (int)cudaErrorInvalidValue;
    if (f32) pair_embed_kernel<float><<<a.n, 256, 0, st>>>(a);
    else pair_embed_kernel<bf16><<<a.n, 256, 0, st>>>(a);
    if (portions) pair_commit_kernel<<<(a.reqs + 127) / 128, 128, 0, st>>>(a);
    return (int)cudaGetLastError();
}

// commit_requests: requests of a fire in which a portion may span several blocks (0: none does)
PIE_API int pie_conv_norm(const ConvNormArgs* args, int f32, int commit_requests, cudaStream_t st) {
    const ConvNormArgs& a = *args;
    if (a.n <= 0) return 0;
    const bool carried = a.conv && a.taps > 1;
    if (a.rows_per_block <= 0 || a.x_out == a.x || (a.y0 && (!a.x_out || !a.y0_norm)) || (!a.y0 && a.x_out) || (a.y1 && (!a.y0 || !a.y1_norm)) ||
        (a.w && (!a.b || !a.h)) || (a.conv && (!a.w || a.taps < 1)) || (carried && (!a.state || (commit_requests > 0 && !a.stage))))
        return (int)cudaErrorInvalidValue;
    auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = a.width % 4 == 0 && a.ldx % 4 == 0 && a.ldy % 4 == 0 && a.ldh % 4 == 0 && aligned(a.x) && aligned(a.x_out) && aligned(a.y0) &&
                     aligned(a.y1) && aligned(a.y0_norm) && aligned(a.y1_norm) && aligned(a.w) && aligned(a.b) && aligned(a.conv) && aligned(a.h) &&
                     (!carried || (aligned(a.state) && aligned(a.stage) && a.slot_stride % 4 == 0));
    const unsigned tiles = (a.n + a.rows_per_block - 1) / a.rows_per_block;
    const size_t smem = (size_t)((carried ? a.taps - 1 : 0) + a.rows_per_block) * sizeof(float2);
    if (smem > 40 * 1024) return (int)cudaErrorInvalidValue;
    cudaError_t e = cudaSuccess;
    auto run = [&](auto whole, auto stats, auto apply, int v) {
        if (!a.stats) {
            e = launch_pdl(whole, dim3(tiles), dim3(256), smem, st, a);
            return;
        }
        e = launch_pdl(stats, dim3((a.n + 7) / 8), dim3(256), 0, st, a);
        if (e == cudaSuccess && a.w) e = launch_pdl(apply, dim3((a.width / v + 255) / 256, tiles), dim3(256), 0, st, a);
    };
#define GO(T_, V_, B_) run(conv_norm_kernel<T_, V_, B_>, conv_stats_kernel<T_, V_>, conv_apply_kernel<T_, V_, B_>, V_)
#define GO_B(T_)                                                                       \
    if (!vec) GO(T_, 1, -1);                                                           \
    else if (!carried || a.taps > 4) GO(T_, 4, -1);                                    \
    else if (a.taps == 2) GO(T_, 4, 1);                                                \
    else if (a.taps == 3) GO(T_, 4, 2);                                                \
    else GO(T_, 4, 3)
    if (f32) { GO_B(float); } else { GO_B(bf16); }
#undef GO_B
#undef GO
    if (e != cudaSuccess) return (int)e;
    if (carried && commit_requests > 0)
        conv_commit_kernel<<<dim3(commit_requests, ((a.taps - 1) * a.width + 255) / 256), 256, 0, st>>>(
            a.stage, a.state, a.qo_indptr, a.slots, a.slot_stride, (a.taps - 1) * a.width, a.rows_per_block);
    return (int)cudaGetLastError();
}
