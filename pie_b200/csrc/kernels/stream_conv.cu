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

// One block walks rows_per_block consecutive tokens. The norm outputs of the last taps - 1 tokens go round in shared memory, every
// thread seeing its own columns only; those before the block's first token are computed again, or read from the state.
template <typename T, int MAXV, int VEC>
__global__ void __launch_bounds__(256) conv_norm_kernel(const ConvNormArgs a) {
    extern __shared__ __align__(16) float hist[];       // [taps - 1][nvec * VEC]
    __shared__ float red[64];
    pdl_trigger();
    pdl_wait();
    const int nvec = a.width / VEC, back = a.conv ? a.taps - 1 : 0;
    auto each = [&](auto f) {
#pragma unroll
        for (int j = 0; j < MAXV; ++j) {
            const int i = threadIdx.x + j * 256;
            if (i < nvec) f(j, i * VEC);
        }
    };
    auto load_stream = [&](int t, float (&v)[MAXV][VEC]) {
        const float* xr = a.x + (size_t)t * a.ldx;
        each([&](int j, int c) { load_vec<VEC>(xr + c, v[j]); });
        if (!a.y0) return;
        float p[MAXV][VEC], q[MAXV][VEC], sp = 0.f, sq = 0.f;
        const T* pr = static_cast<const T*>(a.y0) + (size_t)t * a.ldy;
        const T* qr = static_cast<const T*>(a.y1) + (size_t)t * a.ldy;
        each([&](int j, int c) {
            load_vec<VEC>(pr + c, p[j]);
            if (a.y1) load_vec<VEC>(qr + c, q[j]);
#pragma unroll
            for (int k = 0; k < VEC; ++k) {
                if (!a.y1) q[j][k] = 0.f;
                sp += p[j][k] * p[j][k];
                sq += q[j][k] * q[j][k];
            }
        });
        const float2 s = block_sum2(sp, sq, red);
        const float ip = 1.f / sqrtf(s.x / (float)a.width + a.eps), iq = 1.f / sqrtf(s.y / (float)a.width + a.eps);
        each([&](int j, int c) {
            float g[VEC];
            load_vec<VEC>(a.y0_norm + c, g);
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[j][k] += p[j][k] * ip * g[k];
            if (!a.y1) return;
            load_vec<VEC>(a.y1_norm + c, g);
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[j][k] += q[j][k] * iq * g[k];
        });
    };
    auto normalise = [&](float (&v)[MAXV][VEC]) {
        float s = 0.f;
        each([&](int j, int) {
#pragma unroll
            for (int k = 0; k < VEC; ++k) s += v[j][k];
        });
        const float mean = block_sum(s, red) / (float)a.width;
        s = 0.f;
        each([&](int j, int) {
#pragma unroll
            for (int k = 0; k < VEC; ++k) {
                v[j][k] -= mean;
                s += v[j][k] * v[j][k];
            }
        });
        const float inv = 1.f / sqrtf(block_sum(s, red) / (float)a.width + a.eps);
        each([&](int j, int c) {
            float g[VEC], b[VEC];
            load_vec<VEC>(a.w + c, g);
            load_vec<VEC>(a.b + c, b);
#pragma unroll
            for (int k = 0; k < VEC; ++k) v[j][k] = v[j][k] * inv * g[k] + b[k];
        });
    };
    auto ring = [&](int t) { return hist + (size_t)((t + back) % back) * a.width; };      // t >= -back

    float v[MAXV][VEC];
    const int t0 = blockIdx.x * a.rows_per_block, t1 = min(a.n, t0 + a.rows_per_block);
    for (int t = t0; t < t1; ++t) {
        int r = 0, q0 = 0, q1 = 0, slot = -1;
        if (back) {
            r = a.tok_req[t];
            q0 = a.qo_indptr[r];
            q1 = a.qo_indptr[r + 1];
            slot = a.slots[r];
            if (t == t0 || t == q0) {
                const bool fresh = slot < 0 || a.reset[r] != 0;
                const float* st = a.state + (size_t)max(slot, 0) * a.slot_stride;
                for (int s = t - back; s < t; ++s) {
                    float* dst = ring(s);
                    if (s >= q0) {
                        load_stream(s, v);
                        normalise(v);
                        each([&](int j, int c) { store_vec<VEC>(dst + c, v[j]); });
                    } else {
                        each([&](int, int c) {
                            float f[VEC];
                            load_vec<VEC>(st + (size_t)(back + s - q0) * a.width + c, f);
#pragma unroll
                            for (int k = 0; k < VEC; ++k) f[k] = fresh ? 0.f : f[k];
                            store_vec<VEC>(dst + c, f);
                        });
                    }
                }
            }
        }
        load_stream(t, v);
        if (a.x_out) {
            float* xo = a.x_out + (size_t)t * a.ldx;
            each([&](int j, int c) { store_vec<VEC>(xo + c, v[j]); });
            for (int i = a.width + threadIdx.x; i < a.ldx; i += 256) xo[i] = 0.f;
        }
        if (!a.w) continue;
        normalise(v);
        T* hr = static_cast<T*>(a.h) + (size_t)t * a.ldh;
        float* keep = nullptr;
        if (back && t == q1 - 1 && slot >= 0)
            keep = one_block(q0, q1, a.rows_per_block) ? a.state + (size_t)slot * a.slot_stride : a.stage + (size_t)r * back * a.width;
        each([&](int j, int c) {
            float o[VEC], g[VEC], f[VEC];
            if (a.conv) {
                load_vec<VEC>(a.conv + (size_t)back * a.width + c, g);
#pragma unroll
                for (int k = 0; k < VEC; ++k) o[k] = g[k] * v[j][k];
                for (int s = 0; s < back; ++s) {
                    load_vec<VEC>(ring(t - back + s) + c, f);
                    load_vec<VEC>(a.conv + (size_t)s * a.width + c, g);
#pragma unroll
                    for (int k = 0; k < VEC; ++k) o[k] += g[k] * f[k];
                }
                if (back) store_vec<VEC>(ring(t) + c, v[j]);
                for (int s = 0; keep && s < back; ++s) {
                    load_vec<VEC>(ring(t - back + 1 + s) + c, f);
                    store_vec<VEC>(keep + (size_t)s * a.width + c, f);
                }
                store_vec<VEC>(hr + c, o);
            } else {
                store_vec<VEC>(hr + c, v[j]);
            }
        });
        for (int i = a.width + threadIdx.x; i < a.ldh; i += 256) hr[i] = from_f<T>(0.f);
    }
}

__global__ void __launch_bounds__(256) conv_commit_kernel(const float* __restrict__ stage, float* __restrict__ state,
                                                          const int* __restrict__ qo_indptr, const int* __restrict__ slots,
                                                          long slot_stride, int elems, int rows_per_block) {
    const int r = blockIdx.x, slot = slots[r], q0 = qo_indptr[r], q1 = qo_indptr[r + 1];
    if (slot < 0 || q1 <= q0 || one_block(q0, q1, rows_per_block)) return;
    for (int i = threadIdx.x; i < elems; i += 256) state[(size_t)slot * slot_stride + i] = stage[(size_t)r * elems + i];
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
    const int per = (a.width / (vec ? 4 : 1) + 255) / 256;
    if (per > (vec ? 16 : 32)) return (int)cudaErrorInvalidValue;
    const dim3 grid((a.n + a.rows_per_block - 1) / a.rows_per_block);
    const size_t smem = carried ? (size_t)(a.taps - 1) * a.width * sizeof(float) : 0;
    if (smem > 220 * 1024) return (int)cudaErrorInvalidValue;
#define GO(T_, M_, V_)                                                                                                    \
    {                                                                                                                     \
        auto kern = conv_norm_kernel<T_, M_, V_>;                                                                         \
        cudaError_t e = smem > 47 * 1024 ? cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) : cudaSuccess; \
        if (e == cudaSuccess) e = launch_pdl(kern, grid, dim3(256), smem, st, a);                                         \
        if (e != cudaSuccess) return (int)e;                                                                              \
    }
#define GO_M(T_, V_)                                                                                     \
    if (per <= 1) GO(T_, 1, V_) else if (per <= 2) GO(T_, 2, V_) else if (per <= 4) GO(T_, 4, V_)        \
    else if (per <= 8) GO(T_, 8, V_) else if (per <= 16) GO(T_, 16, V_) else GO(T_, 32, 1)
    if (f32) { if (vec) { GO_M(float, 4) } else { GO_M(float, 1) } }
    else if (vec) { GO_M(bf16, 4) } else { GO_M(bf16, 1) }
#undef GO_M
#undef GO
    if (carried && commit_requests > 0)
        conv_commit_kernel<<<commit_requests, 256, 0, st>>>(a.stage, a.state, a.qo_indptr, a.slots, a.slot_stride, (a.taps - 1) * a.width,
                                                            a.rows_per_block);
    return (int)cudaGetLastError();
}
