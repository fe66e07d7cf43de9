// Kernels of blocks that keep a 32-bit residual stream, shift their mixer's input by one token and attend over a cached
// latent: stream embedding, [token-input residual + grouped RMSNorm + token shift] in one pass, latent rows (RMSNorm,
// rotation, paged write) with the query rotation, latent attention (any sizes, bf16 or 32-bit), xIELU, token-input gate.
//
// T is the activation type: bf16 when serving, float for the 32-bit path. The residual stream, norms, shift state,
// angles, scores and softmax weights are 32-bit in both. Leading dimensions (ld*) are in elements; columns between a
// row's width and its padded width are written as zeros, since the GEMMs read them.
#include "typed.cuh"

namespace pie {

// ---------------------------------------------------------------- embedding
// x[t, :] = table[tokens[t], :] * scale in 32-bit (zeros for an id outside the table and in the padding columns).
template <typename T>
__global__ void stream_embed_kernel(const int* __restrict__ tokens, const T* __restrict__ table, float* __restrict__ x,
                                    int width, int ldx, int vocab, float scale) {
    const int t = blockIdx.x, id = tokens[t];
    const bool ok = id >= 0 && id < vocab;
    const T* src = table + (size_t)(ok ? id : 0) * width;
    float* dst = x + (size_t)t * ldx;
    for (int i = threadIdx.x; i < ldx; i += blockDim.x) dst[i] = ok && i < width ? to_f(src[i]) * scale : 0.f;
}

// ------------------------------------------- stream norm (+ token shift)
struct StreamNormArgs {
    const float* x;             // [n, ldx] residual stream
    const void* y;              // [n, ldy] pending token input, or null: x += y / rms(y) * y_norm
    const void* y_norm;
    float* x_out;               // [n, ldx] updated stream (null when y is null); never aliases x
    const void* norm_w;         // null: only the pending update, and with h a copy of the stream in the activation type
    const void* shift;          // null: no token shift
    void* h;                    // [n, ldh] norm(x); null without norm_w: none
    void* hs;                   // [n, ldh] h + (previous token's h - h) * shift
    const int* tok_req;         // request of a token
    const int* qo_indptr;
    const int* slots;           // state slot of a request (< 0: padding row, no state)
    const int* reset;           // 1: the request's state starts from zeros
    float* state;               // [slots, width] previous token's h
    float* stage;               // [requests, width] last h of a portion of two tokens or more
    int n, width, ldx, ldy, ldh, groups, rows_per_block;
    float eps;
};

// One block walks rows_per_block consecutive tokens. The previous token's h is carried in registers; for the first
// token of a block it comes from the state (start of a portion) or is computed again from the stream. A single-token
// portion updates its state in place (no other block reads it); a longer one leaves its last h in `stage`, because the
// block with its first token may still be reading the state (shift_commit_kernel moves it).
// GT is the type of the gains (norm_w, y_norm).
template <typename T, int MAXV, int VEC, typename GT = T>
__global__ void __launch_bounds__(256) stream_norm_kernel(const StreamNormArgs a) {
    extern __shared__ float sq[];                 // one sum of squares per vector, then one factor per group
    __shared__ float red[32];
    pdl_trigger();
    pdl_wait();
    const int nvec = a.width / VEC, part = a.width / a.groups, part_vec = part / VEC;
    float* factor = sq + nvec;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const GT* y_norm = static_cast<const GT*>(a.y_norm);
    const GT* norm_w = static_cast<const GT*>(a.norm_w);
    const T* shift = static_cast<const T*>(a.shift);

    auto load_stream = [&](int t, float (&v)[MAXV][VEC]) {
        const float* xr = a.x + (size_t)t * a.ldx;
#pragma unroll
        for (int j = 0; j < MAXV; ++j) {
            const int i = threadIdx.x + j * 256;
            if (i < nvec) load_vec<VEC>(xr + i * VEC, v[j]);
        }
        if (!a.y) return;
        const T* yr = static_cast<const T*>(a.y) + (size_t)t * a.ldy;
        float yv[MAXV][VEC], ss = 0.f;
#pragma unroll
        for (int j = 0; j < MAXV; ++j) {
            const int i = threadIdx.x + j * 256;
            if (i < nvec) {
                load_vec<VEC>(yr + i * VEC, yv[j]);
#pragma unroll
                for (int k = 0; k < VEC; ++k) ss += yv[j][k] * yv[j][k];
            }
        }
        const float inv = 1.f / sqrtf(block_sum(ss, red) / (float)a.width + a.eps);
#pragma unroll
        for (int j = 0; j < MAXV; ++j) {
            const int i = threadIdx.x + j * 256;
            if (i < nvec) {
                float w[VEC];
                load_vec<VEC>(y_norm + i * VEC, w);
#pragma unroll
                for (int k = 0; k < VEC; ++k) v[j][k] += yv[j][k] * inv * w[k];
            }
        }
    };
    auto normalise = [&](float (&v)[MAXV][VEC]) {
#pragma unroll
        for (int j = 0; j < MAXV; ++j) {
            const int i = threadIdx.x + j * 256;
            if (i < nvec) {
                float s = 0.f;
#pragma unroll
                for (int k = 0; k < VEC; ++k) s += v[j][k] * v[j][k];
                sq[i] = s;
            }
        }
        __syncthreads();
        for (int g = warp; g < a.groups; g += 8) {
            float s = 0.f;
            for (int i = lane; i < part_vec; i += 32) s += sq[g * part_vec + i];
            s = warp_sum(s);
            if (lane == 0) factor[g] = 1.f / sqrtf(s / (float)part + a.eps);
        }
        __syncthreads();
#pragma unroll
        for (int j = 0; j < MAXV; ++j) {
            const int i = threadIdx.x + j * 256;
            if (i < nvec) {
                float w[VEC];
                load_vec<VEC>(norm_w + i * VEC, w);
                const float f = factor[i / part_vec];
#pragma unroll
                for (int k = 0; k < VEC; ++k) v[j][k] = v[j][k] * f * w[k];
            }
        }
        __syncthreads();
    };

    float prev[MAXV][VEC], v[MAXV][VEC];
    const int t0 = blockIdx.x * a.rows_per_block, t1 = min(a.n, t0 + a.rows_per_block);
    for (int t = t0; t < t1; ++t) {
        int r = 0, slot = -1;
        bool first = false, last = false, single = false;
        if (shift) {
            r = a.tok_req[t];
            const int q0 = a.qo_indptr[r], q1 = a.qo_indptr[r + 1];
            first = t == q0;
            last = t == q1 - 1;
            single = q1 - q0 == 1;
            slot = a.slots[r];
            if (first) {
                const bool zero = slot < 0 || a.reset[r] != 0;
                const float* st = a.state + (size_t)max(slot, 0) * a.width;
#pragma unroll
                for (int j = 0; j < MAXV; ++j) {
                    const int i = threadIdx.x + j * 256;
                    if (i < nvec) {
                        load_vec<VEC>(st + i * VEC, prev[j]);
#pragma unroll
                        for (int k = 0; k < VEC; ++k) prev[j][k] = zero ? 0.f : prev[j][k];
                    }
                }
            } else if (t == t0) {
                load_stream(t - 1, prev);
                normalise(prev);
            }
        }
        load_stream(t, v);
        if (a.x_out) {
            float* xo = a.x_out + (size_t)t * a.ldx;
#pragma unroll
            for (int j = 0; j < MAXV; ++j) {
                const int i = threadIdx.x + j * 256;
                if (i < nvec) store_vec<VEC>(xo + i * VEC, v[j]);
            }
            for (int i = a.width + threadIdx.x; i < a.ldx; i += 256) xo[i] = 0.f;
        }
        if (!a.h) continue;
        if (norm_w) normalise(v);
        T* hr = static_cast<T*>(a.h) + (size_t)t * a.ldh;
        T* hsr = shift ? static_cast<T*>(a.hs) + (size_t)t * a.ldh : nullptr;
        float* keep = nullptr;
        if (last && slot >= 0) keep = single ? a.state + (size_t)slot * a.width : a.stage + (size_t)r * a.width;
#pragma unroll
        for (int j = 0; j < MAXV; ++j) {
            const int i = threadIdx.x + j * 256;
            if (i < nvec) {
                store_vec<VEC>(hr + i * VEC, v[j]);
                if (shift) {
                    float m[VEC], s[VEC];
                    load_vec<VEC>(shift + i * VEC, m);
#pragma unroll
                    for (int k = 0; k < VEC; ++k) {
                        s[k] = v[j][k] + (prev[j][k] - v[j][k]) * m[k];
                        prev[j][k] = v[j][k];
                    }
                    store_vec<VEC>(hsr + i * VEC, s);
                    if (keep) store_vec<VEC>(keep + i * VEC, v[j]);
                }
            }
        }
        for (int i = a.width + threadIdx.x; i < a.ldh; i += 256) {
            hr[i] = from_f<T>(0.f);
            if (hsr) hsr[i] = from_f<T>(0.f);
        }
    }
}

__global__ void shift_commit_kernel(const float* __restrict__ stage, float* __restrict__ state, const int* __restrict__ qo_indptr,
                                    const int* __restrict__ slots, int width) {
    const int r = blockIdx.x, slot = slots[r];
    if (slot < 0 || qo_indptr[r + 1] - qo_indptr[r] < 2) return;
    for (int i = threadIdx.x; i < width; i += blockDim.x) state[(size_t)slot * width + i] = stage[(size_t)r * width + i];
}

// ------------------------------------- query rotation + latent cache rows
struct LatentRowsArgs {
    const void* q;              // [n, ld]: heads x (dim | rot_dim) queries
    const void* kv;             // [n, ld_kv]: latent | shared key part (read if `cache`)
    const int* positions;
    const int* slots;           // cache slot (page * page_size + offset), < 0: no write
    const float* inv_freq;      // [rot_dims / 2]
    const void* norm_w;         // [rank]
    void* q_out;                // rows of q_width per (token, head)
    void* cache;                // [slots, cache_row], null for a layer that borrows another's rows
    int n, ld, ld_kv, heads, dim, rot_dim, rot_dims, rank, rank_pad, cache_row;
    int copy_nope;              // 1: q_out = (dim | rotated part | zeros); 0: (.. | rotated part | zeros), see q_zero
    int q_width, q_rot, q_zero; // row width, column of the rotated part, first column zeroed before it
    int adjacent;               // 1: the halves of a rotated pair are neighbours, 0: rot_dims / 2 apart
    float eps, rot_factor;      // factor on cos and sin
};

// One warp per (token, head) and one more per token for the latent.
template <typename T>
__global__ void __launch_bounds__(256) latent_rows_kernel(const LatentRowsArgs a) {
    pdl_trigger();
    pdl_wait();
    const int units = a.heads + (a.cache ? 1 : 0);
    const long w = (blockIdx.x * 256L + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (w >= (long)a.n * units) return;
    const int t = (int)(w / units), u = (int)(w - (long)t * units);
    const bool is_q = u < a.heads;
    const T* rot_src;
    T *rot_dst, *end;
    if (is_q) {
        const T* src = static_cast<const T*>(a.q) + (size_t)t * a.ld + (size_t)u * (a.dim + a.rot_dim);
        T* dst = static_cast<T*>(a.q_out) + ((size_t)t * a.heads + u) * a.q_width;
        if (a.copy_nope) {
            constexpr int E = 16 / sizeof(T);
            const bool vec = ((uintptr_t)src & 15) == 0 && ((uintptr_t)dst & 15) == 0 && a.dim % E == 0;
            if (vec)
                for (int i = lane; i < a.dim / E; i += 32) reinterpret_cast<uint4*>(dst)[i] = reinterpret_cast<const uint4*>(src)[i];
            else
                for (int i = lane; i < a.dim; i += 32) dst[i] = src[i];
        }
        for (int i = a.q_zero + lane; i < a.q_rot; i += 32) dst[i] = from_f<T>(0.f);
        rot_src = src + a.dim;
        rot_dst = dst + a.q_rot;
        end = dst + a.q_width;
    } else {
        const int slot = a.slots[t];
        if (slot < 0) return;
        const T* src = static_cast<const T*>(a.kv) + (size_t)t * a.ld_kv;
        T* dst = static_cast<T*>(a.cache) + (size_t)slot * a.cache_row;
        const T* nw = static_cast<const T*>(a.norm_w);
        float ss = 0.f;
        for (int i = lane; i < a.rank; i += 32) { const float f = to_f(src[i]); ss += f * f; }
        const float inv = 1.f / sqrtf(warp_sum(ss) / (float)a.rank + a.eps);
        for (int i = lane; i < a.rank_pad; i += 32) dst[i] = from_f<T>(i < a.rank ? to_f(src[i]) * inv * to_f(nw[i]) : 0.f);
        rot_src = src + a.rank;
        rot_dst = dst + a.rank_pad;
        end = dst + a.cache_row;
    }
    const int half = a.rot_dims / 2;
    const float pos = (float)a.positions[t];
    for (int i = lane; i < half; i += 32) {
        float s, c;
        sincosf(pos * a.inv_freq[i], &s, &c);
        s *= a.rot_factor;
        c *= a.rot_factor;
        const int e0 = a.adjacent ? 2 * i : i, e1 = a.adjacent ? e0 + 1 : i + half;
        const float p = to_f(rot_src[e0]), q = to_f(rot_src[e1]);
        rot_dst[e0] = from_f<T>(p * c - q * s);
        rot_dst[e1] = from_f<T>(q * c + p * s);
    }
    for (int i = a.rot_dims + lane; i < a.rot_dim; i += 32) rot_dst[i] = rot_src[i];
    for (T* p = rot_dst + a.rot_dim + lane; p < end; p += 32) *p = from_f<T>(0.f);
}

// ------------------------------------------------------- latent attention
struct LatentAttnArgs {
    const void* q;              // [n, heads, row]: query against the latent, then the rotated part
    const void* cache;          // [pages, page_size, cache_row]
    const int* page_indices;
    const int* kv_page_indptr;
    const int* qo_indptr;
    const int* kv_lens;
    const int* tok_req;
    const int* slots;           // cache slot of every token; < 0: padding row
    const uint32_t* mask_bits;  // custom mask words, or null (causal)
    const long* mask_word_indptr;
    void* out;                  // [n, heads, rank_pad]: softmax-weighted latents
    int n, heads, row, rank_pad, cache_row, page_size, window_left;
    float scale;
};

// Any sizes, either type: one warp per (token, head), one key at a time. ME = elements of a row per lane.
template <typename T, int ME>
__global__ void __launch_bounds__(128) latent_attn_warp_kernel(const LatentAttnArgs a) {
    pdl_trigger();
    pdl_wait();
    const long w = (blockIdx.x * 128L + threadIdx.x) >> 5;
    const int lane = threadIdx.x & 31;
    if (w >= (long)a.n * a.heads) return;
    const int t = (int)(w / a.heads);
    float q[ME], acc[ME], m = -INFINITY, l = 0.f;
    const T* qr = static_cast<const T*>(a.q) + w * a.row;
#pragma unroll
    for (int i = 0; i < ME; ++i) {
        const int e = lane + 32 * i;
        q[i] = e < a.row ? to_f(qr[e]) * a.scale : 0.f;
        acc[i] = 0.f;
    }
    if (a.slots[t] >= 0) {
        const int r = a.tok_req[t], q0 = a.qo_indptr[r], qlen = a.qo_indptr[r + 1] - q0, kv_len = a.kv_lens[r];
        const int pos = kv_len - qlen + (t - q0);
        const uint32_t* bits = nullptr;
        if (a.mask_bits) bits = a.mask_bits + a.mask_word_indptr[r] + (long)(t - q0) * ((kv_len + 31) / 32);
        const int* pages = a.page_indices + a.kv_page_indptr[r];
        const int hi = bits ? kv_len : pos + 1;
        for (int j = max(0, pos - a.window_left); j < hi; ++j) {
            if (bits && !(bits[j >> 5] >> (j & 31) & 1u)) continue;
            const T* kr = static_cast<const T*>(a.cache) +
                          ((size_t)pages[j / a.page_size] * a.page_size + j % a.page_size) * a.cache_row;
            float k[ME], s = 0.f;
#pragma unroll
            for (int i = 0; i < ME; ++i) {
                const int e = lane + 32 * i;
                k[i] = e < a.row ? to_f(kr[e]) : 0.f;
                s += q[i] * k[i];
            }
            s = warp_sum(s);
            const float mn = fmaxf(m, s), c = expf(m - mn), p = expf(s - mn);
            m = mn;
            l = l * c + p;
#pragma unroll
            for (int i = 0; i < ME; ++i) acc[i] = acc[i] * c + p * k[i];
        }
    }
    const float inv = l > 0.f ? 1.f / l : 0.f;
    T* dst = static_cast<T*>(a.out) + w * a.rank_pad;
#pragma unroll
    for (int i = 0; i < ME; ++i) {
        const int e = lane + 32 * i;
        if (e < a.rank_pad) dst[e] = from_f<T>(acc[i] * inv);
    }
}

// ------------------------------------------------------------ activations
__device__ __forceinline__ float softplus(float z) { return log1pf(expf(-fabsf(z))) + fmaxf(z, 0.f); }
// xIELU with a = softplus(p), b = 1/2 + softplus(q): a z^2 + z/2 right of zero, b (e^z - 1 - z) + z/2 left of it
__device__ __forceinline__ float xielu(float z, float a, float b) {
    return (z > 0.f ? a * z * z : b * (expm1f(z) - z)) + 0.5f * z;
}

// y = xIELU(y + bias), in place; act holds the two learned numbers.
template <typename T>
__global__ void bias_xielu_kernel(T* __restrict__ y, int ld, const T* __restrict__ bias, const T* __restrict__ act, long total, int cols) {
    const float a = softplus(to_f(act[0])), b = 0.5f + softplus(to_f(act[1]));
    for (long i = blockIdx.x * (long)blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
        const long r = i / cols;
        const int c = (int)(i - r * cols);
        T* p = y + r * ld + c;
        *p = from_f<T>(xielu(to_f(*p) + to_f(bias[c]), a, b));
    }
}

// x_out = x + d (+ bias), and a copy in the activation type for the product that reads the stream.
template <typename T>
__global__ void stream_add_kernel(const float* __restrict__ x, const T* __restrict__ d, const T* __restrict__ bias,
                                  float* __restrict__ x_out, T* __restrict__ copy, int cols, long total) {
    for (long i = blockIdx.x * (long)blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
        const float v = x[i] + to_f(d[i]) + (bias ? to_f(bias[i % cols]) : 0.f);
        x_out[i] = v;
        if (copy) copy[i] = from_f<T>(v);
    }
}

// g = gelu_tanh(z) * e, e = columns [col0, col0 + dim) of the token's row in the side table; zeros in the padding columns.
// z arrives as `splits` arrays of Z, z_split elements apart, that add up to it (one array: the product itself).
template <typename T, typename Z>
__global__ void side_gate_kernel(const Z* __restrict__ z, int ldz, long z_split, int splits, const T* __restrict__ table, int ldt,
                                 const int* __restrict__ tokens, T* __restrict__ g, int ldg, int dim, int col0, int vocab, long total) {
    pdl_trigger();
    pdl_wait();
    for (long i = blockIdx.x * (long)blockDim.x + threadIdx.x; i < total; i += (long)gridDim.x * blockDim.x) {
        const long t = i / ldg;
        const int c = (int)(i - t * ldg), id = tokens[t];
        float v = 0.f;
        if (c < dim && id >= 0 && id < vocab) {
            const float e = to_f(table[(size_t)id * ldt + col0 + c]);
            float x = 0.f;
#pragma unroll 4
            for (int s = 0; s < splits; ++s) x += to_f(z[s * z_split + t * ldz + c]);
            v = 0.5f * x * (1.f + tanhf(0.7978845608028654f * (x + 0.044715f * x * x * x))) * e;
        }
        g[i] = from_f<T>(v);
    }
}

static int grid_for(long total) {
    const long b = (total + 255) / 256;
    return (int)(b < 4736 ? (b < 1 ? 1 : b) : 4736);
}

}  // namespace pie

using namespace pie;

PIE_API int pie_stream_embed(const int* tokens, const void* table, float* x, int n, int width, int ldx, int vocab, float scale, int f32,
                             cudaStream_t st) {
    if (n <= 0) return 0;
    if (f32) stream_embed_kernel<float><<<n, 256, 0, st>>>(tokens, (const float*)table, x, width, ldx, vocab, scale);
    else stream_embed_kernel<bf16><<<n, 256, 0, st>>>(tokens, (const bf16*)table, x, width, ldx, vocab, scale);
    return (int)cudaGetLastError();
}

// gain_f32: norm_w and y_norm are 32-bit also where the activations are not
PIE_API int pie_stream_norm(const StreamNormArgs* args, int f32, int gain_f32, int commit_requests, cudaStream_t st) {
    const StreamNormArgs& a = *args;
    if (a.n <= 0) return 0;
    if (a.groups <= 0 || a.width % a.groups || a.rows_per_block <= 0 || a.x_out == a.x || (a.y && !a.x_out) ||
        (a.norm_w && !a.h) || (a.shift && (!a.norm_w || !a.hs || !a.state || (commit_requests > 0 && !a.stage))))
        return (int)cudaErrorInvalidValue;
    const int part = a.width / a.groups;
    const bool vec = part % 4 == 0 && a.ldx % 4 == 0 && a.ldy % 4 == 0 && a.ldh % 4 == 0;
    const int per = (a.width / (vec ? 4 : 1) + 255) / 256;
    if (per > (vec ? 16 : 32)) return (int)cudaErrorInvalidValue;
    const dim3 grid((a.n + a.rows_per_block - 1) / a.rows_per_block);
    const size_t smem = ((vec ? a.width / 4 : a.width) + a.groups) * sizeof(float);
#define GO(T_, M_, V_, G_)                                                                   \
    {                                                                                        \
        cudaError_t e = launch_pdl(stream_norm_kernel<T_, M_, V_, G_>, grid, dim3(256), smem, st, a); \
        if (e != cudaSuccess) return (int)e;                                                 \
    }
#define GO_M(T_, V_, G_)                                                                     \
    if (per <= 1) GO(T_, 1, V_, G_) else if (per <= 2) GO(T_, 2, V_, G_) else if (per <= 4) GO(T_, 4, V_, G_) \
    else if (per <= 8) GO(T_, 8, V_, G_) else if (per <= 16) GO(T_, 16, V_, G_) else GO(T_, 32, 1, G_)
    if (f32) { if (vec) { GO_M(float, 4, float) } else { GO_M(float, 1, float) } }
    else if (gain_f32) { if (vec) { GO_M(bf16, 4, float) } else { GO_M(bf16, 1, float) } }
    else { if (vec) { GO_M(bf16, 4, bf16) } else { GO_M(bf16, 1, bf16) } }
#undef GO_M
#undef GO
    if (a.shift && commit_requests > 0)
        shift_commit_kernel<<<commit_requests, 256, 0, st>>>(a.stage, a.state, a.qo_indptr, a.slots, a.width);
    return (int)cudaGetLastError();
}

PIE_API int pie_latent_rows(const LatentRowsArgs* args, int f32, cudaStream_t st) {
    const LatentRowsArgs& a = *args;
    if (a.n <= 0) return 0;
    if (a.rot_dims % 2 || a.rot_dims > a.rot_dim || a.q_rot + a.rot_dim > a.q_width ||
        (a.cache && a.rank_pad + a.rot_dim > a.cache_row))
        return (int)cudaErrorInvalidValue;
    const long warps = (long)a.n * (a.heads + (a.cache ? 1 : 0));
    const dim3 grid((unsigned)((warps + 7) / 8));
    const cudaError_t e = f32 ? launch_pdl(latent_rows_kernel<float>, grid, dim3(256), 0, st, a)
                              : launch_pdl(latent_rows_kernel<bf16>, grid, dim3(256), 0, st, a);
    return (int)(e != cudaSuccess ? e : cudaGetLastError());
}

PIE_API int pie_latent_attn_warp(const LatentAttnArgs* args, int f32, cudaStream_t st) {
    const LatentAttnArgs& a = *args;
    if (a.n <= 0) return 0;
    if (a.rank_pad > a.row || a.row > a.cache_row || a.row > 32 * 40) return (int)cudaErrorInvalidValue;
    const dim3 grid((unsigned)(((long)a.n * a.heads + 3) / 4));
#define GO(T_, M_) latent_attn_warp_kernel<T_, M_><<<grid, 128, 0, st>>>(a)
#define GO_M(T_) \
    if (a.row <= 32 * 5) GO(T_, 5); else if (a.row <= 32 * 10) GO(T_, 10); else if (a.row <= 32 * 20) GO(T_, 20); else GO(T_, 40);
    if (f32) { GO_M(float) } else { GO_M(bf16) }
#undef GO_M
#undef GO
    return (int)cudaGetLastError();
}

PIE_API int pie_bias_xielu(void* y, int ld, const void* bias, const void* act, int rows, int cols, int f32, cudaStream_t st) {
    const long total = (long)rows * cols;
    if (total <= 0) return 0;
    if (f32) bias_xielu_kernel<float><<<grid_for(total), 256, 0, st>>>((float*)y, ld, (const float*)bias, (const float*)act, total, cols);
    else bias_xielu_kernel<bf16><<<grid_for(total), 256, 0, st>>>((bf16*)y, ld, (const bf16*)bias, (const bf16*)act, total, cols);
    return (int)cudaGetLastError();
}

PIE_API int pie_stream_add(const float* x, const void* d, const void* bias, float* x_out, void* copy, int rows, int cols, int f32, cudaStream_t st) {
    const long total = (long)rows * cols;
    if (total <= 0) return 0;
    if (f32)
        stream_add_kernel<float><<<grid_for(total), 256, 0, st>>>(x, (const float*)d, (const float*)bias, x_out, (float*)copy, cols, total);
    else
        stream_add_kernel<bf16><<<grid_for(total), 256, 0, st>>>(x, (const bf16*)d, (const bf16*)bias, x_out, (bf16*)copy, cols, total);
    return (int)cudaGetLastError();
}

// z_f32: the partial products are 32-bit (else they have the type of the others, which f32 gives)
PIE_API int pie_side_gate(const void* z, int ldz, long z_split, int splits, int z_f32, const void* table, int ldt, const int* tokens,
                          void* g, int ldg, int dim, int col0, int vocab, int rows, int f32, cudaStream_t st) {
    const long total = (long)rows * ldg;
    if (total <= 0) return 0;
    if (splits < 1) return (int)cudaErrorInvalidValue;
#define GO(T_, Z_)                                                                                                                 \
    return (int)launch_pdl(side_gate_kernel<T_, Z_>, dim3(grid_for(total)), dim3(256), 0, st, (const Z_*)z, ldz, z_split, splits,   \
                           (const T_*)table, ldt, tokens, (T_*)g, ldg, dim, col0, vocab, total)
    if (f32) GO(float, float);
    if (z_f32) GO(bf16, float);
    GO(bf16, bf16);
#undef GO
}
