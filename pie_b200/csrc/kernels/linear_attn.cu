// Linear attention with a decaying state: per head S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, S in 32-bit
// [dim][vdim], one state per (slot, head), carried from fire to fire. Three decays: one per key channel and token
// (`log_decay`, base-2 logarithms, at most 0), one constant per head, or one per head and token (`tok_decay`) beside a
// factor on the token's key (`tok_input`). The last also carries a normaliser n, n_t = a_t n_(t-1) + k_t, after the states
// of all heads, and returns n_t . q_t per token and head.
//
//   serial   token by token, S in registers: decode steps, and every shape in true 32-bit. A thread holds VEC columns of
//            dim / 8 rows; the eight row groups meet in shared memory once per token.
//   chunked  prompts in bf16: pieces of up to 64 tokens, all pieces at once in three launches:
//              la_chunk_state  U_c = sum_s (k_s * decay from s to the piece's end) v_s^T, and the piece's whole decay
//              la_chunk_scan   S before every piece: S_(c+1) = decay_c * S_c + U_c, elementwise over the pieces
//              la_chunk_out    o = (q_t * decay from the piece's start) S_c + sum_(s <= t) score(t, s) v_s
//            Products run on tf32 tensor-core tiles with 32-bit accumulation. Scores inside a piece are formed 16 x 16:
//            against earlier 16-token blocks relative to the decay at the query block's start, on the diagonal relative
//            to its middle (factors above 1 are bounded by the decay within 8 tokens); where that decay is extreme, pair
//            by pair. Every other factor is at most 1, so nothing overflows whatever the decays.
//
// The form with sub-blocks follows S. Yang et al., "Gated Linear Attention Transformers with Hardware-Efficient Training".
#include "tf32.cuh"
#include "typed.cuh"

namespace pie {

__device__ __forceinline__ float la_silu(float x) { return x / (1.f + expf(-x)); }

struct LinAttnArgs {
    const void *q, *k, *v;       // row t, head h at t * ld + h * dim (h * vdim for v), type T
    float* log_decay;            // [n, heads * dim] base 2, or null; the chunked form leaves running sums of the pieces
    const float* head_decay;     // [heads] the factor itself (null with log_decay)
    const float *tok_decay, *tok_input;   // [heads, n] base-2 logarithms of decay and key factor, at most 0 (null with the others)
    float* den;                  // [heads, n] n_t . q_t (with tok_decay)
    float* out;                  // [n, heads * vdim]
    float* state;                // this layer's part of slot 0: [heads][dim][vdim]
    const int *qo_indptr, *slots, *reset;
    // chunked form
    const int *chunk_req, *chunk_start, *req_chunks;   // request and first row of a piece; pieces of a request (indptr)
    float *u, *piece_decay;      // [chunks][heads][dim][vdim] (with tok_decay then [heads][dim]), [chunks][heads][dim] (base-2 logarithm)
    long slot_stride;
    int n, ld, reqs, heads, dim, vdim, silu, chunks;
    float q_scale;
};

enum LaDecay : int { LA_HEAD = 0, LA_CHANNEL = 1, LA_TOKEN = 2 };
// 32-bit numbers of the state of one slot, or of one piece's update, that decay together
__host__ __device__ __forceinline__ long la_elems(const LinAttnArgs& a) {
    return (long)a.heads * a.dim * a.vdim + (a.tok_decay ? (long)a.heads * a.dim : 0);
}

// ------------------------------------------------------------------ serial
template <typename T, int RPT, int VEC, bool TOK>
__global__ void __launch_bounds__(256) la_serial_kernel(const LinAttnArgs a) {
    constexpr int ROWS = RPT * 8, COLS = 32 * VEC;
    __shared__ float sq[ROWS], sk[ROWS], sa[ROWS];
    __shared__ float red[8][COLS], sn[2][TOK ? ROWS : 1];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, rg = threadIdx.x >> 5;
    const int first = a.qo_indptr[r], len = a.qo_indptr[r + 1] - first, slot = a.slots[r];
    if (len <= 0 || slot < 0) return;          // a padding request of a decode graph: no state, no output
    const int c0 = blockIdx.z * COLS + lane * VEC;
    const bool col = c0 < a.vdim;              // VEC > 1 only where vdim is a multiple of it
    float* sp = a.state + (size_t)slot * a.slot_stride + (size_t)h * a.dim * a.vdim;
    // the first block of a head also keeps the normaliser, the rows each thread stages
    constexpr int NR = (ROWS + 255) / 256;
    const bool norm = TOK && blockIdx.z == 0;
    float* np = a.state + (size_t)slot * a.slot_stride + (size_t)a.heads * a.dim * a.vdim + (size_t)h * a.dim;
    float S[RPT][VEC], N[NR];
    const bool fresh = a.reset[r] != 0;
#pragma unroll
    for (int i = 0; i < NR; ++i) {
        const int d = threadIdx.x + i * 256;
        N[i] = norm && !fresh && d < a.dim ? np[d] : 0.f;
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = rg + 8 * i;
        const bool ok = col && !fresh && d < a.dim;
        if constexpr (VEC == 4) {
            float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
            if (ok) x = *reinterpret_cast<const float4*>(sp + (size_t)d * a.vdim + c0);
            S[i][0] = x.x; S[i][1] = x.y; S[i][2] = x.z; S[i][3] = x.w;
        } else {
            S[i][0] = ok ? sp[(size_t)d * a.vdim + c0] : 0.f;
        }
    }
    const float hd = a.head_decay ? a.head_decay[h] : 1.f;
    for (int t = 0; t < len; ++t) {
        const size_t row = (size_t)(first + t);
        const T* qr = static_cast<const T*>(a.q) + row * a.ld + h * a.dim;
        const T* kr = static_cast<const T*>(a.k) + row * a.ld + h * a.dim;
        const float td = TOK ? exp2f(a.tok_decay[(size_t)h * a.n + row]) : hd;
        const float ti = TOK ? exp2f(a.tok_input[(size_t)h * a.n + row]) : 1.f;
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int d = threadIdx.x + i * 256;
            if (d >= ROWS) break;
            float q = 0.f, k = 0.f, g = 1.f;
            if (d < a.dim) {
                q = to_f(qr[d]);
                k = to_f(kr[d]);
                if (a.silu) { q = la_silu(q); k = la_silu(k); }
                g = a.log_decay ? exp2f(a.log_decay[row * a.heads * a.dim + h * a.dim + d]) : td;
            }
            sq[d] = q * a.q_scale;
            sk[d] = k * ti;
            sa[d] = g;
            if (norm) {
                N[i] = g * N[i] + k * ti;
                sn[t & 1][d] = q * a.q_scale * N[i];
            }
        }
        float v[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
            v[j] = col ? to_f(static_cast<const T*>(a.v)[row * a.ld + h * a.vdim + c0 + j]) : 0.f;
            if (a.silu) v[j] = la_silu(v[j]);
        }
        __syncthreads();
        float o[VEC];
#pragma unroll
        for (int j = 0; j < VEC; ++j) o[j] = 0.f;
#pragma unroll
        for (int i = 0; i < RPT; ++i) {
            const int d = rg + 8 * i;
            const float g = sa[d], k = sk[d], q = sq[d];
#pragma unroll
            for (int j = 0; j < VEC; ++j) {
                S[i][j] = g * S[i][j] + k * v[j];
                o[j] += q * S[i][j];
            }
        }
#pragma unroll
        for (int j = 0; j < VEC; ++j) red[rg][lane * VEC + j] = o[j];
        __syncthreads();
        if (norm && rg == 7) {                 // the other buffer is written before every warp has read this one
            float s = 0.f;
#pragma unroll
            for (int d = lane; d < ROWS; d += 32) s += sn[t & 1][d];
            s = warp_sum(s);
            if (lane == 0) a.den[(size_t)h * a.n + row] = s;
        }
        for (int c = threadIdx.x; c < COLS; c += 256) {
            const int cc = blockIdx.z * COLS + c;
            if (cc >= a.vdim) continue;
            float s = 0.f;
#pragma unroll
            for (int g = 0; g < 8; ++g) s += red[g][c];
            a.out[row * a.heads * a.vdim + h * a.vdim + cc] = s;
        }
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = rg + 8 * i;
        if (!col || d >= a.dim) continue;
        if constexpr (VEC == 4)
            *reinterpret_cast<float4*>(sp + (size_t)d * a.vdim + c0) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
        else
            sp[(size_t)d * a.vdim + c0] = S[i][0];
    }
#pragma unroll
    for (int i = 0; i < NR; ++i)
        if (norm && threadIdx.x + i * 256 < a.dim) np[threadIdx.x + i * 256] = N[i];
}

// ----------------------------------------------------------------- chunked
constexpr int LA_C = 64;                  // tokens per piece
constexpr int LA_VT = 64;                 // value columns per pass
constexpr int LA_VP = LA_VT + 8;          // pitch of a tile read as (row by t, column by g): fragment reads hit 32 banks
constexpr int LA_SP = LA_C + 4;           // pitch of the scores, and of values read at rows 2 t, 2 t + 1
constexpr int LA_THREADS = 256;

__host__ __device__ constexpr int la_dimp(int dim) { return (dim + 15) / 16 * 16; }
// Pitch of a [64][dim] array of bf16 (queries, keys) and of 32-bit decayed keys: 8 (mod 32) words or 4 (mod 16)
__host__ __device__ constexpr int la_pitch(int dim) { return la_dimp(dim) + 8; }

// Eight bf16 of a row of a projection as floats (with the activation, rounded to tf32), zeros outside; VEC: one 16-byte load.
template <bool VEC>
__device__ __forceinline__ void la_load8(const bf16* p, int valid, bool act, float (&f)[8]) {
    if (VEC && valid >= 8) {
        unpack8(*reinterpret_cast<const bf16x8*>(p), f);
    } else {
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = e < valid ? to_f(p[e]) : 0.f;
    }
    if (act) {
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = tf32_f(f[e] / (1.f + __expf(-f[e])));
    }
}

// A tile of values [64 tokens][64 columns] on its way from global to shared memory: two 8-column vectors per thread.
template <bool VEC>
struct ValueTile {
    float f[2][8];
    __device__ __forceinline__ void load(const bf16* v, int ld, int len, int cols, bool act) {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int u = threadIdx.x + i * LA_THREADS, s = u >> 3, j = (u & 7) * 8;
            la_load8<VEC>(v + (size_t)s * ld + j, s < len ? min(8, cols - j) : 0, act, f[i]);
        }
    }
    template <int PITCH>
    __device__ __forceinline__ void store(float* dst) const {
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const int u = threadIdx.x + i * LA_THREADS, s = u >> 3, j = (u & 7) * 8;
            float4* d = reinterpret_cast<float4*>(dst + s * PITCH + j);
            d[0] = make_float4(f[i][0], f[i][1], f[i][2], f[i][3]);
            d[1] = make_float4(f[i][4], f[i][5], f[i][6], f[i][7]);
        }
    }
};

// Running sum of the piece's token decays (sb[t]: decay from before the piece's first token to t) and its key factors, by
// the first two warps; rows past the piece repeat its last sum and have no key.
__device__ __forceinline__ void la_token_sums(const LinAttnArgs& a, int row0, int len, int h, float* sb, float* si, float* half) {
    if (threadIdx.x < LA_C) {
        const int s = threadIdx.x, lane = s & 31;
        const size_t at = (size_t)h * a.n + row0 + s;
        float x = s < len ? a.tok_decay[at] : 0.f;
        si[s] = s < len ? a.tok_input[at] : -INFINITY;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float y = __shfl_up_sync(0xffffffffu, x, o);
            if (lane >= o) x += y;
        }
        if (s == 31) *half = x;
        sb[s] = x;
    }
    __syncthreads();
    if (threadIdx.x >= 32 && threadIdx.x < LA_C) sb[threadIdx.x] += *half;
    __syncthreads();
}

// U and the piece's decay; turns log_decay into its running sum from the piece's start (in place), which la_chunk_out reads.
template <int DEC, bool VEC>
__global__ void __launch_bounds__(LA_THREADS, DEC == LA_CHANNEL ? 2 : 3) la_chunk_state_kernel(const LinAttnArgs a) {
    constexpr bool CHAN = DEC == LA_CHANNEL;
    extern __shared__ __align__(16) float sm[];
    __shared__ float tb[LA_C], ti[LA_C], th;
    const int c = blockIdx.x, h = blockIdx.y, r = a.chunk_req[c];
    const int row0 = a.chunk_start[c], len = min(LA_C, a.qo_indptr[r + 1] - row0);
    const int dimp = la_dimp(a.dim), kp = la_pitch(a.dim);
    float* sk = sm;                        // [64][kp] decayed keys
    float* sv = sk + LA_C * kp;            // [64][LA_VP] a tile of values
    float* tot = sv + LA_C * LA_VP;        // [128] decay of the first 32 tokens
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const bf16* kb = static_cast<const bf16*>(a.k) + (size_t)row0 * a.ld + h * a.dim;
    const bf16* vb = static_cast<const bf16*>(a.v) + (size_t)row0 * a.ld + h * a.vdim;
    ValueTile<VEC> vt;
    vt.load(vb, a.ld, len, a.vdim, a.silu);
    if (CHAN) {
        const int half = threadIdx.x >> 7;
        float* dec = a.piece_decay + ((size_t)c * a.heads + h) * a.dim;
        for (int d0 = 0; d0 < dimp; d0 += 128) {
            const int d = d0 + (threadIdx.x & 127);
            const bool ok = d < a.dim;
            float* lg = a.log_decay + ((size_t)(row0 + half * 32) * a.heads + h) * a.dim + d;
            const size_t step = (size_t)a.heads * a.dim;
            const bf16* kd = kb + (size_t)half * 32 * a.ld + d;
            float b[32], run = 0.f;
#pragma unroll
            for (int s = 0; s < 32; ++s) b[s] = ok && half * 32 + s < len ? lg[s * step] : 0.f;
#pragma unroll
            for (int s = 0; s < 32; ++s) b[s] = run += b[s];
            if (half == 0) tot[threadIdx.x] = run;
            __syncthreads();
            const float base = half ? tot[threadIdx.x & 127] : 0.f;
            __syncthreads();
            if (half) tot[threadIdx.x & 127] = base + run;
            __syncthreads();
            const float all = tot[threadIdx.x & 127];
            if (half && ok) dec[d] = all;
            if (d < dimp) {
#pragma unroll
                for (int s0 = 0; s0 < 32; s0 += 16) {
                    float k[16];
#pragma unroll
                    for (int s = 0; s < 16; ++s) k[s] = ok && half * 32 + s0 + s < len ? to_f(kd[(size_t)(s0 + s) * a.ld]) : 0.f;
#pragma unroll
                    for (int s = 0; s < 16; ++s) {
                        const float x = base + b[s0 + s];
                        if (ok && half * 32 + s0 + s < len) lg[(s0 + s) * step] = x;
                        sk[(half * 32 + s0 + s) * kp + d] = tf32_f((a.silu ? la_silu(k[s]) : k[s]) * exp2f(all - x));
                    }
                }
            }
            __syncthreads();               // `tot` is free for the next channels
        }
    } else {
        if (DEC == LA_TOKEN) la_token_sums(a, row0, len, h, tb, ti, &th);
        const float lh = DEC == LA_TOKEN ? 0.f : log2f(a.head_decay[h]);
        const float whole = DEC == LA_TOKEN ? tb[LA_C - 1] : (float)len * lh;
        for (int u = threadIdx.x; u < LA_C * (dimp / 8); u += LA_THREADS) {
            const int s = u / (dimp / 8), d = (u - s * (dimp / 8)) * 8;
            float f[8];
            la_load8<VEC>(kb + (size_t)s * a.ld + d, s < len ? min(8, a.dim - d) : 0, a.silu, f);
            const float w = s >= len ? 0.f : exp2f(DEC == LA_TOKEN ? whole - tb[s] + ti[s] : (float)(len - 1 - s) * lh);
#pragma unroll
            for (int e = 0; e < 8; ++e) sk[s * kp + d + e] = tf32_f(f[e] * w);
        }
        for (int d = threadIdx.x; d < a.dim; d += LA_THREADS)
            a.piece_decay[((size_t)c * a.heads + h) * a.dim + d] = whole;
    }
    const long elems = la_elems(a);
    float* U = a.u + c * elems + (size_t)h * a.dim * a.vdim;
    if (DEC == LA_TOKEN) {
        __syncthreads();
        for (int d = threadIdx.x; d < a.dim; d += LA_THREADS) {
            float x = 0.f;
#pragma unroll 8
            for (int s = 0; s < LA_C; ++s) x += sk[s * kp + d];
            a.u[c * elems + (long)a.heads * a.dim * a.vdim + h * a.dim + d] = x;
        }
    }
    for (int v0 = 0; v0 < a.vdim; v0 += LA_VT) {
        __syncthreads();
        vt.template store<LA_VP>(sv);
        __syncthreads();
        if (v0 + LA_VT < a.vdim) vt.load(vb + v0 + LA_VT, a.ld, len, a.vdim - v0 - LA_VT, a.silu);
        for (int m = warp; m < dimp / 16; m += LA_THREADS / 32) {
            float acc[8][4];
#pragma unroll
            for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll 2
            for (int ks = 0; ks < LA_C / 8; ++ks) {
                const float* kr = sk + (ks * 8 + t) * kp + m * 16 + g;
                const float fa[4] = {kr[0], kr[8], kr[4 * kp], kr[4 * kp + 8]};
                const float* vr = sv + (ks * 8 + t) * LA_VP + g;
#pragma unroll
                for (int n = 0; n < 8; ++n) mma_tf32(acc[n], fa, vr[n * 8], vr[4 * LA_VP + n * 8]);
            }
#pragma unroll
            for (int n = 0; n < 8; ++n)
#pragma unroll
                for (int e = 0; e < 4; e += 2) {
                    const int d = m * 16 + g + (e >> 1) * 8, j = v0 + n * 8 + 2 * t;
                    if (d >= a.dim) continue;
                    float* u = U + (size_t)d * a.vdim + j;
                    if (VEC && j + 1 < a.vdim) {
                        *reinterpret_cast<float2*>(u) = make_float2(acc[n][e], acc[n][e + 1]);
                    } else {
                        if (j < a.vdim) u[0] = acc[n][e];
                        if (j + 1 < a.vdim) u[1] = acc[n][e + 1];
                    }
                }
        }
    }
}

// One thread per V state elements: U becomes the state before each piece; the state after the last goes back to its slot.
template <int V>
__global__ void __launch_bounds__(256) la_chunk_scan_kernel(const LinAttnArgs a) {
    const int r = blockIdx.y, slot = a.slots[r];
    const int c0 = a.req_chunks[r], c1 = a.req_chunks[r + 1];
    const long elems = la_elems(a), states = (long)a.heads * a.dim * a.vdim, i = (blockIdx.x * 256L + threadIdx.x) * V;
    if (i >= elems || c1 <= c0 || slot < 0) return;
    float* sp = a.state + (size_t)slot * a.slot_stride + i;
    float s[V];
    load_vec<V>(sp, s);
    if (a.reset[r])
#pragma unroll
        for (int e = 0; e < V; ++e) s[e] = 0.f;
    float* u = a.u + i;
    // the V elements share a factor, also in the normaliser, whose neighbours are channels of one head (V divides dim)
    const float* dec = a.piece_decay + (i < states ? i / a.vdim : i - states);
    const long dstep = (long)a.heads * a.dim;
    constexpr int AHEAD = 8;
    for (int c = c0; c < c1; c += AHEAD) {
        float x[AHEAD][V], w[AHEAD];
#pragma unroll
        for (int j = 0; j < AHEAD; ++j)
            if (c + j < c1) {
                load_vec<V>(u + (c + j) * elems, x[j]);
                w[j] = dec[(c + j) * dstep];
            }
#pragma unroll
        for (int j = 0; j < AHEAD; ++j)
            if (c + j < c1) {
                store_vec<V>(u + (c + j) * elems, s);
                const float f = exp2f(w[j]);
#pragma unroll
                for (int e = 0; e < V; ++e) s[e] = f * s[e] + x[j][e];
            }
    }
    store_vec<V>(sp, s);
}

// Shared memory of la_chunk_out, in bytes: decays, then decayed queries | keys, then scores | queries, then values | state tile
struct LaOutSmem {
    int xp, kp;
    size_t k, q, s, total;
    __host__ __device__ explicit LaOutSmem(int dim) {
        const size_t tile = (size_t)LA_C * LA_SP * 4;
        xp = la_dimp(dim) + 4;
        kp = la_pitch(dim);
        const size_t half = (size_t)LA_C * kp * 2;
        k = (size_t)LA_C * xp * 4;
        q = k + (half > tile ? half : tile);
        s = q + (half > tile ? half : tile);
        total = s + (size_t)la_dimp(dim) * LA_VP * 4;
    }
};

template <int DEC, bool VEC>
__global__ void __launch_bounds__(LA_THREADS) la_chunk_out_kernel(const LinAttnArgs a) {
    constexpr bool CHAN = DEC == LA_CHANNEL;
    extern __shared__ __align__(16) float sm[];
    __shared__ float tb[LA_C], ti[LA_C], th;
    const LaOutSmem lay(a.dim);
    const int c = blockIdx.x, h = blockIdx.y, r = a.chunk_req[c];
    const int row0 = a.chunk_start[c], len = min(LA_C, a.qo_indptr[r + 1] - row0);
    const int dimp = la_dimp(a.dim), xp = lay.xp, kp = lay.kp;
    uint8_t* base = reinterpret_cast<uint8_t*>(sm);
    float* sb = sm;                                            // [64][xp]
    bf16* sk = reinterpret_cast<bf16*>(base + lay.k);          // [64][kp]
    float* sc = reinterpret_cast<float*>(base + lay.k);        // [64][LA_SP] scores of query rows
    bf16* sq = reinterpret_cast<bf16*>(base + lay.q);          // [64][kp]
    float* sv = reinterpret_cast<float*>(base + lay.q);        // [64][LA_SP] a tile of values
    float* ss = reinterpret_cast<float*>(base + lay.s);        // [dimp][LA_VP] a tile of the state
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int rb = warp & 3, half = warp >> 2, w0 = rb * 16;   // 16 query rows per warp; two warps share them
    const float lh = DEC == LA_HEAD ? log2f(a.head_decay[h]) : 0.f;
    if (DEC == LA_TOKEN) la_token_sums(a, row0, len, h, tb, ti, &th);
    const bf16* qb = static_cast<const bf16*>(a.q) + (size_t)row0 * a.ld + h * a.dim;
    const bf16* kb = static_cast<const bf16*>(a.k) + (size_t)row0 * a.ld + h * a.dim;
    const bf16* vb = static_cast<const bf16*>(a.v) + (size_t)row0 * a.ld + h * a.vdim;
    const int vecs = dimp / 8;
    for (int u = threadIdx.x; u < LA_C * vecs; u += LA_THREADS) {
        const int s = u / vecs, d = (u - s * vecs) * 8, valid = s < len ? min(8, a.dim - d) : 0;
        float f[8];
        la_load8<VEC>(qb + (size_t)s * a.ld + d, valid, a.silu, f);
        *reinterpret_cast<bf16x8*>(sq + s * kp + d) = pack8(f);
        la_load8<VEC>(kb + (size_t)s * a.ld + d, valid, a.silu, f);
        *reinterpret_cast<bf16x8*>(sk + s * kp + d) = pack8(f);
        if (CHAN) {
            // running sums; rows past the piece repeat its last one
            const float* b = a.log_decay + ((size_t)(row0 + min(s, len - 1)) * a.heads + h) * a.dim + d;
            float* dst = sb + s * xp + d;
            if (VEC && a.dim - d >= 8) {
                reinterpret_cast<float4*>(dst)[0] = reinterpret_cast<const float4*>(b)[0];
                reinterpret_cast<float4*>(dst)[1] = reinterpret_cast<const float4*>(b)[1];
            } else {
#pragma unroll
                for (int e = 0; e < 8; ++e) dst[e] = d + e < a.dim ? b[e] : 0.f;
            }
        }
    }
    // the first tiles of values and state are on their way while the scores are formed
    const float* S = a.u + c * la_elems(a) + (size_t)h * a.dim * a.vdim;
    ValueTile<VEC> vt;
    vt.load(vb, a.ld, len, a.vdim, a.silu);
    __syncthreads();

    // scores of the 16 queries against the keys up to the end of their own 16-token block; this warp takes the 8-key tiles
    // 2 J + half of every block J
    float acc[4][4];
#pragma unroll
    for (int n = 0; n < 4; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
    bool exact = false;
    if (CHAN) {
        float range = 0.f;
        for (int d = lane; d < dimp; d += 32) range = fmaxf(range, (w0 ? sb[(w0 - 1) * xp + d] : 0.f) - sb[(w0 + 15) * xp + d]);
        exact = warp_max(range) > 100.f;
    }
    for (int ks = 0; ks < dimp / 8; ++ks) {
        const int d0 = ks * 8 + t, d1 = d0 + 4;
        const float q4[4] = {to_f(sq[(w0 + g) * kp + d0]), to_f(sq[(w0 + g + 8) * kp + d0]), to_f(sq[(w0 + g) * kp + d1]),
                             to_f(sq[(w0 + g + 8) * kp + d1])};
        float fa[4] = {q4[0], q4[1], q4[2], q4[3]}, b4[4], r0 = 0.f, r1 = 0.f;
        auto key = [&](int s, float& k0, float& k1) {
            k0 = to_f(sk[s * kp + d0]);
            k1 = to_f(sk[s * kp + d1]);
            if (CHAN) {
                k0 = tf32_f(k0 * exp2f(r0 - sb[s * xp + d0]));
                k1 = tf32_f(k1 * exp2f(r1 - sb[s * xp + d1]));
            }
        };
        auto queries = [&]() {
#pragma unroll
            for (int e = 0; e < 4; ++e) fa[e] = tf32_f(q4[e] * exp2f(b4[e] - (e < 2 ? r0 : r1)));
        };
        if (CHAN) {
            b4[0] = sb[(w0 + g) * xp + d0]; b4[1] = sb[(w0 + g + 8) * xp + d0];
            b4[2] = sb[(w0 + g) * xp + d1]; b4[3] = sb[(w0 + g + 8) * xp + d1];
            if (rb) {
                r0 = sb[(w0 - 1) * xp + d0];
                r1 = sb[(w0 - 1) * xp + d1];
                queries();
            }
        }
#pragma unroll
        for (int J = 0; J < 3; ++J) {
            if (J >= rb) break;
            float k0, k1;
            key(J * 16 + half * 8 + g, k0, k1);
            mma_tf32(acc[J], fa, k0, k1);
        }
        if (exact) continue;
        if (CHAN) {
            r0 = sb[(w0 + 7) * xp + d0];
            r1 = sb[(w0 + 7) * xp + d1];
            queries();
        }
        float k0, k1;
        key(w0 + half * 8 + g, k0, k1);
        mma_tf32(acc[3], fa, k0, k1);             // the diagonal block
    }
    // decay between the two tokens (constant per head), causal limit
#pragma unroll
    for (int n = 0; n < 4; ++n) {
        const int J = n < 3 ? n : rb;
        if (n < 3 && n >= rb) continue;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int q = w0 + g + (e >> 1) * 8, s = J * 16 + half * 8 + 2 * t + (e & 1);
            if (s > q) { acc[n][e] = 0.f; continue; }
            if (!CHAN) acc[n][e] *= exp2f(DEC == LA_TOKEN ? tb[q] - tb[s] + ti[s] : (float)(q - s) * lh);
            if (CHAN && exact && n == 3) {
                float x = 0.f;
                for (int d = 0; d < dimp; ++d)
                    x += to_f(sq[q * kp + d]) * to_f(sk[s * kp + d]) * exp2f(sb[q * xp + d] - sb[s * xp + d]);
                acc[n][e] = x;
            }
        }
    }
    __syncthreads();                              // keys are done with: the scores take their place
#pragma unroll
    for (int n = 0; n < 4; ++n) {
        const int J = n < 3 ? n : rb;
        if (n < 3 && n >= rb) continue;
#pragma unroll
        for (int e = 0; e < 4; e += 2)
            *reinterpret_cast<float2*>(sc + (w0 + g + (e >> 1) * 8) * LA_SP + J * 16 + half * 8 + 2 * t) =
                make_float2(tf32_f(acc[n][e]), tf32_f(acc[n][e + 1]));
    }
    // queries with the decay from the start of the piece, for the state before it
    for (int u = threadIdx.x; u < LA_C * vecs; u += LA_THREADS) {
        const int s = u / vecs, d = (u - s * vecs) * 8;
        float f[8];
        unpack8(*reinterpret_cast<const bf16x8*>(sq + s * kp + d), f);
        const float w = CHAN ? 0.f : exp2f(DEC == LA_TOKEN ? tb[s] : (float)(s + 1) * lh);
#pragma unroll
        for (int e = 0; e < 8; ++e) sb[s * xp + d + e] = tf32_f(CHAN ? f[e] * exp2f(sb[s * xp + d + e]) : f[e] * w);
    }
    if (DEC == LA_TOKEN) {
        // n_t . q_t: the row's scores, and its decayed query against the normaliser before the piece; four threads per row
        __syncthreads();
        const int q = threadIdx.x >> 2, part = threadIdx.x & 3;
        const float* N = a.u + c * la_elems(a) + (size_t)a.heads * a.dim * a.vdim + (size_t)h * a.dim;
        float x = 0.f;
        for (int s = part; s <= q; s += 4) x += sc[q * LA_SP + s];
        for (int d = part; d < a.dim; d += 4) x += sb[q * xp + d] * N[d];
        x += __shfl_xor_sync(0xffffffffu, x, 1);
        x += __shfl_xor_sync(0xffffffffu, x, 2);
        if (part == 0 && q < len) a.den[(size_t)h * a.n + row0 + q] = x * a.q_scale;
    }
    constexpr int SV = LA_VT / 4;                 // 16-byte pieces of a state row
    for (int v0 = 0; v0 < a.vdim; v0 += LA_VT) {
        __syncthreads();
        vt.template store<LA_SP>(sv);
        for (int u = threadIdx.x; u < dimp * SV; u += LA_THREADS) {
            const int d = u / SV, j = (u % SV) * 4;
            float f[4] = {0.f, 0.f, 0.f, 0.f};
            if (d < a.dim) {
                const float* src = S + (size_t)d * a.vdim + v0 + j;
                if (VEC && v0 + j + 3 < a.vdim) {
                    load_vec<4>(src, f);
                } else {
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        if (v0 + j + e < a.vdim) f[e] = src[e];
                }
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) f[e] = tf32_f(f[e]);
            store_vec<4>(ss + d * LA_VP + j, f);
        }
        __syncthreads();
        if (v0 + LA_VT < a.vdim) vt.load(vb + v0 + LA_VT, a.ld, len, a.vdim - v0 - LA_VT, a.silu);
        float o[4][4];
#pragma unroll
        for (int n = 0; n < 4; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
        const int col = half * 32 + g;            // this warp's 32 of the tile's columns
#pragma unroll 4
        for (int ks = 0; ks < dimp / 8; ++ks) {
            const float* q0 = sb + (w0 + g) * xp + ks * 8 + t;
            const float fa[4] = {q0[0], q0[8 * xp], q0[4], q0[8 * xp + 4]};
            const float* sr = ss + (ks * 8 + t) * LA_VP + col;
#pragma unroll
            for (int n = 0; n < 4; ++n) mma_tf32(o[n], fa, sr[n * 8], sr[4 * LA_VP + n * 8]);
        }
        // columns t and t + 4 of the A operand stand for the keys 2 t and 2 t + 1
        for (int ks = 0; ks < 2 * rb + 2; ++ks) {
            const float2 x = *reinterpret_cast<const float2*>(sc + (w0 + g) * LA_SP + ks * 8 + 2 * t);
            const float2 y = *reinterpret_cast<const float2*>(sc + (w0 + g + 8) * LA_SP + ks * 8 + 2 * t);
            const float fa[4] = {x.x, y.x, x.y, y.y};
            const float* vr = sv + (ks * 8 + 2 * t) * LA_SP + col;
#pragma unroll
            for (int n = 0; n < 4; ++n) mma_tf32(o[n], fa, vr[n * 8], vr[LA_SP + n * 8]);
        }
#pragma unroll
        for (int n = 0; n < 4; ++n)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int q = w0 + g + (e >> 1) * 8, j = v0 + half * 32 + n * 8 + 2 * t;
                if (q >= len) continue;
                float* dst = a.out + (size_t)(row0 + q) * a.heads * a.vdim + h * a.vdim + j;
                if (VEC && j + 1 < a.vdim) {
                    *reinterpret_cast<float2*>(dst) = make_float2(o[n][e] * a.q_scale, o[n][e + 1] * a.q_scale);
                } else {
                    if (j < a.vdim) dst[0] = o[n][e] * a.q_scale;
                    if (j + 1 < a.vdim) dst[1] = o[n][e + 1] * a.q_scale;
                }
            }
    }
}

// ---------------------------------------------------------- channel decays
// log_decay[t, c] = log2(sigmoid(z)) * factor, z = a2[c, :] . a1[t, :] + bias[c]; x holds a1 at column 0 of rows of ld.
// BOUNDED: -sigmoid(z) * factor * log2(e) with a1 passed through tanh first: a decay between exp(-factor) and 1.
constexpr int LD_TOK = 8;
template <typename T, bool BOUNDED>
__global__ void __launch_bounds__(256) la_decay_kernel(const T* __restrict__ x, int ld, const T* __restrict__ a2, const T* __restrict__ bias,
                                                       float* __restrict__ out, int n, int channels, int rank, float factor) {
    extern __shared__ __align__(16) float sx[];          // [rank][LD_TOK]
    pdl_trigger();
    pdl_wait();
    const int t0 = blockIdx.x * LD_TOK, nt = min(LD_TOK, n - t0);
    for (int i = threadIdx.x; i < LD_TOK * rank; i += 256) {
        const int s = i / rank, j = i - s * rank;
        const float f = s < nt ? to_f(x[(size_t)(t0 + s) * ld + j]) : 0.f;
        sx[j * LD_TOK + s] = BOUNDED ? tanhf(f) : f;
    }
    __syncthreads();
    const int c = blockIdx.y * 256 + threadIdx.x;
    if (c >= channels) return;
    float z[LD_TOK];
    const float b = to_f(bias[c]);
#pragma unroll
    for (int s = 0; s < LD_TOK; ++s) z[s] = b;
    const T* w = a2 + (size_t)c * rank;
#pragma unroll 4
    for (int j = 0; j < rank; ++j) {
        const float wj = to_f(w[j]);
        const float4 p = reinterpret_cast<const float4*>(sx)[2 * j], q = reinterpret_cast<const float4*>(sx)[2 * j + 1];
        z[0] += wj * p.x; z[1] += wj * p.y; z[2] += wj * p.z; z[3] += wj * p.w;
        z[4] += wj * q.x; z[5] += wj * q.y; z[6] += wj * q.z; z[7] += wj * q.w;
    }
#pragma unroll
    for (int s = 0; s < LD_TOK; ++s)
        if (s < nt)
            out[(size_t)(t0 + s) * channels + c] = (BOUNDED ? -1.f / (1.f + expf(-z[s])) : fminf(z[s], 0.f) - log1pf(expf(-fabsf(z[s])))) *
                                                   (1.4426950408889634f * factor);
}

// The bounded decay in bf16: products on mma.sync tiles, tanh(a1) as the sum of two bf16 numbers (16 digits), z in 32-bit. A block
// takes 64 tokens and `tiles` times 64 channels, a warp 16 tokens and 32 channels of a tile. Rows of rank + 8 (rank rounded up to
// a multiple of 32, which makes fragment reads hit 32 banks at an odd multiple of 8 words).
constexpr int BD_MAX_RANK = 256;
__host__ __device__ constexpr int bd_rank(int rank) { return (rank + 31) / 32 * 32; }
__device__ __forceinline__ void bd_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__global__ void __launch_bounds__(256) la_bounded_decay_kernel(const bf16* __restrict__ x, int ld, const bf16* __restrict__ a2,
                                                               const bf16* __restrict__ bias, float* __restrict__ out, int n, int channels,
                                                               int rank, float factor, int tiles) {
    extern __shared__ __align__(16) bf16 bd_smem[];
    const int rp = bd_rank(rank), pitch = rp + 8;
    bf16 *hi = bd_smem, *lo = hi + 64 * pitch, *sw = lo + 64 * pitch;
    pdl_trigger();
    const int t0 = blockIdx.y * 64;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, q = lane & 3, wt = (warp & 3) * 16, wc = (warp >> 2) * 32;
    auto weights = [&](int c0) {
        if (rank % 8 == 0) {                   // eight numbers at a time
            for (int u = threadIdx.x; u < 8 * rp; u += 256) {
                const int row = u / (rp / 8), k = (u - row * (rp / 8)) * 8;
                uint4 w = make_uint4(0, 0, 0, 0);
                if (c0 + row < channels && k < rank) w = *reinterpret_cast<const uint4*>(a2 + (size_t)(c0 + row) * rank + k);
                *reinterpret_cast<uint4*>(sw + row * pitch + k) = w;
            }
        } else {
            for (int u = threadIdx.x; u < 64 * rp; u += 256) {
                const int row = u / rp, k = u - row * rp;
                sw[row * pitch + k] = c0 + row < channels && k < rank ? a2[(size_t)(c0 + row) * rank + k] : __float2bfloat16(0.f);
            }
        }
    };
    weights(blockIdx.x * tiles * 64);          // constants: before the kernel ahead is done
    pdl_wait();
    for (int u = threadIdx.x; u < 64 * rp; u += 256) {
        const int row = u / rp, k = u - row * rp;
        const float f = t0 + row < n && k < rank ? tanhf(to_f(x[(size_t)(t0 + row) * ld + k])) : 0.f;
        const bf16 h = __float2bfloat16(f);
        hi[row * pitch + k] = h;
        lo[row * pitch + k] = __float2bfloat16(f - __bfloat162float(h));
    }
    for (int tile = 0; tile < tiles; ++tile) {
        const int c0 = (blockIdx.x * tiles + tile) * 64;
        if (c0 >= channels) break;
        if (tile) {
            __syncthreads();
            weights(c0);
        }
        __syncthreads();
        float acc[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
        for (int ks = 0; ks < rp; ks += 16) {
            auto word = [&](const bf16* m, int row, int col) { return *reinterpret_cast<const uint32_t*>(m + row * pitch + ks + col); };
            const int r0 = wt + g, r1 = r0 + 8, k0 = 2 * q, k1 = k0 + 8;
            const uint32_t ah[4] = {word(hi, r0, k0), word(hi, r1, k0), word(hi, r0, k1), word(hi, r1, k1)};
            const uint32_t al[4] = {word(lo, r0, k0), word(lo, r1, k0), word(lo, r0, k1), word(lo, r1, k1)};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const uint32_t b0 = word(sw, wc + i * 8 + g, 2 * q), b1 = word(sw, wc + i * 8 + g, 2 * q + 8);
                bd_mma(acc[i], ah, b0, b1);
                bd_mma(acc[i], al, b0, b1);
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int c = c0 + wc + i * 8 + 2 * q;
            const float b0 = c < channels ? to_f(bias[c]) : 0.f, b1 = c + 1 < channels ? to_f(bias[c + 1]) : 0.f;
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int t = t0 + wt + g + (e >> 1) * 8;
                if (t >= n) continue;
                const float f = -1.4426950408889634f * factor;
                const float y0 = __fdividef(f, 1.f + __expf(-(acc[i][e] + b0))), y1 = __fdividef(f, 1.f + __expf(-(acc[i][e + 1] + b1)));
                float* dst = out + (size_t)t * channels + c;
                if (c + 1 < channels && channels % 2 == 0) {
                    *reinterpret_cast<float2*>(dst) = make_float2(y0, y1);
                } else {
                    if (c < channels) dst[0] = y0;
                    if (c + 1 < channels) dst[1] = y1;
                }
            }
        }
    }
}

// ------------------------------------------- exponential gates of a matrix memory
// Per head logarithms i = cap tanh(z_i / cap) and f = logsigmoid(cap tanh(z_f / cap)) of the input and forget gates, and a
// running maximum m_t = max(f_t + m_(t-1), i_t), m from 0, that takes the size out of the state: decay exp(f_t + m_(t-1) -
// m_t), key factor exp(i_t - m_t), both at most 1.
struct MemoryGatesArgs {
    const float *z, *bias;          // `splits` arrays [n, ldz] that add up to (z_i | z_f), heads columns each; [2 * heads]
    const int *qo_indptr, *slots, *reset;
    float* m;                       // this layer's maxima of slot 0, [heads]
    float *decay, *input, *floor;   // [heads, n] base-2 logarithms; exp(-m_t)
    long slot_stride, split_stride;
    int n, reqs, heads, ldz, splits;
    float cap;
};

struct MemoryGate { float i, f; };
__device__ __forceinline__ MemoryGate memory_gate(const MemoryGatesArgs& a, size_t t, int h) {
    float zi = a.bias[h], zf = a.bias[a.heads + h];
#pragma unroll 8
    for (int s = 0; s < a.splits; ++s) {
        zi += a.z[s * a.split_stride + t * a.ldz + h];
        zf += a.z[s * a.split_stride + t * a.ldz + a.heads + h];
    }
    const float x = a.cap * tanhf(zf / a.cap);
    return {a.cap * tanhf(zi / a.cap), fminf(x, 0.f) - log1pf(expf(-fabsf(x)))};
}
// A token's factors and the new maximum.
__device__ __forceinline__ float memory_step(MemoryGate g, float m, float& decay, float& input, float& floor) {
    const float kept = g.f + m, next = fmaxf(kept, g.i);
    decay = (kept - next) * 1.4426950408889634f;
    input = (g.i - next) * 1.4426950408889634f;
    floor = expf(-next);
    return next;
}

// One token per request: a thread per (request, head). Rows without a slot (padding of a decode graph) get zeros.
__global__ void __launch_bounds__(128) memory_gates_step_kernel(const MemoryGatesArgs a) {
    pdl_trigger();
    pdl_wait();
    const int i = blockIdx.x * 128 + threadIdx.x;
    if (i >= a.reqs * a.heads) return;
    const int r = i / a.heads, h = i - r * a.heads, t = a.qo_indptr[r], slot = a.slots[r];
    if (a.qo_indptr[r + 1] <= t) return;
    const size_t at = (size_t)h * a.n + t;
    if (slot < 0) { a.decay[at] = a.input[at] = a.floor[at] = 0.f; return; }
    float* m = a.m + (size_t)slot * a.slot_stride + h;
    *m = memory_step(memory_gate(a, t, h), a.reset[r] ? 0.f : *m, a.decay[at], a.input[at], a.floor[at]);
}

// Portions, first pass: the gates' logarithms of every token, f into `decay` and i into `input`.
__global__ void __launch_bounds__(256) memory_gates_log_kernel(const MemoryGatesArgs a) {
    pdl_trigger();
    pdl_wait();
    const long i = blockIdx.x * 256L + threadIdx.x;
    if (i >= (long)a.n * a.heads) return;
    const long t = i / a.heads;
    const int h = (int)(i - t * a.heads);
    const MemoryGate g = memory_gate(a, t, h);
    a.decay[(size_t)h * a.n + t] = g.f;
    a.input[(size_t)h * a.n + t] = g.i;
}

// Second pass: a block per (request, head). m_t is a composition of maps m -> max(m + F, B): over tiles of 1024 tokens the
// threads compose those of four tokens each, a scan gives each the maximum before its tokens, which it then walks.
constexpr int MG_RUN = 4;
__global__ void __launch_bounds__(256) memory_gates_scan_kernel(const MemoryGatesArgs a) {
    __shared__ float sF[2][8], sB[2][8];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, h = blockIdx.y, first = a.qo_indptr[r], len = a.qo_indptr[r + 1] - first, slot = a.slots[r];
    if (len <= 0 || slot < 0) return;
    const size_t at = (size_t)h * a.n + first;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float* mp = a.m + (size_t)slot * a.slot_stride + h;
    float m = a.reset[r] ? 0.f : *mp;
    float f[MG_RUN], g[MG_RUN];
    auto load = [&](int s0) {
#pragma unroll
        for (int j = 0; j < MG_RUN; ++j) {
            f[j] = s0 + j < len ? a.decay[at + s0 + j] : 0.f;
            g[j] = s0 + j < len ? a.input[at + s0 + j] : -INFINITY;
        }
    };
    load(threadIdx.x * MG_RUN);
    for (int tile = 0, b = 0; tile < len; tile += 256 * MG_RUN, b ^= 1) {
        const int s0 = tile + threadIdx.x * MG_RUN;
        MemoryGate own[MG_RUN];
        float F = 0.f, B = -INFINITY;
#pragma unroll
        for (int j = 0; j < MG_RUN; ++j) {
            own[j] = {g[j], f[j]};
            B = fmaxf(B + f[j], g[j]);
            F += f[j];
        }
        if (tile + 256 * MG_RUN < len) load(s0 + 256 * MG_RUN);
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {           // after the maps of earlier lanes
            const float pF = __shfl_up_sync(0xffffffffu, F, o), pB = __shfl_up_sync(0xffffffffu, B, o);
            if (lane >= o) { B = fmaxf(pB + F, B); F += pF; }
        }
        if (lane == 31) { sF[b][warp] = F; sB[b][warp] = B; }
        const float eF = __shfl_up_sync(0xffffffffu, F, 1), eB = __shfl_up_sync(0xffffffffu, B, 1);
        __syncthreads();
        float x = m;
#pragma unroll
        for (int w = 0; w < 8; ++w) {
            if (w == warp) x = m;
            m = fmaxf(m + sF[b][w], sB[b][w]);
        }
        if (lane) x = fmaxf(x + eF, eB);
#pragma unroll
        for (int j = 0; j < MG_RUN; ++j)
            if (s0 + j < len) {
                const size_t o = at + s0 + j;
                x = memory_step(own[j], x, a.decay[o], a.input[o], a.floor[o]);
            }
        if (s0 < len && s0 + MG_RUN >= len) *mp = x;
    }
}

// -------------------------------------------------------- norm and gate of a mixer's output
// dst[t, :] = scale * act(gate) * (rms-normed x) [* w]; the mean square runs over `norm_cols` consecutive columns (0: no
// norm). gate: one number per `gate_cols` columns, or null. den / floor [groups of norm_cols, n]: what is normed is
// x / (max(|den|, floor) + 1e-6), whose division the norm takes up. Column j of the output is column
// (head / group * group_pad + head % group) * head_ld + j % head_cols of x, so that x may hold padded heads. Columns from cols
// to dst_cols are written as zeros.
struct GatedNormPart {
    const void* x;
    const void *w, *gate;
    void* dst;
    const float *den, *floor;
    int x_f32, ldx, head_cols, head_ld, group, group_pad, norm_cols, w_cols, ldg, gate_cols, ldd, cols, dst_cols, act;   // act 0: sigmoid, 1: SiLU
    float eps, scale;
};
struct GatedNormArgs {
    GatedNormPart part[2];
    int n;
};

template <typename T, int VEC>
__global__ void __launch_bounds__(256) la_gated_norm_kernel(const GatedNormArgs args) {
    extern __shared__ __align__(16) float buf[];
    pdl_trigger();
    pdl_wait();
    const GatedNormPart& p = args.part[blockIdx.y];
    const int t = blockIdx.x;
    const T* gate = static_cast<const T*>(p.gate) + (size_t)t * p.ldg;
    const T* w = static_cast<const T*>(p.w);
    T* dst = static_cast<T*>(p.dst) + (size_t)t * p.ldd;
    auto source = [&](int j, float (&v)[VEC]) {
        size_t at = (size_t)t * p.ldx + j;
        if (p.head_ld != p.head_cols || p.group != p.group_pad) {
            const int h = j / p.head_cols;
            at = (size_t)t * p.ldx + (size_t)(h / p.group * p.group_pad + h % p.group) * p.head_ld + (j - h * p.head_cols);
        }
        if (p.x_f32) load_vec<VEC>(static_cast<const float*>(p.x) + at, v);
        else load_vec<VEC>(static_cast<const T*>(p.x) + at, v);
    };
    auto finish = [&](int j, float (&v)[VEC], float inv, int wcol) {
        float z[VEC], gain[VEC];
        if (!p.gate) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) z[e] = 0.f;
        } else if (p.gate_cols == 1) {
            load_vec<VEC>(gate + j, z);
        } else {                                // VEC divides gate_cols
            const float g = to_f(gate[j / p.gate_cols]);
#pragma unroll
            for (int e = 0; e < VEC; ++e) z[e] = g;
        }
        if (w) load_vec<VEC>(w + wcol, gain);
#pragma unroll
        for (int e = 0; e < VEC; ++e) {
            const float s = 1.f / (1.f + __expf(-z[e]));
            v[e] = v[e] * (w ? inv * gain[e] : 1.f) * (p.gate ? (p.act ? z[e] * s : s) : 1.f) * p.scale;
        }
        store_vec<VEC>(dst + j, v);
    };
    auto squared_size = [&](int group) {
        if (!p.den) return 1.f;
        const size_t at = (size_t)group * args.n + t;
        const float d = fmaxf(fabsf(p.den[at]), p.floor[at]) + 1e-6f;
        return d * d;
    };
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (p.norm_cols == 0) {
        for (int j = threadIdx.x * VEC; j < p.cols; j += blockDim.x * VEC) {
            float v[VEC];
            source(j, v);
            finish(j, v, 1.f, 0);
        }
    } else if (p.norm_cols == p.cols) {
        float ss = 0.f;
        for (int j = threadIdx.x * VEC; j < p.cols; j += blockDim.x * VEC) {
            float v[VEC];
            source(j, v);
            store_vec<VEC>(buf + 32 + j, v);
#pragma unroll
            for (int e = 0; e < VEC; ++e) ss += v[e] * v[e];
        }
        const float inv = 1.f / sqrtf(block_sum(ss, buf) / (float)p.cols + p.eps * squared_size(0));
        for (int j = threadIdx.x * VEC; j < p.cols; j += blockDim.x * VEC) {
            float v[VEC];
            load_vec<VEC>(buf + 32 + j, v);
            finish(j, v, inv, j);
        }
    } else {
        for (int gr = warp; gr < p.cols / p.norm_cols; gr += blockDim.x / 32) {
            float ss = 0.f;
            for (int j = lane * VEC; j < p.norm_cols; j += 32 * VEC) {
                float v[VEC];
                source(gr * p.norm_cols + j, v);
#pragma unroll
                for (int e = 0; e < VEC; ++e) ss += v[e] * v[e];
            }
            const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.norm_cols + p.eps * squared_size(gr));
            for (int j = lane * VEC; j < p.norm_cols; j += 32 * VEC) {
                float v[VEC];
                source(gr * p.norm_cols + j, v);
                finish(gr * p.norm_cols + j, v, inv, (gr * p.norm_cols + j) % p.w_cols);
            }
        }
    }
    for (int j = p.cols + threadIdx.x; j < p.dst_cols; j += blockDim.x) dst[j] = from_f<T>(0.f);
}

}  // namespace pie

using namespace pie;

static bool la_decay_ok(const LinAttnArgs& a) {
    return (a.log_decay != nullptr) + (a.head_decay != nullptr) + (a.tok_decay != nullptr) == 1 && (!a.tok_decay || (a.tok_input && a.den));
}

PIE_API int pie_linear_attn_serial(const LinAttnArgs* args, int f32, cudaStream_t st) {
    const LinAttnArgs& a = *args;
    if (a.n <= 0 || a.reqs <= 0) return 0;
    if (a.dim <= 0 || a.dim > 512 || a.vdim <= 0 || !la_decay_ok(a)) return (int)cudaErrorInvalidValue;
    const bool vec = a.vdim % 4 == 0 && a.vdim >= 64 && a.dim <= 256 && a.slot_stride % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    const int cols = vec ? 128 : 32, rpt = (a.dim + 7) / 8;
    const dim3 grid(a.reqs, a.heads, (a.vdim + cols - 1) / cols);
#define GO(T_, R_, V_)                                                                                  \
    return (int)launch_pdl(a.tok_decay ? la_serial_kernel<T_, R_, V_, true> : la_serial_kernel<T_, R_, V_, false>, grid, dim3(256), 0, st, a)
#define GO_R(T_)                                                                                        \
    if (vec) {                                                                                          \
        if (rpt <= 4) GO(T_, 4, 4);                                                                     \
        if (rpt <= 8) GO(T_, 8, 4);                                                                     \
        if (rpt <= 16) GO(T_, 16, 4);                                                                   \
        GO(T_, 32, 4);                                                                                  \
    }                                                                                                   \
    if (rpt <= 4) GO(T_, 4, 1);                                                                         \
    if (rpt <= 8) GO(T_, 8, 1);                                                                         \
    if (rpt <= 16) GO(T_, 16, 1);                                                                       \
    if (rpt <= 32) GO(T_, 32, 1);                                                                       \
    GO(T_, 64, 1)
    if (f32) { GO_R(float); }
    GO_R(bf16);
#undef GO_R
#undef GO
}

static size_t la_state_smem(int dim) { return ((size_t)LA_C * (la_pitch(dim) + LA_VP) + 128) * 4; }
// 1 when the chunked form takes heads of this key size.
PIE_API int pie_linear_attn_chunk_supported(int dim) {
    return dim > 0 && LaOutSmem(dim).total <= 226 * 1024 && la_state_smem(dim) <= 226 * 1024 ? 1 : 0;
}
PIE_API int pie_linear_attn_chunk_tokens() { return LA_C; }

PIE_API int pie_linear_attn_chunked(const LinAttnArgs* args, cudaStream_t st) {
    const LinAttnArgs& a = *args;
    if (a.n <= 0 || a.reqs <= 0 || a.chunks <= 0) return 0;
    if (!pie_linear_attn_chunk_supported(a.dim) || a.vdim <= 0 || !la_decay_ok(a) || !a.u || !a.piece_decay)
        return (int)cudaErrorInvalidValue;
    auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = a.dim % 8 == 0 && a.vdim % 8 == 0 && a.ld % 8 == 0 && aligned(a.q) && aligned(a.k) && aligned(a.v) && aligned(a.log_decay) &&
                     aligned(a.u) && aligned(a.out) && aligned(a.state) && a.slot_stride % 4 == 0;
    const dim3 grid(a.chunks, a.heads);
    const size_t s1 = la_state_smem(a.dim), s3 = LaOutSmem(a.dim).total;
    auto k1 = a.tok_decay ? (vec ? la_chunk_state_kernel<LA_TOKEN, true> : la_chunk_state_kernel<LA_TOKEN, false>)
            : a.log_decay ? (vec ? la_chunk_state_kernel<LA_CHANNEL, true> : la_chunk_state_kernel<LA_CHANNEL, false>)
                          : (vec ? la_chunk_state_kernel<LA_HEAD, true> : la_chunk_state_kernel<LA_HEAD, false>);
    auto k3 = a.tok_decay ? (vec ? la_chunk_out_kernel<LA_TOKEN, true> : la_chunk_out_kernel<LA_TOKEN, false>)
            : a.log_decay ? (vec ? la_chunk_out_kernel<LA_CHANNEL, true> : la_chunk_out_kernel<LA_CHANNEL, false>)
                          : (vec ? la_chunk_out_kernel<LA_HEAD, true> : la_chunk_out_kernel<LA_HEAD, false>);
    cudaError_t e = cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(k3, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);
    if (e != cudaSuccess) return (int)e;
    k1<<<grid, LA_THREADS, s1, st>>>(a);
    const long elems = la_elems(a) / (vec ? 4 : 1);
    const dim3 sgrid((unsigned)((elems + 255) / 256), a.reqs);
    if (vec) la_chunk_scan_kernel<4><<<sgrid, 256, 0, st>>>(a);
    else la_chunk_scan_kernel<1><<<sgrid, 256, 0, st>>>(a);
    k3<<<grid, LA_THREADS, s3, st>>>(a);
    return (int)cudaGetLastError();
}

PIE_API int pie_linear_decay(const void* x, int ld, const void* a2, const void* bias, float* out, int n, int channels, int rank, float factor,
                             int bounded, int f32, cudaStream_t st) {
    if (n <= 0) return 0;
    if (rank <= 0 || rank > 1024 || channels <= 0) return (int)cudaErrorInvalidValue;
    const dim3 grid((n + LD_TOK - 1) / LD_TOK, (channels + 255) / 256);
    const size_t sm = (size_t)LD_TOK * rank * 4;
#define GO(T_, B_) \
    return (int)launch_pdl(la_decay_kernel<T_, B_>, grid, dim3(256), sm, st, (const T_*)x, ld, (const T_*)a2, (const T_*)bias, out, n, channels, \
                           rank, factor)
    if (f32 && bounded) GO(float, true);
    if (f32) GO(float, false);
    if (bounded && rank > BD_MAX_RANK) GO(bf16, true);
    if (bounded) {
        const int bytes = 3 * 64 * (bd_rank(rank) + 8) * 2, tiles = n >= 1024 ? 4 : 1;
        const cudaError_t e = cudaFuncSetAttribute(la_bounded_decay_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);
        if (e != cudaSuccess) return (int)e;
        return (int)launch_pdl(la_bounded_decay_kernel, dim3((channels + 64 * tiles - 1) / (64 * tiles), (n + 63) / 64), dim3(256), bytes, st,
                               (const bf16*)x, ld, (const bf16*)a2, (const bf16*)bias, out, n, channels, rank, factor, tiles);
    }
    GO(bf16, false);
#undef GO
}

// single: every request brings one token.
PIE_API int pie_memory_gates(const MemoryGatesArgs* args, int single, cudaStream_t st) {
    const MemoryGatesArgs& a = *args;
    if (a.n <= 0 || a.reqs <= 0) return 0;
    if (a.heads <= 0 || a.cap <= 0.f || a.splits < 1) return (int)cudaErrorInvalidValue;
    if (single) return (int)launch_pdl(memory_gates_step_kernel, dim3((a.reqs * a.heads + 127) / 128), dim3(128), 0, st, a);
    const cudaError_t e = launch_pdl(memory_gates_log_kernel, dim3((unsigned)(((long)a.n * a.heads + 255) / 256)), dim3(256), 0, st, a);
    if (e != cudaSuccess) return (int)e;
    return (int)launch_pdl(memory_gates_scan_kernel, dim3(a.reqs, a.heads), dim3(256), 0, st, a);
}

// One or two parts (parts: 1 or 2) over the same tokens.
PIE_API int pie_gated_norm(const GatedNormArgs* args, int parts, int f32, cudaStream_t st) {
    const GatedNormArgs& a = *args;
    if (a.n <= 0) return 0;
    if (parts < 1 || parts > 2) return (int)cudaErrorInvalidValue;
    size_t sm = 0;
    int widest = 0;
    bool vec = true;
    auto aligned = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    for (int i = 0; i < parts; ++i) {
        const GatedNormPart& p = a.part[i];
        if (p.head_cols <= 0 || p.group <= 0 || p.cols <= 0 || p.gate_cols <= 0 || (p.den && (!p.floor || !p.norm_cols)) ||
            (p.norm_cols && (p.cols % p.norm_cols || !p.w || p.w_cols <= 0)))
            return (int)cudaErrorInvalidValue;
        widest = p.cols > widest ? p.cols : widest;
        if (p.norm_cols == p.cols) sm = (size_t)(32 + p.cols) * 4 > sm ? (size_t)(32 + p.cols) * 4 : sm;
        vec = vec && p.head_cols % 4 == 0 && p.head_ld % 4 == 0 && p.norm_cols % 4 == 0 && (!p.w || p.w_cols % 4 == 0) &&
              (p.gate_cols == 1 || p.gate_cols % 4 == 0) && p.cols % 4 == 0 && p.ldx % 4 == 0 &&
              (p.gate_cols > 1 || (p.ldg % 4 == 0 && aligned(p.gate))) && p.ldd % 4 == 0 && aligned(p.x) &&
              aligned(p.dst) && aligned(p.w);
    }
    if (sm > 227 * 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid(a.n, parts);
    auto kern = f32 ? (vec ? la_gated_norm_kernel<float, 4> : la_gated_norm_kernel<float, 1>)
                    : (vec ? la_gated_norm_kernel<bf16, 4> : la_gated_norm_kernel<bf16, 1>);
    if (sm > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
        if (e != cudaSuccess) return (int)e;
    }
    return (int)launch_pdl(kern, grid, dim3(widest <= 2048 ? 128 : 256), sm, st, a);
}
