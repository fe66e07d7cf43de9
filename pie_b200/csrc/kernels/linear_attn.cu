// Linear attention with a decaying state: per head S_t = diag(a_t) S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, S in 32-bit
// [dim][vdim], one state per (slot, head), carried from fire to fire. Two decays: one per key channel and token
// (`log_decay`, base-2 logarithms, at most 0), or one constant per head.
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
#include "typed.cuh"

namespace pie {

__device__ __forceinline__ float la_silu(float x) { return x / (1.f + expf(-x)); }

struct LinAttnArgs {
    const void *q, *k, *v;       // row t, head h at t * ld + h * dim (h * vdim for v), type T
    const float* log_decay;      // [n, heads * dim] base 2, or null
    const float* head_decay;     // [heads] the factor itself (null with log_decay)
    float* out;                  // [n, heads * vdim]
    float* state;                // this layer's part of slot 0: [heads][dim][vdim]
    const int *qo_indptr, *slots, *reset;
    // chunked form
    const int *chunk_req, *chunk_start, *req_chunks;   // request and first row of a piece; pieces of a request (indptr)
    float *u, *piece_decay;      // [chunks][heads][dim][vdim], [chunks][heads][dim] (base-2 logarithm)
    long slot_stride;
    int n, ld, reqs, heads, dim, vdim, silu, chunks;
    float q_scale;
};

// ------------------------------------------------------------------ serial
template <typename T, int RPT, int VEC>
__global__ void __launch_bounds__(256) la_serial_kernel(const LinAttnArgs a) {
    constexpr int ROWS = RPT * 8, COLS = 32 * VEC;
    __shared__ float sq[ROWS], sk[ROWS], sa[ROWS];
    __shared__ float red[8][COLS];
    pdl_trigger();
    pdl_wait();
    const int r = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, rg = threadIdx.x >> 5;
    const int first = a.qo_indptr[r], len = a.qo_indptr[r + 1] - first, slot = a.slots[r];
    if (len <= 0 || slot < 0) return;          // a padding request of a decode graph: no state, no output
    const int c0 = blockIdx.z * COLS + lane * VEC;
    const bool col = c0 < a.vdim;              // VEC > 1 only where vdim is a multiple of it
    float* sp = a.state + (size_t)slot * a.slot_stride + (size_t)h * a.dim * a.vdim;
    float S[RPT][VEC];
    const bool fresh = a.reset[r] != 0;
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
        for (int d = threadIdx.x; d < ROWS; d += 256) {
            float q = 0.f, k = 0.f, g = 1.f;
            if (d < a.dim) {
                q = to_f(qr[d]);
                k = to_f(kr[d]);
                if (a.silu) { q = la_silu(q); k = la_silu(k); }
                g = a.log_decay ? exp2f(a.log_decay[row * a.heads * a.dim + h * a.dim + d]) : hd;
            }
            sq[d] = q * a.q_scale;
            sk[d] = k;
            sa[d] = g;
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
}

// ----------------------------------------------------------------- chunked
constexpr int LA_C = 64;                  // tokens per piece
constexpr int LA_VT = 32;                 // value columns per pass of the output kernel

__device__ __forceinline__ uint32_t tf32(float x) {
    uint32_t r;
    asm("cvt.rna.tf32.f32 %0, %1;" : "=r"(r) : "f"(x));
    return r;
}
// C (16 x 8) += A (16 x 8, row) B (8 x 8, col); lane (g = lane / 4, t = lane % 4) holds A (g | g + 8, t | t + 4),
// B (t | t + 4, g) and C (g | g + 8, 2 t | 2 t + 1)
__device__ __forceinline__ void mma_tf32(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// Rows of a chunk in shared memory: pitch of the [64][dim] arrays, in elements
__host__ __device__ constexpr int la_pitch(int dim) { return (dim + 15) / 16 * 16 + 8; }

template <bool CHAN>
__global__ void __launch_bounds__(128) la_chunk_state_kernel(const LinAttnArgs a) {
    extern __shared__ float sm[];
    const int c = blockIdx.x, h = blockIdx.y, r = a.chunk_req[c];
    const int row0 = a.chunk_start[c], len = min(LA_C, a.qo_indptr[r + 1] - row0);
    const int dimp = (a.dim + 15) / 16 * 16, kp = la_pitch(a.dim), vp = 72;
    float* sk = sm;                        // [64][kp] decayed keys
    float* sv = sk + LA_C * kp;            // [64][72] a tile of values
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const float lh = CHAN ? 0.f : log2f(a.head_decay[h]);
    const bf16* kb = static_cast<const bf16*>(a.k) + h * a.dim;
    for (int d = threadIdx.x; d < dimp; d += 128) {
        float w = 0.f;                     // base-2 decay from this token to the end of the piece
        for (int s = LA_C - 1; s >= 0; --s) {
            float k = 0.f;
            if (s < len && d < a.dim) {
                const size_t row = (size_t)(row0 + s);
                k = to_f(kb[row * a.ld + d]);
                if (a.silu) k = la_silu(k);
                k *= exp2f(w);
                w += CHAN ? a.log_decay[row * a.heads * a.dim + h * a.dim + d] : lh;
            }
            sk[s * kp + d] = k;
        }
        if (d < a.dim) a.piece_decay[((size_t)c * a.heads + h) * a.dim + d] = w;
    }
    float* U = a.u + ((size_t)c * a.heads + h) * a.dim * a.vdim;
    const bf16* vb = static_cast<const bf16*>(a.v) + h * a.vdim;
    for (int v0 = 0; v0 < a.vdim; v0 += 64) {
        __syncthreads();
        for (int i = threadIdx.x; i < LA_C * 64; i += 128) {
            const int s = i >> 6, j = i & 63;
            float v = 0.f;
            if (s < len && v0 + j < a.vdim) {
                v = to_f(vb[(size_t)(row0 + s) * a.ld + v0 + j]);
                if (a.silu) v = la_silu(v);
            }
            sv[s * vp + j] = v;
        }
        __syncthreads();
        const int nt = min(8, (a.vdim - v0 + 7) / 8);
        for (int m = warp; m < dimp / 16; m += 4) {
            float acc[8][4];
#pragma unroll
            for (int n = 0; n < 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < LA_C / 8; ++ks) {
                const float* kr = sk + (ks * 8 + t) * kp + m * 16 + g;
                const uint32_t fa[4] = {tf32(kr[0]), tf32(kr[8]), tf32(kr[4 * kp]), tf32(kr[4 * kp + 8])};
#pragma unroll
                for (int n = 0; n < 8; ++n) {
                    if (n >= nt) break;
                    const float* vr = sv + (ks * 8 + t) * vp + n * 8 + g;
                    mma_tf32(acc[n], fa, tf32(vr[0]), tf32(vr[4 * vp]));
                }
            }
#pragma unroll
            for (int n = 0; n < 8; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int d = m * 16 + g + (e >> 1) * 8, j = v0 + n * 8 + 2 * t + (e & 1);
                    if (d < a.dim && j < a.vdim) U[(size_t)d * a.vdim + j] = acc[n][e];
                }
        }
    }
}

// One thread per state element: U becomes the state before each piece; the state after the last goes back to its slot.
__global__ void __launch_bounds__(256) la_chunk_scan_kernel(const LinAttnArgs a) {
    const int r = blockIdx.y, slot = a.slots[r];
    const int c0 = a.req_chunks[r], c1 = a.req_chunks[r + 1];
    const long elems = (long)a.heads * a.dim * a.vdim, i = blockIdx.x * 256L + threadIdx.x;
    if (i >= elems || c1 <= c0 || slot < 0) return;
    float* sp = a.state + (size_t)slot * a.slot_stride + i;
    float s = a.reset[r] ? 0.f : *sp;
    float* u = a.u + i;
    const float* dec = a.piece_decay + i / a.vdim;
    const long dstep = (long)a.heads * a.dim;
    int c = c0;
    for (; c + 4 <= c1; c += 4) {
        float x[4], w[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) { x[j] = u[(c + j) * elems]; w[j] = dec[(c + j) * dstep]; }
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            u[(c + j) * elems] = s;
            s = exp2f(w[j]) * s + x[j];
        }
    }
    for (; c < c1; ++c) {
        const float x = u[c * elems], w = dec[c * dstep];
        u[c * elems] = s;
        s = exp2f(w) * s + x;
    }
    *sp = s;
}

template <bool CHAN>
__global__ void __launch_bounds__(128) la_chunk_out_kernel(const LinAttnArgs a) {
    extern __shared__ float sm[];
    const int c = blockIdx.x, h = blockIdx.y, r = a.chunk_req[c];
    const int row0 = a.chunk_start[c], len = min(LA_C, a.qo_indptr[r + 1] - row0);
    const int dimp = (a.dim + 15) / 16 * 16, kp = la_pitch(a.dim), xp = dimp + 4, sp = LA_VT + 8, vp = LA_VT + 4;
    // xp (row index by g, column by t) and sp (row by t, column by g) keep fragment reads off each other's banks
    float* sb = sm;                                        // [64][xp] decay from the piece's start (CHAN), then decayed queries
    float* ss = sb + LA_C * xp;                            // [dimp][sp] a tile of the state
    float* sv = ss + dimp * sp;                            // [64][vp] a tile of values
    bf16* sq = reinterpret_cast<bf16*>(sv + LA_C * vp);    // [64][kp]
    bf16* sk = sq + LA_C * kp;                             // [64][kp]
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const float lh = CHAN ? 0.f : log2f(a.head_decay[h]);
    const bf16* qb = static_cast<const bf16*>(a.q) + h * a.dim;
    const bf16* kb = static_cast<const bf16*>(a.k) + h * a.dim;
    for (int i = threadIdx.x; i < LA_C * dimp; i += 128) {
        const int s = i / dimp, d = i - s * dimp;
        bf16 q = __float2bfloat16(0.f), k = q;
        if (s < len && d < a.dim) {
            const size_t o = (size_t)(row0 + s) * a.ld + d;
            q = qb[o];
            k = kb[o];
            if (a.silu) {
                q = __float2bfloat16(la_silu(to_f(q)));
                k = __float2bfloat16(la_silu(to_f(k)));
            }
        }
        sq[s * kp + d] = q;
        sk[s * kp + d] = k;
    }
    if (CHAN) {
        for (int d = threadIdx.x; d < dimp; d += 128) {
            float w = 0.f;
            for (int s = 0; s < LA_C; ++s) {
                if (s < len && d < a.dim) w += a.log_decay[(size_t)(row0 + s) * a.heads * a.dim + h * a.dim + d];
                sb[s * xp + d] = w;
            }
        }
    }
    __syncthreads();

    // scores of this warp's 16 queries against the keys up to the end of their own 16-token block
    const int w0 = warp * 16;
    float sc[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) sc[n][0] = sc[n][1] = sc[n][2] = sc[n][3] = 0.f;
    bool exact = false;
    if (CHAN) {
        float range = 0.f;
        for (int d = lane; d < dimp; d += 32) range = fmaxf(range, (w0 ? sb[(w0 - 1) * xp + d] : 0.f) - sb[(w0 + 15) * xp + d]);
        exact = warp_max(range) > 100.f;
    }
    for (int ks = 0; ks < dimp / 8; ++ks) {
        const int d0 = ks * 8 + t, d1 = d0 + 4;
        float q4[4] = {to_f(sq[(w0 + g) * kp + d0]), to_f(sq[(w0 + g + 8) * kp + d0]), to_f(sq[(w0 + g) * kp + d1]),
                       to_f(sq[(w0 + g + 8) * kp + d1])};
        uint32_t fa[4];
        float b4[4], r0 = 0.f, r1 = 0.f;
        if (CHAN) {
            b4[0] = sb[(w0 + g) * xp + d0]; b4[1] = sb[(w0 + g + 8) * xp + d0];
            b4[2] = sb[(w0 + g) * xp + d1]; b4[3] = sb[(w0 + g + 8) * xp + d1];
            if (w0) { r0 = sb[(w0 - 1) * xp + d0]; r1 = sb[(w0 - 1) * xp + d1]; }
#pragma unroll
            for (int e = 0; e < 4; ++e) fa[e] = tf32(q4[e] * exp2f(b4[e] - (e < 2 ? r0 : r1)));
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) fa[e] = __float_as_uint(q4[e]);
        }
#pragma unroll
        for (int n = 0; n < 6; ++n) {
            if (n >= 2 * warp) break;
            const int s = n * 8 + g;
            float k0 = to_f(sk[s * kp + d0]), k1 = to_f(sk[s * kp + d1]);
            if (CHAN) {
                k0 *= exp2f(r0 - sb[s * xp + d0]);
                k1 *= exp2f(r1 - sb[s * xp + d1]);
            }
            mma_tf32(sc[n], fa, tf32(k0), tf32(k1));
        }
        if (exact) continue;
        if (CHAN) {
            r0 = sb[(w0 + 7) * xp + d0];
            r1 = sb[(w0 + 7) * xp + d1];
#pragma unroll
            for (int e = 0; e < 4; ++e) fa[e] = tf32(q4[e] * exp2f(b4[e] - (e < 2 ? r0 : r1)));
        }
#pragma unroll
        for (int n2 = 0; n2 < 2; ++n2) {
            const int s = w0 + n2 * 8 + g;
            float k0 = to_f(sk[s * kp + d0]), k1 = to_f(sk[s * kp + d1]);
            if (CHAN) {
                k0 *= exp2f(r0 - sb[s * xp + d0]);
                k1 *= exp2f(r1 - sb[s * xp + d1]);
            }
            const uint32_t b0 = tf32(k0), b1 = tf32(k1);
#pragma unroll
            for (int w = 0; w < 4; ++w)
                if (w == warp) mma_tf32(sc[2 * w + n2], fa, b0, b1);
        }
    }
    // decay between the two tokens (constant per head), causal limit
#pragma unroll
    for (int n = 0; n < 8; ++n) {
        if (n >= 2 * warp + 2) break;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int q = w0 + g + (e >> 1) * 8, s = n * 8 + 2 * t + (e & 1);
            if (s > q) { sc[n][e] = 0.f; continue; }
            if (!CHAN) sc[n][e] *= exp2f((float)(q - s) * lh);
            if (CHAN && exact && n >= 2 * warp) {
                float x = 0.f;
                for (int d = 0; d < dimp; ++d)
                    x += to_f(sq[q * kp + d]) * to_f(sk[s * kp + d]) * exp2f(sb[q * xp + d] - sb[s * xp + d]);
                sc[n][e] = x;
            }
        }
    }
    // queries with the decay from the start of the piece, for the state before it
    __syncthreads();
    for (int i = threadIdx.x; i < LA_C * dimp; i += 128) {
        const int s = i / dimp, d = i - s * dimp;
        const float q = to_f(sq[s * kp + d]);
        sb[s * xp + d] = CHAN ? q * exp2f(sb[s * xp + d]) : q * exp2f((float)(s + 1) * lh);
    }

    const float* S = a.u + ((size_t)c * a.heads + h) * a.dim * a.vdim;
    const bf16* vb = static_cast<const bf16*>(a.v) + h * a.vdim;
    for (int v0 = 0; v0 < a.vdim; v0 += LA_VT) {
        __syncthreads();
        for (int i = threadIdx.x; i < dimp * LA_VT; i += 128) {
            const int d = i / LA_VT, j = i % LA_VT;
            ss[d * sp + j] = d < a.dim && v0 + j < a.vdim ? S[(size_t)d * a.vdim + v0 + j] : 0.f;
        }
        for (int i = threadIdx.x; i < LA_C * LA_VT; i += 128) {
            const int s = i / LA_VT, j = i % LA_VT;
            float v = 0.f;
            if (s < len && v0 + j < a.vdim) {
                v = to_f(vb[(size_t)(row0 + s) * a.ld + v0 + j]);
                if (a.silu) v = la_silu(v);
            }
            sv[s * vp + j] = v;
        }
        __syncthreads();
        float acc[LA_VT / 8][4];
#pragma unroll
        for (int n = 0; n < LA_VT / 8; ++n) acc[n][0] = acc[n][1] = acc[n][2] = acc[n][3] = 0.f;
        for (int ks = 0; ks < dimp / 8; ++ks) {
            const float* q0 = sb + (w0 + g) * xp + ks * 8 + t;
            const float* q1 = q0 + 8 * xp;
            const uint32_t fa[4] = {tf32(q0[0]), tf32(q1[0]), tf32(q0[4]), tf32(q1[4])};
            const float* sr = ss + (ks * 8 + t) * sp + g;
#pragma unroll
            for (int n = 0; n < LA_VT / 8; ++n) mma_tf32(acc[n], fa, tf32(sr[n * 8]), tf32(sr[4 * sp + n * 8]));
        }
        // scores as the A operand: its columns t and t + 4 stand for the keys 2 t and 2 t + 1 that this lane holds
#pragma unroll
        for (int ks = 0; ks < 8; ++ks) {
            if (ks >= 2 * warp + 2) break;
            const uint32_t fa[4] = {tf32(sc[ks][0]), tf32(sc[ks][2]), tf32(sc[ks][1]), tf32(sc[ks][3])};
            const float* vr = sv + (ks * 8 + 2 * t) * vp + g;
#pragma unroll
            for (int n = 0; n < LA_VT / 8; ++n) mma_tf32(acc[n], fa, tf32(vr[n * 8]), tf32(vr[vp + n * 8]));
        }
#pragma unroll
        for (int n = 0; n < LA_VT / 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int q = w0 + g + (e >> 1) * 8, j = v0 + n * 8 + 2 * t + (e & 1);
                if (q < len && j < a.vdim) a.out[(size_t)(row0 + q) * a.heads * a.vdim + h * a.vdim + j] = acc[n][e] * a.q_scale;
            }
    }
}

// ---------------------------------------------------------- channel decays
// log_decay[t, c] = log2(sigmoid(z)) / tau, z = a2[c, :] . a1[t, :] + bias[c]; x holds a1 at column 0 of rows of ld.
constexpr int LD_TOK = 8;
template <typename T>
__global__ void __launch_bounds__(256) la_decay_kernel(const T* __restrict__ x, int ld, const T* __restrict__ a2, const T* __restrict__ bias,
                                                       float* __restrict__ out, int n, int channels, int rank, float inv_tau) {
    extern __shared__ float sx[];          // [LD_TOK][rank]
    pdl_trigger();
    pdl_wait();
    const int t0 = blockIdx.x * LD_TOK, nt = min(LD_TOK, n - t0);
    for (int i = threadIdx.x; i < LD_TOK * rank; i += 256) {
        const int s = i / rank, j = i - s * rank;
        sx[i] = s < nt ? to_f(x[(size_t)(t0 + s) * ld + j]) : 0.f;
    }
    __syncthreads();
    const int c = blockIdx.y * 256 + threadIdx.x;
    if (c >= channels) return;
    float z[LD_TOK];
    const float b = to_f(bias[c]);
#pragma unroll
    for (int s = 0; s < LD_TOK; ++s) z[s] = b;
    const T* w = a2 + (size_t)c * rank;
    for (int j = 0; j < rank; ++j) {
        const float wj = to_f(w[j]);
#pragma unroll
        for (int s = 0; s < LD_TOK; ++s) z[s] += wj * sx[s * rank + j];
    }
#pragma unroll
    for (int s = 0; s < LD_TOK; ++s)
        if (s < nt) out[(size_t)(t0 + s) * channels + c] = (fminf(z[s], 0.f) - log1pf(expf(-fabsf(z[s])))) * (1.4426950408889634f * inv_tau);
}

// -------------------------------------------------------- norm and gate of a mixer's output
// dst[t, :] = scale * act(gate) * (rms-normed x) [* w]; the mean square runs over `norm_cols` consecutive columns (0: no
// norm). Column j of the output is column (head / group * group_pad + head % group) * head_ld + j % head_cols of x, so that
// x may hold padded heads. Columns from cols to dst_cols are written as zeros.
struct GatedNormPart {
    const void* x;
    const void *w, *gate;
    void* dst;
    int x_f32, ldx, head_cols, head_ld, group, group_pad, norm_cols, w_cols, ldg, ldd, cols, dst_cols, act;   // act 0: sigmoid, 1: SiLU
    float eps, scale;
};
struct GatedNormArgs {
    GatedNormPart part[2];
    int n;
};

template <typename T>
__global__ void __launch_bounds__(256) la_gated_norm_kernel(const GatedNormArgs args) {
    extern __shared__ float buf[];
    pdl_trigger();
    pdl_wait();
    const GatedNormPart& p = args.part[blockIdx.y];
    const int t = blockIdx.x;
    const T* gate = static_cast<const T*>(p.gate) + (size_t)t * p.ldg;
    T* dst = static_cast<T*>(p.dst) + (size_t)t * p.ldd;
    auto source = [&](int j) {
        const int h = j / p.head_cols;
        const size_t at = (size_t)t * p.ldx + (size_t)(h / p.group * p.group_pad + h % p.group) * p.head_ld + (j - h * p.head_cols);
        return p.x_f32 ? static_cast<const float*>(p.x)[at] : to_f(static_cast<const T*>(p.x)[at]);
    };
    auto finish = [&](int j, float v) {
        const float z = to_f(gate[j]), s = 1.f / (1.f + expf(-z));
        dst[j] = from_f<T>(v * (p.act ? z * s : s) * p.scale);
    };
    if (p.norm_cols == 0) {
        for (int j = threadIdx.x; j < p.cols; j += 256) finish(j, source(j));
    } else {
        const T* w = static_cast<const T*>(p.w);
        const int groups = p.cols / p.norm_cols, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
        if (groups == 1) {
            float ss = 0.f;
            for (int j = threadIdx.x; j < p.cols; j += 256) {
                const float v = source(j);
                buf[32 + j] = v;
                ss += v * v;
            }
            const float inv = 1.f / sqrtf(block_sum(ss, buf) / (float)p.cols + p.eps);
            for (int j = threadIdx.x; j < p.cols; j += 256) finish(j, buf[32 + j] * inv * to_f(w[j]));
        } else {
            for (int gr = warp; gr < groups; gr += 8) {
                float ss = 0.f;
                for (int j = lane; j < p.norm_cols; j += 32) {
                    const float v = source(gr * p.norm_cols + j);
                    ss += v * v;
                }
                const float inv = 1.f / sqrtf(warp_sum(ss) / (float)p.norm_cols + p.eps);
                for (int j = lane; j < p.norm_cols; j += 32) {
                    const int c = gr * p.norm_cols + j;
                    finish(c, source(c) * inv * to_f(w[c % p.w_cols]));
                }
            }
        }
    }
    for (int j = p.cols + threadIdx.x; j < p.dst_cols; j += 256) dst[j] = from_f<T>(0.f);
}

}  // namespace pie

using namespace pie;

PIE_API int pie_linear_attn_serial(const LinAttnArgs* args, int f32, cudaStream_t st) {
    const LinAttnArgs& a = *args;
    if (a.n <= 0 || a.reqs <= 0) return 0;
    if (a.dim <= 0 || a.dim > 512 || a.vdim <= 0 || (!a.log_decay && !a.head_decay)) return (int)cudaErrorInvalidValue;
    const bool vec = a.vdim % 4 == 0 && a.vdim >= 64 && a.dim <= 256 && a.slot_stride % 4 == 0 && ((uintptr_t)a.state & 15) == 0;
    const int cols = vec ? 128 : 32, rpt = (a.dim + 7) / 8;
    const dim3 grid(a.reqs, a.heads, (a.vdim + cols - 1) / cols);
#define GO(T_, R_, V_)                                                                                  \
    return (int)launch_pdl(la_serial_kernel<T_, R_, V_>, grid, dim3(256), 0, st, a)
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

static size_t la_state_smem(int dim) { return (size_t)LA_C * (la_pitch(dim) + 72) * 4; }
static size_t la_out_smem(int dim) {
    const int dimp = (dim + 15) / 16 * 16;
    return ((size_t)LA_C * (dimp + 4) + (size_t)dimp * (LA_VT + 8) + (size_t)LA_C * (LA_VT + 4)) * 4 + 2ul * LA_C * la_pitch(dim) * 2;
}
// 1 when the chunked form takes heads of this key size.
PIE_API int pie_linear_attn_chunk_supported(int dim) {
    return dim > 0 && la_out_smem(dim) <= 227 * 1024 && la_state_smem(dim) <= 227 * 1024 ? 1 : 0;
}
PIE_API int pie_linear_attn_chunk_tokens() { return LA_C; }

PIE_API int pie_linear_attn_chunked(const LinAttnArgs* args, cudaStream_t st) {
    const LinAttnArgs& a = *args;
    if (a.n <= 0 || a.reqs <= 0 || a.chunks <= 0) return 0;
    if (!pie_linear_attn_chunk_supported(a.dim) || a.vdim <= 0 || (!a.log_decay && !a.head_decay) || !a.u || !a.piece_decay)
        return (int)cudaErrorInvalidValue;
    const dim3 grid(a.chunks, a.heads);
    const size_t s1 = la_state_smem(a.dim), s3 = la_out_smem(a.dim);
    auto k1 = a.log_decay ? la_chunk_state_kernel<true> : la_chunk_state_kernel<false>;
    auto k3 = a.log_decay ? la_chunk_out_kernel<true> : la_chunk_out_kernel<false>;
    cudaError_t e = cudaFuncSetAttribute(k1, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s1);
    if (e == cudaSuccess) e = cudaFuncSetAttribute(k3, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)s3);
    if (e != cudaSuccess) return (int)e;
    k1<<<grid, 128, s1, st>>>(a);
    const long elems = (long)a.heads * a.dim * a.vdim;
    la_chunk_scan_kernel<<<dim3((unsigned)((elems + 255) / 256), a.reqs), 256, 0, st>>>(a);
    k3<<<grid, 128, s3, st>>>(a);
    return (int)cudaGetLastError();
}

PIE_API int pie_linear_decay(const void* x, int ld, const void* a2, const void* bias, float* out, int n, int channels, int rank, float inv_tau,
                             int f32, cudaStream_t st) {
    if (n <= 0) return 0;
    if (rank <= 0 || rank > 1024 || channels <= 0) return (int)cudaErrorInvalidValue;
    const dim3 grid((n + LD_TOK - 1) / LD_TOK, (channels + 255) / 256);
    const size_t sm = (size_t)LD_TOK * rank * 4;
    if (f32)
        return (int)launch_pdl(la_decay_kernel<float>, grid, dim3(256), sm, st, (const float*)x, ld, (const float*)a2, (const float*)bias, out, n,
                               channels, rank, inv_tau);
    return (int)launch_pdl(la_decay_kernel<bf16>, grid, dim3(256), sm, st, (const bf16*)x, ld, (const bf16*)a2, (const bf16*)bias, out, n,
                           channels, rank, inv_tau);
}

// One or two parts (parts: 1 or 2) over the same tokens.
PIE_API int pie_gated_norm(const GatedNormArgs* args, int parts, int f32, cudaStream_t st) {
    const GatedNormArgs& a = *args;
    if (a.n <= 0) return 0;
    if (parts < 1 || parts > 2) return (int)cudaErrorInvalidValue;
    size_t sm = 0;
    for (int i = 0; i < parts; ++i) {
        const GatedNormPart& p = a.part[i];
        if (p.head_cols <= 0 || p.group <= 0 || p.cols <= 0 || (p.norm_cols && (p.cols % p.norm_cols || !p.w || p.w_cols <= 0)))
            return (int)cudaErrorInvalidValue;
        if (p.norm_cols == p.cols) sm = (size_t)(32 + p.cols) * 4 > sm ? (size_t)(32 + p.cols) * 4 : sm;
    }
    if (sm > 227 * 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid(a.n, parts);
    auto kern = f32 ? la_gated_norm_kernel<float> : la_gated_norm_kernel<bf16>;
    if (sm > 48 * 1024) {
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sm);
        if (e != cudaSuccess) return (int)e;
    }
    return (int)launch_pdl(kern, grid, dim3(256), sm, st, a);
}
