// Delta rule with a decay and a removal rate per key channel: per head, with the unit key u = k / sqrt(sum k^2 + 1e-6),
//   S_t = diag(w_t) S_(t-1) - (a_t * u_t) (u_t^T S_(t-1)) + k_t v_t^T,   o_t = S_t^T r_t,
// S in 32-bit [dim][dim], one state per (slot, head), carried from fire to fire. Everything but the projections (r, k, v and the
// product behind a) is 32-bit. Both sums of a token run over the old state:
//   y = S^T u,  z = S^T (r * w),   o = z - (r . (a * u)) y + (r . k) v,
// so that columns of the state never meet, and a column's rows once per token.
//
//   step       one token per request: a block holds 128 columns (VEC per lane) of a head, an eighth of the rows per warp
//   portions   any lengths: LPC lanes share CPT columns, each with R rows of them; a token's sums meet by halving (a lane ends up
//              with one of them); the tokens' vectors are prepared CT at a time in shared memory while the tokens before run
//   chunked    prompts in bf16, heads of up to 128: 16 tokens at a time on tf32 tensor-core tiles, see below
#include "tf32.cuh"
#include "typed.cuh"

namespace pie {

struct DeltaArgs {
    const void *r, *k, *v, *a;      // row t, head h at t * ld + h * dim, type T; a: the removal rate's product
    const float* a_bias;            // [heads * dim]
    const float* log_decay;         // [n, heads * dim] base 2
    float* out;                     // [n, heads * dim]
    float* state;                   // this layer's part of slot 0: [heads][dim][dim]
    const int *qo_indptr, *slots, *reset;
    // chunked form: request and first row of a piece of 16 tokens; pieces of a request (indptr)
    const int *chunk_req, *chunk_start, *req_chunks;
    void* pieces;                   // [chunks][heads] DeltaPiece
    long slot_stride;
    int n, ld, reqs, heads, dim, chunks;
};

__device__ __forceinline__ float delta_rate(float z) { return 1.f / (1.f + expf(-z)); }

template <typename T, int RPT, int VEC>
__global__ void __launch_bounds__(256) delta_step_kernel(const DeltaArgs a) {
    constexpr int ROWS = RPT * 8, COLS = 32 * VEC;
    __shared__ float su[ROWS], sau[ROWS], sw[ROWS], srw[ROWS], sk[ROWS], red[32];
    __shared__ __align__(16) float ry[8][COLS], rz[8][COLS];
    pdl_trigger();
    pdl_wait();
    const int q = blockIdx.x, h = blockIdx.y, lane = threadIdx.x & 31, rg = threadIdx.x >> 5;
    const int t = a.qo_indptr[q], slot = a.slots[q];
    if (a.qo_indptr[q + 1] <= t || slot < 0) return;       // a padding request of a decode graph: no state, no output
    const int c0 = blockIdx.z * COLS + lane * VEC;
    const bool col = c0 < a.dim;                           // VEC > 1 only where dim is a multiple of it
    float* sp = a.state + (size_t)slot * a.slot_stride + (size_t)h * a.dim * a.dim;
    const bool fresh = a.reset[q] != 0;
    float S[RPT][VEC];
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = rg + 8 * i;
#pragma unroll
        for (int j = 0; j < VEC; ++j) S[i][j] = 0.f;
        if (col && !fresh && d < a.dim) load_vec<VEC>(sp + (size_t)d * a.dim + c0, S[i]);
    }
    const size_t row = (size_t)t * a.ld + h * a.dim;
    float v[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) v[j] = 0.f;
    if (col) load_vec<VEC>(static_cast<const T*>(a.v) + row + c0, v);
    constexpr int PER = (ROWS + 255) / 256;
    float k[PER], ss = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int d = threadIdx.x + i * 256;
        k[i] = d < a.dim ? to_f(static_cast<const T*>(a.k)[row + d]) : 0.f;
        ss += k[i] * k[i];
    }
    const float inv = 1.f / sqrtf(block_sum(ss, red) + 1e-6f);
    float rau = 0.f, rk = 0.f;
#pragma unroll
    for (int i = 0; i < PER; ++i) {
        const int d = threadIdx.x + i * 256;
        if (d >= ROWS) break;
        float r = 0.f, w = 1.f, rate = 0.f;
        if (d < a.dim) {
            r = to_f(static_cast<const T*>(a.r)[row + d]);
            w = exp2f(a.log_decay[((size_t)t * a.heads + h) * a.dim + d]);
            rate = delta_rate(to_f(static_cast<const T*>(a.a)[row + d]) + a.a_bias[h * a.dim + d]);
        }
        const float u = k[i] * inv, au = rate * u;
        su[d] = u; sau[d] = au; sw[d] = w; srw[d] = r * w; sk[d] = k[i];
        rau += r * au;
        rk += r * k[i];
    }
    rau = block_sum(rau, red);
    rk = block_sum(rk, red);
    float y[VEC], z[VEC];
#pragma unroll
    for (int j = 0; j < VEC; ++j) y[j] = z[j] = 0.f;
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const float u = su[rg + 8 * i], rw = srw[rg + 8 * i];
#pragma unroll
        for (int j = 0; j < VEC; ++j) {
            y[j] += u * S[i][j];
            z[j] += rw * S[i][j];
        }
    }
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
        ry[rg][lane * VEC + j] = y[j];
        rz[rg][lane * VEC + j] = z[j];
    }
    __syncthreads();
#pragma unroll
    for (int j = 0; j < VEC; ++j) {
        y[j] = z[j] = 0.f;
#pragma unroll
        for (int g = 0; g < 8; ++g) {
            y[j] += ry[g][lane * VEC + j];
            if (rg == 0) z[j] += rz[g][lane * VEC + j];
        }
    }
    if (!col) return;
    if (rg == 0) {
        float* dst = a.out + ((size_t)t * a.heads + h) * a.dim + c0;
#pragma unroll
        for (int j = 0; j < VEC; ++j) dst[j] = z[j] - rau * y[j] + rk * v[j];
    }
#pragma unroll
    for (int i = 0; i < RPT; ++i) {
        const int d = rg + 8 * i;
        if (d >= a.dim) continue;
        const float w = sw[d], au = sau[d], kk = sk[d];
#pragma unroll
        for (int j = 0; j < VEC; ++j) S[i][j] = w * S[i][j] - au * y[j] + kk * v[j];
        store_vec<VEC>(sp + (size_t)d * a.dim + c0, S[i]);
    }
}

constexpr int DELTA_WARPS = 4;
constexpr int DELTA_CT = 8;                // tokens prepared at a time

template <int R, int LPC, int CPT>
struct DeltaSmem {
    static constexpr int DP = R * LPC, COLS = DELTA_WARPS * (32 / LPC) * CPT;
    float vec[2][DELTA_CT][5 * DP];        // u, r * w, w, a * u, k of a token
    float v[2][DELTA_CT][COLS], o[2][DELTA_CT][COLS];
    float2 dots[2][DELTA_CT];              // r . (a * u), r . k
};

// Sums of NV values over LPC lanes: halves change hands until a lane is left with one value (of index `which`, the lane's own
// number in bits from the top); further lanes then add up copies of it.
template <int NV, int LPC>
__device__ __forceinline__ float halving_sum(float (&x)[NV], int g) {
    if constexpr (NV == 1) {
        float y = x[0];
#pragma unroll
        for (int o = LPC / 2; o; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
        return y;
    } else {
        const bool up = g & (LPC / 2);
        float y[NV / 2];
#pragma unroll
        for (int i = 0; i < NV / 2; ++i) {
            const float keep = up ? x[i + NV / 2] : x[i], give = up ? x[i] : x[i + NV / 2];
            y[i] = keep + __shfl_xor_sync(0xffffffffu, give, LPC / 2);
        }
        return halving_sum<NV / 2, LPC / 2>(y, g);
    }
}

// Lane g of a column group holds the rows 4 (g + LPC i) + e.
template <typename T, int R, int LPC, int CPT>
__global__ void __launch_bounds__(DELTA_WARPS * 32) delta_portion_kernel(const DeltaArgs a) {
    using Smem = DeltaSmem<R, LPC, CPT>;
    constexpr int THREADS = DELTA_WARPS * 32, CT = DELTA_CT, DP = Smem::DP, COLS = Smem::COLS, TPW = CT / DELTA_WARPS, EPL = DP / 32;
    constexpr int VPT = (CT * COLS + THREADS - 1) / THREADS, NV = 2 * CPT;
    static_assert(NV <= LPC && R % 4 == 0 && CPT % 2 == 0, "");
    extern __shared__ __align__(16) uint8_t raw[];
    Smem& sm = *reinterpret_cast<Smem*>(raw);
    const int q = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int first = a.qo_indptr[q], len = a.qo_indptr[q + 1] - first, slot = a.slots[q];
    if (len <= 0 || slot < 0) return;
    const int g = lane % LPC, cl = (warp * (32 / LPC) + lane / LPC) * CPT, c0 = blockIdx.z * COLS + cl;
    float* sp = a.state + (size_t)slot * a.slot_stride + (size_t)h * a.dim * a.dim;
    const bool fresh = a.reset[q] != 0;
    F2 S[CPT][R / 2];
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int i = 0; i < R / 2; ++i) {
            const int d = 4 * (g + LPC * (i / 2)) + 2 * (i & 1);
            const bool ok = !fresh && c0 + c < a.dim;
            S[c][i] = f2(ok && d < a.dim ? sp[(size_t)d * a.dim + c0 + c] : 0.f, ok && d + 1 < a.dim ? sp[(size_t)(d + 1) * a.dim + c0 + c] : 0.f);
        }
    const T* Rp = static_cast<const T*>(a.r) + (size_t)first * a.ld + h * a.dim;
    const T* Kp = static_cast<const T*>(a.k) + (size_t)first * a.ld + h * a.dim;
    const T* Vp = static_cast<const T*>(a.v) + (size_t)first * a.ld + h * a.dim;
    const T* Ap = static_cast<const T*>(a.a) + (size_t)first * a.ld + h * a.dim;
    const float* Wp = a.log_decay + ((size_t)first * a.heads + h) * a.dim;
    float* O = a.out + ((size_t)first * a.heads + h) * a.dim;
    const size_t step = (size_t)a.heads * a.dim;
    float bias[EPL];
#pragma unroll
    for (int i = 0; i < EPL; ++i) bias[i] = lane + 32 * i < a.dim ? a.a_bias[h * a.dim + lane + 32 * i] : 0.f;

    T pr[TPW][EPL], pk[TPW][EPL], pa[TPW][EPL], pv[VPT];
    float pw[TPW][EPL];
    auto load = [&](int t0) {
#pragma unroll
        for (int s = 0; s < TPW; ++s) {
            const int t = t0 + warp * TPW + s;
#pragma unroll
            for (int i = 0; i < EPL; ++i) {
                const int d = lane + 32 * i;
                const bool ok = t < len && d < a.dim;
                const size_t at = (size_t)t * a.ld + d;
                pr[s][i] = ok ? Rp[at] : from_f<T>(0.f);
                pk[s][i] = ok ? Kp[at] : from_f<T>(0.f);
                pa[s][i] = ok ? Ap[at] : from_f<T>(0.f);
                pw[s][i] = ok ? Wp[(size_t)t * step + d] : 0.f;
            }
        }
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            const int x = threadIdx.x + i * THREADS, t = t0 + x / COLS, cc = blockIdx.z * COLS + x % COLS;
            pv[i] = x < CT * COLS && t < len && cc < a.dim ? Vp[(size_t)t * a.ld + cc] : from_f<T>(0.f);
        }
    };
    auto prepare = [&](int b) {
#pragma unroll
        for (int s = 0; s < TPW; ++s) {
            float ss = 0.f, rau = 0.f, rk = 0.f;
#pragma unroll
            for (int i = 0; i < EPL; ++i) ss += to_f(pk[s][i]) * to_f(pk[s][i]);
            const float inv = 1.f / sqrtf(warp_sum(ss) + 1e-6f);
            float* dst = sm.vec[b][warp * TPW + s] + lane;
#pragma unroll
            for (int i = 0; i < EPL; ++i) {
                const float k = to_f(pk[s][i]), r = to_f(pr[s][i]), w = exp2f(pw[s][i]), u = k * inv;
                const float au = delta_rate(to_f(pa[s][i]) + bias[i]) * u;
                dst[32 * i] = u;
                dst[DP + 32 * i] = r * w;
                dst[2 * DP + 32 * i] = w;
                dst[3 * DP + 32 * i] = au;
                dst[4 * DP + 32 * i] = k;
                rau += r * au;
                rk += r * k;
            }
            rau = warp_sum(rau);
            rk = warp_sum(rk);
            if (lane == 0) sm.dots[b][warp * TPW + s] = make_float2(rau, rk);
        }
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            const int x = threadIdx.x + i * THREADS;
            if (x < CT * COLS) sm.v[b][x / COLS][x % COLS] = to_f(pv[i]);
        }
    };
    // the sum a lane ends up with: y of column `which`, or z of column `which - CPT`
    constexpr int SPAN = LPC / NV;
    const int which = g / SPAN, mine = which % CPT, base = lane - g;
    auto run = [&](int b, int count) {
        for (int t = 0; t < count; ++t) {
            const float4* p = reinterpret_cast<const float4*>(sm.vec[b][t]) + g;
            F2 y[CPT], z[CPT];
#pragma unroll
            for (int c = 0; c < CPT; ++c) y[c] = z[c] = f2(0.f);
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const float4 u = p[LPC * i], rw = p[DP / 4 + LPC * i];
                const F2 u0 = f2(u.x, u.y), u1 = f2(u.z, u.w), w0 = f2(rw.x, rw.y), w1 = f2(rw.z, rw.w);
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    y[c] = fma2(u1, S[c][2 * i + 1], fma2(u0, S[c][2 * i], y[c]));
                    z[c] = fma2(w1, S[c][2 * i + 1], fma2(w0, S[c][2 * i], z[c]));
                }
            }
            float x[NV];
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                float lo, hi;
                unpack2(y[c], lo, hi);
                x[c] = lo + hi;
                unpack2(z[c], lo, hi);
                x[CPT + c] = lo + hi;
            }
            const float sum = halving_sum<NV, LPC>(x, g);
            float v[CPT], gone[CPT], my_v = 0.f, my_y = 0.f;
#pragma unroll
            for (int c = 0; c < CPT; ++c) {
                v[c] = sm.v[b][t][cl + c];
                gone[c] = __shfl_sync(0xffffffffu, sum, base + c * SPAN);
                if (c == mine) { my_v = v[c]; my_y = gone[c]; }
            }
            if (which >= CPT && g % SPAN == 0) {
                const float2 dots = sm.dots[b][t];
                sm.o[b][t][cl + mine] = sum - dots.x * my_y + dots.y * my_v;
            }
#pragma unroll
            for (int i = 0; i < R / 4; ++i) {
                const float4 w = p[2 * DP / 4 + LPC * i], au = p[3 * DP / 4 + LPC * i], k = p[4 * DP / 4 + LPC * i];
                const F2 w0 = f2(w.x, w.y), w1 = f2(w.z, w.w), a0 = f2(au.x, au.y), a1 = f2(au.z, au.w), k0 = f2(k.x, k.y), k1 = f2(k.z, k.w);
#pragma unroll
                for (int c = 0; c < CPT; ++c) {
                    const F2 ny = f2(-gone[c]), vv = f2(v[c]);
                    S[c][2 * i] = fma2(a0, ny, fma2(w0, S[c][2 * i], mul2(k0, vv)));
                    S[c][2 * i + 1] = fma2(a1, ny, fma2(w1, S[c][2 * i + 1], mul2(k1, vv)));
                }
            }
        }
    };
    auto flush = [&](int b, int t0, int count) {
        for (int x = threadIdx.x; x < count * COLS; x += THREADS) {
            const int cc = blockIdx.z * COLS + x % COLS;
            if (cc < a.dim) O[(size_t)(t0 + x / COLS) * step + cc] = sm.o[b][x / COLS][x % COLS];
        }
    };
    load(0);
    prepare(0);
    __syncthreads();
    int b = 0;
    for (int t0 = 0; t0 < len; t0 += CT, b ^= 1) {
        const bool more = t0 + CT < len;
        if (more) load(t0 + CT);
        run(b, min(CT, len - t0));
        if (more) prepare(b ^ 1);
        __syncthreads();
        flush(b, t0, min(CT, len - t0));       // written again two rounds on, past the next barrier
    }
#pragma unroll
    for (int c = 0; c < CPT; ++c)
#pragma unroll
        for (int i = 0; i < R / 2; ++i) {
            const int d = 4 * (g + LPC * (i / 2)) + 2 * (i & 1);
            float lo, hi;
            unpack2(S[c][i], lo, hi);
            if (c0 + c >= a.dim) continue;
            if (d < a.dim) sp[(size_t)d * a.dim + c0 + c] = lo;
            if (d + 1 < a.dim) sp[(size_t)(d + 1) * a.dim + c0 + c] = hi;
        }
}

// ----------------------------------------------------------------- chunked
// Sixteen tokens from a state S0. With G_t the product of the decays up to t and
//   c_t = G_(t-1) u_t,  R_t = G_t r_t,  K_t = k_t / G_t,  B_t = (a_t u_t) / G_t      (1 / G_t <= e^9.8: decays are at least 0.54)
// the rows p_t = u_t^T S_(t-1) that the tokens remove solve p_t + sum_(s < t) (c_t.B_s) p_s = c_t S0 + sum_(s < t) (c_t.K_s) v_s, and
//   o_t = R_t S0 + sum_(s <= t) (R_t.K_s) v_s - (R_t.B_s) p_s,    S_16 = G_16 (S0 + sum_s K_s v_s^T - B_s p_s^T).
//   delta_piece   all pieces at once: those vectors, the four 16 x 16 score matrices, the inverse of the triangular one
//   delta_walk    piece by piece: a warp holds 16 value columns of S0 transposed, [columns][keys], as the accumulators of the
//                 update, which are at the same time the A operand of c S0 and R S0 (a key step's columns t and t + 4 stand for the
//                 keys 2 t and 2 t + 1); the next piece is on its way meanwhile
// The state stays 32-bit; product operands are rounded to tf32.
constexpr int DC_T = 16, DC_WARPS = 4, DC_COLS = DC_WARPS * 16, DC_SMALL = 24;

template <int DP>
struct DeltaPiece {
    static constexpr int XP = DP + 8, KP = DP + 4;          // pitches: fragment reads hit 32 banks
    float x[2 * DC_T][XP];                                  // c, then R
    float k[DC_T][KP], b[DC_T][KP];
    float m[DC_T][DC_SMALL], q[DC_T][DC_SMALL], nb[DC_T][DC_SMALL], t[DC_T][DC_SMALL];   // c.K, R.K, -R.B, inverse less 1
    float g[DP];
};

template <int DP>
__global__ void __launch_bounds__(128) delta_piece_kernel(const DeltaArgs a) {
    using Piece = DeltaPiece<DP>;
    extern __shared__ __align__(16) uint8_t raw[];
    Piece& B = *reinterpret_cast<Piece*>(raw);
    __shared__ __align__(16) float l[DC_T][DC_T + 4];       // c.B
    __shared__ float squares[4][DC_T];
    const int pc = blockIdx.x, h = blockIdx.y, hw = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3, d = threadIdx.x;
    const int row0 = a.chunk_start[pc], len = min(DC_T, a.qo_indptr[a.chunk_req[pc] + 1] - row0);
    const bool own = d < a.dim;
    const size_t step = (size_t)a.heads * a.dim, at0 = (size_t)row0 * a.ld + h * a.dim + d;
    const float* W = a.log_decay + (size_t)row0 * step + h * a.dim + d;
    const bf16 none = __float2bfloat16(0.f);
    bf16 pk[DC_T], pr[DC_T], pa[DC_T];
    float pw[DC_T], sq[DC_T];
#pragma unroll
    for (int s = 0; s < DC_T; ++s) {
        const bool ok = own && s < len;
        const size_t at = at0 + (size_t)s * a.ld;
        pk[s] = ok ? static_cast<const bf16*>(a.k)[at] : none;
        pr[s] = ok ? static_cast<const bf16*>(a.r)[at] : none;
        pa[s] = ok ? static_cast<const bf16*>(a.a)[at] : none;
        pw[s] = ok ? W[s * step] : 0.f;
    }
#pragma unroll
    for (int s = 0; s < DC_T; ++s) sq[s] = to_f(pk[s]) * to_f(pk[s]);
    const float part = halving_sum<DC_T, 32>(sq, lane);     // of token lane / 2
    if ((lane & 1) == 0) squares[hw][lane >> 1] = part;
    __syncthreads();
    const float inv = 1.f / sqrtf(squares[0][lane & 15] + squares[1][lane & 15] + squares[2][lane & 15] + squares[3][lane & 15] + 1e-6f);
    const float bias = own ? a.a_bias[h * a.dim + d] : 0.f;
    float sum = 0.f, before = 1.f;
#pragma unroll
    for (int s = 0; s < DC_T; ++s) {
        const float unit = __shfl_sync(0xffffffffu, inv, s);
        if (d >= DP) continue;
        sum += pw[s];
        const float now = exp2f(sum), back = exp2f(-sum), k = to_f(pk[s]), u = k * unit;
        B.x[s][d] = tf32_f(before * u);
        B.x[DC_T + s][d] = tf32_f(now * to_f(pr[s]));
        B.k[s][d] = tf32_f(back * k);
        B.b[s][d] = tf32_f(back * u * __fdividef(1.f, 1.f + __expf(-(to_f(pa[s]) + bias))));
        before = now;
    }
    if (d < DP) B.g[d] = before;
    __syncthreads();
    // scores: this warp's eight keys (K of tokens 0-7, 8-15, then B) against c and R
    float acc[2][4];
#pragma unroll
    for (int i = 0; i < 2; ++i) acc[i][0] = acc[i][1] = acc[i][2] = acc[i][3] = 0.f;
    const float* row = (hw < 2 ? B.k : B.b)[(hw & 1) * 8 + g];
#pragma unroll
    for (int j = 0; j < DP / 8; ++j) {
        const float2 f = *reinterpret_cast<const float2*>(row + j * 8 + 2 * t);
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const float2 x0 = *reinterpret_cast<const float2*>(&B.x[i * DC_T + g][j * 8 + 2 * t]);
            const float2 x1 = *reinterpret_cast<const float2*>(&B.x[i * DC_T + g + 8][j * 8 + 2 * t]);
            const float fa[4] = {x0.x, x1.x, x0.y, x1.y};
            mma_tf32(acc[i], fa, f.x, f.y);
        }
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const int i = g + (e >> 1) * 8, s = (hw & 1) * 8 + 2 * t + (e & 1);
        const float c = s < i ? acc[0][e] : 0.f, r = s <= i ? acc[1][e] : 0.f;
        if (hw < 2) {
            B.m[i][s] = tf32_f(c);
            B.q[i][s] = tf32_f(r);
        } else {
            l[i][s] = c;
            B.nb[i][s] = tf32_f(-r);
        }
    }
    __syncthreads();
    if (hw == 0) {
        // column `lane` of the inverse of 1 + l
        float y[DC_T];
#pragma unroll
        for (int i = 0; i < DC_T; ++i) {
            float z0 = i == lane ? 1.f : 0.f, z1 = 0.f;
#pragma unroll
            for (int s = 0; s < i; ++s) {
                if (s & 1) z1 -= l[i][s] * y[s];
                else z0 -= l[i][s] * y[s];
            }
            y[i] = z0 + z1;
            if (lane < DC_T) B.t[i][lane] = i > lane ? tf32_f(y[i]) : 0.f;
        }
    }
    __syncthreads();
    float4* dst = reinterpret_cast<float4*>(static_cast<Piece*>(a.pieces) + (size_t)pc * a.heads + h);
    const float4* src = reinterpret_cast<const float4*>(raw);
    for (int i = threadIdx.x; i < (int)(sizeof(Piece) / 16); i += 128) dst[i] = src[i];
}

__device__ __forceinline__ void copy16(void* dst, const void* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src));
}

template <int DP>
__global__ void __launch_bounds__(DC_WARPS * 32) delta_walk_kernel(const DeltaArgs a) {
    using Piece = DeltaPiece<DP>;
    constexpr int NT = DP / 8;
    extern __shared__ __align__(16) uint8_t raw[];
    Piece* buf = reinterpret_cast<Piece*>(raw);
    const int q = blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int first = a.qo_indptr[q], len = a.qo_indptr[q + 1] - first, slot = a.slots[q];
    if (len <= 0 || slot < 0) return;
    const int pieces = (len + DC_T - 1) / DC_T, c0 = blockIdx.z * DC_COLS + warp * 16;
    const Piece* src = static_cast<const Piece*>(a.pieces) + (size_t)a.req_chunks[q] * a.heads + h;
    auto fetch = [&](int pc) {
        const uint8_t* from = reinterpret_cast<const uint8_t*>(src + (size_t)pc * a.heads);
        uint8_t* to = reinterpret_cast<uint8_t*>(buf + (pc & 1));
        for (int i = threadIdx.x * 16; i < (int)sizeof(Piece); i += DC_WARPS * 32 * 16) copy16(to + i, from + i);
    };
    // values of a piece as A operands: [key step][token 2 t | 2 t + 1, column g | g + 8]
    const bf16* V = static_cast<const bf16*>(a.v) + (size_t)first * a.ld + h * a.dim;
    bf16 pv[2][4];
    auto values = [&](int pc) {
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int tok = pc * DC_T + j * 8 + 2 * t + (e >> 1), c = c0 + g + (e & 1) * 8;
                pv[j][e] = tok < len && c < a.dim ? V[(size_t)tok * a.ld + c] : __float2bfloat16(0.f);
            }
    };
    fetch(0);
    asm volatile("cp.async.commit_group;\n");
    values(0);
    float* sp = a.state + (size_t)slot * a.slot_stride + (size_t)h * a.dim * a.dim;
    const size_t step = (size_t)a.heads * a.dim;
    float* O = a.out + ((size_t)first * a.heads + h) * a.dim;
    const bool fresh = a.reset[q] != 0;
    float S[NT][4];
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = j * 8 + 2 * t + (e & 1), c = c0 + g + (e >> 1) * 8;
            S[j][e] = !fresh && d < a.dim && c < a.dim ? sp[(size_t)d * a.dim + c] : 0.f;
        }
    for (int pc = 0; pc < pieces; ++pc) {
        if (pc + 1 < pieces) fetch(pc + 1);
        asm volatile("cp.async.commit_group;\n");
        float va[2][4];
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) va[j][e] = to_f(pv[j][e]);
        if (pc + 1 < pieces) values(pc + 1);
        asm volatile("cp.async.wait_group 1;\n" ::: "memory");
        __syncthreads();
        const Piece& B = buf[pc & 1];
        float x[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i) x[i][0] = x[i][1] = x[i][2] = x[i][3] = 0.f;
#pragma unroll
        for (int j = 0; j < NT; ++j) {
            const float fa[4] = {tf32_f(S[j][0]), tf32_f(S[j][2]), tf32_f(S[j][1]), tf32_f(S[j][3])};
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float2 f = *reinterpret_cast<const float2*>(&B.x[i * 8 + g][j * 8 + 2 * t]);
                mma_tf32(x[i], fa, f.x, f.y);
            }
        }
        float ya[2][4], p[2][4];
        auto lower = [&](float (&acc)[4], const float (&m)[DC_T][DC_SMALL], int i, int j, const float (&fa)[4]) {
            const float2 f = *reinterpret_cast<const float2*>(&m[i * 8 + g][j * 8 + 2 * t]);
            mma_tf32(acc, fa, f.x, f.y);
        };
        auto operand = [&](float (&fa)[4], const float (&acc)[4]) {
            fa[0] = tf32_f(acc[0]); fa[1] = tf32_f(acc[2]); fa[2] = tf32_f(acc[1]); fa[3] = tf32_f(acc[3]);
        };
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j <= i; ++j) {
                lower(x[i], B.m, i, j, va[j]);
                lower(x[2 + i], B.q, i, j, va[j]);
            }
#pragma unroll
        for (int j = 0; j < 2; ++j) {
#pragma unroll
            for (int e = 0; e < 4; ++e) p[j][e] = x[j][e];
            operand(ya[j], x[j]);
        }
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j <= i; ++j) lower(p[i], B.t, i, j, ya[j]);
        operand(ya[0], p[0]);
        operand(ya[1], p[1]);
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int j = 0; j <= i; ++j) lower(x[2 + i], B.nb, i, j, ya[j]);
#pragma unroll
        for (int i = 0; i < 2; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int tok = pc * DC_T + i * 8 + 2 * t + (e & 1), c = c0 + g + (e >> 1) * 8;
                if (tok < len && c < a.dim) O[(size_t)tok * step + c] = x[2 + i][e];
                ya[i][e] = -ya[i][e];
            }
#pragma unroll
        for (int n = 0; n < NT; ++n) {
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                mma_tf32(S[n], va[j], B.k[j * 8 + 2 * t][n * 8 + g], B.k[j * 8 + 2 * t + 1][n * 8 + g]);
                mma_tf32(S[n], ya[j], B.b[j * 8 + 2 * t][n * 8 + g], B.b[j * 8 + 2 * t + 1][n * 8 + g]);
            }
            const float2 f = *reinterpret_cast<const float2*>(&B.g[n * 8 + 2 * t]);
            S[n][0] *= f.x; S[n][1] *= f.y; S[n][2] *= f.x; S[n][3] *= f.y;
        }
        __syncthreads();
    }
#pragma unroll
    for (int j = 0; j < NT; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = j * 8 + 2 * t + (e & 1), c = c0 + g + (e >> 1) * 8;
            if (d < a.dim && c < a.dim) sp[(size_t)d * a.dim + c] = S[j][e];
        }
}

}  // namespace pie

using namespace pie;

static bool delta_ok(const DeltaArgs& a) {
    return a.dim > 0 && a.dim <= 512 && a.heads > 0 && a.a_bias && a.log_decay && a.state;
}

// One token per request.
PIE_API int pie_delta_step(const DeltaArgs* args, int f32, cudaStream_t st) {
    const DeltaArgs& a = *args;
    if (a.n <= 0 || a.reqs <= 0) return 0;
    if (!delta_ok(a)) return (int)cudaErrorInvalidValue;
    const bool vec = a.dim % 4 == 0 && a.dim >= 64 && a.dim <= 256 && a.slot_stride % 4 == 0 && ((uintptr_t)a.state & 15) == 0 &&
                     ((uintptr_t)a.v & 15) == 0 && a.ld % 4 == 0;
    const int cols = vec ? 128 : 32, rpt = (a.dim + 7) / 8;
    const dim3 grid(a.reqs, a.heads, (a.dim + cols - 1) / cols);
#define GO(T_, R_, V_) return (int)launch_pdl(delta_step_kernel<T_, R_, V_>, grid, dim3(256), 0, st, a)
#define GO_R(T_)                            \
    if (vec) {                              \
        if (rpt <= 8) GO(T_, 8, 4);         \
        if (rpt <= 16) GO(T_, 16, 4);       \
        GO(T_, 32, 4);                      \
    }                                       \
    if (rpt <= 4) GO(T_, 4, 1);             \
    if (rpt <= 8) GO(T_, 8, 1);             \
    if (rpt <= 16) GO(T_, 16, 1);           \
    if (rpt <= 32) GO(T_, 32, 1);           \
    GO(T_, 64, 1)
    if (f32) { GO_R(float); }
    GO_R(bf16);
#undef GO_R
#undef GO
}

// Bytes of one piece of one head in the chunked form; 0: no such form for this head size.
PIE_API int pie_delta_piece_bytes(int dim) {
    if (dim <= 0 || dim > 128) return 0;
    return dim <= 32 ? (int)sizeof(DeltaPiece<32>) : dim <= 64 ? (int)sizeof(DeltaPiece<64>) : (int)sizeof(DeltaPiece<128>);
}
PIE_API int pie_delta_piece_tokens() { return DC_T; }

// Prompts in bf16, head sizes with a piece.
PIE_API int pie_delta_chunked(const DeltaArgs* args, cudaStream_t st) {
    const DeltaArgs& a = *args;
    if (a.n <= 0 || a.reqs <= 0 || a.chunks <= 0) return 0;
    if (!delta_ok(a) || a.dim > 128 || !a.pieces || !a.chunk_req || !a.chunk_start || !a.req_chunks) return (int)cudaErrorInvalidValue;
    const dim3 grid(a.reqs, a.heads, (a.dim + DC_COLS - 1) / DC_COLS);
#define GO(D_)                                                                                                              \
    {                                                                                                                       \
        constexpr int bytes = (int)sizeof(DeltaPiece<D_>);                                                                  \
        static_assert(bytes % 16 == 0, "");                                                                                 \
        cudaError_t e = cudaFuncSetAttribute(delta_piece_kernel<D_>, cudaFuncAttributeMaxDynamicSharedMemorySize, bytes);   \
        if (e == cudaSuccess) e = cudaFuncSetAttribute(delta_walk_kernel<D_>, cudaFuncAttributeMaxDynamicSharedMemorySize, 2 * bytes); \
        if (e != cudaSuccess) return (int)e;                                                                                \
        delta_piece_kernel<D_><<<dim3(a.chunks, a.heads), 128, bytes, st>>>(a);                                             \
        delta_walk_kernel<D_><<<grid, DC_WARPS * 32, 2 * bytes, st>>>(a);                                                   \
        return (int)cudaGetLastError();                                                                                     \
    }
    if (a.dim <= 32) GO(32)
    if (a.dim <= 64) GO(64)
    GO(128)
#undef GO
}

PIE_API int pie_delta_portions(const DeltaArgs* args, int f32, cudaStream_t st) {
    const DeltaArgs& a = *args;
    if (a.n <= 0 || a.reqs <= 0) return 0;
    if (!delta_ok(a)) return (int)cudaErrorInvalidValue;
#define GO(T_, R_, L_, C_)                                                                                        \
    {                                                                                                             \
        using Smem = DeltaSmem<R_, L_, C_>;                                                                       \
        auto kern = delta_portion_kernel<T_, R_, L_, C_>;                                                         \
        const cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)sizeof(Smem)); \
        if (e != cudaSuccess) return (int)e;                                                                      \
        kern<<<dim3(a.reqs, a.heads, (a.dim + Smem::COLS - 1) / Smem::COLS), DELTA_WARPS * 32, sizeof(Smem), st>>>(a); \
        return (int)cudaGetLastError();                                                                           \
    }
#define GO_R(T_)                            \
    if (a.dim <= 32) GO(T_, 4, 8, 4)        \
    if (a.dim <= 64) GO(T_, 4, 16, 4)       \
    if (a.dim <= 128) GO(T_, 8, 16, 4)      \
    if (a.dim <= 256) GO(T_, 8, 32, 4)      \
    GO(T_, 16, 32, 2)
    if (f32) { GO_R(float) }
    GO_R(bf16)
#undef GO_R
#undef GO
}
