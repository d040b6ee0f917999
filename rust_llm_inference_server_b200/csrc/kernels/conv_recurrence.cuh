// Linear recurrences behind short causal convolutions, over a float32 state per request and head.  One set of
// kernels, three recurrences (MODE):
//
//   x      = the rows of one stacked projection: C convolved channels (q and k: n_qk heads of d each, v: nh heads of dv,
//            in any order) and nh logits b
//   q, k, v = silu(conv(x) + conv_bias): a causal convolution over the request's tokens per channel, `taps` long, the
//            last tap on the current token, zeros before the request's start
//
//   HEAD_DECAY, the gated delta rule:    q = q / sqrt(sum(q^2) + unit_eps) * q_scale, k = k / sqrt(sum(k^2) + unit_eps)
//            per head; beta = sigmoid(x_b), g = exp(-exp(A_log_h) softplus(x_a + dt_bias_h)) per head;
//            S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q                per head, S [d, dv]
//   CHANNEL_DECAY, the same with one decay a head and key channel: g = exp(-exp(A_log_h) softplus(a + dt_bias)), a and
//            dt_bias [nh, d] (a from rows of their own);  S <- diag(g) S, the rest as above
//   STATE_SPACE (the state-space dual form of Mamba-2): beta = softplus(x_b + dt_bias_h), g = exp(-exp(A_log_h) beta);
//            S <- g S + beta k v^T;  o = S^T q + D_h v
//
// (head h reads q and k of head h / (nh / n_qk)).  Everything after the projection is float32.
//
// A request's state slot holds S transposed ([nh, dv, d], a column's entries contiguous) followed by the last
// taps - 1 rows of x's convolved columns, [taps - 1, C] as float32 (exact for either element type); a request
// whose first token is in this step starts from zeros in both.
//
// prepare: one warp a (token, head of q, k or v, or head of decays), and one more a token for the numbers a head;
//          writes float32 rows [convolved channels | beta | ln g].  It reads the convolution's tail from the slot and
//          leaves it as it is.
// scan:    (steps of single tokens and short portions) columns of S evolve independently: a CTA takes (request,
//          head, 16 columns), 16 threads share a column (each a contiguous share of its entries in registers) and
//          walk the request's tokens of this step in order; the column's dot product with k is summed over the 16
//          threads by shuffles, the read-out's partial sums after each tile of tokens.  The request's CTAs also
//          move the slot's convolution tail on, a share of the channels each (every reader of the old one is
//          done: the prepare kernel has finished).
// chunks:  (steps with prompts) the same CTAs and threads take 16 tokens at a time.  With L_t the sum of ln g
//          over the chunk's tokens up to t and S0 the state before the chunk,
//              u_t = beta_t (v_t - e^{L_t} S0^T k_t) - sum_{i<t} beta_t e^{L_t - L_i} (k_t . k_i) u_i
//              o_t = e^{L_t} S0^T q_t + sum_{i<=t} e^{L_t - L_i} (q_t . k_i) u_i
//              S   = e^{L_15} S0 + sum_t e^{L_15 - L_t} k_t u_t^T
//          which is the recurrence written out (STATE_SPACE: u_t = beta_t v_t, nothing to solve).  The products with S0
//          of all 16 tokens are independent (summed over a column's 16 threads by a transposing butterfly, after which
//          thread t of the column holds token t's), the triangular system is solved beforehand for all columns, and the
//          state takes the 16 outer products at once: the chain from token to token shrinks from a shuffle reduction a
//          token to one broadcast and one multiply-add.  The dot products k_t . k_i and q_t . k_i of tokens in the
//          same chunk do not depend on S: a kernel before (gram: a warp a (token, head)) leaves them by
//          (token, tokens back).  With a decay a channel the factors e^{L_t - L_i} sit inside the dot products, so gram
//          forms them there, and also leaves e^{L_t} q_t, e^{L_t} k_t and e^{L_15 - L_t} k_t for the walk.  Every
//          exponent is a sum of ln g over tokens in between, so <= 0.
#pragma once
#include "common.cuh"
#include <math.h>

namespace convrec {
constexpr int HEAD_DECAY = 0, CHANNEL_DECAY = 1, STATE_SPACE = 2;
constexpr int MAX_D = 512;                       // head sizes of q and k up to 512 (16 entries a lane in prepare)
constexpr int MAX_TAPS = 8;
constexpr int PREP_WARPS = 4;

__device__ __forceinline__ float silu_f(float z) { return z / (1.0f + expf(-z)); }
__device__ __forceinline__ float softplus_f(float z) { return z > 20.0f ? z : log1pf(expf(z)); }

struct Seqs {
    const int* cu_seqlens;      // [B + 1] first row of every request among the step's tokens
    const int* ctx_lens;        // [B] tokens of the request once this step is done
    const int* state_slots;     // [B]
    const int* seq_of_token;    // [T]
};

// Sizes, and where the first q, k and v head lie among the convolved channels.
struct Shape {
    int nh, n_qk, d, dv, taps;
    int q_at, k_at, v_at;
    __host__ __device__ int channels() const { return 2 * n_qk * d + nh * dv; }
};

// Floats of a row that `prepare` leaves a token.
template <int MODE> __host__ __device__ __forceinline__ int act_width(const Shape& z) {
    return z.channels() + z.nh + (MODE == CHANNEL_DECAY ? z.nh * z.d : z.nh);
}

// Floats of scratch a token that the chunk kernels' predecessors leave (`gram`): 16 products k . k and 16 q . k a head
// (of q / k, or of v where the decays sit inside), then, with a delta rule, a row of 16 of the solved system a head.
template <int MODE> __host__ __device__ __forceinline__ int gram_width(const Shape& z) {
    return (MODE == CHANNEL_DECAY ? z.nh : z.n_qk) * 32 + (MODE == STATE_SPACE ? 0 : z.nh * 16);
}

// The input of channel c (of C) that lies `back` tokens before local index `li` of a request's portion that
// starts at row `row0`: from this step's rows, from the slot's tail, or zero before the request's start.
template <typename T>
__device__ __forceinline__ float conv_input(const T* __restrict__ x, long long stride, int row0, int src, int c, int C,
                                            const float* __restrict__ tail, int taps, bool fresh) {
    if (src >= 0) return to_f<T>(x[(size_t)(row0 + src) * stride + c]);
    return fresh ? 0.f : tail[(size_t)(taps - 1 + src) * C + c];
}

// ln g, kept finite so that differences of its sums are defined (e^x is 0 long before)
__device__ __forceinline__ float log_decay(float a_log, float step) { return fmaxf(-expf(a_log) * step, -1e30f); }

// x: the convolved columns of the projection's rows; b: the logits a head of the same rows; a: the decay logits (HEAD_DECAY:
// one a head; CHANNEL_DECAY: d a head), rows a_stride apart.
template <int MODE, typename T>
__global__ __launch_bounds__(PREP_WARPS * 32) void prepare_kernel(
    const T* __restrict__ x, long long stride, const T* __restrict__ bl, const T* __restrict__ al, long long a_stride,
    const float* __restrict__ conv_w, const float* __restrict__ conv_b, const float* __restrict__ a_log,
    const float* __restrict__ dt_bias, const float* __restrict__ state, long long state_stride, long long tail_off, Seqs sq,
    float* __restrict__ act, int n_units, Shape z, float unit_eps, float q_scale) {
    pdl_wait_and_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int unit = blockIdx.x * PREP_WARPS + warp;
    if (unit >= n_units) return;
    const int nh = z.nh, n_qk = z.n_qk, d = z.d, taps = z.taps;
    const int per = 2 * n_qk + nh + (MODE == CHANNEL_DECAY ? nh : 0) + 1;
    const int t = unit / per, u = unit - t * per;
    const int C = z.channels();
    float* arow = act + (size_t)t * act_width<MODE>(z);
    if (u == per - 1) {
        for (int h = lane; h < nh; h += 32) {
            const float b = to_f<T>(bl[(size_t)t * stride + h]);
            if (MODE == STATE_SPACE) {
                const float dt = softplus_f(b + dt_bias[h]);
                arow[C + h] = dt;
                arow[C + nh + h] = log_decay(a_log[h], dt);
            } else {
                arow[C + h] = 1.0f / (1.0f + expf(-b));
                if (MODE == HEAD_DECAY)
                    arow[C + nh + h] = log_decay(a_log[h], softplus_f(to_f<T>(al[(size_t)t * a_stride + h]) + dt_bias[h]));
            }
        }
        return;
    }
    if (MODE == CHANNEL_DECAY && u >= 2 * n_qk + nh) {
        const int h = u - 2 * n_qk - nh;
        const float alog = a_log[h];
        for (int j = lane; j < d; j += 32)
            arow[C + nh + h * d + j] =
                log_decay(alog, softplus_f(to_f<T>(al[(size_t)t * a_stride + h * d + j]) + dt_bias[h * d + j]));
        return;
    }
    const int b = sq.seq_of_token[t];
    const int row0 = sq.cu_seqlens[b], n = sq.cu_seqlens[b + 1] - row0;
    const int li = t - row0;
    const bool fresh = sq.ctx_lens[b] - n == 0;
    const float* tail = state + (size_t)sq.state_slots[b] * state_stride + tail_off;
    const bool of_qk = u < 2 * n_qk;
    const bool unit_norm = of_qk && MODE != STATE_SPACE;
    const int width = of_qk ? d : z.dv;
    const int c0 = u < n_qk ? z.q_at + u * d : of_qk ? z.k_at + (u - n_qk) * d : z.v_at + (u - 2 * n_qk) * z.dv;
    float ss = 0.f;
    for (int j = lane; j < width; j += 32) {
        const int c = c0 + j;
        float acc = 0.f;
        for (int k = 0; k < taps; ++k)
            acc = fmaf(conv_w[(size_t)c * taps + k], conv_input<T>(x, stride, row0, li - (taps - 1 - k), c, C, tail, taps, fresh), acc);
        if (conv_b != nullptr) acc += conv_b[c];
        const float y = silu_f(acc);
        ss = fmaf(y, y, ss);
        arow[c] = y;
    }
    if (unit_norm) {                               // every lane scales what it wrote itself
        ss = warp_sum(ss);
        const float r = (u < n_qk ? q_scale : 1.0f) / sqrtf(ss + unit_eps);
        for (int j = lane; j < width; j += 32) arow[c0 + j] *= r;
    }
}

constexpr int COLS = 16, SLICES = 16, MAX_E = 32;
constexpr int THREADS = COLS * SLICES;

// The tail of the convolution after this step: the last taps - 1 inputs of the request, the channels shared out among
// the request's CTAs (a channel's old tail is read by the thread that replaces it).
template <typename T, int NT>
__device__ __forceinline__ void move_tail(float* __restrict__ tail, const T* __restrict__ x, long long stride, int row0, int n,
                                          int C, int taps, bool fresh, int first_cta, int n_ctas) {
    for (int c = first_cta * NT + threadIdx.x; c < C; c += n_ctas * NT) {
        float nv[MAX_TAPS - 1];
#pragma unroll
        for (int j = 0; j < MAX_TAPS - 1; ++j)
            nv[j] = j < taps - 1 ? conv_input<T>(x, stride, row0, n - (taps - 1) + j, c, C, tail, taps, fresh) : 0.f;
#pragma unroll
        for (int j = 0; j < MAX_TAPS - 1; ++j)
            if (j < taps - 1) tail[(size_t)j * C + c] = nv[j];
    }
}

// A thread's entries i0 .. i0 + E - 1 of a column of S (those at or beyond d are zero and stay unwritten); `quads`: d is
// a multiple of 4 and the column starts on a 16-byte boundary.
template <int E>
__device__ __forceinline__ void load_column(float (&s)[E], const float* __restrict__ S, int i0, int d, bool there, bool quads) {
    if (quads) {
#pragma unroll
        for (int e = 0; e < E; e += 4) {
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
            if (there && i0 + e < d) v = *reinterpret_cast<const float4*>(S + i0 + e);
            s[e] = v.x; s[e + 1] = v.y; s[e + 2] = v.z; s[e + 3] = v.w;
        }
    } else {
#pragma unroll
        for (int e = 0; e < E; ++e) s[e] = there && i0 + e < d ? S[i0 + e] : 0.f;
    }
}
template <int E>
__device__ __forceinline__ void store_column(const float (&s)[E], float* __restrict__ S, int i0, int d, bool quads) {
    if (quads) {
#pragma unroll
        for (int e = 0; e < E; e += 4)
            if (i0 + e < d) *reinterpret_cast<float4*>(S + i0 + e) = make_float4(s[e], s[e + 1], s[e + 2], s[e + 3]);
    } else {
#pragma unroll
        for (int e = 0; e < E; ++e)
            if (i0 + e < d) S[i0 + e] = s[e];
    }
}

// E = entries of a column that one thread holds (a multiple of 4; thread `slice` owns slice * E .. + E - 1).
template <int MODE, typename T, int E>
__global__ __launch_bounds__(THREADS) void scan_kernel(
    const float* __restrict__ act, float* __restrict__ out, float* __restrict__ state, long long state_stride,
    long long tail_off, const T* __restrict__ x, long long stride, const float* __restrict__ skip, Seqs sq, Shape z) {
    pdl_wait();     // (the next kernel is let in at the end: this one runs long on few warps)
    constexpr bool VEC = MODE == CHANNEL_DECAY;    // a third staged array: the decays
    constexpr int TOK = VEC ? (E > 16 ? 4 : E > 4 ? 8 : 16) : (E > 8 ? 8 : 16);
    constexpr int DP = SLICES * E;
    constexpr int ES = E + 4;                      // shares sit 4 floats apart: no bank conflicts
    constexpr int DPS = SLICES * ES;
    __shared__ __align__(16) float qs[TOK * DPS];
    __shared__ __align__(16) float ks[TOK * DPS];
    __shared__ __align__(16) float as[VEC ? TOK * DPS : 4];
    __shared__ float vs[TOK * COLS];
    __shared__ float bg[TOK * 2];
    __shared__ __align__(16) float os[TOK * COLS * SLICES];
    const int nh = z.nh, n_qk = z.n_qk, d = z.d, dv = z.dv;
    const int b = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS;
    const int row0 = sq.cu_seqlens[b], n = sq.cu_seqlens[b + 1] - row0;
    const int slice = threadIdx.x % SLICES, col = threadIdx.x / SLICES;
    const bool live = c0 + col < dv;
    const bool fresh = sq.ctx_lens[b] - n == 0;
    float* slot = state + (size_t)sq.state_slots[b] * state_stride;
    const int C = z.channels();
    const int AW = act_width<MODE>(z);
    if (z.taps > 1)
        move_tail<T, THREADS>(slot + tail_off, x, stride, row0, n, C, z.taps, fresh, h * gridDim.z + blockIdx.z, nh * gridDim.z);
    float* S = slot + ((size_t)h * dv + c0 + col) * d;     // this thread's column: d contiguous entries
    const int hq = h / (nh / n_qk);
    const int q_col = z.q_at + hq * d, k_col = z.k_at + hq * d, v_col = z.v_at + h * dv;
    const bool quads = ((d | (int)(state_stride & 3)) & 3) == 0;
    float s[E];
    load_column<E>(s, S, slice * E, d, !fresh && live, quads);
    constexpr int PER = TOK * DP / THREADS;
    float rq[PER], rk[PER], ra[VEC ? PER : 1], rv;
    float rb = 0.f;
    auto fetch = [&](int t0) {
        const int nt = min(TOK, n - t0);
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int idx = threadIdx.x + j * THREADS, tt = idx / DP, i = idx - tt * DP;
            const bool ok = tt < nt && i < d;
            const float* r = act + (size_t)(row0 + t0 + (ok ? tt : 0)) * AW + (ok ? i : 0);
            rq[j] = ok ? r[q_col] : 0.f;
            rk[j] = ok ? r[k_col] : 0.f;
            if (VEC) ra[j] = ok ? r[C + nh + h * d] : 0.f;
        }
        {
            const int tt = threadIdx.x / COLS, c = threadIdx.x - tt * COLS;     // TOK * COLS <= THREADS
            const bool ok = tt < nt && c0 + c < dv;
            rv = ok ? act[(size_t)(row0 + t0 + tt) * AW + v_col + c0 + c] : 0.f;
        }
        if (threadIdx.x < 2 * TOK) {
            const int tt = threadIdx.x >> 1, which = threadIdx.x & 1;
            rb = tt < nt && !(VEC && which) ? act[(size_t)(row0 + t0 + tt) * AW + C + which * nh + h] : 0.f;
            if (which) rb = expf(rb);       // g from ln g
        }
    };
    if (n > 0) fetch(0);
    for (int t0 = 0; t0 < n; t0 += TOK) {
        const int nt = min(TOK, n - t0);
        __syncthreads();
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int idx = threadIdx.x + j * THREADS, tt = idx / DP, i = idx - tt * DP;
            const int at = tt * DPS + (i / E) * ES + i % E;
            qs[at] = rq[j];
            ks[at] = rk[j];
            if (VEC) as[at] = expf(ra[j]);
        }
        if (threadIdx.x < TOK * COLS) vs[threadIdx.x] = rv;
        if (threadIdx.x < 2 * TOK) bg[threadIdx.x] = rb;
        __syncthreads();
        if (t0 + TOK < n) fetch(t0 + TOK);
#pragma unroll 2
        for (int tt = 0; tt < nt; ++tt) {
            const float v = vs[tt * COLS + col];
            const float beta = bg[2 * tt], g = bg[2 * tt + 1];
            const float4* kr = reinterpret_cast<const float4*>(ks + tt * DPS + slice * ES);
            const float4* qr = reinterpret_cast<const float4*>(qs + tt * DPS + slice * ES);
            const float4* ar = reinterpret_cast<const float4*>(as + (VEC ? tt * DPS + slice * ES : 0));
            float4 k4[E / 4];
            float p[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int e4 = 0; e4 < E / 4; ++e4) {
                k4[e4] = kr[e4];
                if (VEC) {
                    const float4 a4 = ar[e4];
                    s[4 * e4 + 0] *= a4.x;
                    s[4 * e4 + 1] *= a4.y;
                    s[4 * e4 + 2] *= a4.z;
                    s[4 * e4 + 3] *= a4.w;
                }
                if (MODE != STATE_SPACE) {
                    p[0] = fmaf(s[4 * e4 + 0], k4[e4].x, p[0]);
                    p[1] = fmaf(s[4 * e4 + 1], k4[e4].y, p[1]);
                    p[2] = fmaf(s[4 * e4 + 2], k4[e4].z, p[2]);
                    p[3] = fmaf(s[4 * e4 + 3], k4[e4].w, p[3]);
                }
            }
            float u;
            if (MODE == STATE_SPACE) {
                u = beta * v;
            } else {
                float dot = (p[0] + p[1]) + (p[2] + p[3]);
#pragma unroll
                for (int o = SLICES / 2; o > 0; o >>= 1) dot += __shfl_xor_sync(0xffffffffu, dot, o);    // the column's 16 threads
                // a decay a head: S^T k of the decayed state is g times that of the old one
                u = VEC ? beta * (v - dot) : beta * (v - g * dot);
            }
            float o4[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int e4 = 0; e4 < E / 4; ++e4) {
                const float4 q4 = qr[e4];
                if (VEC) {
                    s[4 * e4 + 0] = fmaf(k4[e4].x, u, s[4 * e4 + 0]);
                    s[4 * e4 + 1] = fmaf(k4[e4].y, u, s[4 * e4 + 1]);
                    s[4 * e4 + 2] = fmaf(k4[e4].z, u, s[4 * e4 + 2]);
                    s[4 * e4 + 3] = fmaf(k4[e4].w, u, s[4 * e4 + 3]);
                } else {
                    s[4 * e4 + 0] = fmaf(g, s[4 * e4 + 0], k4[e4].x * u);
                    s[4 * e4 + 1] = fmaf(g, s[4 * e4 + 1], k4[e4].y * u);
                    s[4 * e4 + 2] = fmaf(g, s[4 * e4 + 2], k4[e4].z * u);
                    s[4 * e4 + 3] = fmaf(g, s[4 * e4 + 3], k4[e4].w * u);
                }
                o4[0] = fmaf(s[4 * e4 + 0], q4.x, o4[0]);
                o4[1] = fmaf(s[4 * e4 + 1], q4.y, o4[1]);
                o4[2] = fmaf(s[4 * e4 + 2], q4.z, o4[2]);
                o4[3] = fmaf(s[4 * e4 + 3], q4.w, o4[3]);
            }
            os[(tt * COLS + col) * SLICES + slice] = (o4[0] + o4[1]) + (o4[2] + o4[3]);
        }
        __syncthreads();
        for (int idx = threadIdx.x; idx < nt * COLS; idx += THREADS) {
            const int tt = idx / COLS, c = idx - tt * COLS;
            const float4* p4 = reinterpret_cast<const float4*>(os + idx * SLICES);
            float sum = 0.f;
#pragma unroll
            for (int j = 0; j < SLICES / 4; ++j) {
                const float4 a = p4[j];
                sum += (a.x + a.y) + (a.z + a.w);
            }
            if (MODE == STATE_SPACE) sum = fmaf(skip[h], vs[idx], sum);
            if (c0 + c < dv) out[(size_t)(row0 + t0 + tt) * nh * dv + h * dv + c0 + c] = sum;
        }
    }
    if (live) store_column<E>(s, S, slice * E, d, quads);
    pdl_trigger();
}

// ---- steps with prompts: 16 tokens at a time ------------------------------------------------------------------
constexpr int CH = 16;                 // tokens a chunk; equal to SLICES, so thread t of a column takes token t
constexpr int MS = CH + 4;             // row stride of the chunk's 16 x 16 matrices: rows read by 16-byte loads
constexpr int GRAM_WARPS = 4;

// gram[t][hq][0][j] = k_t . k_{t-j},  gram[t][hq][1][j] = q_t . k_{t-j}  for the tokens t - j of t's own chunk
// (chunks count from the first row of the request's portion); entries of other chunks are left as they are.
// STATE_SPACE needs q . k only.
template <int MODE>
__global__ __launch_bounds__(GRAM_WARPS * 32) void gram_kernel(const float* __restrict__ act, float* __restrict__ gram, Seqs sq,
                                                               int n_units, Shape z) {
    pdl_wait();     // no early trigger: the chunk kernel's few CTAs are to find the SMs empty, one each
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int unit = blockIdx.x * GRAM_WARPS + warp;
    if (unit >= n_units) return;
    const int d = z.d;
    const int t = unit / z.n_qk, hq = unit - t * z.n_qk;
    const int b = sq.seq_of_token[t];
    const int back = (t - sq.cu_seqlens[b]) & (CH - 1);
    const int AW = act_width<MODE>(z);
    const float* qt = act + (size_t)t * AW + z.q_at + hq * d;
    const float* kt = act + (size_t)t * AW + z.k_at + hq * d;
    float qr[MAX_D / 32], kr[MAX_D / 32];
#pragma unroll
    for (int i = 0; i < MAX_D / 32; ++i) {
        const int e = lane + 32 * i;
        qr[i] = e < d ? qt[e] : 0.f;
        kr[i] = MODE != STATE_SPACE && e < d ? kt[e] : 0.f;
    }
    float* g = gram + (size_t)t * gram_width<MODE>(z) + hq * 2 * CH;
    for (int j = 0; j <= back; ++j) {
        const float* ki = kt - (size_t)j * AW;
        float a = 0.f, c = 0.f;
#pragma unroll
        for (int i = 0; i < MAX_D / 32; ++i) {
            const int e = lane + 32 * i;
            const float kv = e < d ? ki[e] : 0.f;
            if (MODE != STATE_SPACE) a = fmaf(kr[i], kv, a);
            c = fmaf(qr[i], kv, c);
        }
        if (MODE != STATE_SPACE) a = warp_sum(a);
        c = warp_sum(c);
        if (lane == 0) {
            if (MODE != STATE_SPACE) g[j] = a;
            g[CH + j] = c;
        }
    }
}

// CHANNEL_DECAY: a warp a (token, head).  gram[t][h][0][j] = sum_c k_t[c] k_{t-j}[c] e^{L_t[c] - L_{t-j}[c]}, gram[t][h][1][j]
// the same with q_t; scaled[t][h] = [e^{L_t} q_t | e^{L_t} k_t | e^{L_end - L_t} k_t | e^{L_end}], L counted from the
// chunk's start, `end` the last token of the chunk in this step (the last part is written by that token alone).
// NE: entries a lane.
template <int NE>
__global__ __launch_bounds__(GRAM_WARPS * 32) void gram_channel_kernel(const float* __restrict__ act, float* __restrict__ gram,
                                                                       float* __restrict__ scaled, Seqs sq, int n_units, Shape z) {
    pdl_wait();     // no early trigger, see gram_kernel
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int unit = blockIdx.x * GRAM_WARPS + warp;
    if (unit >= n_units) return;
    const int d = z.d, nh = z.nh;
    const int t = unit / nh, h = unit - t * nh;
    const int hq = h / (nh / z.n_qk);
    const int b = sq.seq_of_token[t];
    const int row0 = sq.cu_seqlens[b], n = sq.cu_seqlens[b + 1] - row0;
    const int back = (t - row0) & (CH - 1);
    const int ahead = min(CH - 1 - back, n - 1 - (t - row0));     // tokens of the chunk after this one
    const int AW = act_width<CHANNEL_DECAY>(z);
    const float* qt = act + (size_t)t * AW + z.q_at + hq * d;
    const float* kt = act + (size_t)t * AW + z.k_at + hq * d;
    const float* lt = act + (size_t)t * AW + z.channels() + nh + h * d;
    float qr[NE], kr[NE], D[NE];
#pragma unroll
    for (int i = 0; i < NE; ++i) {
        const int e = lane + 32 * i;
        qr[i] = e < d ? qt[e] : 0.f;
        kr[i] = e < d ? kt[e] : 0.f;
        D[i] = 0.f;
    }
    float* g = gram + (size_t)t * gram_width<CHANNEL_DECAY>(z) + h * 2 * CH;
    for (int j = 0; j <= back; ++j) {
        const float* ki = kt - (size_t)j * AW;
        const float* li = lt - (size_t)j * AW;
        float a = 0.f, c = 0.f;
#pragma unroll
        for (int i = 0; i < NE; ++i) {
            const int e = lane + 32 * i;
            const float kv = (e < d ? ki[e] : 0.f) * expf(D[i]);
            a = fmaf(kr[i], kv, a);
            c = fmaf(qr[i], kv, c);
            D[i] += e < d ? li[e] : 0.f;           // from here on e^{L_t - L_{t-j-1}}
        }
        a = warp_sum(a);
        c = warp_sum(c);
        if (lane == 0) {
            g[j] = a;
            g[CH + j] = c;
        }
    }
    float* sc = scaled + ((size_t)t * nh + h) * 4 * d;
    float F[NE];
#pragma unroll
    for (int i = 0; i < NE; ++i) F[i] = 0.f;
    for (int j = 1; j <= ahead; ++j) {
        const float* li = lt + (size_t)j * AW;
#pragma unroll
        for (int i = 0; i < NE; ++i) {
            const int e = lane + 32 * i;
            F[i] += e < d ? li[e] : 0.f;
        }
    }
#pragma unroll
    for (int i = 0; i < NE; ++i) {
        const int e = lane + 32 * i;
        if (e >= d) continue;
        const float el = expf(D[i]);
        sc[e] = qr[i] * el;
        sc[d + e] = kr[i] * el;
        sc[2 * d + e] = kr[i] * expf(F[i]);
        if (ahead == 0) sc[3 * d + e] = el;
    }
}

// w[t][h][i] = row (t's place in its chunk) of (I + M)^-1 for the chunk's matrix M[a][i] = beta_a e^{L_a - L_i}
// k_a . k_i (i < a; with a decay a channel the factor sits inside the product), so that the chunk's u are W (beta (v -
// e^L S0^T k)): a triangular system solved once a (token, head) for all columns, and for all chunks at once, outside the
// kernel that walks the chunks in order.
// One warp a (token, head): lane j keeps column j of the rows so far; row a = e_a - sum_{i<a} M[a][i] row_i.
template <int MODE>
__global__ __launch_bounds__(GRAM_WARPS * 32) void solve_kernel(const float* __restrict__ act, float* __restrict__ gram, Seqs sq,
                                                                int n_units, Shape z) {
    pdl_wait();     // no early trigger: the chunk kernel's few CTAs are to find the SMs empty, one each
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int unit = blockIdx.x * GRAM_WARPS + warp;
    if (unit >= n_units) return;
    const int nh = z.nh;
    const int t = unit / nh, h = unit - t * nh;
    const int hg = MODE == CHANNEL_DECAY ? h : h / (nh / z.n_qk);
    const int b = sq.seq_of_token[t];
    const int back = (t - sq.cu_seqlens[b]) & (CH - 1);
    const int C = z.channels();
    const int AW = act_width<MODE>(z), GW = gram_width<MODE>(z);
    const int r0 = t - back;                        // the chunk's first row
    const int j = lane & (CH - 1);
    const bool in = j <= back;
    const float* arow = act + (size_t)(r0 + (in ? j : 0)) * AW + C;
    const float beta = in ? arow[h] : 0.f;
    float L = 0.f;
    if (MODE == HEAD_DECAY) {
        L = in ? arow[nh + h] : 0.f;
#pragma unroll
        for (int o = 1; o < CH; o <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, L, o, CH);
            if (j >= o) L += up;
        }
    }
    float col[CH], kk[CH];                          // col[a] = W[a][j];  kk[a] = k_a . k_j
#pragma unroll
    for (int a = 0; a < CH; ++a)
        kk[a] = j < a && a <= back ? gram[(size_t)(r0 + a) * GW + hg * 2 * CH + (a - j)] : 0.f;
#pragma unroll
    for (int a = 0; a < CH; ++a) {
        col[a] = 0.f;
        if (a <= back) {                            // the same for the whole warp
            // lane i < a: M[a][i]
            const float La = MODE == HEAD_DECAY ? __shfl_sync(0xffffffffu, L, a) : 0.f;
            const float ba = __shfl_sync(0xffffffffu, beta, a);
            const float mi = j < a ? (MODE == HEAD_DECAY ? ba * expf(La - L) * kk[a] : ba * kk[a]) : 0.f;
            float acc = j == a ? 1.f : 0.f;
#pragma unroll
            for (int i = 0; i < a; ++i) acc = fmaf(-__shfl_sync(0xffffffffu, mi, i), col[i], acc);
            col[a] = acc;
        }
    }
    float mine = 0.f;
#pragma unroll
    for (int a = 0; a < CH; ++a) mine = a == back ? col[a] : mine;
    if (lane < CH) gram[(size_t)t * GW + (MODE == CHANNEL_DECAY ? nh : z.n_qk) * 2 * CH + h * CH + j] = in ? mine : 0.f;
}

// Sums a[0..15] over the 16 lanes of a half-warp; lane `slice` returns the sum of index `slice`.  Halving
// exchanges: 8 + 4 + 2 + 1 shuffles, always the same order of additions.
__device__ __forceinline__ float reduce_scatter16(float (&a)[CH], int slice) {
#pragma unroll
    for (int off = CH / 2; off >= 1; off >>= 1) {
        const bool up = (slice & off) != 0;
#pragma unroll
        for (int m = 0; m < off; ++m) {
            const float send = up ? a[m] : a[m + off];
            const float keep = up ? a[m + off] : a[m];
            a[m] = keep + __shfl_xor_sync(0xffffffffu, send, off);
        }
    }
    return a[0];
}

template <int MODE> constexpr size_t chunk_smem_floats(int E) {
    return (size_t)(MODE == CHANNEL_DECAY ? 3 : 2) * CH * SLICES * (E + 4) + CH * COLS + 2 * CH * MS + 4 * CH + COLS * (CH + 1);
}

constexpr int NC = 2;                          // columns a thread: a share of k or q read once serves both
constexpr int CGROUPS = COLS / NC;             // thread (slice, cg) holds columns cg and cg + CGROUPS
constexpr int CTHREADS = SLICES * CGROUPS;
constexpr int FT = CTHREADS / SLICES;          // tokens that the CTA's threads stage at a time

template <int MODE, typename T, int E>
__global__ __launch_bounds__(CTHREADS) void chunk_kernel(
    const float* __restrict__ act, const float* __restrict__ gram, const float* __restrict__ scaled, float* __restrict__ out,
    float* __restrict__ state, long long state_stride, long long tail_off, const T* __restrict__ x_in, long long stride,
    const float* __restrict__ skip, Seqs sq, Shape z) {
    pdl_wait();     // (the next kernel is let in at the end: this one runs long on few warps)
    constexpr bool DELTA = MODE != STATE_SPACE;
    constexpr bool VEC = MODE == CHANNEL_DECAY;    // staged: e^L q, e^L k and e^{L_15 - L} k instead of q and k
    constexpr int ES = E + 4;                      // shares sit 4 floats apart: no bank conflicts
    constexpr int DPS = SLICES * ES;
    constexpr bool AHEAD = E <= 8;                 // the next chunk's rows wait in registers while this one runs
    constexpr int GRP = E <= 8 ? 4 : 1;            // tokens whose shares are loaded before the arithmetic on them
    constexpr int NF = CH / FT;
    extern __shared__ __align__(16) float sm[];
    float* qs = sm;                                // [CH][DPS]
    float* ks = qs + CH * DPS;                     // [CH][DPS]
    float* kw = VEC ? ks + CH * DPS : ks;          // [CH][DPS] what the state takes
    float* vs = kw + CH * DPS;                     // [CH][COLS]
    float* Ws = vs + CH * COLS;                    // [CH][MS] (I + M)^-1, see solve_kernel
    float* Bs = Ws + CH * MS;                      // [CH][MS] e^{L_t - L_i} q_t . k_i, i <= t, else 0
    float* eL = Bs + CH * MS;                      // [CH] e^{L_t}
    float* wL = eL + CH;                           // [CH] e^{L_15 - L_t}
    float* bs = wL + CH;                           // [CH] beta_t
    float* Ls = bs + CH;                           // [CH] L_t
    float* os = Ls + CH;                           // [COLS][CH + 1]
    const int nh = z.nh, n_qk = z.n_qk, d = z.d, dv = z.dv;
    const int b = blockIdx.x, h = blockIdx.y, c0 = blockIdx.z * COLS;
    const int row0 = sq.cu_seqlens[b], n = sq.cu_seqlens[b + 1] - row0;
    const int slice = threadIdx.x % SLICES, cg = threadIdx.x / SLICES;
    const bool fresh = sq.ctx_lens[b] - n == 0;
    float* slot = state + (size_t)sq.state_slots[b] * state_stride;
    const int C = z.channels();
    const int AW = act_width<MODE>(z), GW = gram_width<MODE>(z);
    if (z.taps > 1)
        move_tail<T, CTHREADS>(slot + tail_off, x_in, stride, row0, n, C, z.taps, fresh, h * gridDim.z + blockIdx.z, nh * gridDim.z);
    const int hq = h / (nh / n_qk);
    const int hg = VEC ? h : hq, w_at = (VEC ? nh : n_qk) * 2 * CH;
    const int v_col = z.v_at + h * dv;
    const float d_skip = MODE == STATE_SPACE ? skip[h] : 0.f;
    const bool quads = ((d | (int)(state_stride & 3)) & 3) == 0;
    float* S[NC];                                  // this thread's columns: d contiguous entries each
    bool live[NC];
    float s[NC][E];
#pragma unroll
    for (int x = 0; x < NC; ++x) {
        live[x] = c0 + cg + x * CGROUPS < dv;
        S[x] = slot + ((size_t)h * dv + c0 + cg + x * CGROUPS) * d;
        load_column<E>(s[x], S[x], slice * E, d, !fresh && live[x], quads);
    }
    // What a thread brings to shared memory for a chunk, as thread (ft = tid / 16, fj = tid % 16), of the tokens ft,
    // ft + FT, ..: share fj of the token's q and k, its v of column fj, entry fj of its rows of W and of q . k; and in
    // warp 0 beta (lanes 0..15) or ln g (16..31) of token tid % 16.  A token past the portion's end: zeros, beta 0, g 1.
    const int ft = threadIdx.x / SLICES, fj = threadIdx.x % SLICES;
    float rq[NF][E], rk[NF][E], r3[VEC ? NF : 1][E], rv[NF], rw[NF], rgq[NF], rb = 0.f;
    float rd[VEC ? E : 1];                         // the chunk's whole decay of this thread's entries
    auto fetch = [&](int t0) {
#pragma unroll
        for (int x = 0; x < NF; ++x) {
            const int tt = ft + x * FT;
            const bool tok = t0 + tt < n;
            const size_t trow = (size_t)(row0 + t0 + (tok ? tt : 0));
            const float* arow = act + trow * AW;
            const float* grow = gram + trow * GW;
            const float* srow = VEC ? scaled + (trow * nh + h) * 4 * d : nullptr;
#pragma unroll
            for (int e = 0; e < E; ++e) {
                const int i = fj * E + e;
                const bool ok = tok && i < d;
                if (VEC) {
                    rq[x][e] = ok ? srow[i] : 0.f;
                    rk[x][e] = ok ? srow[d + i] : 0.f;
                    r3[x][e] = ok ? srow[2 * d + i] : 0.f;
                } else {
                    rq[x][e] = ok ? arow[z.q_at + hq * d + i] : 0.f;
                    rk[x][e] = ok ? arow[z.k_at + hq * d + i] : 0.f;
                }
            }
            rv[x] = tok && c0 + fj < dv ? arow[v_col + c0 + fj] : 0.f;
            if (DELTA) rw[x] = tok ? grow[w_at + h * CH + fj] : 0.f;
            rgq[x] = tok && fj <= tt ? grow[hg * 2 * CH + CH + fj] : 0.f;
        }
        if (threadIdx.x < 2 * CH) {
            const int tt = threadIdx.x & (CH - 1), which = threadIdx.x >> 4;
            rb = t0 + tt < n && !(VEC && which) ? act[(size_t)(row0 + t0 + tt) * AW + C + which * nh + h] : 0.f;
        }
        if (VEC) {
            const float* srow = scaled + ((size_t)(row0 + t0 + min(CH, n - t0) - 1) * nh + h) * 4 * d + 3 * d;
#pragma unroll
            for (int e = 0; e < E; ++e) rd[e] = slice * E + e < d ? srow[slice * E + e] : 1.f;
        }
    };
    if (AHEAD && n > 0) fetch(0);
    for (int t0 = 0; t0 < n; t0 += CH) {
        const int nt = min(CH, n - t0);
        __syncthreads();
        if (!AHEAD) fetch(t0);
#pragma unroll
        for (int x = 0; x < NF; ++x) {
            const int tt = ft + x * FT;
            float4* q4 = reinterpret_cast<float4*>(qs + tt * DPS + fj * ES);
            float4* k4 = reinterpret_cast<float4*>(ks + tt * DPS + fj * ES);
            float4* w4 = reinterpret_cast<float4*>(kw + tt * DPS + fj * ES);
#pragma unroll
            for (int e4 = 0; e4 < E / 4; ++e4) {
                q4[e4] = make_float4(rq[x][4 * e4], rq[x][4 * e4 + 1], rq[x][4 * e4 + 2], rq[x][4 * e4 + 3]);
                k4[e4] = make_float4(rk[x][4 * e4], rk[x][4 * e4 + 1], rk[x][4 * e4 + 2], rk[x][4 * e4 + 3]);
                if (VEC) w4[e4] = make_float4(r3[x][4 * e4], r3[x][4 * e4 + 1], r3[x][4 * e4 + 2], r3[x][4 * e4 + 3]);
            }
            vs[tt * COLS + fj] = rv[x];
            if (DELTA) Ws[tt * MS + fj] = rw[x];
        }
        if (threadIdx.x < 32) {
            float L = rb;                           // lanes 16..31: running sum of ln g
#pragma unroll
            for (int o = 1; o < CH; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, L, o, CH);
                if ((threadIdx.x & (CH - 1)) >= o) L += up;
            }
            const float last = __shfl_sync(0xffffffffu, L, 31);
            if (threadIdx.x < CH) bs[threadIdx.x] = rb;
            else if (!VEC) {
                const int tt = threadIdx.x - CH;
                Ls[tt] = L;
                eL[tt] = expf(L);
                wL[tt] = expf(last - L);
            }
        }
        float dec[VEC ? E : 1];
        if (VEC) {
#pragma unroll
            for (int e = 0; e < E; ++e) dec[e] = rd[e];
        }
        __syncthreads();
#pragma unroll
        for (int x = 0; x < NF; ++x) {
            const int tt = ft + x * FT, i = tt - fj;                  // fj tokens back
            if (i >= 0) Bs[tt * MS + i] = VEC ? rgq[x] : expf(Ls[tt] - Ls[i]) * rgq[x];
            else Bs[tt * MS + CH + i] = 0.f;
        }
        if (AHEAD && t0 + CH < n) fetch(t0 + CH);
        // S0^T k_t and S0^T q_t of the 16 tokens: this thread's share, then the sum over the column's threads
        float pk[DELTA ? NC : 1][CH], pq[NC][CH];
#pragma unroll
        for (int tt0 = 0; tt0 < CH; tt0 += GRP) {
            float4 kk[GRP][E / 4], qq[GRP][E / 4];
#pragma unroll
            for (int g = 0; g < GRP; ++g) {
                const float4* kr = reinterpret_cast<const float4*>(ks + (tt0 + g) * DPS + slice * ES);
                const float4* qr = reinterpret_cast<const float4*>(qs + (tt0 + g) * DPS + slice * ES);
#pragma unroll
                for (int e4 = 0; e4 < E / 4; ++e4) {
                    if (DELTA) kk[g][e4] = kr[e4];
                    qq[g][e4] = qr[e4];
                }
            }
#pragma unroll
            for (int g = 0; g < GRP; ++g) {
#pragma unroll
                for (int x = 0; x < NC; ++x) {
                    float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
#pragma unroll
                    for (int e4 = 0; e4 < E / 4; ++e4) {
                        if (DELTA) {
                            a0 = fmaf(s[x][4 * e4 + 0], kk[g][e4].x, a0);
                            a1 = fmaf(s[x][4 * e4 + 1], kk[g][e4].y, a1);
                            a0 = fmaf(s[x][4 * e4 + 2], kk[g][e4].z, a0);
                            a1 = fmaf(s[x][4 * e4 + 3], kk[g][e4].w, a1);
                        }
                        b0 = fmaf(s[x][4 * e4 + 0], qq[g][e4].x, b0);
                        b1 = fmaf(s[x][4 * e4 + 1], qq[g][e4].y, b1);
                        b0 = fmaf(s[x][4 * e4 + 2], qq[g][e4].z, b0);
                        b1 = fmaf(s[x][4 * e4 + 3], qq[g][e4].w, b1);
                    }
                    if (DELTA) pk[x][tt0 + g] = a0 + a1;
                    pq[x][tt0 + g] = b0 + b1;
                }
            }
        }
        float sk[NC], sqt[NC];
#pragma unroll
        for (int x = 0; x < NC; ++x) {
            if (DELTA) sk[x] = reduce_scatter16(pk[x], slice);        // token `slice`'s
            sqt[x] = reduce_scatter16(pq[x], slice);
        }
        __syncthreads();                                   // Bs is written
        const int t = slice;
        const float el = VEC ? 1.0f : eL[t], bt = bs[t];
        float u[NC][CH];
        if (DELTA) {
            // u_t = sum_i W[t][i] r_i, then every thread of the column takes all 16
            float w[CH];
            const float4* wr = reinterpret_cast<const float4*>(Ws + t * MS);
#pragma unroll
            for (int j = 0; j < CH / 4; ++j) {
                const float4 a = wr[j];
                w[4 * j] = a.x, w[4 * j + 1] = a.y, w[4 * j + 2] = a.z, w[4 * j + 3] = a.w;
            }
#pragma unroll
            for (int x = 0; x < NC; ++x) {
                const float r = bt * (vs[t * COLS + cg + x * CGROUPS] - el * sk[x]);
                float u0 = 0.f, u1 = 0.f;
#pragma unroll
                for (int i = 0; i < CH; i += 2) {
                    u0 = fmaf(w[i], __shfl_sync(0xffffffffu, r, i, CH), u0);
                    u1 = fmaf(w[i + 1], __shfl_sync(0xffffffffu, r, i + 1, CH), u1);
                }
                const float ut = u0 + u1;
#pragma unroll
                for (int i = 0; i < CH; ++i) u[x][i] = __shfl_sync(0xffffffffu, ut, i, CH);
            }
        } else {
#pragma unroll
            for (int i = 0; i < CH; ++i) {
                const float bi = bs[i];
#pragma unroll
                for (int x = 0; x < NC; ++x) u[x][i] = bi * vs[i * COLS + cg + x * CGROUPS];
            }
        }
        {
            float bq[CH];
            const float4* br = reinterpret_cast<const float4*>(Bs + t * MS);
#pragma unroll
            for (int j = 0; j < CH / 4; ++j) {
                const float4 a = br[j];
                bq[4 * j] = a.x, bq[4 * j + 1] = a.y, bq[4 * j + 2] = a.z, bq[4 * j + 3] = a.w;
            }
#pragma unroll
            for (int x = 0; x < NC; ++x) {
                float o0 = el * sqt[x], o1 = MODE == STATE_SPACE ? d_skip * vs[t * COLS + cg + x * CGROUPS] : 0.f;
#pragma unroll
                for (int i = 0; i < CH; i += 2) {
                    o0 = fmaf(bq[i], u[x][i], o0);
                    o1 = fmaf(bq[i + 1], u[x][i + 1], o1);
                }
                os[(cg + x * CGROUPS) * (CH + 1) + t] = o0 + o1;
            }
        }
        {
            if (VEC) {
#pragma unroll
                for (int x = 0; x < NC; ++x)
#pragma unroll
                    for (int e = 0; e < E; ++e) s[x][e] *= dec[e];
            } else {
                const float dall = eL[CH - 1];
                const float4* wr = reinterpret_cast<const float4*>(wL);
#pragma unroll
                for (int j = 0; j < CH / 4; ++j) {
                    const float4 a = wr[j];
#pragma unroll
                    for (int x = 0; x < NC; ++x)
                        u[x][4 * j] *= a.x, u[x][4 * j + 1] *= a.y, u[x][4 * j + 2] *= a.z, u[x][4 * j + 3] *= a.w;
                }
#pragma unroll
                for (int x = 0; x < NC; ++x)
#pragma unroll
                    for (int e = 0; e < E; ++e) s[x][e] *= dall;
            }
#pragma unroll
            for (int tt0 = 0; tt0 < CH; tt0 += GRP) {
                float4 kk[GRP][E / 4];
#pragma unroll
                for (int g = 0; g < GRP; ++g) {
                    const float4* kr = reinterpret_cast<const float4*>(kw + (tt0 + g) * DPS + slice * ES);
#pragma unroll
                    for (int e4 = 0; e4 < E / 4; ++e4) kk[g][e4] = kr[e4];
                }
#pragma unroll
                for (int g = 0; g < GRP; ++g) {
#pragma unroll
                    for (int x = 0; x < NC; ++x) {
#pragma unroll
                        for (int e4 = 0; e4 < E / 4; ++e4) {
                            s[x][4 * e4 + 0] = fmaf(kk[g][e4].x, u[x][tt0 + g], s[x][4 * e4 + 0]);
                            s[x][4 * e4 + 1] = fmaf(kk[g][e4].y, u[x][tt0 + g], s[x][4 * e4 + 1]);
                            s[x][4 * e4 + 2] = fmaf(kk[g][e4].z, u[x][tt0 + g], s[x][4 * e4 + 2]);
                            s[x][4 * e4 + 3] = fmaf(kk[g][e4].w, u[x][tt0 + g], s[x][4 * e4 + 3]);
                        }
                    }
                }
            }
        }
        __syncthreads();
#pragma unroll
        for (int x = 0; x < NF; ++x) {
            const int tt = ft + x * FT;
            if (tt < nt && c0 + fj < dv) out[(size_t)(row0 + t0 + tt) * nh * dv + h * dv + c0 + fj] = os[fj * (CH + 1) + tt];
        }
    }
#pragma unroll
    for (int x = 0; x < NC; ++x)
        if (live[x]) store_column<E>(s[x], S[x], slice * E, d, quads);
    pdl_trigger();
}

// What a launch gets.  x, b, a: the convolved columns, the logits a head and the decay logits of the first token, in the
// element type.  act float32 [T, act_width]; gram null: token by token, else float32 [T, gram_width] and 16 tokens at a
// time; scaled float32 [T, nh, 4 d] (CHANNEL_DECAY in chunks); out float32 [T, nh dv].
struct Args {
    const void *x, *b, *a;
    long long stride, a_stride;
    const float *conv_w, *conv_b, *a_log, *dt_bias, *skip;
    float* state;
    long long state_stride;
    Seqs sq;
    float *act, *gram, *scaled, *out;
    int n_tokens, n_seqs;
    Shape z;
    float unit_eps, q_scale;
};

// Floats of a request's state slot: S of every head, then the convolution's tail, rounded up to whole 16-byte vectors.
static inline int state_floats(int nh, int n_qk, int d, int dv, int taps) {
    return (nh * dv * d + (taps - 1) * (2 * n_qk * d + nh * dv) + 3) & ~3;
}

template <int MODE, typename T>
static int launch_typed(const Args& g, cudaStream_t stream) {
    const Shape& z = g.z;
    const long long tail_off = (long long)z.nh * z.dv * z.d;
    const long long units = (long long)g.n_tokens * (2 * z.n_qk + z.nh + (MODE == CHANNEL_DECAY ? z.nh : 0) + 1);
    if (units > 0x7fffffffLL) return RLIS_ERR_UNSUPPORTED;
    rlis_launch(prepare_kernel<MODE, T>, (unsigned)((units + PREP_WARPS - 1) / PREP_WARPS), PREP_WARPS * 32, 0, stream,
                (const T*)g.x, g.stride, (const T*)g.b, (const T*)g.a, g.a_stride, g.conv_w, g.conv_b, g.a_log, g.dt_bias,
                (const float*)g.state, g.state_stride, tail_off, g.sq, g.act, (int)units, z, g.unit_eps, g.q_scale);
    dim3 grid(g.n_seqs, z.nh, (z.dv + COLS - 1) / COLS);
    // few CTAs that run long: shared memory asked for beyond the need keeps them one an SM
    static int sms = 0;
    if (!sms) {
        int dev = 0;
        cudaGetDevice(&dev);
        cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev);
    }
    const bool spread = (long long)grid.x * grid.y * grid.z <= sms;
    const int e = (z.d + SLICES - 1) / SLICES;
#define RLIS_SCAN(E)                                                                                                     \
    do {                                                                                                                 \
        const size_t bytes = spread && g.n_tokens > g.n_seqs ? 120 * 1024 : 0;                                           \
        if (bytes) cudaFuncSetAttribute(scan_kernel<MODE, T, E>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes); \
        rlis_launch(scan_kernel<MODE, T, E>, grid, THREADS, bytes, stream, (const float*)g.act, g.out, g.state,          \
                    g.state_stride, tail_off, (const T*)g.x, g.stride, g.skip, g.sq, z);                                 \
    } while (0)
#define RLIS_CHUNK(E)                                                                                                    \
    do {                                                                                                                 \
        size_t bytes = chunk_smem_floats<MODE>(E) * sizeof(float);                                                       \
        if (spread && bytes < 120 * 1024) bytes = 120 * 1024;                                                            \
        cudaFuncSetAttribute(chunk_kernel<MODE, T, E>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);         \
        rlis_launch(chunk_kernel<MODE, T, E>, grid, CTHREADS, bytes, stream, (const float*)g.act, (const float*)g.gram,  \
                    (const float*)g.scaled, g.out, g.state, g.state_stride, tail_off, (const T*)g.x, g.stride, g.skip,   \
                    g.sq, z);                                                                                            \
    } while (0)
    if (g.gram == nullptr) {
        if (e <= 4) RLIS_SCAN(4);
        else if (e <= 8) RLIS_SCAN(8);
        else if (e <= 16) RLIS_SCAN(16);
        else RLIS_SCAN(32);
        return RLIS_LAUNCH_CHECK();
    }
    const int heads = MODE == CHANNEL_DECAY ? z.nh : z.n_qk;
    const int gunits = g.n_tokens * heads, sunits = g.n_tokens * z.nh;
    const unsigned gblocks = (unsigned)((gunits + GRAM_WARPS - 1) / GRAM_WARPS);
    if constexpr (MODE == CHANNEL_DECAY) {
        if (z.d <= 128)
            rlis_launch(gram_channel_kernel<4>, gblocks, GRAM_WARPS * 32, 0, stream, (const float*)g.act, g.gram, g.scaled, g.sq, gunits, z);
        else
            rlis_launch(gram_channel_kernel<MAX_D / 32>, gblocks, GRAM_WARPS * 32, 0, stream, (const float*)g.act, g.gram, g.scaled, g.sq, gunits, z);
    } else {
        rlis_launch(gram_kernel<MODE>, gblocks, GRAM_WARPS * 32, 0, stream, (const float*)g.act, g.gram, g.sq, gunits, z);
    }
    if constexpr (MODE != STATE_SPACE)
        rlis_launch(solve_kernel<MODE>, (unsigned)((sunits + GRAM_WARPS - 1) / GRAM_WARPS), GRAM_WARPS * 32, 0, stream,
                    (const float*)g.act, g.gram, g.sq, sunits, z);
    if (e <= 4) RLIS_CHUNK(4);
    else if (e <= 8) RLIS_CHUNK(8);
    else if (e <= 16) RLIS_CHUNK(16);
    else RLIS_CHUNK(32);
#undef RLIS_CHUNK
#undef RLIS_SCAN
    return RLIS_LAUNCH_CHECK();
}

template <int MODE>
static int launch(const Args& g, int dtype, cudaStream_t stream) {
    if (g.n_tokens <= 0 || g.n_seqs <= 0) return 0;
    const Shape& z = g.z;
    if (z.d <= 0 || z.d > MAX_D || z.d > SLICES * MAX_E || z.dv <= 0 || z.nh <= 0 || z.nh > 65535 ||
        z.n_qk <= 0 || z.nh % z.n_qk != 0 || z.taps < 1 || z.taps > MAX_TAPS || (z.dv + COLS - 1) / COLS > 65535)
        return RLIS_ERR_UNSUPPORTED;
    if (g.state_stride < state_floats(z.nh, z.n_qk, z.d, z.dv, z.taps)) return RLIS_ERR_UNSUPPORTED;
    if (MODE == CHANNEL_DECAY && g.gram != nullptr && g.scaled == nullptr) return RLIS_ERR_UNSUPPORTED;
    if (dtype == RLIS_F32) return launch_typed<MODE, float>(g, stream);
    if (dtype == RLIS_BF16) return launch_typed<MODE, bf16>(g, stream);
    return RLIS_ERR_UNSUPPORTED;
}
}  // namespace convrec
