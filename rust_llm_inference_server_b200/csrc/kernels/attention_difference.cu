// Causal grouped-query attention with two maps a head whose outputs are taken off each other.  A query head holds two
// vectors and so does a key head (a cached key row is [map 1 | map 2], 2 d entries), both maps weigh the same values:
//
//   s_m(i, j) = scale * q_m(i) . k_m(j), then cap * tanh(s / cap) where a cap is given,  j <= i (and i - j < window)
//   a_m(i)    = sum_j softmax_j(s_m(i, j)) v(j)                                             m = 1, 2
//   o(i)      = a_1 - lambda a_2,   o / sqrt(mean(o^2) + eps) * out_scale * sigmoid(gate_h(i))   mean over the dv entries
//
// lambda is one number for the layer, out_scale a constant, the gate one logit a head (or none).  Scores, softmax, value
// sums and everything after them are float32 whatever the element type.
//
// This file: one warp per (token, query head), both maps, keys in blocks of 32 that start at multiples of 32, so the order of
// every sum depends on the query's position only.  The kernel of the float32 path and of bfloat16 sizes that the
// tensor-core kernels (attention_prefill_tcgen05.cu, attention_bias_mma.cu) refuse.
#include "common.cuh"
#include <math.h>

namespace {
constexpr int WARPS = 4;
constexpr int MAX_DV = 256;

template <typename T>
__global__ __launch_bounds__(WARPS * 32) void attn_difference_kernel(
    const T* __restrict__ q, const T* __restrict__ k_cache, const T* __restrict__ v_cache, T* __restrict__ out,
    const T* __restrict__ gate, long long gate_stride, const int* __restrict__ seq_of_token, const int* __restrict__ positions,
    const int* __restrict__ block_tables, const int* __restrict__ token_rows, int max_blocks, int n_rows, int nh, int nkv, int d,
    int dv, int page_size, float scale, float cap, int window, float lambda, float out_scale, float eps) {
    pdl_wait();
    extern __shared__ float qs_all[];
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int gw = blockIdx.x * WARPS + warp;
    if (gw >= n_rows) return;  // no block-wide barrier below
    const int ti = gw / nh, h = gw - ti * nh;
    const int t = token_rows != nullptr ? token_rows[ti] : ti;
    const int kvh = h / (nh / nkv);
    const int pos = positions[t];
    const int* table = block_tables + (size_t)seq_of_token[t] * max_blocks;
    float* qs = qs_all + warp * 2 * d;
    const T* qrow = q + ((size_t)t * nh + h) * 2 * d;
    for (int j = lane; j < 2 * d; j += 32) qs[j] = to_f<T>(qrow[j]);
    __syncwarp();

    const int lo = window > 0 ? max(0, pos - window + 1) : 0;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    float acc[2][MAX_DV / 32];
#pragma unroll
    for (int i = 0; i < MAX_DV / 32; ++i) acc[0][i] = acc[1][i] = 0.f;

    for (int kb = lo - (lo & 31); kb <= pos; kb += 32) {
        const int key = kb + lane;
        const bool valid = key >= lo && key <= pos;
        float s[2] = {-INFINITY, -INFINITY};
        long long row = -1;      // row of this lane's key in the pools, or -1: hidden, or a page the host did not map
        if (valid) {
            const int page = table[key / page_size];
            if (page < 0) {
                s[0] = s[1] = NAN;
            } else {
                row = ((long long)page * nkv + kvh) * page_size + key % page_size;
                const T* krow = k_cache + row * 2 * d;
#pragma unroll
                for (int mp = 0; mp < 2; ++mp) {
                    float dot = 0.f;
                    for (int j = 0; j < d; ++j) dot = fmaf(qs[mp * d + j], to_f<T>(krow[mp * d + j]), dot);
                    s[mp] = dot * scale;
                    if (cap > 0.f) s[mp] = cap * tanhf(s[mp] / cap);
                }
            }
        }
        float p[2];
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
            const float m_new = fmaxf(m[mp], warp_max(s[mp]));
            p[mp] = valid ? expf(s[mp] - m_new) : 0.f;
            const float corr = expf(m[mp] - m_new);
            l[mp] = l[mp] * corr + warp_sum(p[mp]);
#pragma unroll
            for (int i = 0; i < MAX_DV / 32; ++i) acc[mp][i] *= corr;
            m[mp] = m_new;
        }
#pragma unroll 8
        for (int kk = 0; kk < 32; ++kk) {
            const float p0 = __shfl_sync(0xffffffffu, p[0], kk), p1 = __shfl_sync(0xffffffffu, p[1], kk);
            const long long r = __shfl_sync(0xffffffffu, row, kk);
            if (r < 0) continue;               // uniform over the warp
            const T* vrow = v_cache + r * dv;
#pragma unroll
            for (int i = 0; i < MAX_DV / 32; ++i) {
                const int c = lane + 32 * i;
                if (c < dv) {
                    const float v = to_f<T>(vrow[c]);
                    acc[0][i] = fmaf(p0, v, acc[0][i]);
                    acc[1][i] = fmaf(p1, v, acc[1][i]);
                }
            }
        }
    }
    const float i0 = 1.0f / l[0], i1 = lambda / l[1];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < MAX_DV / 32; ++i) {
        acc[0][i] = lane + 32 * i < dv ? acc[0][i] * i0 - acc[1][i] * i1 : 0.f;
        ss = fmaf(acc[0][i], acc[0][i], ss);
    }
    ss = warp_sum(ss);
    float r = out_scale / sqrtf(ss / (float)dv + eps);
    if (gate != nullptr) r *= 1.0f / (1.0f + expf(-to_f<T>(gate[(size_t)t * gate_stride + h])));
    T* orow = out + ((size_t)t * nh + h) * dv;
#pragma unroll
    for (int i = 0; i < MAX_DV / 32; ++i) {
        const int c = lane + 32 * i;
        if (c < dv) orow[c] = from_f<T>(acc[0][i] * r);
    }
    pdl_trigger();
}
}  // namespace

// q [T, nh, 2 d]; k_cache [pages, nkv, page_size, 2 d]; v_cache [pages, nkv, page_size, dv]; out [T, nh dv]; gate (null:
// none): logits, head h of token t at gate[t * gate_stride + h]; cap 0: scores are not capped.
extern "C" int rlis_attention_difference(const void* q, const void* k_cache, const void* v_cache, void* out, const void* gate,
                                         long long gate_stride, const int* seq_of_token, const int* positions,
                                         const int* block_tables, const int* token_rows, int max_blocks, int n_tokens, int nh,
                                         int nkv, int d, int dv, int page_size, float scale, float cap, int window, float lambda,
                                         float out_scale, float eps, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (d <= 0 || d > 1024 || dv <= 0 || dv > MAX_DV || nkv <= 0 || nh % nkv != 0 || cap < 0.f) return RLIS_ERR_UNSUPPORTED;
    const long long n_rows = (long long)n_tokens * nh;
    if (n_rows > 0x7fffffffLL) return RLIS_ERR_UNSUPPORTED;
    const unsigned blocks = (unsigned)((n_rows + WARPS - 1) / WARPS);
    const size_t smem = (size_t)WARPS * 2 * d * sizeof(float);
#define RLIS_DIFF(T) rlis_launch(attn_difference_kernel<T>, blocks, WARPS * 32, smem, stream, (const T*)q, (const T*)k_cache,   \
                                 (const T*)v_cache, (T*)out, (const T*)gate, gate_stride, seq_of_token, positions, block_tables, \
                                 token_rows, max_blocks, (int)n_rows, nh, nkv, d, dv, page_size, scale, cap, window, lambda,     \
                                 out_scale, eps)
    if (dtype == RLIS_F32) RLIS_DIFF(float);
    else if (dtype == RLIS_BF16) RLIS_DIFF(bf16);
    else return RLIS_ERR_UNSUPPORTED;
#undef RLIS_DIFF
    return RLIS_LAUNCH_CHECK();
}
