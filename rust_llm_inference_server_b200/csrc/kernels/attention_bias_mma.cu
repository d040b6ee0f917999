// Tensor-core kernels (bfloat16) for the attention that attention_bias.cu describes: normed queries and
// keys, score = scale * q . k + bias[min(distance, n_dist - 1), head], keys of width D and values of
// width DV, a gate on every head's result; optionally slope_h * distance is subtracted from a score and
// exp(sink_h) joins the denominator of head h's softmax.  mma.sync m16n8k16 with float32 sums; keys and values reach
// shared memory by 16-byte asynchronous copies, two or three stages deep, in tiles of 64 keys; rows padded by 8
// elements so that ldmatrix is free of bank conflicts; softmax in float32 in units of log2(e).
//
// Portions of prompts: one CTA = one query head x 64 tokens of one request (4 warps x 16 rows); the
// causal edge is aligned to the end of the keys.  The bias of a tile depends on query - key only: the
// 127 distances of a 64 x 64 tile are brought to shared memory with the tile (times log2(e)); a tile
// that lies wholly beyond the table's reach adds the last row's constant instead.
//
// Single tokens: one CTA = one key/value head x one request x one piece of its context; the query
// heads of the group are the 16 rows of the products, so keys and values are read once a group.
// Each of the 4 warps takes 16 of a tile's 64 keys with a running softmax of its own; the warps are
// merged through shared memory at the end, pieces of a context by a second kernel.
//
// Single tokens with two maps a head (attention_difference.cu): the same, with rows 0..7 of the products the query heads' first
// maps and rows 8..15 their second ones (groups of up to 8).  A key row is [map 1 | map 2], each padded to 64 entries; a query
// row is its map's vector and zeros over the other's entries, so one set of products gives both maps' scores and the values
// are multiplied once.  The maps meet where the warps (or the pieces) are merged: up to 16 pieces of a context are a
// thread-block cluster, which merges through distributed shared memory (a CTA a head of the group, a warp a quarter of its
// columns), more by a second kernel.
#include "common.cuh"
#include "mma_utils.cuh"
#include <math.h>

namespace {
constexpr int WARPS = 4;
constexpr int THREADS = WARPS * 32;
constexpr int BM = 64;   // query tokens per CTA (prompts)
static_assert(BM == RLIS_PREFILL_TILE, "the host's tile list is cut for another tile size");
constexpr int BN = 64;   // keys per tile
constexpr float LOG2E = 1.4426950408889634f;

// 2^x in one instruction (relative error 2^-22; arguments here are at most 0, and -inf gives 0).
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

template <int D, int DV> struct Stage { static constexpr int ELEMS = BN * (D + 8) + BN * (DV + 8); };
template <int D, int DV> constexpr size_t smem_bytes() {
    return (size_t)2 * Stage<D, DV>::ELEMS * sizeof(bf16) + 2 * 128 * sizeof(float);
}
// single tokens: three stages (two tiles of keys in flight while one is used: the kernel lives on bytes in flight)
constexpr int DEC_STAGES = 3;
template <int D, int DV> constexpr size_t decode_smem_bytes() {
    return (size_t)DEC_STAGES * Stage<D, DV>::ELEMS * sizeof(bf16);
}

// Brings tile `kt` of a request's keys and values into stage memory (ks_, vs_); keys outside [k_lo, k_hi) are zeros.
template <int D, int DV>
__device__ __forceinline__ void issue_tile(bf16* ks_, bf16* vs_, const bf16* kbase, const bf16* vbase,
                                           const int* table, int kt, int k_lo, int k_hi, int page_size,
                                           int page_shift, size_t page_stride_k, size_t page_stride_v) {
    // (page_shift: log2 of a power-of-two page size, or -1; a shift instead of a division a row)
    constexpr int CK = D / 8, CV = DV / 8;
#pragma unroll
    for (int i = 0; i < (BN * CK) / THREADS; ++i) {
        const int idx = threadIdx.x + i * THREADS;
        const int kin = idx / CK, c16 = idx % CK;
        const int key = kt * BN + kin;
        const bool valid = key < k_hi && key >= k_lo;
        size_t off = 0;
        if (valid) {
            const int pi = page_shift >= 0 ? key >> page_shift : key / page_size;
            off = (size_t)table[pi] * page_stride_k + (size_t)((key - pi * page_size) * D + c16 * 8);
        }
        cp_async16(ks_ + kin * (D + 8) + c16 * 8, kbase + off, valid);
    }
#pragma unroll
    for (int i = 0; i < (BN * CV) / THREADS; ++i) {
        const int idx = threadIdx.x + i * THREADS;
        const int kin = idx / CV, c16 = idx % CV;
        const int key = kt * BN + kin;
        const bool valid = key < k_hi && key >= k_lo;
        size_t off = 0;
        if (valid) {
            const int pi = page_shift >= 0 ? key >> page_shift : key / page_size;
            off = (size_t)table[pi] * page_stride_v + (size_t)((key - pi * page_size) * DV + c16 * 8);
        }
        cp_async16(vs_ + kin * (DV + 8) + c16 * 8, vbase + off, valid);
    }
}

// (four CTAs an SM for the narrow heads, three for the wide ones: the bound keeps the registers under that)
template <int D, int DV>
__global__ __launch_bounds__(THREADS, (D + DV <= 128) ? 4 : 3) void attn_bias_prefill_kernel(
    const bf16* __restrict__ q, const bf16* __restrict__ k_cache, const bf16* __restrict__ v_cache,
    bf16* __restrict__ out, const float* __restrict__ bias, int n_dist, const bf16* __restrict__ gate,
    long long gate_stride, const int* __restrict__ tiles, const int* __restrict__ cu_seqlens,
    const int* __restrict__ ctx_lens, const int* __restrict__ block_tables, int max_blocks, int nh, int nkv,
    int page_size, float scale, int window, const float* __restrict__ sinks, const float* __restrict__ slopes,
    int gate_cols) {
    pdl_wait();
    constexpr int SK = D + 8, SV = DV + 8;
    constexpr int KS = D / 16, ND = DV / 8;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* sbase = reinterpret_cast<bf16*>(smem_raw);
    float* bias_s = reinterpret_cast<float*>(sbase + 2 * Stage<D, DV>::ELEMS);     // [stage][128]

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, c = lane & 3;
    const int b = tiles[2 * blockIdx.y], t0 = tiles[2 * blockIdx.y + 1];
    const int head = blockIdx.x;
    const int kvh = head / (nh / nkv);
    const int q_start = cu_seqlens[b];
    const int q_len = cu_seqlens[b + 1] - q_start;
    const int ctx = ctx_lens[b];
    const int start_pos = ctx - q_len;
    const int* table = block_tables + (size_t)b * max_blocks;

    const int r0 = warp * 16 + g, r1 = r0 + 8;            // this lane's two rows of the tile
    const int ti0 = t0 + r0, ti1 = t0 + r1;
    const bool rv0 = ti0 < q_len, rv1 = ti1 < q_len;
    const int pos0 = start_pos + ti0, pos1 = start_pos + ti1;
    const int lo0 = window > 0 ? max(0, pos0 - window + 1) : 0;
    const int lo1 = window > 0 ? max(0, pos1 - window + 1) : 0;

    uint32_t qa[KS][4];
    {
        const bf16* q0 = q + ((size_t)(q_start + (rv0 ? ti0 : 0)) * nh + head) * D;
        const bf16* q1 = q + ((size_t)(q_start + (rv1 ? ti1 : 0)) * nh + head) * D;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            qa[ks][0] = rv0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 2 * c) : 0u;
            qa[ks][1] = rv1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 2 * c) : 0u;
            qa[ks][2] = rv0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 2 * c + 8) : 0u;
            qa[ks][3] = rv1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 2 * c + 8) : 0u;
        }
    }
    const int last_tok = min(t0 + BM, q_len) - 1;
    const int k_hi = start_pos + last_tok + 1;                                  // exclusive
    const int k_lo = window > 0 ? max(0, start_pos + t0 - window + 1) : 0;
    const int kt0 = k_lo / BN, kt1 = (k_hi + BN - 1) / BN;
    const size_t psk = (size_t)nkv * page_size * D, psv = (size_t)nkv * page_size * DV;
    const int page_shift = (page_size & (page_size - 1)) == 0 ? 31 - __clz(page_size) : -1;
    const bf16* kbase = k_cache + (size_t)kvh * page_size * D;
    const bf16* vbase = v_cache + (size_t)kvh * page_size * DV;
    const float far_bias = bias != nullptr ? bias[(size_t)(n_dist - 1) * nh + head] * LOG2E : 0.f;
    const float slope_l2 = slopes != nullptr ? slopes[head] * LOG2E : 0.f;

    auto issue = [&](int kt, int stage) {
        bf16* ks_ = sbase + (size_t)stage * Stage<D, DV>::ELEMS;
        issue_tile<D, DV>(ks_, ks_ + BN * SK, kbase, vbase, table, kt, k_lo, k_hi, page_size, page_shift, psk, psv);
        // the tile's distances: row r, key column j are dist0 + r + (BN - 1 - j) apart
        const int dist0 = start_pos + t0 - (kt * BN + BN - 1);
        if (bias != nullptr && dist0 < n_dist - 1 && threadIdx.x < 2 * BN - 1) {
            const int dist = min(max(dist0 + (int)threadIdx.x, 0), n_dist - 1);
            bias_s[stage * 128 + threadIdx.x] = bias[(size_t)dist * nh + head] * LOG2E;
        }
        cp_async_commit();
    };

    const float scale_log2 = scale * LOG2E;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    float oacc[ND][4];
#pragma unroll
    for (int nd = 0; nd < ND; ++nd)
#pragma unroll
        for (int e = 0; e < 4; ++e) oacc[nd][e] = 0.f;

    int stage = 0;
    if (kt0 < kt1) issue(kt0, 0);
    for (int kt = kt0; kt < kt1; ++kt) {
        if (kt + 1 < kt1) {
            issue(kt + 1, stage ^ 1);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        const bf16* ks_ = sbase + (size_t)stage * Stage<D, DV>::ELEMS;
        const bf16* vs_ = ks_ + BN * SK;
        const float* bs = bias_s + stage * 128;

        float sacc[8][4];
#pragma unroll
        for (int nt = 0; nt < 8; ++nt) {
#pragma unroll
            for (int e = 0; e < 4; ++e) sacc[nt][e] = 0.f;
#pragma unroll
            for (int ks2 = 0; ks2 < KS / 2; ++ks2) {
                uint32_t kb[4];
                ldmatrix_x4(kb, ks_ + (nt * 8 + (lane & 7)) * SK + ks2 * 32 + (lane >> 3) * 8);
                mma_bf16_16816(sacc[nt], qa[2 * ks2], kb[0], kb[1]);
                mma_bf16_16816(sacc[nt], qa[2 * ks2 + 1], kb[2], kb[3]);
            }
        }
        const bool edge = (kt + 1) * BN - 1 > start_pos + t0 + warp * 16 || window > 0;
        const bool near = bias != nullptr && start_pos + t0 - (kt * BN + BN - 1) < n_dist - 1;
        float mx0 = -INFINITY, mx1 = -INFINITY;
        if (!edge && !near && slopes == nullptr) {
            // most tiles of a long prompt: every key is seen by every row, and all share the table's last row
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float s0 = fmaf(sacc[nt][e], scale_log2, far_bias);
                    const float s1 = fmaf(sacc[nt][2 + e], scale_log2, far_bias);
                    sacc[nt][e] = s0;
                    sacc[nt][2 + e] = s1;
                    mx0 = fmaxf(mx0, s0);
                    mx1 = fmaxf(mx1, s1);
                }
        } else {
#pragma unroll
            for (int nt = 0; nt < 8; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int j = nt * 8 + 2 * c + e;
                    float s0 = fmaf(sacc[nt][e], scale_log2, near ? bs[r0 + BN - 1 - j] : far_bias);
                    float s1 = fmaf(sacc[nt][2 + e], scale_log2, near ? bs[r1 + BN - 1 - j] : far_bias);
                    const int key = kt * BN + j;
                    s0 = fmaf(slope_l2, (float)(key - pos0), s0);       // minus slope * distance
                    s1 = fmaf(slope_l2, (float)(key - pos1), s1);
                    if (edge) {
                        if (!(key <= pos0 && key >= lo0)) s0 = -INFINITY;
                        if (!(key <= pos1 && key >= lo1)) s1 = -INFINITY;
                    }
                    sacc[nt][e] = s0;
                    sacc[nt][2 + e] = s1;
                    mx0 = fmaxf(mx0, s0);
                    mx1 = fmaxf(mx1, s1);
                }
        }
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
        mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
        mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
        const float mn0 = fmaxf(m_run[0], mx0), mn1 = fmaxf(m_run[1], mx1);
        const float ms0 = mn0 == -INFINITY ? 0.f : mn0, ms1 = mn1 == -INFINITY ? 0.f : mn1;
        const float corr0 = ex2(m_run[0] - ms0), corr1 = ex2(m_run[1] - ms1);
        float ls0 = 0.f, ls1 = 0.f;
#pragma unroll
        for (int nt = 0; nt < 8; ++nt)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const float p0 = ex2(sacc[nt][e] - ms0), p1 = ex2(sacc[nt][2 + e] - ms1);
                sacc[nt][e] = p0;
                sacc[nt][2 + e] = p1;
                ls0 += p0;
                ls1 += p1;
            }
        ls0 += __shfl_xor_sync(0xffffffffu, ls0, 1);
        ls0 += __shfl_xor_sync(0xffffffffu, ls0, 2);
        ls1 += __shfl_xor_sync(0xffffffffu, ls1, 1);
        ls1 += __shfl_xor_sync(0xffffffffu, ls1, 2);
        l_run[0] = l_run[0] * corr0 + ls0;
        l_run[1] = l_run[1] * corr1 + ls1;
        m_run[0] = mn0;
        m_run[1] = mn1;
#pragma unroll
        for (int nd = 0; nd < ND; ++nd) {
            oacc[nd][0] *= corr0;
            oacc[nd][1] *= corr0;
            oacc[nd][2] *= corr1;
            oacc[nd][3] *= corr1;
        }
#pragma unroll
        for (int kk = 0; kk < BN / 16; ++kk) {
            uint32_t pa[4];
            pa[0] = pack_bf16(sacc[2 * kk][0], sacc[2 * kk][1]);
            pa[1] = pack_bf16(sacc[2 * kk][2], sacc[2 * kk][3]);
            pa[2] = pack_bf16(sacc[2 * kk + 1][0], sacc[2 * kk + 1][1]);
            pa[3] = pack_bf16(sacc[2 * kk + 1][2], sacc[2 * kk + 1][3]);
#pragma unroll
            for (int nd2 = 0; nd2 < ND / 2; ++nd2) {
                uint32_t vb[4];
                const int mat = lane >> 3;
                ldmatrix_x4_trans(vb, vs_ + (kk * 16 + (mat & 1) * 8 + (lane & 7)) * SV + (nd2 * 2 + (mat >> 1)) * 8);
                mma_bf16_16816(oacc[2 * nd2], pa, vb[0], vb[1]);
                mma_bf16_16816(oacc[2 * nd2 + 1], pa, vb[2], vb[3]);
            }
        }
        __syncthreads();       // everyone is done with this stage before the next copies land in it
        stage ^= 1;
    }

    if (sinks != nullptr) {
        // one more term of the denominator, without a key or a value (a sink far above every score gives inf, and 0)
        const float sink_l2 = sinks[head] * LOG2E;
        l_run[0] += ex2(sink_l2 - m_run[0]);
        l_run[1] += ex2(sink_l2 - m_run[1]);
    }
    float inv0 = l_run[0] > 0.f ? 1.0f / l_run[0] : 0.f;
    float inv1 = l_run[1] > 0.f ? 1.0f / l_run[1] : 0.f;
    const bool by_channel = gate != nullptr && gate_cols > 1;      // a logit a channel: gate[t, head * DV + col]
    if (gate != nullptr && !by_channel) {
        if (rv0) inv0 *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)(q_start + ti0) * gate_stride + head])));
        if (rv1) inv1 *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)(q_start + ti1) * gate_stride + head])));
    }
    if (rv0) {
        bf16* o = out + ((size_t)(q_start + ti0) * nh + head) * DV;
        const bf16* gr = by_channel ? gate + (size_t)(q_start + ti0) * gate_stride + (size_t)head * DV : nullptr;
#pragma unroll
        for (int nd = 0; nd < ND; ++nd) {
            float g0 = 1.0f, g1 = 1.0f;
            if (by_channel) {
                g0 = 1.0f / (1.0f + expf(-__bfloat162float(gr[nd * 8 + 2 * c])));
                g1 = 1.0f / (1.0f + expf(-__bfloat162float(gr[nd * 8 + 2 * c + 1])));
            }
            *reinterpret_cast<uint32_t*>(o + nd * 8 + 2 * c) = pack_bf16(oacc[nd][0] * inv0 * g0, oacc[nd][1] * inv0 * g1);
        }
    }
    if (rv1) {
        bf16* o = out + ((size_t)(q_start + ti1) * nh + head) * DV;
        const bf16* gr = by_channel ? gate + (size_t)(q_start + ti1) * gate_stride + (size_t)head * DV : nullptr;
#pragma unroll
        for (int nd = 0; nd < ND; ++nd) {
            float g0 = 1.0f, g1 = 1.0f;
            if (by_channel) {
                g0 = 1.0f / (1.0f + expf(-__bfloat162float(gr[nd * 8 + 2 * c])));
                g1 = 1.0f / (1.0f + expf(-__bfloat162float(gr[nd * 8 + 2 * c + 1])));
            }
            *reinterpret_cast<uint32_t*>(o + nd * 8 + 2 * c) = pack_bf16(oacc[nd][2] * inv1 * g0, oacc[nd][3] * inv1 * g1);
        }
    }
    pdl_trigger();
}

// partial [n_dec][nh][pieces][DV + 2] float32: unnormalised sums, then the maximum (log2 units) and the denominator.
template <int D, int DV>
__global__ __launch_bounds__(THREADS) void attn_bias_decode_kernel(
    const bf16* __restrict__ q, const bf16* __restrict__ k_cache, const bf16* __restrict__ v_cache,
    bf16* __restrict__ out, float* __restrict__ partial, const float* __restrict__ bias, int n_dist,
    const bf16* __restrict__ gate, long long gate_stride, const int* __restrict__ dec_rows,
    const int* __restrict__ dec_seqs, const int* __restrict__ ctx_lens, const int* __restrict__ block_tables,
    int max_blocks, int nh, int nkv, int page_size, float scale, int window, int pieces,
    const float* __restrict__ sinks, const float* __restrict__ slopes, int gate_cols) {
    pdl_wait();
    constexpr int SK = D + 8, SV = DV + 8;
    constexpr int KS = D / 16, ND = DV / 8;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* sbase = reinterpret_cast<bf16*>(smem_raw);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, c = lane & 3;
    const int kvh = blockIdx.x, bi = blockIdx.y, piece = blockIdx.z;
    const int nrep = nh / nkv;
    const int row = dec_rows[bi], seq = dec_seqs[bi];
    const int ctx = ctx_lens[seq];
    const int pos = ctx - 1;
    const int* table = block_tables + (size_t)seq * max_blocks;
    const int h0 = kvh * nrep + g, h1 = h0 + 8;            // this lane's two rows: heads of the group
    const bool rv0 = g < nrep, rv1 = g + 8 < nrep;

    uint32_t qa[KS][4];
    {
        const bf16* q0 = q + ((size_t)row * nh + (rv0 ? h0 : kvh * nrep)) * D;
        const bf16* q1 = q + ((size_t)row * nh + (rv1 ? h1 : kvh * nrep)) * D;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            qa[ks][0] = rv0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 2 * c) : 0u;
            qa[ks][1] = rv1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 2 * c) : 0u;
            qa[ks][2] = rv0 ? *reinterpret_cast<const uint32_t*>(q0 + ks * 16 + 2 * c + 8) : 0u;
            qa[ks][3] = rv1 ? *reinterpret_cast<const uint32_t*>(q1 + ks * 16 + 2 * c + 8) : 0u;
        }
    }
    const int k_lo = window > 0 ? max(0, ctx - window) : 0;
    const int k_hi = ctx;
    const int t_first = k_lo / BN, t_all = (k_hi + BN - 1) / BN - t_first;
    const int per = (t_all + pieces - 1) / pieces;
    const int kt0 = t_first + piece * per, kt1 = min(kt0 + per, t_first + t_all);
    const size_t psk = (size_t)nkv * page_size * D, psv = (size_t)nkv * page_size * DV;
    const int page_shift = (page_size & (page_size - 1)) == 0 ? 31 - __clz(page_size) : -1;
    const bf16* kbase = k_cache + (size_t)kvh * page_size * D;
    const bf16* vbase = v_cache + (size_t)kvh * page_size * DV;
    const float* brow0 = bias != nullptr ? bias + (rv0 ? h0 : 0) : nullptr;
    const float* brow1 = bias != nullptr ? bias + (rv1 ? h1 : 0) : nullptr;
    const float far0 = bias != nullptr ? brow0[(size_t)(n_dist - 1) * nh] * LOG2E : 0.f;
    const float far1 = bias != nullptr ? brow1[(size_t)(n_dist - 1) * nh] * LOG2E : 0.f;
    const float slope0 = slopes != nullptr && rv0 ? slopes[h0] * LOG2E : 0.f;
    const float slope1 = slopes != nullptr && rv1 ? slopes[h1] * LOG2E : 0.f;

    auto issue = [&](int kt, int stage) {
        bf16* ks_ = sbase + (size_t)stage * Stage<D, DV>::ELEMS;
        issue_tile<D, DV>(ks_, ks_ + BN * SK, kbase, vbase, table, kt, k_lo, k_hi, page_size, page_shift, psk, psv);
        cp_async_commit();
    };

    const float scale_log2 = scale * LOG2E;
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    float oacc[ND][4];
#pragma unroll
    for (int nd = 0; nd < ND; ++nd)
#pragma unroll
        for (int e = 0; e < 4; ++e) oacc[nd][e] = 0.f;

#pragma unroll
    for (int s = 0; s < DEC_STAGES - 1; ++s) {
        if (kt0 + s < kt1) issue(kt0 + s, s);
        else cp_async_commit();                      // an empty group keeps the count of groups in step
    }
    for (int kt = kt0; kt < kt1; ++kt) {
        const int stage = (kt - kt0) % DEC_STAGES;
        cp_async_wait<DEC_STAGES - 2>();
        __syncthreads();                             // tile kt has landed, and everyone is done with the stage of tile kt - 1
        if (kt + DEC_STAGES - 1 < kt1) issue(kt + DEC_STAGES - 1, (kt - kt0 + DEC_STAGES - 1) % DEC_STAGES);
        else cp_async_commit();
        const bf16* ks_ = sbase + (size_t)stage * Stage<D, DV>::ELEMS;
        const bf16* vs_ = ks_ + BN * SK;
        const int key0 = kt * BN + warp * 16;              // this warp's 16 keys of the tile
        if (key0 < k_hi && key0 + 15 >= k_lo) {
            float sacc[2][4];
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
                for (int e = 0; e < 4; ++e) sacc[nt][e] = 0.f;
#pragma unroll
                for (int ks2 = 0; ks2 < KS / 2; ++ks2) {
                    uint32_t kb[4];
                    ldmatrix_x4(kb, ks_ + (warp * 16 + nt * 8 + (lane & 7)) * SK + ks2 * 32 + (lane >> 3) * 8);
                    mma_bf16_16816(sacc[nt], qa[2 * ks2], kb[0], kb[1]);
                    mma_bf16_16816(sacc[nt], qa[2 * ks2 + 1], kb[2], kb[3]);
                }
            }
            const bool near = bias != nullptr && pos - (key0 + 15) < n_dist - 1;
            float mx0 = -INFINITY, mx1 = -INFINITY;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int key = key0 + nt * 8 + 2 * c + e;
                    const bool seen = key < k_hi && key >= k_lo;
                    float b0 = far0, b1 = far1;
                    if (near && seen) {
                        const size_t at = (size_t)min(pos - key, n_dist - 1) * nh;
                        b0 = brow0[at] * LOG2E;
                        b1 = brow1[at] * LOG2E;
                    }
                    const float dist = (float)(key - pos);                   // minus the distance
                    const float s0 = seen ? fmaf(slope0, dist, fmaf(sacc[nt][e], scale_log2, b0)) : -INFINITY;
                    const float s1 = seen ? fmaf(slope1, dist, fmaf(sacc[nt][2 + e], scale_log2, b1)) : -INFINITY;
                    sacc[nt][e] = s0;
                    sacc[nt][2 + e] = s1;
                    mx0 = fmaxf(mx0, s0);
                    mx1 = fmaxf(mx1, s1);
                }
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 1));
            mx0 = fmaxf(mx0, __shfl_xor_sync(0xffffffffu, mx0, 2));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 1));
            mx1 = fmaxf(mx1, __shfl_xor_sync(0xffffffffu, mx1, 2));
            const float mn0 = fmaxf(m_run[0], mx0), mn1 = fmaxf(m_run[1], mx1);
            const float ms0 = mn0 == -INFINITY ? 0.f : mn0, ms1 = mn1 == -INFINITY ? 0.f : mn1;
            const float corr0 = exp2f(m_run[0] - ms0), corr1 = exp2f(m_run[1] - ms1);
            float ls0 = 0.f, ls1 = 0.f;
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float p0 = exp2f(sacc[nt][e] - ms0), p1 = exp2f(sacc[nt][2 + e] - ms1);
                    sacc[nt][e] = p0;
                    sacc[nt][2 + e] = p1;
                    ls0 += p0;
                    ls1 += p1;
                }
            ls0 += __shfl_xor_sync(0xffffffffu, ls0, 1);
            ls0 += __shfl_xor_sync(0xffffffffu, ls0, 2);
            ls1 += __shfl_xor_sync(0xffffffffu, ls1, 1);
            ls1 += __shfl_xor_sync(0xffffffffu, ls1, 2);
            l_run[0] = l_run[0] * corr0 + ls0;
            l_run[1] = l_run[1] * corr1 + ls1;
            m_run[0] = mn0;
            m_run[1] = mn1;
#pragma unroll
            for (int nd = 0; nd < ND; ++nd) {
                oacc[nd][0] *= corr0;
                oacc[nd][1] *= corr0;
                oacc[nd][2] *= corr1;
                oacc[nd][3] *= corr1;
            }
            uint32_t pa[4];
            pa[0] = pack_bf16(sacc[0][0], sacc[0][1]);
            pa[1] = pack_bf16(sacc[0][2], sacc[0][3]);
            pa[2] = pack_bf16(sacc[1][0], sacc[1][1]);
            pa[3] = pack_bf16(sacc[1][2], sacc[1][3]);
#pragma unroll
            for (int nd2 = 0; nd2 < ND / 2; ++nd2) {
                uint32_t vb[4];
                const int mat = lane >> 3;
                ldmatrix_x4_trans(vb, vs_ + (warp * 16 + (mat & 1) * 8 + (lane & 7)) * SV + (nd2 * 2 + (mat >> 1)) * 8);
                mma_bf16_16816(oacc[2 * nd2], pa, vb[0], vb[1]);
                mma_bf16_16816(oacc[2 * nd2 + 1], pa, vb[2], vb[3]);
            }
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    pdl_trigger();
    // the four warps' states meet in shared memory (the stages are free now): [warp][row][DV + 2]
    float* mg = reinterpret_cast<float*>(smem_raw);
    constexpr int MW = DV + 2;
    {
        float* a0 = mg + ((size_t)warp * 16 + g) * MW;
        float* a1 = a0 + 8 * MW;
#pragma unroll
        for (int nd = 0; nd < ND; ++nd) {
            a0[nd * 8 + 2 * c] = oacc[nd][0];
            a0[nd * 8 + 2 * c + 1] = oacc[nd][1];
            a1[nd * 8 + 2 * c] = oacc[nd][2];
            a1[nd * 8 + 2 * c + 1] = oacc[nd][3];
        }
        if (c == 0) {
            a0[DV] = m_run[0]; a0[DV + 1] = l_run[0];
            a1[DV] = m_run[1]; a1[DV + 1] = l_run[1];
        }
    }
    __syncthreads();
    for (int idx = threadIdx.x; idx < nrep * DV; idx += THREADS) {
        const int r = idx / DV, col = idx - r * DV;
        float m = -INFINITY;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) m = fmaxf(m, mg[((size_t)w * 16 + r) * MW + DV]);
        float l = 0.f, o = 0.f;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) {
            const float* a = mg + ((size_t)w * 16 + r) * MW;
            const float f = a[DV] == -INFINITY ? 0.f : exp2f(a[DV] - m);
            l = fmaf(a[DV + 1], f, l);
            o = fmaf(a[col], f, o);
        }
        const int head = kvh * nrep + r;
        if (pieces == 1) {
            if (sinks != nullptr) l += exp2f(sinks[head] * LOG2E - m);
            float inv = l > 0.f ? 1.0f / l : 0.f;
            if (gate != nullptr)
                inv *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)row * gate_stride + (gate_cols > 1 ? head * DV + col : head)])));
            out[((size_t)row * nh + head) * DV + col] = __float2bfloat16_rn(o * inv);
        } else {
            float* p = partial + (((size_t)bi * nh + head) * pieces + piece) * MW;
            p[col] = o;
            if (col == 0) { p[DV] = m; p[DV + 1] = l; }
        }
    }
}

// Pieces of a context into one result: one warp a (token, head).
__global__ __launch_bounds__(128) void attn_bias_decode_merge_kernel(
    const float* __restrict__ partial, bf16* __restrict__ out, const bf16* __restrict__ gate, long long gate_stride,
    const int* __restrict__ dec_rows, int n_units, int nh, int dv, int pieces, const float* __restrict__ sinks,
    int gate_cols) {
    pdl_wait_and_trigger();
    const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= n_units) return;
    const int bi = unit / nh, head = unit - bi * nh;
    const int row = dec_rows[bi];
    const int mw = dv + 2;
    const float* p = partial + (size_t)unit * pieces * mw;
    float m = -INFINITY;
    for (int s = 0; s < pieces; ++s) m = fmaxf(m, p[(size_t)s * mw + dv]);
    float l = 0.f;
    for (int s = 0; s < pieces; ++s) {
        const float ms = p[(size_t)s * mw + dv];
        l = fmaf(p[(size_t)s * mw + dv + 1], ms == -INFINITY ? 0.f : exp2f(ms - m), l);
    }
    if (sinks != nullptr) l += exp2f(sinks[head] * LOG2E - m);
    float inv = l > 0.f ? 1.0f / l : 0.f;
    const bool by_channel = gate != nullptr && gate_cols > 1;
    if (gate != nullptr && !by_channel) inv *= 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)row * gate_stride + head])));
    for (int col = lane; col < dv; col += 32) {
        float o = 0.f;
        for (int s = 0; s < pieces; ++s) {
            const float ms = p[(size_t)s * mw + dv];
            o = fmaf(p[(size_t)s * mw + col], ms == -INFINITY ? 0.f : exp2f(ms - m), o);
        }
        float gc = 1.0f;
        if (by_channel) gc = 1.0f / (1.0f + expf(-__bfloat162float(gate[(size_t)row * gate_stride + (size_t)head * dv + col])));
        out[((size_t)row * nh + head) * dv + col] = __float2bfloat16_rn(o * inv * gc);
    }
}

constexpr int MAX_CLUSTER_PIECES = 16;
constexpr int TABLE_SLICE = 512;       // page numbers of a CTA's piece kept in shared memory (longer pieces look them up as they go)
template <int DV> constexpr size_t difference_smem_bytes() { return decode_smem_bytes<128, DV>() + TABLE_SLICE * sizeof(int); }
struct DiffDecode {
    const bf16 *q, *k_cache, *v_cache;
    bf16* out;
    float* partial;           // several pieces: [n_dec][nh][map][pieces][DV + 2]
    const bf16* gate;         // logits, one a head, or null
    long long gate_stride;
    const int *dec_rows, *dec_seqs, *ctx_lens, *block_tables;
    int max_blocks, nh, nkv, d, dv, page_size, window, pieces;
    int cluster;              // 1: the pieces are a cluster and merge themselves
    float scale, cap, lambda, out_scale, eps;
};

// log2(e) cap tanh(s scale / cap), or log2(e) s scale without a cap.
__device__ __forceinline__ float capped_log2(float s, float scale, float cap) {
    if (cap <= 0.f) return s * scale * LOG2E;
    const float e = ex2(s * (2.0f * LOG2E * scale / cap)), top = cap * LOG2E;         // e^{2u}: tanh(u) = 1 - 2 / (1 + e^{2u})
    return fmaf(-2.0f * top, __fdividef(1.0f, 1.0f + fminf(e, 1e30f)), top);
}

// One head's result from its maps' sums (unnormalised, over `n` parts of MW floats each, maximum and denominator at the end of a
// part; part p of map m at base + (m * n + p) * part_stride): a warp a head.
template <int NC>
__device__ __forceinline__ void store_difference(const float* base, int n, size_t part_stride, size_t map_stride, int mcol, int dv,
                                                 float lambda, float out_scale, float eps, const bf16* gate, bf16* out, int lane) {
    float o[NC];
#pragma unroll
    for (int i = 0; i < NC; ++i) o[i] = 0.f;
#pragma unroll
    for (int mp = 0; mp < 2; ++mp) {
        const float* b = base + mp * map_stride;
        float m = -INFINITY, l = 0.f;
        for (int p = lane; p < n; p += 32) m = fmaxf(m, b[p * part_stride + mcol]);
        m = warp_max(m);
        float a[NC];
#pragma unroll
        for (int i = 0; i < NC; ++i) a[i] = 0.f;
#pragma unroll 4
        for (int p = 0; p < n; ++p) {
            const float* r = b + p * part_stride;
            const float f = r[mcol] == -INFINITY ? 0.f : exp2f(r[mcol] - m);
            l = fmaf(r[mcol + 1], f, l);
#pragma unroll
            for (int i = 0; i < NC; ++i)
                if (lane + 32 * i < dv) a[i] = fmaf(r[lane + 32 * i], f, a[i]);
        }
        const float inv = (mp == 0 ? 1.0f : -lambda) / l;
#pragma unroll
        for (int i = 0; i < NC; ++i) o[i] = fmaf(a[i], inv, o[i]);
    }
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < NC; ++i) ss = fmaf(o[i], o[i], ss);
    ss = warp_sum(ss);
    float r = out_scale / sqrtf(ss / (float)dv + eps);
    if (gate != nullptr) r /= 1.0f + expf(-__bfloat162float(*gate));
#pragma unroll
    for (int i = 0; i < NC; ++i)
        if (lane + 32 * i < dv) out[lane + 32 * i] = __float2bfloat16_rn(o[i] * r);
}

template <int DV>
__global__ __launch_bounds__(THREADS) void attn_difference_decode_kernel(const DiffDecode a) {
    pdl_wait();
    constexpr int D = 128, SK = D + 8, SV = DV + 8, KS = D / 16, ND = DV / 8;
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* sbase = reinterpret_cast<bf16*>(smem_raw);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, c = lane & 3;
    const int kvh = blockIdx.x, bi = blockIdx.y, piece = blockIdx.z;
    const int nrep = a.nh / a.nkv;
    const int row = a.dec_rows[bi], seq = a.dec_seqs[bi];
    const int ctx = a.ctx_lens[seq];
    const int* table = a.block_tables + (size_t)seq * a.max_blocks;
    const bool live = g < nrep;                            // this lane's two rows: both maps of head kvh * nrep + g
    const int d = a.d, dv = a.dv, page_size = a.page_size;

    uint32_t qa[KS][4];
    {
        const bf16* q0 = a.q + ((size_t)row * a.nh + kvh * nrep + (live ? g : 0)) * 2 * d;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            const int mp = ks / (KS / 2), col = (ks % (KS / 2)) * 16 + 2 * c;
            const bool in0 = live && col < d, in8 = live && col + 8 < d;
            const uint32_t x0 = in0 ? *reinterpret_cast<const uint32_t*>(q0 + mp * d + col) : 0u;
            const uint32_t x8 = in8 ? *reinterpret_cast<const uint32_t*>(q0 + mp * d + col + 8) : 0u;
            qa[ks][0] = mp == 0 ? x0 : 0u;
            qa[ks][1] = mp == 0 ? 0u : x0;
            qa[ks][2] = mp == 0 ? x8 : 0u;
            qa[ks][3] = mp == 0 ? 0u : x8;
        }
    }
    const int k_lo = a.window > 0 ? max(0, ctx - a.window) : 0;
    const int k_hi = ctx;
    const int t_first = k_lo / BN, t_all = (k_hi + BN - 1) / BN - t_first;
    const int per = (t_all + a.pieces - 1) / a.pieces;
    const int kt0 = t_first + piece * per, kt1 = min(kt0 + per, t_first + t_all);
    const int page_shift = (page_size & (page_size - 1)) == 0 ? 31 - __clz(page_size) : -1;
    // a look-up in global memory before every copy is most of a tile's time: the piece's page numbers come to shared memory once
    int* pages = reinterpret_cast<int*>(sbase + (size_t)DEC_STAGES * Stage<D, DV>::ELEMS);
    const int p_first = kt0 * BN / page_size, p_count = kt1 > kt0 ? (min(kt1 * BN, k_hi) - 1) / page_size - p_first + 1 : 0;
    const bool sliced = p_count <= TABLE_SLICE;
    if (sliced) {
        for (int i = threadIdx.x; i < p_count; i += THREADS) pages[i] = table[p_first + i];
        __syncthreads();
    }

    auto issue = [&](int kt, int stage) {
        bf16* ks_ = sbase + (size_t)stage * Stage<D, DV>::ELEMS;
        bf16* vs_ = ks_ + BN * SK;
        constexpr int CK = D / 8, CV = DV / 8;
#pragma unroll
        for (int i = 0; i < BN * (CK + CV) / THREADS; ++i) {
            const bool is_v = i >= BN * CK / THREADS;
            const int idx = threadIdx.x + (is_v ? i - BN * CK / THREADS : i) * THREADS;
            const int chunks = is_v ? CV : CK;
            const int kin = idx / chunks, c16 = idx % chunks;
            const int key = kt * BN + kin;
            const int col = is_v ? c16 * 8 : (c16 % (CK / 2)) * 8;
            const bool valid = key < k_hi && key >= k_lo && col < (is_v ? dv : d);
            size_t off = 0;
            if (valid) {
                const int pi = page_shift >= 0 ? key >> page_shift : key / page_size;
                const int page = sliced ? pages[pi - p_first] : table[pi];
                const size_t r = ((size_t)page * a.nkv + kvh) * page_size + (key - pi * page_size);
                off = is_v ? r * dv + col : (r * 2 + c16 / (CK / 2)) * d + col;
            }
            if (is_v) cp_async16(vs_ + kin * SV + c16 * 8, a.v_cache + off, valid);
            else cp_async16(ks_ + kin * SK + c16 * 8, a.k_cache + off, valid);
        }
        cp_async_commit();
    };

    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    float oacc[ND][4];
#pragma unroll
    for (int nd = 0; nd < ND; ++nd)
#pragma unroll
        for (int e = 0; e < 4; ++e) oacc[nd][e] = 0.f;
#pragma unroll
    for (int s = 0; s < DEC_STAGES - 1; ++s) {
        if (kt0 + s < kt1) issue(kt0 + s, s);
        else cp_async_commit();                      // an empty group keeps the count of groups in step
    }
    for (int kt = kt0; kt < kt1; ++kt) {
        const int stage = (kt - kt0) % DEC_STAGES;
        cp_async_wait<DEC_STAGES - 2>();
        __syncthreads();                             // tile kt has landed, and everyone is done with the stage of tile kt - 1
        if (kt + DEC_STAGES - 1 < kt1) issue(kt + DEC_STAGES - 1, (kt - kt0 + DEC_STAGES - 1) % DEC_STAGES);
        else cp_async_commit();
        const bf16* ks_ = sbase + (size_t)stage * Stage<D, DV>::ELEMS;
        const bf16* vs_ = ks_ + BN * SK;
        const int key0 = kt * BN + warp * 16;              // this warp's 16 keys of the tile
        if (key0 < k_hi && key0 + 15 >= k_lo) {
            float sacc[2][4];
#pragma unroll
            for (int nt = 0; nt < 2; ++nt) {
#pragma unroll
                for (int e = 0; e < 4; ++e) sacc[nt][e] = 0.f;
#pragma unroll
                for (int ks2 = 0; ks2 < KS / 2; ++ks2) {
                    uint32_t kb[4];
                    ldmatrix_x4(kb, ks_ + (warp * 16 + nt * 8 + (lane & 7)) * SK + ks2 * 32 + (lane >> 3) * 8);
                    mma_bf16_16816(sacc[nt], qa[2 * ks2], kb[0], kb[1]);
                    mma_bf16_16816(sacc[nt], qa[2 * ks2 + 1], kb[2], kb[3]);
                }
            }
            float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int key = key0 + nt * 8 + 2 * c + (e & 1);
                    const bool seen = key < k_hi && key >= k_lo;
                    sacc[nt][e] = seen ? capped_log2(sacc[nt][e], a.scale, a.cap) : -INFINITY;
                    mx[e >> 1] = fmaxf(mx[e >> 1], sacc[nt][e]);
                }
            float ms[2], corr[2], ls[2] = {0.f, 0.f};
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
                const float mn = fmaxf(m_run[r], mx[r]);
                ms[r] = mn == -INFINITY ? 0.f : mn;
                corr[r] = exp2f(m_run[r] - ms[r]);
                m_run[r] = mn;
            }
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    sacc[nt][e] = exp2f(sacc[nt][e] - ms[e >> 1]);
                    ls[e >> 1] += sacc[nt][e];
                }
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                ls[r] += __shfl_xor_sync(0xffffffffu, ls[r], 1);
                ls[r] += __shfl_xor_sync(0xffffffffu, ls[r], 2);
                l_run[r] = l_run[r] * corr[r] + ls[r];
            }
#pragma unroll
            for (int nd = 0; nd < ND; ++nd)
#pragma unroll
                for (int e = 0; e < 4; ++e) oacc[nd][e] *= corr[e >> 1];
            uint32_t pa[4];
            pa[0] = pack_bf16(sacc[0][0], sacc[0][1]);
            pa[1] = pack_bf16(sacc[0][2], sacc[0][3]);
            pa[2] = pack_bf16(sacc[1][0], sacc[1][1]);
            pa[3] = pack_bf16(sacc[1][2], sacc[1][3]);
#pragma unroll
            for (int nd2 = 0; nd2 < ND / 2; ++nd2) {
                uint32_t vb[4];
                const int mat = lane >> 3;
                ldmatrix_x4_trans(vb, vs_ + (warp * 16 + (mat & 1) * 8 + (lane & 7)) * SV + (nd2 * 2 + (mat >> 1)) * 8);
                mma_bf16_16816(oacc[2 * nd2], pa, vb[0], vb[1]);
                mma_bf16_16816(oacc[2 * nd2 + 1], pa, vb[2], vb[3]);
            }
        }
    }
    cp_async_wait<0>();
    __syncthreads();
    pdl_trigger();
    // the four warps' states meet in shared memory (the stages are free now): [warp][row][DV + 2]
    constexpr int MW = DV + 2;
    float* mg = reinterpret_cast<float*>(smem_raw);
    {
        float* a0 = mg + ((size_t)warp * 16 + g) * MW;
        float* a1 = a0 + 8 * MW;
#pragma unroll
        for (int nd = 0; nd < ND; ++nd) {
            a0[nd * 8 + 2 * c] = oacc[nd][0];
            a0[nd * 8 + 2 * c + 1] = oacc[nd][1];
            a1[nd * 8 + 2 * c] = oacc[nd][2];
            a1[nd * 8 + 2 * c + 1] = oacc[nd][3];
        }
        if (c == 0) {
            a0[DV] = m_run[0]; a0[DV + 1] = l_run[0];
            a1[DV] = m_run[1]; a1[DV + 1] = l_run[1];
        }
    }
    __syncthreads();
    if (a.pieces == 1) {
        for (int r = warp; r < nrep; r += WARPS) {
            const int head = kvh * nrep + r;
            store_difference<DV / 32>(mg + (size_t)r * MW, WARPS, (size_t)16 * MW, (size_t)8 * MW, DV, dv, a.lambda, a.out_scale, a.eps,
                                      a.gate != nullptr ? a.gate + (size_t)row * a.gate_stride + head : nullptr,
                                      a.out + ((size_t)row * a.nh + head) * dv, lane);
        }
        return;
    }
    // (in a cluster: this CTA's merged rows [head][map][MW], behind the warps' rows)
    float* mine = mg + (size_t)WARPS * 16 * MW;
    for (int idx = threadIdx.x; idx < 2 * nrep * DV; idx += THREADS) {
        const int u = idx / DV, col = idx - u * DV, r = u >> 1, mp = u & 1;
        const float* b = mg + (size_t)(mp * 8 + r) * MW;
        float m = -INFINITY, l = 0.f, o = 0.f;
#pragma unroll
        for (int w = 0; w < WARPS; ++w) m = fmaxf(m, b[(size_t)w * 16 * MW + DV]);
#pragma unroll
        for (int w = 0; w < WARPS; ++w) {
            const float* x = b + (size_t)w * 16 * MW;
            const float f = x[DV] == -INFINITY ? 0.f : exp2f(x[DV] - m);
            l = fmaf(x[DV + 1], f, l);
            o = fmaf(x[col], f, o);
        }
        float* dst = a.cluster ? mine + (size_t)u * MW : a.partial + ((((size_t)bi * a.nh + kvh * nrep + r) * 2 + mp) * a.pieces + piece) * MW;
        dst[col] = o;
        if (col == 0) { dst[DV] = m; dst[DV + 1] = l; }
    }
    if (!a.cluster) return;
    cluster_sync_all();
    __shared__ float red[WARPS];
    for (int r = piece; r < nrep; r += a.pieces) {         // the same for all threads of the CTA
        // warp w takes columns w, w + 4, ... blocks of 32; every lane reads its columns from all pieces
        constexpr int NC = DV / 32 / WARPS > 0 ? DV / 32 / WARPS : 1;
        float o[NC];
#pragma unroll
        for (int i = 0; i < NC; ++i) o[i] = 0.f;
#pragma unroll
        for (int mp = 0; mp < 2; ++mp) {
            const float* b = mine + (size_t)(2 * r + mp) * MW;
            // lane p holds piece p's maximum and denominator (up to 16 pieces)
            const float pm = lane < a.pieces ? ld_dsmem(b + DV, (uint32_t)lane) : -INFINITY;
            const float pl = lane < a.pieces ? ld_dsmem(b + DV + 1, (uint32_t)lane) : 0.f;
            const float m = warp_max(pm);
            const float pf = pm == -INFINITY ? 0.f : exp2f(pm - m);
            const float inv = (mp == 0 ? 1.0f : -a.lambda) / warp_sum(pl * pf);
            float x[NC][16];
#pragma unroll
            for (int p = 0; p < 16; ++p)
#pragma unroll
                for (int i = 0; i < NC; ++i) {
                    const int col = (warp + i * WARPS) * 32 + lane;
                    x[i][p] = p < a.pieces && col < DV ? ld_dsmem(b + col, (uint32_t)p) : 0.f;
                }
#pragma unroll
            for (int p = 0; p < 16; ++p) {
                const float f = __shfl_sync(0xffffffffu, pf, p) * inv;
#pragma unroll
                for (int i = 0; i < NC; ++i) o[i] = fmaf(x[i][p], f, o[i]);
            }
        }
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < NC; ++i) ss = fmaf(o[i], o[i], ss);
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        const int head = kvh * nrep + r;
        float f = a.out_scale / sqrtf(((red[0] + red[1]) + (red[2] + red[3])) / (float)dv + a.eps);
        if (a.gate != nullptr) f /= 1.0f + expf(-__bfloat162float(a.gate[(size_t)row * a.gate_stride + head]));
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const int col = (warp + i * WARPS) * 32 + lane;
            if (col < dv) a.out[((size_t)row * a.nh + head) * dv + col] = __float2bfloat16_rn(o[i] * f);
        }
        __syncthreads();
    }
    cluster_sync_all();        // nobody leaves while its rows may still be read
}

// Pieces of a context into one result: one warp a (token, head), both maps.
template <int DV>
__global__ __launch_bounds__(128) void attn_difference_merge_kernel(const DiffDecode a, int n_units) {
    pdl_wait_and_trigger();
    const int unit = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (unit >= n_units) return;
    const int bi = unit / a.nh, head = unit - bi * a.nh, row = a.dec_rows[bi];
    constexpr int MW = DV + 2;
    store_difference<DV / 32>(a.partial + (size_t)unit * 2 * a.pieces * MW, a.pieces, MW, (size_t)a.pieces * MW, DV, a.dv, a.lambda,
                              a.out_scale, a.eps, a.gate != nullptr ? a.gate + (size_t)row * a.gate_stride + head : nullptr,
                              a.out + ((size_t)row * a.nh + head) * a.dv, lane);
}

bool sizes_taken(int d, int dv) { return (d == 64 || d == 128) && (dv == 32 || dv == 64 || dv == 128); }

template <int D, int DV> void raise_smem_limits() {
    cudaFuncSetAttribute(attn_bias_prefill_kernel<D, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_bytes<D, DV>());
    cudaFuncSetAttribute(attn_bias_decode_kernel<D, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)decode_smem_bytes<D, DV>());
}
void raise_all_once() {
    static bool done = false;
    if (done) return;
    raise_smem_limits<64, 32>(); raise_smem_limits<64, 64>(); raise_smem_limits<64, 128>();
    raise_smem_limits<128, 32>(); raise_smem_limits<128, 64>(); raise_smem_limits<128, 128>();
    done = true;
}
}  // namespace

// Whether the kernels of this file exist for keys of width d and values of width dv (bfloat16).
extern "C" int rlis_attention_bias_mma_takes(int d, int dv) { return sizes_taken(d, dv) ? 1 : 0; }

#define RLIS_AB_DISPATCH(CALL)                                                         \
    if (d == 64 && dv == 32) { CALL(64, 32); } else if (d == 64 && dv == 64) { CALL(64, 64); } \
    else if (d == 64) { CALL(64, 128); } else if (dv == 32) { CALL(128, 32); }             \
    else if (dv == 64) { CALL(128, 64); } else { CALL(128, 128); }

// tiles: int32 [n_tiles][2] = (batch entry, first token of the tile within the entry's portion).
extern "C" int rlis_attention_bias_prefill(const void* q, const void* k_cache, const void* v_cache, void* out,
                                           const float* bias, int n_dist, const void* gate, long long gate_stride,
                                           const int* tiles, int n_tiles, const int* cu_seqlens, const int* ctx_lens,
                                           const int* block_tables, int max_blocks, int nh, int nkv, int d, int dv,
                                           int page_size, float scale, int window, const float* sinks,
                                           const float* slopes, int gate_cols, cudaStream_t stream) {
    if (n_tiles <= 0) return 0;
    if (!sizes_taken(d, dv) || nkv <= 0 || nh % nkv != 0 || n_tiles > 65535 || (bias != nullptr && n_dist <= 0) ||
        (gate != nullptr && gate_cols != 1 && gate_cols != dv))
        return RLIS_ERR_UNSUPPORTED;
    raise_all_once();
    dim3 grid(nh, n_tiles);
#define RLIS_AB_PF(D_, DV_) rlis_launch(attn_bias_prefill_kernel<D_, DV_>, grid, THREADS, smem_bytes<D_, DV_>(), stream, \
        (const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, (bf16*)out, bias, n_dist, (const bf16*)gate,      \
        gate_stride, tiles, cu_seqlens, ctx_lens, block_tables, max_blocks, nh, nkv, page_size, scale, window,        \
        sinks, slopes, gate_cols)
    RLIS_AB_DISPATCH(RLIS_AB_PF)
#undef RLIS_AB_PF
    return RLIS_LAUNCH_CHECK();
}

// partial: float32, at least n_dec * nh * pieces * (dv + 2) elements when pieces > 1.  sinks, slopes: float32 [nh] or null.
extern "C" int rlis_attention_bias_decode(const void* q, const void* k_cache, const void* v_cache, void* out,
                                          float* partial, const float* bias, int n_dist, const void* gate,
                                          long long gate_stride, const int* dec_rows, const int* dec_seqs,
                                          const int* ctx_lens, const int* block_tables, int max_blocks, int n_dec,
                                          int nh, int nkv, int d, int dv, int page_size, float scale, int window,
                                          int pieces, const float* sinks, const float* slopes, int gate_cols,
                                          cudaStream_t stream) {
    if (n_dec <= 0) return 0;
    if (!sizes_taken(d, dv) || nkv <= 0 || nh % nkv != 0 || nh / nkv > 16 || pieces < 1 || pieces > 65535 ||
        n_dec > 65535 || (bias != nullptr && n_dist <= 0) || (pieces > 1 && partial == nullptr) ||
        (gate != nullptr && gate_cols != 1 && gate_cols != dv))
        return RLIS_ERR_UNSUPPORTED;
    raise_all_once();
    dim3 grid(nkv, n_dec, pieces);
#define RLIS_AB_DEC(D_, DV_) rlis_launch(attn_bias_decode_kernel<D_, DV_>, grid, THREADS, decode_smem_bytes<D_, DV_>(), stream, \
        (const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, (bf16*)out, partial, bias, n_dist,                 \
        (const bf16*)gate, gate_stride, dec_rows, dec_seqs, ctx_lens, block_tables, max_blocks, nh, nkv, page_size,   \
        scale, window, pieces, sinks, slopes, gate_cols)
    RLIS_AB_DISPATCH(RLIS_AB_DEC)
#undef RLIS_AB_DEC
    int err = RLIS_LAUNCH_CHECK();
    if (err != 0 || pieces == 1) return err;
    const int units = n_dec * nh;
    rlis_launch(attn_bias_decode_merge_kernel, (units + 3) / 4, 128, 0, stream, (const float*)partial, (bf16*)out,
                (const bf16*)gate, gate_stride, dec_rows, units, nh, dv, pieces, sinks, gate_cols);
    return RLIS_LAUNCH_CHECK();
}

// Whether the kernel for single tokens with two maps a head takes these sizes (bfloat16).
extern "C" int rlis_attention_difference_decode_takes(int nh, int nkv, int d, int dv) {
    return nkv > 0 && nh % nkv == 0 && nh / nkv <= 8 && d > 0 && d <= 64 && d % 8 == 0 && dv > 0 && dv <= 128 && dv % 8 == 0;
}
// Width of a value row in the partial sums (values are padded to it).
extern "C" int rlis_attention_difference_decode_width(int dv) { return dv <= 64 ? 64 : 128; }

static void raise_difference_limits() {
    static bool done = false;
    if (done) return;
    cudaFuncSetAttribute(attn_difference_decode_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)difference_smem_bytes<64>());
    cudaFuncSetAttribute(attn_difference_decode_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)difference_smem_bytes<128>());
    cudaFuncSetAttribute(attn_difference_decode_kernel<64>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    cudaFuncSetAttribute(attn_difference_decode_kernel<128>, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    done = true;
}

// How many clusters of `pieces` CTAs the device holds at a time (0: none, or the query failed).
extern "C" int rlis_attention_difference_decode_resident(int dv, int pieces) {
    if (pieces < 1 || pieces > MAX_CLUSTER_PIECES) return 0;
    raise_difference_limits();
    const bool narrow = rlis_attention_difference_decode_width(dv) == 64;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(1, 1, (unsigned)pieces);
    cfg.blockDim = THREADS;
    cfg.dynamicSmemBytes = narrow ? difference_smem_bytes<64>() : difference_smem_bytes<128>();
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1;
    attr[0].val.clusterDim.y = 1;
    attr[0].val.clusterDim.z = (unsigned)pieces;
    cfg.attrs = attr;
    cfg.numAttrs = 1;
    int n = 0;
    const cudaError_t e = narrow ? cudaOccupancyMaxActiveClusters(&n, attn_difference_decode_kernel<64>, &cfg)
                                 : cudaOccupancyMaxActiveClusters(&n, attn_difference_decode_kernel<128>, &cfg);
    if (e != cudaSuccess) {
        cudaGetLastError();
        return 0;
    }
    return n;
}

// Up to this many pieces of a context merge inside a cluster.
extern "C" int rlis_attention_difference_decode_cluster() { return MAX_CLUSTER_PIECES; }

// partial: float32, at least n_dec * nh * 2 * pieces * (width(dv) + 2) elements when the pieces do not merge in a cluster; the rest as
// rlis_attention_difference.
extern "C" int rlis_attention_difference_decode(const void* q, const void* k_cache, const void* v_cache, void* out, float* partial,
                                                const void* gate, long long gate_stride, const int* dec_rows, const int* dec_seqs,
                                                const int* ctx_lens, const int* block_tables, int max_blocks, int n_dec, int nh,
                                                int nkv, int d, int dv, int page_size, float scale, float cap, int window, int pieces,
                                                float lambda, float out_scale, float eps, cudaStream_t stream) {
    if (n_dec <= 0) return 0;
    if (!rlis_attention_difference_decode_takes(nh, nkv, d, dv) || pieces < 1 || pieces > 65535 || n_dec > 65535 || cap < 0.f ||
        (pieces > MAX_CLUSTER_PIECES && partial == nullptr) ||
        ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache)) & 15) != 0)
        return RLIS_ERR_UNSUPPORTED;
    raise_difference_limits();
    const DiffDecode a{(const bf16*)q, (const bf16*)k_cache, (const bf16*)v_cache, (bf16*)out, partial, (const bf16*)gate, gate_stride,
                       dec_rows, dec_seqs, ctx_lens, block_tables, max_blocks, nh, nkv, d, dv, page_size, window, pieces,
                       pieces > 1 && pieces <= MAX_CLUSTER_PIECES ? 1 : 0, scale, cap, lambda, out_scale, eps};
    const dim3 grid(nkv, n_dec, pieces);
    const bool narrow = rlis_attention_difference_decode_width(dv) == 64;
    const dim3 cluster(1, 1, a.cluster ? (unsigned)pieces : 1u);
    if (narrow) rlis_launch_cluster(attn_difference_decode_kernel<64>, grid, THREADS, difference_smem_bytes<64>(), stream, cluster, a);
    else rlis_launch_cluster(attn_difference_decode_kernel<128>, grid, THREADS, difference_smem_bytes<128>(), stream, cluster, a);
    const int err = RLIS_LAUNCH_CHECK();
    if (err != 0 || pieces == 1 || a.cluster) return err;
    const int units = n_dec * nh;
    if (narrow) rlis_launch(attn_difference_merge_kernel<64>, (units + 3) / 4, 128, 0, stream, a, units);
    else rlis_launch(attn_difference_merge_kernel<128>, (units + 3) / 4, 128, 0, stream, a, units);
    return RLIS_LAUNCH_CHECK();
}
