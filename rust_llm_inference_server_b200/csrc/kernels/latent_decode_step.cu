// What a step of a few single tokens needs around attention over latent rows (bfloat16, up to 16 tokens), where the library's
// batched product and three small kernels would each cost a launch:
//
//   per_head_small : out[t, h, n] = sum_k W[h, n, k] a[t, h, k], one small matrix a head (the key map folded into queries, the
//                    value map applied to the sums over latents).  mma.sync m16n8k16: 16 rows of a head's matrix are the M
//                    side, the tokens the N side, so every weight is read once, by 16-byte loads straight into the operand
//                    registers: a lane takes 8 consecutive k of its rows and tokens and hands them to the products as pairs (a
//                    product does not mind in which order it sums, as long as both sides agree).  The weights do not depend on
//                    the kernel before and are requested before the wait for it.
//   latent_step    : the folding of the key map into the queries, the rotation of the queries' other part, and the row that the
//                    cache keeps of every token (norm of the latent, rotation of the shared key part), in one launch: behind the
//                    CTAs that fold come one a token for its row and some for the queries' rotations, a pair a thread.
//
// Sums are float32.  Rotation and norm are those of attention_latent.cu.
#include "common.cuh"
#include "mma_utils.cuh"
#include <math.h>

namespace {
constexpr int MAX_T = 16;
constexpr int AHEAD = 4;        // blocks of 32 k whose weights are requested before the wait

struct SmallProduct {
    const bf16* a;              // [T, H, K]: token rows a_row apart, heads a_head apart
    long long a_row, a_head;
    const bf16* w;              // [H, N, K]
    bf16* out;                  // [T, H, N]: token rows o_row apart, heads o_head apart
    long long o_row, o_head;
    int T, H, N, K;
};

__device__ __forceinline__ uint4 ld16(const bf16* p, bool valid) {
    return valid ? *reinterpret_cast<const uint4*>(p) : make_uint4(0u, 0u, 0u, 0u);
}

// The four warps of a CTA and the 16-row tiles of head h: SPLIT, all four take tile `tile` and a quarter of k each; else warp w
// takes tile `tile` * 4 + w.  `red` holds 4 * 16 * 16 floats when SPLIT.
template <bool SPLIT>
__device__ __forceinline__ void small_product(const SmallProduct& s, int h, int tile, float* red) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, c = lane & 3;
    const int n0 = (SPLIT ? tile : tile * 4 + warp) * 16;
    const int blocks = (s.K + 31) / 32;
    const int per = SPLIT ? (blocks + 3) / 4 : blocks;
    const int kb0 = SPLIT ? warp * per : 0, kb1 = min(kb0 + per, blocks);
    const bf16* w0 = s.w + ((size_t)h * s.N + n0 + g) * s.K + 8 * c;
    const bf16* w1 = w0 + (size_t)8 * s.K;
    const bool r0 = n0 + g < s.N, r1 = n0 + g + 8 < s.N;
    uint4 x0[AHEAD], x1[AHEAD];
#pragma unroll
    for (int i = 0; i < AHEAD; ++i) {
        const int k = (kb0 + i) * 32;
        const bool in = kb0 + i < kb1 && k + 8 * c < s.K;
        x0[i] = ld16(w0 + k, in && r0);
        x1[i] = ld16(w1 + k, in && r1);
    }
    pdl_wait_and_trigger();
    const bf16* a0 = s.a + (size_t)g * s.a_row + (size_t)h * s.a_head + 8 * c;
    const bf16* a1 = a0 + (size_t)8 * s.a_row;
    const bool t0 = g < s.T, t1 = g + 8 < s.T;
    const bool wide = s.T > 8;
    float acc[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
    auto block = [&](const uint4& p0, const uint4& p1, int k) {
        const bool in = k + 8 * c < s.K;
        const uint4 b = ld16(a0 + k, in && t0);
        const uint32_t f0[4] = {p0.x, p1.x, p0.y, p1.y}, f1[4] = {p0.z, p1.z, p0.w, p1.w};
        mma_bf16_16816(acc[0], f0, b.x, b.y);
        mma_bf16_16816(acc[0], f1, b.z, b.w);
        if (wide) {
            const uint4 b2 = ld16(a1 + k, in && t1);
            mma_bf16_16816(acc[1], f0, b2.x, b2.y);
            mma_bf16_16816(acc[1], f1, b2.z, b2.w);
        }
    };
#pragma unroll
    for (int i = 0; i < AHEAD; ++i)
        if (kb0 + i < kb1) block(x0[i], x1[i], (kb0 + i) * 32);
    for (int kb = kb0 + AHEAD; kb < kb1; ++kb) {
        const int k = kb * 32;
        const bool in = k + 8 * c < s.K;
        block(ld16(w0 + k, in && r0), ld16(w1 + k, in && r1), k);
    }
    if constexpr (SPLIT) {
        // rows of 16 features a token, added in the order of the warps
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e)
                red[(warp * MAX_T + j * 8 + 2 * c + (e & 1)) * 16 + g + 8 * (e >> 1)] = acc[j][e];
        __syncthreads();
        for (int i = threadIdx.x; i < MAX_T * 16; i += 128) {
            const int t = i >> 4, n = n0 + (i & 15);
            const float v = (red[i] + red[MAX_T * 16 + i]) + (red[2 * MAX_T * 16 + i] + red[3 * MAX_T * 16 + i]);
            if (t < s.T && n < s.N) s.out[(size_t)t * s.o_row + (size_t)h * s.o_head + n] = __float2bfloat16_rn(v);
        }
    } else {
#pragma unroll
        for (int j = 0; j < 2; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = j * 8 + 2 * c + (e & 1), n = n0 + g + 8 * (e >> 1);
                if (t < s.T && n < s.N) s.out[(size_t)t * s.o_row + (size_t)h * s.o_head + n] = __float2bfloat16_rn(acc[j][e]);
            }
    }
}

template <bool SPLIT>
__global__ __launch_bounds__(128) void per_head_small_kernel(const SmallProduct s, int tiles) {
    __shared__ float red[SPLIT ? 4 * MAX_T * 16 : 1];
    small_product<SPLIT>(s, blockIdx.x / tiles, blockIdx.x % tiles, red);
}

struct LatentStep {
    SmallProduct fold;          // a: the queries' plain parts, out: the first `rank` entries of qa
    int fold_ctas, tiles;
    const bf16* q_rot;          // [T, H, rot]: strides as fold.a's
    const bf16* z;              // [T, rank + rot]: the latent and the shared key part of the same rows
    long long z_row;
    const float *w, *inv_freq;
    const int *positions, *slots;
    bf16* cache;
    int rank, rot, rot_dims;
    float mag, eps;
    int units;                  // of a head's rotated part: its pairs, and the entries that pass
};

__device__ __forceinline__ float turned(const bf16* x, int i, int rot_dims, const float* inv_freq, float pos, float mag) {
    const float v = __bfloat162float(x[i]);
    if (i >= rot_dims) return v;
    const int half = rot_dims / 2, j = i < half ? i : i - half;
    float s, c;
    sincosf(pos * inv_freq[j], &s, &c);
    s *= mag;
    c *= mag;
    const float a = __bfloat162float(x[j]), b = __bfloat162float(x[j + half]);
    return i < half ? rope_first(a, b, c, s) : rope_second(a, b, c, s);
}

__global__ __launch_bounds__(128) void latent_step_kernel(const LatentStep s) {
    if ((int)blockIdx.x < s.fold_ctas) {
        small_product<false>(s.fold, blockIdx.x / s.tiles, blockIdx.x % s.tiles, nullptr);
        return;
    }
    pdl_wait_and_trigger();
    if ((int)blockIdx.x >= s.fold_ctas + s.fold.T) {
        const int idx = (blockIdx.x - s.fold_ctas - s.fold.T) * 128 + threadIdx.x, u = idx % s.units, th = idx / s.units;
        if (th >= s.fold.T * s.fold.H) return;
        const int t = th / s.fold.H, h = th - t * s.fold.H, half = s.rot_dims / 2;
        const bf16* x = s.q_rot + (size_t)t * s.fold.a_row + (size_t)h * s.fold.a_head;
        bf16* o = s.fold.out + (size_t)t * s.fold.o_row + (size_t)h * s.fold.o_head + s.rank;
        if (u >= half) {
            o[half + u] = x[half + u];
            return;
        }
        float sn, cs;
        sincosf((float)s.positions[t] * s.inv_freq[u], &sn, &cs);
        sn *= s.mag;
        cs *= s.mag;
        const float a = __bfloat162float(x[u]), b = __bfloat162float(x[u + half]);
        o[u] = __float2bfloat16_rn(rope_first(a, b, cs, sn));
        o[u + half] = __float2bfloat16_rn(rope_second(a, b, cs, sn));
        return;
    }
    __shared__ float scratch[33];
    const int t = blockIdx.x - s.fold_ctas;
    const float pos = (float)s.positions[t];
    const bf16* zr = s.z + (size_t)t * s.z_row;
    const int slot = s.slots != nullptr ? s.slots[t] : -1;
    float ss = 0.f;
    for (int i = threadIdx.x; i < s.rank; i += 128) {
        const float v = __bfloat162float(zr[i]);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    if (slot >= 0) {
        const float r = 1.0f / sqrtf(ss / (float)s.rank + s.eps);
        bf16* row = s.cache + (size_t)slot * (s.rank + s.rot);
        for (int i = threadIdx.x; i < s.rank; i += 128) row[i] = __float2bfloat16_rn(__bfloat162float(zr[i]) * r * s.w[i]);
        for (int i = threadIdx.x; i < s.rot; i += 128)
            row[s.rank + i] = __float2bfloat16_rn(turned(zr + s.rank, i, s.rot_dims, s.inv_freq, pos, s.mag));
    }
}

bool takes(const SmallProduct& s) {
    return s.T > 0 && s.T <= MAX_T && s.H > 0 && s.N > 0 && s.K > 0 && s.K % 8 == 0 && s.a_row % 8 == 0 && s.a_head % 8 == 0 &&
           ((reinterpret_cast<uintptr_t>(s.a) | reinterpret_cast<uintptr_t>(s.w)) & 15) == 0;
}
}  // namespace

// a [T, H, K] (rows a_row, heads a_head elements apart: multiples of 8), w [H, N, K], out [T, H, N] (o_row, o_head); bfloat16, T
// up to 16, K a multiple of 8, a and w on 16-byte boundaries.
extern "C" int rlis_per_head_small(const void* a, long long a_row, long long a_head, const void* w, void* out, long long o_row,
                                   long long o_head, int T, int H, int N, int K, cudaStream_t stream) {
    if (T == 0) return 0;
    const SmallProduct s{(const bf16*)a, a_row, a_head, (const bf16*)w, (bf16*)out, o_row, o_head, T, H, N, K};
    if (!takes(s)) return RLIS_ERR_UNSUPPORTED;
    const bool split = K >= 256;
    const int tiles = split ? (N + 15) / 16 : (N + 63) / 64;
    if (split) rlis_launch(per_head_small_kernel<true>, (unsigned)(H * tiles), 128, 0, stream, s, tiles);
    else rlis_launch(per_head_small_kernel<false>, (unsigned)(H * tiles), 128, 0, stream, s, tiles);
    return RLIS_LAUNCH_CHECK();
}

// q [T, H (d + rot)] (rows q_row apart, a multiple of 8), z [T, rank + rot] (rows z_row apart); k_fold [H, rank, d]; qa [T, H,
// rank + rot]; slots null: nothing is stored.  d, d + rot multiples of 8.
extern "C" int rlis_latent_step(const void* q, long long q_row, const void* z, long long z_row, const void* k_fold, const float* w,
                                const float* inv_freq, const int* positions, const int* slots, void* cache, void* qa, int T, int H,
                                int d, int rank, int rot, int rot_dims, float mag, float eps, cudaStream_t stream) {
    if (T == 0) return 0;
    if (rot < 0 || rot_dims < 0 || rot_dims > rot || rot_dims % 2) return RLIS_ERR_UNSUPPORTED;
    const long long dk = rank + rot;
    LatentStep s;
    s.fold = SmallProduct{(const bf16*)q, q_row, d + rot, (const bf16*)k_fold, (bf16*)qa, H * dk, dk, T, H, rank, d};
    if (!takes(s.fold)) return RLIS_ERR_UNSUPPORTED;
    s.tiles = (rank + 63) / 64;
    s.fold_ctas = H * s.tiles;
    s.q_rot = (const bf16*)q + d;
    s.z = (const bf16*)z;
    s.z_row = z_row;
    s.w = w;
    s.inv_freq = inv_freq;
    s.positions = positions;
    s.slots = slots;
    s.cache = (bf16*)cache;
    s.rank = rank;
    s.rot = rot;
    s.rot_dims = rot_dims;
    s.mag = mag;
    s.eps = eps;
    s.units = rot_dims / 2 + (rot - rot_dims);
    rlis_launch(latent_step_kernel, (unsigned)(s.fold_ctas + T + (T * H * s.units + 127) / 128), 128, 0, stream, s);
    return RLIS_LAUNCH_CHECK();
}
