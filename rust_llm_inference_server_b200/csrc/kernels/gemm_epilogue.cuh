// What the epilogue warps of the tcgen05 products do with 32 consecutive float32 sums of one row.
#pragma once
#include "common.cuh"
#include "mma_utils.cuh"
#include <math.h>

namespace tc {

// Parameters of the gated epilogue with clipping (EPI 3): g' sigmoid(slope g') (u' + shift) with g' = min(g,
// limit) and u' = clamp(u, -limit, limit); limit +inf clips nothing; slope +inf: max(g', 0) (u' + shift); the gate's
// argument is g' + cubic g'^3.  bias (float32, one
// a column; null: none) is added to g and u first.
struct GluParams {
    float slope, limit, shift;
    const float* bias;
    float cubic;
};

// The bias of 32 columns, one a lane (requested before the sums are read), and its addition to every lane's row of sums.
__device__ __forceinline__ float bias_of_lane(const GluParams& gp, int col, int lane, int N) {
    return gp.bias != nullptr && col + lane < N ? gp.bias[col + lane] : 0.f;
}
__device__ __forceinline__ void add_bias32(uint32_t (&r)[32], float bias) {
#pragma unroll
    for (int i = 0; i < 32; ++i) r[i] = __float_as_uint(__uint_as_float(r[i]) + __shfl_sync(0xffffffffu, bias, i));
}

// EPI 0: bf16 y [M, N].  EPI 1: SwiGLU over a gate|up matrix whose rows are interleaved in blocks of
// 4 (columns 8 t .. 8 t + 3 gate, 8 t + 4 .. 8 t + 7 up), y [M, N / 2] bf16.  EPI 2: float32 y [M, N].
// EPI 3: the layout of EPI 1 with the clipped gating of GluParams.
// r: the sums of columns col .. col + 31 of row `row`; columns from N on are not stored.
template <int EPI>
__device__ __forceinline__ void store_sums32(const uint32_t (&r)[32], void* __restrict__ y, int row, int col, int N,
                                             const GluParams& gp) {
    if (EPI == 0) {
        bf16* o = reinterpret_cast<bf16*>(y) + (size_t)row * N + col;
#pragma unroll
        for (int v = 0; v < 4; ++v) {
            if (col + v * 8 >= N) break;
            uint4 pk;
            pk.x = pack_bf16(__uint_as_float(r[v * 8 + 0]), __uint_as_float(r[v * 8 + 1]));
            pk.y = pack_bf16(__uint_as_float(r[v * 8 + 2]), __uint_as_float(r[v * 8 + 3]));
            pk.z = pack_bf16(__uint_as_float(r[v * 8 + 4]), __uint_as_float(r[v * 8 + 5]));
            pk.w = pack_bf16(__uint_as_float(r[v * 8 + 6]), __uint_as_float(r[v * 8 + 7]));
            *reinterpret_cast<uint4*>(o + v * 8) = pk;
        }
    } else if (EPI == 1 || EPI == 3) {
        bf16* o = reinterpret_cast<bf16*>(y) + (size_t)row * (N >> 1) + (col >> 1);
        float res[16];
        if (EPI == 3 && gp.cubic != 0.f && gp.limit == INFINITY && gp.shift == 0.f) {
            // a gate of the gelu kind, without the branches of the general one: its result is rounded to bfloat16, so the
            // fast exponential and division serve
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                const float g = __uint_as_float(r[(i >> 2) * 8 + (i & 3)]), u = __uint_as_float(r[(i >> 2) * 8 + 4 + (i & 3)]);
                const float z = fmaf(gp.cubic * g * g, g, g);
                res[i] = __fdividef(g, 1.0f + __expf(-gp.slope * z)) * u;
            }
        } else
#pragma unroll
        for (int tt = 0; tt < 4; ++tt)
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float gt = __uint_as_float(r[tt * 8 + j]), up = __uint_as_float(r[tt * 8 + 4 + j]);
                if (EPI == 1) {
                    res[tt * 4 + j] = gt / (1.0f + expf(-gt)) * up;
                } else {
                    const float g = fminf(gt, gp.limit), u = fminf(fmaxf(up, -gp.limit), gp.limit);
                    res[tt * 4 + j] = glu_gate(g, gp.slope, gp.cubic) * (u + gp.shift);
                }
            }
#pragma unroll
        for (int v = 0; v < 2; ++v) {
            if (col + v * 16 >= N) break;
            uint4 pk;
            pk.x = pack_bf16(res[v * 8 + 0], res[v * 8 + 1]);
            pk.y = pack_bf16(res[v * 8 + 2], res[v * 8 + 3]);
            pk.z = pack_bf16(res[v * 8 + 4], res[v * 8 + 5]);
            pk.w = pack_bf16(res[v * 8 + 6], res[v * 8 + 7]);
            *reinterpret_cast<uint4*>(o + v * 8) = pk;
        }
    } else {
        float* o = reinterpret_cast<float*>(y) + (size_t)row * N + col;
#pragma unroll
        for (int v = 0; v < 8; ++v) {
            if (col + v * 4 >= N) break;
            *reinterpret_cast<float4*>(o + v * 4) = make_float4(
                __uint_as_float(r[v * 4]), __uint_as_float(r[v * 4 + 1]), __uint_as_float(r[v * 4 + 2]),
                __uint_as_float(r[v * 4 + 3]));
        }
    }
}

}  // namespace tc
