// RMSNorm, or layer norm (CENTRE), over the float32 residual stream, fused with the residual addition that precedes it.
//
//   resid[t, :] += delta[t, :] (+ delta2[t, :])   (only what is given; float32 sums, stored as float32)
//   x            = resid[t, :], for the layer norm minus its mean over the row
//   out[t, :]    = x / sqrt(mean(x^2) + eps) * w                         (rounded once to T)
//
// The layer norm takes its variance from the squared deviations (a second pass over the row, held in registers), so a
// mean far from zero costs no digits.
//
// With a row list, output row i is computed from source row rows[i] (the rows whose logits are
// wanted) and the residual stream is left as it is.
//
// Formula: crates/model/src/layers.rs:141-146 (weight multiplies directly, eps as float32);
// the residual additions are crates/model/src/llama.rs:267,270.  Sum of squares and scale in
// float32; the order of the sum depends only on the width, never on the batch.
#include "common.cuh"

template <typename T, bool CENTRE>
__global__ void rmsnorm_kernel(float* __restrict__ resid, const T* __restrict__ delta, const T* __restrict__ delta2,
                               const float* __restrict__ w, T* __restrict__ out,
                               const int* __restrict__ rows, int hidden, float eps) {
    pdl_wait_and_trigger();
    __shared__ float scratch[33];
    const size_t obase = (size_t)blockIdx.x * hidden;
    const size_t base = rows != nullptr ? (size_t)rows[blockIdx.x] * hidden : obase;
    auto value = [&](int i) {
        float v = resid[base + i];
        if (delta != nullptr) v += to_f<T>(delta[base + i]) + (delta2 != nullptr ? to_f<T>(delta2[base + i]) : 0.f);
        return v;
    };
    // whole rows are stored back, and a thread reads its own entries again; with a row list the sum is formed again
    const bool keep = rows == nullptr && delta != nullptr;
    float ss = 0.f, sum = 0.f;
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
        const float v = value(i);
        if (keep) resid[base + i] = v;
        ss += v * v;
        sum += v;
    }
    auto again = [&](int i) { return keep ? resid[base + i] : value(i); };
    float mean = 0.f;
    if constexpr (CENTRE) {
        mean = block_sum(sum, scratch) / (float)hidden;
        ss = 0.f;
        for (int i = threadIdx.x; i < hidden; i += blockDim.x) {
            const float d = again(i) - mean;
            ss += d * d;
        }
    }
    ss = block_sum(ss, scratch);
    const float rstd = 1.0f / sqrtf(ss / (float)hidden + eps);
    for (int i = threadIdx.x; i < hidden; i += blockDim.x) out[obase + i] = from_f<T>((again(i) - mean) * rstd * w[i]);
}

// The same for widths that are multiples of 4: 16-byte accesses, and the row is kept
// in registers between the sum of squares and the scaling (up to 4 vectors a thread).
template <typename T> struct Delta4;
template <> struct Delta4<float> {
    static __device__ __forceinline__ float4 load(const float* p) { return *reinterpret_cast<const float4*>(p); }
    static __device__ __forceinline__ void store(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
};
template <> struct Delta4<bf16> {
    static __device__ __forceinline__ float4 load(const bf16* p) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
        const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        return make_float4(a.x, a.y, b.x, b.y);
    }
    static __device__ __forceinline__ void store(bf16* p, float4 v) {
        __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
        uint2 raw;
        raw.x = *reinterpret_cast<uint32_t*>(&a);
        raw.y = *reinterpret_cast<uint32_t*>(&b);
        *reinterpret_cast<uint2*>(p) = raw;
    }
};

template <typename T, bool CENTRE>
__global__ void rmsnorm_vec4_kernel(float* __restrict__ resid, const T* __restrict__ delta, const T* __restrict__ delta2,
                                    const float* __restrict__ w, T* __restrict__ out,
                                    const int* __restrict__ rows, int hidden, float eps) {
    __shared__ float scratch[33];
    constexpr int MAXV = 4;
    const size_t obase = (size_t)blockIdx.x * hidden;
    const size_t base = rows != nullptr ? (size_t)rows[blockIdx.x] * hidden : obase;
    const int nvec = hidden >> 2;
    float4 v[MAXV];
    pdl_wait_and_trigger();
    float ss = 0.f, sum = 0.f;
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = it * blockDim.x + threadIdx.x;
        if (i < nvec) {
            float4 x = *reinterpret_cast<const float4*>(resid + base + 4 * (size_t)i);
            if (delta != nullptr) {
                float4 dl = Delta4<T>::load(delta + base + 4 * (size_t)i);
                if (delta2 != nullptr) {
                    const float4 d2 = Delta4<T>::load(delta2 + base + 4 * (size_t)i);
                    dl.x += d2.x; dl.y += d2.y; dl.z += d2.z; dl.w += d2.w;
                }
                x.x += dl.x; x.y += dl.y; x.z += dl.z; x.w += dl.w;
                if (rows == nullptr) *reinterpret_cast<float4*>(resid + base + 4 * (size_t)i) = x;
            }
            v[it] = x;
            if constexpr (CENTRE) {
                sum += (x.x + x.y) + (x.z + x.w);
            } else {
                ss += x.x * x.x;
                ss += x.y * x.y;
                ss += x.z * x.z;
                ss += x.w * x.w;
            }
        }
    }
    if constexpr (CENTRE) {
        const float mean = block_sum(sum, scratch) / (float)hidden;
#pragma unroll
        for (int it = 0; it < MAXV; ++it) {
            if (it * blockDim.x + threadIdx.x < nvec) {
                float4& x = v[it];
                x.x -= mean; x.y -= mean; x.z -= mean; x.w -= mean;
                ss += (x.x * x.x + x.y * x.y) + (x.z * x.z + x.w * x.w);
            }
        }
    }
    ss = block_sum(ss, scratch);
    const float rstd = 1.0f / sqrtf(ss / (float)hidden + eps);
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = it * blockDim.x + threadIdx.x;
        if (i < nvec) {
            const float4 ww = *reinterpret_cast<const float4*>(w + 4 * (size_t)i);
            const float4 x = v[it];
            Delta4<T>::store(out + obase + 4 * (size_t)i,
                             make_float4(x.x * rstd * ww.x, x.y * rstd * ww.y, x.z * rstd * ww.z, x.w * rstd * ww.w));
        }
    }
}

// delta2: a second addition of the same row (a block whose sublayers stand side by side leaves two).
template <bool CENTRE>
static int launch_norm(float* resid, const void* delta, const void* delta2, const float* w, void* out, const int* rows, int n_tokens,
                       int hidden, float eps, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (delta == nullptr && delta2 != nullptr) return RLIS_ERR_UNSUPPORTED;
    int threads = hidden >= 2048 ? 512 : (hidden >= 512 ? 256 : 128);
    // many rows (portions of prompts): fewer threads with four vectors each keep more loads in
    // flight an SM (2048 rows of 2048: a 2048-token prefill of 16 layers 4.72 -> 4.64 ms)
    if (n_tokens > 64 && (hidden & 3) == 0) threads = min(threads, max(128, ((hidden + 15) / 16 + 31) / 32 * 32));
    const bool vec = (hidden & 3) == 0 && hidden <= threads * 16;
#define RLIS_NORM(KERNEL, T) rlis_launch(KERNEL<T, CENTRE>, n_tokens, threads, 0, stream, resid, (const T*)delta, (const T*)delta2, w, \
                                         (T*)out, rows, hidden, eps)
    if (dtype == RLIS_F32) { if (vec) RLIS_NORM(rmsnorm_vec4_kernel, float); else RLIS_NORM(rmsnorm_kernel, float); }
    else if (dtype == RLIS_BF16) { if (vec) RLIS_NORM(rmsnorm_vec4_kernel, bf16); else RLIS_NORM(rmsnorm_kernel, bf16); }
    else return RLIS_ERR_UNSUPPORTED;
#undef RLIS_NORM
    return RLIS_LAUNCH_CHECK();
}

extern "C" int rlis_rmsnorm(float* resid, const void* delta, const void* delta2, const float* w, void* out, const int* rows,
                            int n_tokens, int hidden, float eps, int dtype, cudaStream_t stream) {
    return launch_norm<false>(resid, delta, delta2, w, out, rows, n_tokens, hidden, eps, dtype, stream);
}

extern "C" int rlis_layer_norm(float* resid, const void* delta, const void* delta2, const float* w, void* out, const int* rows,
                               int n_tokens, int hidden, float eps, int dtype, cudaStream_t stream) {
    return launch_norm<true>(resid, delta, delta2, w, out, rows, n_tokens, hidden, eps, dtype, stream);
}
