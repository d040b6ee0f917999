// Residual streams side by side (hyper-connections), and norms without statistics.  One pass over a token's row joins a
// sublayer's result to the streams and makes the input of the sublayer that follows:
//
//   x_t <- sum_s mix[s, t] x_s + out[t] (y + y_bias)     with the old x_s on the right (only when y is given)
//   u    = sum_t in[t] x_t                               (in null: the plain sum)
//   h    = norm(u)                                       rounded once to the activation type
//
// norm 0: u itself; 1: tanh(alpha u) * w + b (dynamic tanh: no mean, no variance); 2: u / sqrt(mean(u^2) + eps) * w.
// mix null: the streams stay themselves (x_t <- x_t + out[t] y); out null: ones.  With one stream and neither, this is the
// residual addition and the norm of an ordinary pre-norm block.
//
// x is float32 [token, stream, width]; a stream stride of 0 reads one row as every stream (what an embedding leaves: the
// streams start equal and are written apart by the first update).  With a row list, output row i is made from source row
// rows[i] and the streams stay as they are.  Everything is float32; a thread owns its columns of all streams, so the
// update is in place, and the order of every sum depends on S (and, for norm 2, the width) only.
#include "common.cuh"
#include <math.h>

namespace {
constexpr int THREADS = 256;
constexpr int MAX_STREAMS = 8;

struct NormArgs {
    int kind;
    float alpha, eps;
    const float *w, *b;
};

template <typename T, int VN> __device__ __forceinline__ void load_n(const T* p, float (&v)[VN]);
template <> __device__ __forceinline__ void load_n<float, 1>(const float* p, float (&v)[1]) { v[0] = *p; }
template <> __device__ __forceinline__ void load_n<bf16, 1>(const bf16* p, float (&v)[1]) { v[0] = __bfloat162float(*p); }
template <> __device__ __forceinline__ void load_n<float, 4>(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
template <> __device__ __forceinline__ void load_n<bf16, 4>(const bf16* p, float (&v)[4]) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
template <typename T, int VN> __device__ __forceinline__ void store_n(T* p, const float (&v)[VN]);
template <> __device__ __forceinline__ void store_n<float, 1>(float* p, const float (&v)[1]) { *p = v[0]; }
template <> __device__ __forceinline__ void store_n<bf16, 1>(bf16* p, const float (&v)[1]) { *p = __float2bfloat16_rn(v[0]); }
template <> __device__ __forceinline__ void store_n<float, 4>(float* p, const float (&v)[4]) {
    *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
}
template <> __device__ __forceinline__ void store_n<bf16, 4>(bf16* p, const float (&v)[4]) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    uint2 raw;
    raw.x = *reinterpret_cast<uint32_t*>(&a);
    raw.y = *reinterpret_cast<uint32_t*>(&b);
    *reinterpret_cast<uint2*>(p) = raw;
}

// SM: streams kept in registers (S <= SM).  A row is shared by gridDim.y CTAs unless the norm needs its mean square.
template <typename T, int SM, int VN>
__global__ __launch_bounds__(THREADS) void stream_mix_kernel(
    const float* x, long long x_row, long long x_stream, int S, const T* __restrict__ y, const float* __restrict__ y_bias,
    const float* __restrict__ mix, const float* __restrict__ out_c, float* x_out, const float* __restrict__ in_c,
    const NormArgs nm, T* __restrict__ h, float* u_out, const int* __restrict__ rows, int width) {
    pdl_wait_and_trigger();
    extern __shared__ float row_u[];               // norm 2: the row of u
    __shared__ float scratch[33];
    __shared__ float cm[SM * SM], co[SM], ci[SM];
    if (threadIdx.x < SM * SM) {
        const int s = threadIdx.x / SM, t = threadIdx.x % SM;
        cm[threadIdx.x] = s < S && t < S ? (mix != nullptr ? mix[s * S + t] : (s == t ? 1.f : 0.f)) : 0.f;
    }
    if (threadIdx.x < SM) {
        co[threadIdx.x] = threadIdx.x < S ? (out_c != nullptr ? out_c[threadIdx.x] : 1.f) : 0.f;
        ci[threadIdx.x] = threadIdx.x < S ? (in_c != nullptr ? in_c[threadIdx.x] : 1.f) : 0.f;
    }
    __syncthreads();
    const size_t src = rows != nullptr ? (size_t)rows[blockIdx.x] : (size_t)blockIdx.x;
    const float* xr = x + src * x_row;
    float ss = 0.f;
    for (int c = (blockIdx.y * THREADS + threadIdx.x) * VN; c < width; c += gridDim.y * THREADS * VN) {
        float v[SM][VN], u[VN];
#pragma unroll
        for (int s = 0; s < SM; ++s) {
            if (s < S) {
                load_n<float, VN>(xr + s * x_stream + c, v[s]);
            } else {
#pragma unroll
                for (int i = 0; i < VN; ++i) v[s][i] = 0.f;
            }
        }
#pragma unroll
        for (int i = 0; i < VN; ++i) u[i] = 0.f;
        if (y != nullptr) {
            float yv[VN];
            load_n<T, VN>(y + src * width + c, yv);
            if (y_bias != nullptr) {
                float bv[VN];
                load_n<float, VN>(y_bias + c, bv);
#pragma unroll
                for (int i = 0; i < VN; ++i) yv[i] += bv[i];
            }
#pragma unroll
            for (int t = 0; t < SM; ++t) {
                if (t >= S) break;
                float a[VN];
#pragma unroll
                for (int i = 0; i < VN; ++i) a[i] = 0.f;
#pragma unroll
                for (int s = 0; s < SM; ++s)
#pragma unroll
                    for (int i = 0; i < VN; ++i) a[i] = fmaf(cm[s * SM + t], v[s][i], a[i]);
#pragma unroll
                for (int i = 0; i < VN; ++i) {
                    a[i] = fmaf(co[t], yv[i], a[i]);
                    u[i] = fmaf(ci[t], a[i], u[i]);
                }
                if (x_out != nullptr && rows == nullptr) store_n<float, VN>(x_out + (src * S + t) * width + c, a);
            }
        } else {
#pragma unroll
            for (int t = 0; t < SM; ++t)
#pragma unroll
                for (int i = 0; i < VN; ++i) u[i] = fmaf(ci[t], v[t][i], u[i]);
        }
        if (u_out != nullptr) store_n<float, VN>(u_out + (size_t)blockIdx.x * width + c, u);
        if (h == nullptr) continue;
        if (nm.kind == 2) {
#pragma unroll
            for (int i = 0; i < VN; ++i) {
                ss = fmaf(u[i], u[i], ss);
                row_u[c + i] = u[i];
            }
            continue;
        }
        if (nm.kind == 1) {
            float w[VN], b[VN];
            load_n<float, VN>(nm.w + c, w);
            load_n<float, VN>(nm.b + c, b);
#pragma unroll
            for (int i = 0; i < VN; ++i) u[i] = fmaf(tanhf(nm.alpha * u[i]), w[i], b[i]);
        }
        store_n<T, VN>(h + (size_t)blockIdx.x * width + c, u);
    }
    if (nm.kind == 2 && h != nullptr) {
        const float r = 1.0f / sqrtf(block_sum(ss, scratch) / (float)width + nm.eps);
        for (int c = threadIdx.x * VN; c < width; c += THREADS * VN) {     // what this thread wrote itself
            float w[VN], o[VN];
            load_n<float, VN>(nm.w + c, w);
#pragma unroll
            for (int i = 0; i < VN; ++i) o[i] = row_u[c + i] * r * w[i];
            store_n<T, VN>(h + (size_t)blockIdx.x * width + c, o);
        }
    }
}

// out[t, part] = g / sqrt(mean over the part of g^2 + eps) * w with g = x silu(z): first gated, then normed, each of
// gridDim.y equal parts of a row has a root mean square of its own.  One CTA a (token, part).
template <typename T, int VN>
__global__ __launch_bounds__(THREADS) void gate_group_norm_kernel(
    const float* __restrict__ x, const T* __restrict__ z, long long z_stride, const float* __restrict__ w, T* __restrict__ out,
    int width, int part, float eps) {
    pdl_wait_and_trigger();
    __shared__ float scratch[33];
    const float* xr = x + (size_t)blockIdx.x * width + blockIdx.y * part;
    const T* zr = z + (size_t)blockIdx.x * z_stride + blockIdx.y * part;
    const float* wr = w + blockIdx.y * part;
    T* orow = out + (size_t)blockIdx.x * width + blockIdx.y * part;
    constexpr int KEEP = 4;                        // vectors a thread keeps; wider parts are gated again in the second pass
    float kept[KEEP][VN];
    float ss = 0.f;
    auto gated = [&](int c, float (&g)[VN]) {
        float zv[VN];
        load_n<float, VN>(xr + c, g);
        load_n<T, VN>(zr + c, zv);
#pragma unroll
        for (int i = 0; i < VN; ++i) g[i] *= zv[i] / (1.0f + expf(-zv[i]));
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int c = (k * blockDim.x + threadIdx.x) * VN;
        if (c < part) {
            gated(c, kept[k]);
#pragma unroll
            for (int i = 0; i < VN; ++i) ss = fmaf(kept[k][i], kept[k][i], ss);
        }
    }
    for (int c = (KEEP * blockDim.x + threadIdx.x) * VN; c < part; c += blockDim.x * VN) {
        float g[VN];
        gated(c, g);
#pragma unroll
        for (int i = 0; i < VN; ++i) ss = fmaf(g[i], g[i], ss);
    }
    const float r = 1.0f / sqrtf(block_sum(ss, scratch) / (float)part + eps);
    auto write = [&](int c, const float (&g)[VN]) {
        float wv[VN], o[VN];
        load_n<float, VN>(wr + c, wv);
#pragma unroll
        for (int i = 0; i < VN; ++i) o[i] = g[i] * r * wv[i];
        store_n<T, VN>(orow + c, o);
    };
#pragma unroll
    for (int k = 0; k < KEEP; ++k) {
        const int c = (k * blockDim.x + threadIdx.x) * VN;
        if (c < part) write(c, kept[k]);
    }
    for (int c = (KEEP * blockDim.x + threadIdx.x) * VN; c < part; c += blockDim.x * VN) {
        float g[VN];
        gated(c, g);
        write(c, g);
    }
}

bool aligned16(const void* p) { return ((uintptr_t)p & 15) == 0; }
}  // namespace

// x float32 rows x_row floats apart, streams x_stream apart (0: one row is every stream); y, h [T, width] in the element
// type (h null: not made); y_bias, w, b float32 [width]; mix float32 [S, S] (from, to), out_c, in_c float32 [S]; x_out
// float32 [T, S, width] (null: not written; may be x itself); u_out float32 (null: not wanted).
extern "C" int rlis_stream_mix(const float* x, long long x_row, long long x_stream, int n_streams, const void* y,
                               const float* y_bias, const float* mix, const float* out_c, float* x_out, const float* in_c,
                               int norm, float alpha, float eps, const float* w, const float* b, void* h, float* u_out,
                               const int* rows, int n_rows, int width, int dtype, cudaStream_t stream) {
    if (n_rows <= 0) return 0;
    if (n_streams < 1 || n_streams > MAX_STREAMS || width <= 0 || norm < 0 || norm > 2 || (norm > 0 && h != nullptr && w == nullptr) ||
        (norm == 1 && h != nullptr && b == nullptr))
        return RLIS_ERR_UNSUPPORTED;
    const NormArgs nm{norm, alpha, eps, w, b};
    const bool rms = norm == 2 && h != nullptr;
    const size_t smem = rms ? (size_t)width * sizeof(float) : 0;
    if (smem > 40 * 1024) return RLIS_ERR_UNSUPPORTED;
    const bool quads = width % 4 == 0 && x_row % 4 == 0 && x_stream % 4 == 0 && aligned16(x) && aligned16(y) && aligned16(h) &&
                       aligned16(x_out) && aligned16(u_out) && aligned16(y_bias) && aligned16(w) && aligned16(b);
    const int vn = quads ? 4 : 1;
    // few rows: a row is cut into pieces so that its loads are spread over the SMs
    const int pieces = rms ? 1 : n_rows >= 512 ? 1 : (width + THREADS * vn - 1) / (THREADS * vn);
    const dim3 grid(n_rows, pieces);
#define RLIS_MIX(T, SM, VN) rlis_launch(stream_mix_kernel<T, SM, VN>, grid, THREADS, smem, stream, x, x_row, x_stream, n_streams, \
                                        (const T*)y, y_bias, mix, out_c, x_out, in_c, nm, (T*)h, u_out, rows, width)
#define RLIS_MIX_S(T, VN)                                \
    do {                                                 \
        if (n_streams == 1) RLIS_MIX(T, 1, VN);          \
        else if (n_streams == 2) RLIS_MIX(T, 2, VN);     \
        else if (n_streams <= 4) RLIS_MIX(T, 4, VN);     \
        else RLIS_MIX(T, 8, VN);                         \
    } while (0)
    if (dtype == RLIS_F32) { if (quads) RLIS_MIX_S(float, 4); else RLIS_MIX_S(float, 1); }
    else if (dtype == RLIS_BF16) { if (quads) RLIS_MIX_S(bf16, 4); else RLIS_MIX_S(bf16, 1); }
    else return RLIS_ERR_UNSUPPORTED;
#undef RLIS_MIX_S
#undef RLIS_MIX
    return RLIS_LAUNCH_CHECK();
}

// x float32 [T, width]; z [T, width] in the element type, rows z_stride apart; w float32 [width]; out [T, width].
extern "C" int rlis_gate_group_norm(const float* x, const void* z, long long z_stride, const float* w, void* out, int n_tokens,
                                    int width, int groups, float eps, int dtype, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (width <= 0 || groups <= 0 || groups > 65535 || width % groups != 0) return RLIS_ERR_UNSUPPORTED;
    const int part = width / groups;
    const bool quads = part % 4 == 0 && z_stride % 4 == 0 && aligned16(x) && aligned16(w) && aligned16(out) &&
                       ((uintptr_t)z & (dtype == RLIS_F32 ? 15 : 7)) == 0;
    const int per = (part + (quads ? 3 : 0)) / (quads ? 4 : 1);
    const int threads = per <= 64 ? 64 : per <= 128 ? 128 : THREADS;
    const dim3 grid(n_tokens, groups);
#define RLIS_GGN(T, VN) rlis_launch(gate_group_norm_kernel<T, VN>, grid, threads, 0, stream, x, (const T*)z, z_stride, w, (T*)out, \
                                    width, part, eps)
    if (dtype == RLIS_F32) { if (quads) RLIS_GGN(float, 4); else RLIS_GGN(float, 1); }
    else if (dtype == RLIS_BF16) { if (quads) RLIS_GGN(bf16, 4); else RLIS_GGN(bf16, 1); }
    else return RLIS_ERR_UNSUPPORTED;
#undef RLIS_GGN
    return RLIS_LAUNCH_CHECK();
}
