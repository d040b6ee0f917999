// Single decoded tokens of attention with two maps a head (attention_difference.cu has the formulas), on mma.sync m16n8k16 with
// float32 sums.  One CTA of four warps = one key/value head x one request x one piece of its context.  Rows 0..7 of the products
// are the group's query heads' first maps, rows 8..15 their second ones; a cached key row is [map 1 | map 2], each padded to 64
// entries, and a query row is its map's vector with zeros over the other's entries, so one set of products gives both maps'
// scores and the values are read and multiplied once.
//
// Tiles of 64 keys arrive page by page by bulk tensor copies (TMA, 128-byte swizzle: K as two sub-tiles of 64 columns, V as one
// or two; a box a lane of the first warp; tensor maps of three dimensions fill maps narrower than 64 with zeros), three tiles
// deep; the first ones, if they hold none of this step's keys, are requested before the wait for the kernel before.  (By 16-byte
// asynchronous copies, the addresses of 32 copies a thread and tile were most of what a warp issued: 35 us for 8 requests at
// 4,096 keys and four key/value heads, 22 % of the memory's rate.)  Each warp takes 16 of a tile's keys with a running softmax of
// its own; the warps meet in shared memory.  Up to 16 pieces of a context are a thread-block cluster, which merges through
// distributed shared memory: a CTA a head of the group, a warp a quarter of its columns.  More pieces are merged by a second
// kernel.
//
// Every mbarrier wait is bounded (a fifth of a second); a wait that runs out sets the error word
// (rlis_attention_difference_decode_error) and the kernel runs to its end.
#include "tcgen05_utils.cuh"
#include <math.h>

namespace {
using namespace tc;
constexpr int WARPS = 4;
constexpr int THREADS = WARPS * 32;
constexpr int BN = 64;                 // keys per tile
constexpr int STAGES = 3;
constexpr int SUB = BN * 128;          // bytes of a swizzled sub-tile: 64 keys x 64 columns
constexpr float LOG2E = 1.4426950408889634f;
constexpr int MAX_CLUSTER_PIECES = 16;
constexpr int TABLE_SLICE = 512;       // page numbers of a CTA's piece kept in shared memory (longer pieces look them up as they go)

template <int DV> struct Tile {
    static constexpr int SUBS = 2 + DV / 64;
    static constexpr int BYTES = SUBS * SUB;
};
struct Ctrl {
    uint64_t full[STAGES];
    int abort;
    float red[WARPS];
    int pages[TABLE_SLICE];
};
template <int DV> constexpr size_t smem_bytes() { return (size_t)STAGES * Tile<DV>::BYTES + sizeof(Ctrl) + 1024 /* alignment */; }

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* map, int x, int y, int z, uint64_t* bar) {
    asm volatile(
        "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];"
        ::"r"(smem_u32(dst)), "l"(map), "r"(smem_u32(bar)), "r"(x), "r"(y), "r"(z)
        : "memory");
}

// 16-byte chunk `chunk` of row `row` of a swizzled sub-tile.
__device__ __forceinline__ const unsigned char* swizzled(const unsigned char* sub, int row, int chunk) {
    return sub + row * 128 + ((chunk ^ (row & 7)) << 4);
}

struct DiffDecode {
    const bf16* q;
    bf16* out;
    float* partial;           // several pieces: [n_dec][nh][map][pieces][DV + 2]
    const bf16* gate;         // logits, one a head, or null
    long long gate_stride;
    const int *dec_rows, *dec_seqs, *ctx_lens, *block_tables;
    int max_blocks, nh, nkv, d, dv, page_size, window, pieces;
    int cluster;              // 1: the pieces are a cluster and merge themselves
    int cache_rows;           // rows of the pools seen as [rows, ...]: pages * nkv * page_size
    float slope, top;         // with a cap: 2 log2(e) scale / cap and log2(e) cap; without: log2(e) scale and 0
    float lambda, out_scale, eps;
};

// A score in units of log2(e): log2(e) cap tanh(s scale / cap), or log2(e) s scale without a cap.
__device__ __forceinline__ float capped_log2(float s, const DiffDecode& a) {
    if (a.top <= 0.f) return s * a.slope;
    const float e = ex2(s * a.slope);                                                 // e^{2u}: tanh(u) = 1 - 2 / (1 + e^{2u})
    return fmaf(-2.0f * a.top, __fdividef(1.0f, 1.0f + fminf(e, 1e30f)), a.top);
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
            const float f = r[mcol] == -INFINITY ? 0.f : ex2(r[mcol] - m);
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
__global__ __launch_bounds__(THREADS) void attn_difference_decode_kernel(const __grid_constant__ CUtensorMap map_k,
                                                                         const __grid_constant__ CUtensorMap map_v, const DiffDecode a) {
    constexpr int KS = 8, ND = DV / 8;                     // k-steps of 16 over both maps; output tiles of 8 columns
    using TL = Tile<DV>;
    extern __shared__ unsigned char dd_smem_raw[];
    unsigned char* tiles = reinterpret_cast<unsigned char*>((reinterpret_cast<uintptr_t>(dd_smem_raw) + 1023) & ~(uintptr_t)1023);
    Ctrl* ctrl = reinterpret_cast<Ctrl*>(tiles + STAGES * TL::BYTES);

    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int g = lane >> 2, c = lane & 3;
    const int kvh = blockIdx.x, bi = blockIdx.y, piece = blockIdx.z;
    const int nrep = a.nh / a.nkv;
    // (the step's index arrays were there before any of its kernels)
    const int row = a.dec_rows[bi], seq = a.dec_seqs[bi];
    const int ctx = a.ctx_lens[seq];
    const int* table = a.block_tables + (size_t)seq * a.max_blocks;
    const bool live = g < nrep;                            // this lane's two rows: both maps of head kvh * nrep + g
    const int d = a.d, dv = a.dv, page_size = a.page_size;
    const int k_lo = a.window > 0 ? max(0, ctx - a.window) : 0;
    const int k_hi = ctx;
    const int t_first = k_lo / BN, t_all = (k_hi + BN - 1) / BN - t_first;
    const int per = (t_all + a.pieces - 1) / a.pieces;
    const int kt0 = t_first + piece * per, kt1 = min(kt0 + per, t_first + t_all);
    const int per_tile = BN / page_size, p_first = kt0 * per_tile;
    const int p_count = kt1 > kt0 ? (min(kt1 * BN, k_hi) - 1) / page_size - p_first + 1 : 0;
    const bool sliced = p_count <= TABLE_SLICE;

    if (threadIdx.x == 0) {
        ctrl->abort = 0;
        for (int s = 0; s < STAGES; ++s) bar_init(&ctrl->full[s], 1);
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_k) : "memory");
        asm volatile("prefetch.tensormap [%0];" ::"l"(&map_v) : "memory");
    }
    if (sliced)
        for (int i = threadIdx.x; i < p_count; i += THREADS) ctrl->pages[i] = table[p_first + i];
    __syncthreads();

    // tile `kt` into its stage, by warp 0: lane = (page of the tile, sub-tile).  A page past the context, or wholly behind the
    // window (it may have been given back), is asked for past the end of the tensor and arrives as zeros.
    auto issue = [&](int kt) {
        const int s = (kt - kt0) % STAGES;
        if (lane == 0) bar_expect_tx(&ctrl->full[s], TL::BYTES);
        __syncwarp();
        if (lane < per_tile * TL::SUBS) {
            const int pg = lane % per_tile, sub = lane / per_tile;
            const int key = kt * BN + pg * page_size;
            int z = a.cache_rows;
            if (key < k_hi && key + page_size > k_lo) {
                const int pi = kt * per_tile + pg;
                z = ((sliced ? ctrl->pages[pi - p_first] : table[pi]) * a.nkv + kvh) * page_size;
            }
            unsigned char* dst = tiles + s * TL::BYTES + sub * SUB + pg * page_size * 128;
            if (sub < 2) tma_load_3d(dst, &map_k, 0, sub, z, &ctrl->full[s]);
            else tma_load_2d(dst, &map_v, (sub - 2) * 64, z, &ctrl->full[s]);
        }
        __syncwarp();
    };
    // the first tiles: those below the step's own key hold nothing that a kernel of this step writes
    int issued = kt0;
    if (warp == 0)
        for (; issued < min(kt0 + STAGES - 1, kt1) && (issued + 1) * BN < ctx; ++issued) issue(issued);
    pdl_wait();
    if (warp == 0)
        for (; issued < min(kt0 + STAGES - 1, kt1); ++issued) issue(issued);

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
    float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
    float oacc[ND][4];
#pragma unroll
    for (int nd = 0; nd < ND; ++nd)
#pragma unroll
        for (int e = 0; e < 4; ++e) oacc[nd][e] = 0.f;
    for (int kt = kt0; kt < kt1; ++kt) {
        const int stage = (kt - kt0) % STAGES;
        unsigned char* tile = tiles + stage * TL::BYTES;
        bar_wait(&ctrl->full[stage], ((kt - kt0) / STAGES) & 1, &ctrl->abort);
        if ((kt + 1) * BN > ctx) {
            // slots of the last page past the context hold whatever was there before, and a weight of zero times a NaN would
            // still be a NaN: those rows of V are cleared
            for (int i = threadIdx.x; i < BN * 8 * (TL::SUBS - 2); i += THREADS) {
                const int r = (i >> 3) % BN;
                if (kt * BN + r >= ctx)
                    *reinterpret_cast<uint4*>(tile + (2 + (i >> 3) / BN) * SUB + r * 128 + (i & 7) * 16) = make_uint4(0u, 0u, 0u, 0u);
            }
        }
        __syncthreads();                             // everyone sees tile kt, and is done with the stage of tile kt - 1
        if (warp == 0 && kt + STAGES - 1 < kt1) issue(kt + STAGES - 1);
        const int key0 = kt * BN + warp * 16;              // this warp's 16 keys of the tile
        if (key0 < k_hi && key0 + 15 >= k_lo) {
            float sacc[2][4];
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) sacc[nt][e] = 0.f;
#pragma unroll
            for (int ks2 = 0; ks2 < KS / 2; ++ks2) {
#pragma unroll
                for (int nt = 0; nt < 2; ++nt) {
                    uint32_t kb[4];
                    ldmatrix_x4(kb, swizzled(tile + (ks2 / 2) * SUB, warp * 16 + nt * 8 + (lane & 7), (ks2 & 1) * 4 + (lane >> 3)));
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
                    sacc[nt][e] = seen ? capped_log2(sacc[nt][e], a) : -INFINITY;
                    mx[e >> 1] = fmaxf(mx[e >> 1], sacc[nt][e]);
                }
            float ms[2], corr[2], ls[2] = {0.f, 0.f};
#pragma unroll
            for (int r = 0; r < 2; ++r) {
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 1));
                mx[r] = fmaxf(mx[r], __shfl_xor_sync(0xffffffffu, mx[r], 2));
                const float mn = fmaxf(m_run[r], mx[r]);
                ms[r] = mn == -INFINITY ? 0.f : mn;
                corr[r] = ex2(m_run[r] - ms[r]);
                m_run[r] = mn;
            }
#pragma unroll
            for (int nt = 0; nt < 2; ++nt)
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    sacc[nt][e] = ex2(sacc[nt][e] - ms[e >> 1]);
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
                const int mat = lane >> 3, chunk = nd2 * 2 + (mat >> 1);
                ldmatrix_x4_trans(vb, swizzled(tile + (2 + nd2 / 4) * SUB, warp * 16 + (mat & 1) * 8 + (lane & 7), chunk & 7));
                mma_bf16_16816(oacc[2 * nd2], pa, vb[0], vb[1]);
                mma_bf16_16816(oacc[2 * nd2 + 1], pa, vb[2], vb[3]);
            }
        }
    }
    __syncthreads();
    pdl_trigger();
    // the four warps' states meet in shared memory (the stages are free now): [warp][row][DV + 2]
    constexpr int MW = DV + 2;
    float* mg = reinterpret_cast<float*>(tiles);
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
            const float f = x[DV] == -INFINITY ? 0.f : ex2(x[DV] - m);
            l = fmaf(x[DV + 1], f, l);
            o = fmaf(x[col], f, o);
        }
        float* dst = a.cluster ? mine + (size_t)u * MW : a.partial + ((((size_t)bi * a.nh + kvh * nrep + r) * 2 + mp) * a.pieces + piece) * MW;
        dst[col] = o;
        if (col == 0) { dst[DV] = m; dst[DV + 1] = l; }
    }
    if (!a.cluster) return;
    cluster_sync_all();
    float* red = ctrl->red;
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
            const float pf = pm == -INFINITY ? 0.f : ex2(pm - m);
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

// A [rows, mid, cols] bf16 row-major tensor with boxes of 64 columns (zeros past `cols`) x 1 x box_rows (mid 0: [rows, cols]).
bool make_pool_map(CUtensorMap* map, const void* ptr, long long rows, int mid, int cols, int box_rows) {
    EncodeTiledFn fn = encode_fn();
    if (fn == nullptr) return false;
    const int m = mid > 0 ? mid : 1;
    const cuuint64_t dims3[3] = {(cuuint64_t)cols, (cuuint64_t)m, (cuuint64_t)rows}, dims2[2] = {(cuuint64_t)cols, (cuuint64_t)rows};
    const cuuint64_t strides3[2] = {(cuuint64_t)cols * 2, (cuuint64_t)cols * m * 2}, strides2[1] = {(cuuint64_t)cols * 2};
    const cuuint32_t box3[3] = {64u, 1u, (cuuint32_t)box_rows}, box2[2] = {64u, (cuuint32_t)box_rows}, estr[3] = {1, 1, 1};
    return fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, mid > 0 ? 3 : 2, const_cast<void*>(ptr), mid > 0 ? dims3 : dims2,
              mid > 0 ? strides3 : strides2, mid > 0 ? box3 : box2, estr, CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B,
              CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE) == CUDA_SUCCESS;
}
}  // namespace

extern "C" int rlis_attention_difference_decode_error(void) { return tc::read_error_word(); }
extern "C" int* rlis_attention_difference_decode_error_addr(void) { return tc::error_word_addr(); }

// Whether the kernel for single tokens with two maps a head takes these sizes (bfloat16).
extern "C" int rlis_attention_difference_decode_takes(int nh, int nkv, int d, int dv, int page_size) {
    return nkv > 0 && nh % nkv == 0 && nh / nkv <= 8 && d > 0 && d <= 64 && d % 8 == 0 && dv > 0 && dv <= 128 && dv % 8 == 0 &&
           page_size >= 8 && page_size <= BN && BN % page_size == 0;
}
// Width of a value row in the partial sums (values are padded to it).
extern "C" int rlis_attention_difference_decode_width(int dv) { return dv <= 64 ? 64 : 128; }

static void raise_difference_limits() {
    static bool done = false;
    if (done) return;
    cudaFuncSetAttribute(attn_difference_decode_kernel<64>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_bytes<64>());
    cudaFuncSetAttribute(attn_difference_decode_kernel<128>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem_bytes<128>());
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
    cfg.dynamicSmemBytes = narrow ? smem_bytes<64>() : smem_bytes<128>();
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
                                                const int* ctx_lens, const int* block_tables, int max_blocks, int n_dec, int n_pages, int nh,
                                                int nkv, int d, int dv, int page_size, float scale, float cap, int window, int pieces,
                                                float lambda, float out_scale, float eps, cudaStream_t stream) {
    if (n_dec <= 0) return 0;
    if (!rlis_attention_difference_decode_takes(nh, nkv, d, dv, page_size) || pieces < 1 || pieces > 65535 || n_dec > 65535 || cap < 0.f ||
        (pieces > MAX_CLUSTER_PIECES && partial == nullptr) ||
        ((reinterpret_cast<uintptr_t>(q) | reinterpret_cast<uintptr_t>(k_cache) | reinterpret_cast<uintptr_t>(v_cache)) & 15) != 0)
        return RLIS_ERR_UNSUPPORTED;
    raise_difference_limits();
    const long long cache_rows = (long long)n_pages * nkv * page_size;
    if (cache_rows >= (1ll << 31)) return RLIS_ERR_UNSUPPORTED;
    CUtensorMap map_k, map_v;
    if (!make_pool_map(&map_k, k_cache, cache_rows, 2, d, page_size) || !make_pool_map(&map_v, v_cache, cache_rows, 0, dv, page_size))
        return RLIS_ERR_UNSUPPORTED;
    const float slope = cap > 0.f ? 2.0f * LOG2E * scale / cap : LOG2E * scale, top = cap > 0.f ? LOG2E * cap : 0.f;
    DiffDecode a;
    a.q = (const bf16*)q;
    a.out = (bf16*)out;
    a.partial = partial;
    a.gate = (const bf16*)gate;
    a.gate_stride = gate_stride;
    a.dec_rows = dec_rows;
    a.dec_seqs = dec_seqs;
    a.ctx_lens = ctx_lens;
    a.block_tables = block_tables;
    a.max_blocks = max_blocks;
    a.nh = nh;
    a.nkv = nkv;
    a.d = d;
    a.dv = dv;
    a.page_size = page_size;
    a.window = window;
    a.pieces = pieces;
    a.cluster = pieces > 1 && pieces <= MAX_CLUSTER_PIECES ? 1 : 0;
    a.cache_rows = (int)cache_rows;
    a.slope = slope;
    a.top = top;
    a.lambda = lambda;
    a.out_scale = out_scale;
    a.eps = eps;
    const dim3 grid(nkv, n_dec, pieces);
    const bool narrow = rlis_attention_difference_decode_width(dv) == 64;
    const dim3 cluster(1, 1, a.cluster ? (unsigned)pieces : 1u);
    if (narrow) rlis_launch_cluster(attn_difference_decode_kernel<64>, grid, THREADS, smem_bytes<64>(), stream, cluster, map_k, map_v, a);
    else rlis_launch_cluster(attn_difference_decode_kernel<128>, grid, THREADS, smem_bytes<128>(), stream, cluster, map_k, map_v, a);
    const int err = RLIS_LAUNCH_CHECK();
    if (err != 0 || pieces == 1 || a.cluster) return err;
    const int units = n_dec * nh;
    if (narrow) rlis_launch(attn_difference_merge_kernel<64>, (units + 3) / 4, 128, 0, stream, a, units);
    else rlis_launch(attn_difference_merge_kernel<128>, (units + 3) / 4, 128, 0, stream, a, units);
    return RLIS_LAUNCH_CHECK();
}
