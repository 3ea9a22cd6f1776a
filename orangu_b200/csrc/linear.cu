// Products with bfloat16 weights for models given as a list of layers, with the operator that follows as the epilogue.
//
//   gemv_act_kernel      a few tokens: a group of lanes per pair of rows streams the weights once, HBM-bound
//   linear_tc5_kernel    bf16 activations: tcgen05.mma (kind::f16) with fp32 accumulators in tensor memory, operands by TMA
//   linear_simt_kernel   fp32 activations: plain fp32 multiply-add tiles
// Each also runs grouped products (a mixture of experts), the rows of which have batch entries of their own.
// All three end in epilogue_store, so a product means the same whichever kernel runs it.
#include <algorithm>

#include "layered.h"
#include "pdl.cuh"
#include "tc5_common.cuh"

namespace ob {

namespace {

// ---- activations -------------------------------------------------------------------------------------------------------
__device__ __forceinline__ void unpack8(const uint4 &w, float (&f)[8]) {  // eight bfloat16
    const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        f[2 * i] = __uint_as_float(u[i] << 16);
        f[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
    }
}
__device__ __forceinline__ void load8(const __nv_bfloat16 *p, float (&f)[8]) { unpack8(*reinterpret_cast<const uint4 *>(p), f); }
__device__ __forceinline__ void load8(const float *p, float (&f)[8]) {
    const float4 a = reinterpret_cast<const float4 *>(p)[0], b = reinterpret_cast<const float4 *>(p)[1];
    f[0] = a.x, f[1] = a.y, f[2] = a.z, f[3] = a.w, f[4] = b.x, f[5] = b.y, f[6] = b.z, f[7] = b.w;
}

// N consecutive values to p, the first n of which exist.
template <int N>
__device__ __forceinline__ void store_row(float *p, const float *v, uint32_t n) {
    if (N % 4 == 0 && n == N && (reinterpret_cast<uintptr_t>(p) & 15) == 0) {
#pragma unroll
        for (int i = 0; i < N / 4; ++i) reinterpret_cast<float4 *>(p)[i] = make_float4(v[4 * i], v[4 * i + 1], v[4 * i + 2], v[4 * i + 3]);
        return;
    }
#pragma unroll
    for (int i = 0; i < N; ++i)
        if (i < n) p[i] = v[i];
}
__device__ __forceinline__ uint32_t pack2(float a, float b) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const uint32_t *>(&h);
}
template <int N>
__device__ __forceinline__ void store_row(__nv_bfloat16 *p, const float *v, uint32_t n) {
    if (N % 8 == 0 && n == N && (reinterpret_cast<uintptr_t>(p) & 15) == 0) {
#pragma unroll
        for (int i = 0; i < N / 8; ++i)
            reinterpret_cast<uint4 *>(p)[i] = make_uint4(pack2(v[8 * i], v[8 * i + 1]), pack2(v[8 * i + 2], v[8 * i + 3]), pack2(v[8 * i + 4], v[8 * i + 5]), pack2(v[8 * i + 6], v[8 * i + 7]));
        return;
    }
#pragma unroll
    for (int i = 0; i < N; ++i)
        if (i < n) p[i] = __float2bfloat16_rn(v[i]);
}

// ---- epilogues -----------------------------------------------------------------------------------------------------------
__device__ __forceinline__ float sigmoidf(float z) { return 1.0f / (1.0f + expf(-z)); }
__device__ __forceinline__ float gelu_tanhf(float z) {
    constexpr float c = 0.7978845608028654f;  // sqrt(2 / pi)
    return 0.5f * z * (1.0f + tanhf(c * (z + 0.044715f * z * z * z)));
}

// N consecutive weight rows starting at r (within one 32-row group, r even) of token t: v holds the products.
template <typename TA, int N>
__device__ __forceinline__ void epilogue_store(const LinArgs &a, uint32_t batch, uint32_t t, uint32_t r, float *v) {
    if (a.bias) {
        const float *b = a.bias + (uint64_t)batch * a.n_rows + r;
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] += __ldg(b + i);
    }
#pragma unroll 1
    for (int s = 0; s < a.n_seg; ++s) {
        const LinSegment &g = a.seg[s];
        if (r < g.row0 || r >= g.row0 + g.n) continue;
        const uint32_t k = r - g.row0, n = min((uint32_t)N, g.n - k);
        const uint64_t row = g.page_pitch ? (uint64_t)(t / KV_PAGE) * g.page_pitch + t % KV_PAGE * g.pitch : (uint64_t)t * g.pitch;
        const uint64_t base = row + g.col0 + (uint64_t)batch * g.batch_cols;
        switch (g.epi) {
        case LE_F32: store_row<N>(static_cast<float *>(g.out) + base + k, v, n); break;
        case LE_ACT: store_row<N>(static_cast<TA *>(g.out) + base + k, v, n); break;
        case LE_GLU: {
            float o[N / 2 > 0 ? N / 2 : 1];
#pragma unroll
            for (int j = 0; j < N / 2; ++j) {
                const float gt = fminf(v[2 * j], a.glu_limit), up = fminf(fmaxf(v[2 * j + 1], -a.glu_limit), a.glu_limit);
                o[j] = gt * sigmoidf(a.glu_alpha * gt) * (up + 1.0f);
            }
            store_row<(N / 2 > 0 ? N / 2 : 1)>(static_cast<TA *>(g.out) + base + k / 2, o, n / 2);
            break;
        }
        case LE_RESIDUAL: {
            float *x = static_cast<float *>(g.out) + base + k;
            if (N % 4 == 0 && n == N && (reinterpret_cast<uintptr_t>(x) & 15) == 0) {
#pragma unroll
                for (int i = 0; i < N / 4; ++i) {
                    const float4 o = reinterpret_cast<const float4 *>(x)[i];
                    v[4 * i] += o.x, v[4 * i + 1] += o.y, v[4 * i + 2] += o.z, v[4 * i + 3] += o.w;
                }
            } else {
#pragma unroll
                for (int i = 0; i < N; ++i)
                    if (i < n) v[i] += x[i];
            }
            store_row<N>(x, v, n);
            if (a.out2) store_row<N>(static_cast<TA *>(a.out2) + (uint64_t)t * a.out2_pitch + k, v, n);
            break;
        }
        case LE_GELU_EMB: {
            const __nv_bfloat16 *e = a.emb + (uint64_t)a.tokens[t] * a.emb_pitch + a.emb_col0 + k;
#pragma unroll
            for (int i = 0; i < N; ++i)
                if (i < n) v[i] = gelu_tanhf(v[i]) * __bfloat162float(e[i]);
            store_row<N>(static_cast<TA *>(g.out) + base + k, v, n);
            break;
        }
        case LE_RELU2: {
#pragma unroll
            for (int i = 0; i < N; ++i) {
                const float p = fmaxf(v[i], 0.0f);
                v[i] = p * p;
            }
            store_row<N>(static_cast<TA *>(g.out) + base + k, v, n);
            break;
        }
        case LE_SWIGLU: {
            const float w = a.row_scale ? a.row_scale[t] : 1.0f;
            float o[N / 2 > 0 ? N / 2 : 1];
#pragma unroll
            for (int j = 0; j < N / 2; ++j) {
                const float gt = v[2 * j] * w;
                o[j] = gt * sigmoidf(gt) * (v[2 * j + 1] * w);
            }
            if (a.out_scale) {
                const float f = a.out_scale[t];
#pragma unroll
                for (int j = 0; j < N / 2; ++j) o[j] *= f;
            }
            store_row<(N / 2 > 0 ? N / 2 : 1)>(static_cast<TA *>(g.out) + base + k / 2, o, n / 2);
            break;
        }
        case LE_GELU_GLU: {
            float o[N / 2 > 0 ? N / 2 : 1];
#pragma unroll
            for (int j = 0; j < N / 2; ++j) o[j] = gelu_tanhf(v[2 * j]) * v[2 * j + 1];
            store_row<(N / 2 > 0 ? N / 2 : 1)>(static_cast<TA *>(g.out) + base + k / 2, o, n / 2);
            break;
        }
        case LE_TANH: {
#pragma unroll
            for (int i = 0; i < N; ++i) v[i] = tanhf(v[i]);
            store_row<N>(static_cast<TA *>(g.out) + base + k, v, n);
            break;
        }
        case LE_DECAY: {
#pragma unroll
            for (int i = 0; i < N; ++i) v[i] = expf(-expf(v[i]));
            store_row<N>(static_cast<float *>(g.out) + base + k, v, n);
            break;
        }
        case LE_GATED_EACH: {
            const TA *gate = static_cast<const TA *>(a.gate_act) + (uint64_t)t * a.gate_pitch + (uint64_t)batch * g.batch_cols + k;
            if (N % 8 == 0 && n == N && (reinterpret_cast<uintptr_t>(gate) & 15) == 0) {
#pragma unroll
                for (int i = 0; i < N / 8; ++i) {
                    float f[8];
                    load8(gate + 8 * i, f);
#pragma unroll
                    for (int j = 0; j < 8; ++j) v[8 * i + j] *= sigmoidf(f[j]);
                }
            } else {
#pragma unroll
                for (int i = 0; i < N; ++i)
                    if (i < n) v[i] *= sigmoidf((float)gate[i]);
            }
            store_row<N>(static_cast<TA *>(g.out) + base + k, v, n);
            break;
        }
        default: {  // LE_GATED
            const float s = sigmoidf(a.gate[(uint64_t)t * a.gate_pitch + batch]);
#pragma unroll
            for (int i = 0; i < N; ++i) v[i] *= s;
            store_row<N>(static_cast<TA *>(g.out) + base + k, v, n);
        }
        }
        return;
    }
}

// ---- a few tokens ----------------------------------------------------------------------------------------------------------
// G lanes own a pair of rows (2p, 2p+1); with KS > 1 (then G = 32) KS warps share a pair and split its columns.  A lane's weights
// are requested UNROLL chunks of 16 bytes per row ahead; the first of them before the wait for the predecessor kernel.
constexpr int GV_THREADS = 256, GV_UNROLL = 4;

template <typename TA, int NT>
__global__ void __launch_bounds__(GV_THREADS, NT == 1 ? 3 : 2) gemv_act_kernel(LinArgs a, uint32_t G, uint32_t KS) {
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, per_warp = 32 / G;
    const uint32_t ks = KS > 1 ? warp % KS : 0, unit = KS > 1 ? warp / KS : warp * per_warp + lane / G;
    const uint32_t units = KS > 1 ? 8 / KS : 8 * per_warp;
    const uint32_t pair = blockIdx.x * units + unit, r = 2 * pair;
    const bool live = r < a.n_rows, grouped = NT == 1 && a.row_batch != nullptr;  // grouped: a token per blockIdx.z, its weights known once the predecessor is done
    uint32_t batch = blockIdx.z;
    if (grouped) {
        pdl_release();
        pdl_wait();
        batch = a.row_batch[blockIdx.z];
    }
    const uint32_t n_chunk = a.kp / 8, step = G * KS, c_first = ks * G + lane % G;
    const uint4 *wa = reinterpret_cast<const uint4 *>(a.w + ((uint64_t)batch * a.n_rows + (live ? r : 0)) * a.kp);
    const uint4 *wb = wa + n_chunk;
    uint4 na[GV_UNROLL], nb[GV_UNROLL];
    auto fetch = [&](uint32_t c0) {
#pragma unroll
        for (int u = 0; u < GV_UNROLL; ++u) {
            const uint32_t c = c0 + u * step;
            const bool in = live && c < n_chunk;
            na[u] = in ? ldg128_stream(wa + c) : make_uint4(0, 0, 0, 0);
            nb[u] = in ? ldg128_stream(wb + c) : make_uint4(0, 0, 0, 0);
        }
    };
    fetch(c_first);
    if (!grouped) {
        pdl_release();
        pdl_wait();
    }
    const TA *x = static_cast<const TA *>(a.x) + (grouped ? (uint64_t)(blockIdx.z / a.x_div) * a.x_pitch : (uint64_t)batch * a.x_step);
    float acc[NT][2];
#pragma unroll
    for (int t = 0; t < NT; ++t) acc[t][0] = acc[t][1] = 0.0f;
    for (uint32_t c0 = c_first; c0 < n_chunk; c0 += GV_UNROLL * step) {
        uint4 ca[GV_UNROLL], cb[GV_UNROLL];
#pragma unroll
        for (int u = 0; u < GV_UNROLL; ++u) ca[u] = na[u], cb[u] = nb[u];
        fetch(c0 + GV_UNROLL * step);
#pragma unroll
        for (int u = 0; u < GV_UNROLL; ++u) {
            const uint32_t c = c0 + u * step;
            if (c >= n_chunk) continue;
            float fa[8], fb[8];
            unpack8(ca[u], fa);
            unpack8(cb[u], fb);
#pragma unroll
            for (int t = 0; t < NT; ++t) {
                float xv[8];
                load8(x + (uint64_t)t * a.x_pitch + 8 * c, xv);
#pragma unroll
                for (int i = 0; i < 8; ++i) {
                    acc[t][0] = fmaf(fa[i], xv[i], acc[t][0]);
                    acc[t][1] = fmaf(fb[i], xv[i], acc[t][1]);
                }
            }
        }
    }
#pragma unroll
    for (int t = 0; t < NT; ++t)
        for (uint32_t o = G / 2; o > 0; o >>= 1) {
            acc[t][0] += __shfl_xor_sync(0xffffffffu, acc[t][0], o);
            acc[t][1] += __shfl_xor_sync(0xffffffffu, acc[t][1], o);
        }
    if (KS > 1) {
        __shared__ float red[8][NT][2];
        if (lane == 0)
#pragma unroll
            for (int t = 0; t < NT; ++t) red[warp][t][0] = acc[t][0], red[warp][t][1] = acc[t][1];
        __syncthreads();
        if (ks) return;
#pragma unroll
        for (int t = 0; t < NT; ++t)
            for (uint32_t k = 1; k < KS; ++k) acc[t][0] += red[warp + k][t][0], acc[t][1] += red[warp + k][t][1];
    }
    if (!live) return;
#pragma unroll
    for (int t = 0; t < NT; ++t)  // G may be smaller than NT: lanes take tokens in turn
        if ((t % G) == lane % G) epilogue_store<TA, 2>(a, batch, grouped ? blockIdx.z : t, r, acc[t]);
}

// ---- fp32 tiles -----------------------------------------------------------------------------------------------------------
// 64 tokens x 64 rows per CTA, 16 columns per step, 4 x 4 results per thread.
template <typename TA>
__global__ void __launch_bounds__(256) linear_simt_kernel(LinArgs a) {
    __shared__ float xs[16][68], ws[16][68];
    pdl_release();
    pdl_wait();
    uint32_t t0 = blockIdx.y * 64, batch = blockIdx.z, t_end = a.T;
    if (a.tiles) {
        if (blockIdx.y >= *a.n_tiles) return;
        const LinTile tile = a.tiles[blockIdx.y];
        t0 = tile.row0, batch = tile.batch, t_end = tile.row0 + tile.n;
    }
    const uint32_t r0 = blockIdx.x * 64;
    const uint32_t tx = threadIdx.x % 16, ty = threadIdx.x / 16;
    const TA *x = static_cast<const TA *>(a.x) + (a.tiles ? 0 : (uint64_t)batch * a.x_step);
    const __nv_bfloat16 *w = a.w + (uint64_t)batch * a.n_rows * a.kp;
    float acc[4][4] = {};
    for (uint32_t k0 = 0; k0 < a.kp; k0 += 16) {
        {   // each half of the CTA fills one operand: thread = (row, 8 columns)
            const uint32_t i = threadIdx.x & 127, row = i >> 1, c = (i & 1) * 8;
            float f[8];
            if (threadIdx.x < 128) {
                if (t0 + row < t_end) load8(x + (uint64_t)(t0 + row) * a.x_pitch + k0 + c, f);
                else
#pragma unroll
                    for (int j = 0; j < 8; ++j) f[j] = 0.0f;
#pragma unroll
                for (int j = 0; j < 8; ++j) xs[c + j][row] = f[j];
            } else {
                if (r0 + row < a.n_rows) load8(w + (uint64_t)(r0 + row) * a.kp + k0 + c, f);
                else
#pragma unroll
                    for (int j = 0; j < 8; ++j) f[j] = 0.0f;
#pragma unroll
                for (int j = 0; j < 8; ++j) ws[c + j][row] = f[j];
            }
        }
        __syncthreads();
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            const float4 xv = *reinterpret_cast<const float4 *>(&xs[k][4 * ty]), wv = *reinterpret_cast<const float4 *>(&ws[k][4 * tx]);
            const float xa[4] = {xv.x, xv.y, xv.z, xv.w}, wa[4] = {wv.x, wv.y, wv.z, wv.w};
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(xa[i], wa[j], acc[i][j]);
        }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
        if (t0 + 4 * ty + i < t_end && r0 + 4 * tx < a.n_rows) epilogue_store<TA, 4>(a, batch, t0 + 4 * ty + i, r0 + 4 * tx, acc[i]);
}

// ---- tcgen05 ---------------------------------------------------------------------------------------------------------------
// Tiles of 128 tokens (the lanes of tensor memory) x BN weight rows (its columns), K in steps of 64 columns = one 128-byte
// swizzled row per operand row.  Warps 0-3 epilogue (warp w reads lane quadrant w), warp 4 issues the TMA loads, warp 5 owns
// tensor memory and issues the MMAs.  The weight tiles of the first stages are requested before the wait for the predecessor.
// BN = 256 is persistent with two accumulators, so a tile's epilogue runs under the next tile's products; narrower tiles are one
// per CTA, two CTAs per SM.  AR: token rows that are loaded.  With few tokens the other rows of the operand are whatever the
// shared memory holds -- they only reach tensor-memory lanes nobody reads -- and the room goes into more stages of weights.
// An MMA costs its 128 token rows however narrow the tile, so small batches keep wide tiles and fill the GPU by splitting K: the
// splits of a tile leave fp32 partial sums, which linear_finish_kernel adds up in split order before it runs the epilogue.
constexpr int LT_M = 128, LT_EPI_WARPS = 4, LT_TMA_WARP = 4, LT_MMA_WARP = 5, LT_THREADS = 6 * 32;
constexpr uint32_t LT_GROUP = 16;  // token tiles that share the weight tiles of a wave: both operands stay in L2

template <int BN, int AR>
struct LtSmem {
    static constexpr uint32_t A_BYTES = AR * 128, B_BYTES = BN * 128, SLACK = LT_M * 128 - A_BYTES;  // the MMA reads 128 rows from every stage's base
    static constexpr uint32_t STAGES = BN == 256 ? 4 : (104 * 1024 - SLACK) / (A_BYTES + B_BYTES);
    static constexpr uint32_t NBUF = BN == 256 ? 2 : 1;
    static constexpr uint32_t COLS = NBUF * BN;
    static constexpr uint32_t B = 0, A = STAGES * B_BYTES, FULL = A + STAGES * A_BYTES + SLACK, EMPTY = FULL + 8 * STAGES, ACC_FULL = EMPTY + 8 * STAGES,
                              ACC_EMPTY = ACC_FULL + 8 * NBUF, SLOT = ACC_EMPTY + 8 * NBUF, ABORT = SLOT + 8, BYTES = ABORT + 8, ALLOC = BYTES + 1024;
    static_assert(STAGES >= 3 && ALLOC <= (BN == 256 ? 227 : 113) * 1024, "shared memory plan does not fit");
};

struct LtTiles {
    uint32_t rows, toks, total;  // weight tiles and token tiles of one batch entry, tiles of all (splits counted)
    uint32_t splits;             // > 1: one token tile of at most LT_SPLIT_TOKENS rows, a CTA per tile and split
    float *part;                 // [tile][split][LT_SPLIT_TOKENS][BN]
    const LinTile *table;        // grouped: the token tiles (rows of x and their batch entry), *n_table of them; toks and total are bounds
    const uint32_t *n_table;
};
constexpr uint32_t LT_SPLIT_TOKENS = 64;
__device__ __forceinline__ void lt_tile(const LtTiles &g, uint32_t tile, uint32_t *batch, uint32_t *rt, uint32_t *tt) {
    const uint32_t per = g.rows * g.toks;
    *batch = tile / per;
    uint32_t i = tile - *batch * per;
    const uint32_t grp = i / (LT_GROUP * g.rows), width = min(LT_GROUP, g.toks - grp * LT_GROUP);
    i -= grp * LT_GROUP * g.rows;
    *rt = i / width;
    *tt = grp * LT_GROUP + i % width;
}
// Grouped: how many tiles there are in truth; then tile -> weight rows of its batch entry and rows [t0, t_end) of x.
__device__ __forceinline__ void lt_count(LtTiles &g) {
    if (!g.table) return;
    g.toks = *g.n_table;
    g.total = g.rows * g.toks;
}
__device__ __forceinline__ void lt_rows(const LtTiles &g, uint32_t T, uint32_t tt, uint32_t *batch, uint32_t *t0, uint32_t *t_end) {
    *t0 = tt * LT_M, *t_end = T;
    if (!g.table) return;
    const LinTile tile = g.table[tt];
    *batch = tile.batch, *t0 = tile.row0, *t_end = tile.row0 + tile.n;
}

template <int BN, int AR>
__global__ void __launch_bounds__(LT_THREADS, BN == 256 ? 1 : 2)
linear_tc5_kernel(const __grid_constant__ CUtensorMap tm_x, const __grid_constant__ CUtensorMap tm_w, const __grid_constant__ LinArgs a, const LtTiles g_in) {
    using S = LtSmem<BN, AR>;
    extern __shared__ uint8_t smem_raw[];
    const uint32_t sbase = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t *smem = smem_raw + (sbase - smem_u32(smem_raw));
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    volatile uint32_t *abort = reinterpret_cast<volatile uint32_t *>(smem + S::ABORT);
    LtTiles g = g_in;
    const uint32_t split = blockIdx.x % g.splits, k0 = a.kp / 64 * split / g.splits, k1 = a.kp / 64 * (split + 1) / g.splits, n_steps = k1 - k0;

    if (threadIdx.x == 0) {
        for (uint32_t s = 0; s < S::STAGES; ++s) {
            mbar_init(sbase + S::FULL + 8 * s, 1);
            mbar_init(sbase + S::EMPTY + 8 * s, 1);
        }
        for (uint32_t b = 0; b < S::NBUF; ++b) {
            mbar_init(sbase + S::ACC_FULL + 8 * b, 1);
            mbar_init(sbase + S::ACC_EMPTY + 8 * b, LT_EPI_WARPS);
        }
        *abort = 0u;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == LT_MMA_WARP) tmem_alloc(sbase + S::SLOT, S::COLS);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t *>(smem + S::SLOT);
    pdl_release();

    if (warp == LT_TMA_WARP) {
        if (lane == 0) {
            if (g.table) {  // which weights is known once the predecessor is done
                pdl_wait();
                lt_count(g);
            }
            const uint32_t ahead = min(n_steps, S::STAGES);
            uint32_t it = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; ok && tile < g.total; tile += gridDim.x) {
                uint32_t batch, rt, tt, t0, t_end;
                lt_tile(g, tile / g.splits, &batch, &rt, &tt);
                lt_rows(g, a.T, tt, &batch, &t0, &t_end);
                const int32_t wy = (int32_t)(batch * a.n_rows + rt * BN), xc = g.table ? 0 : (int32_t)(batch * a.x_step), xy = (int32_t)t0;
                auto weights = [&](uint32_t k, uint32_t s) {
                    mbar_expect_tx(sbase + S::FULL + 8 * s, S::A_BYTES + S::B_BYTES);
                    tma_load_2d(sbase + S::B + s * S::B_BYTES, &tm_w, (int32_t)(k * 64), wy, sbase + S::FULL + 8 * s);
                };
                if (tile == blockIdx.x) {
                    for (uint32_t k = 0; k < ahead; ++k) weights(k0 + k, k);
                    if (!g.table) pdl_wait();
                }
                for (uint32_t k = k0; k < k1; ++k, ++it) {
                    const uint32_t s = it % S::STAGES;
                    if (it >= S::STAGES && !mbar_wait(sbase + S::EMPTY + 8 * s, ((it / S::STAGES) & 1u) ^ 1u, abort)) {
                        ok = false;
                        break;
                    }
                    if (it >= ahead) weights(k, s);
                    tma_load_2d(sbase + S::A + s * S::A_BYTES, &tm_x, xc + (int32_t)(k * 64), xy, sbase + S::FULL + 8 * s);
                }
            }
        }
    } else if (warp == LT_MMA_WARP) {
        pdl_wait();
        lt_count(g);
        if (lane == 0) {
            constexpr uint32_t idesc = umma_idesc_bf16(BN);
            uint32_t it = 0, n = 0;
            bool ok = true;
            for (uint32_t tile = blockIdx.x; ok && tile < g.total; tile += gridDim.x, ++n) {
                const uint32_t buf = n % S::NBUF;
                if (n >= S::NBUF && !mbar_wait(sbase + S::ACC_EMPTY + 8 * buf, ((n / S::NBUF) & 1u) ^ 1u, abort)) break;
                for (uint32_t k = k0; k < k1; ++k, ++it) {
                    const uint32_t s = it % S::STAGES;
                    if (!mbar_wait(sbase + S::FULL + 8 * s, (it / S::STAGES) & 1u, abort)) {
                        ok = false;
                        break;
                    }
                    tc_fence_after();
                    const uint64_t da = umma_desc_sw128(sbase + S::A + s * S::A_BYTES), db = umma_desc_sw128(sbase + S::B + s * S::B_BYTES);
#pragma unroll
                    for (uint32_t j = 0; j < 4; ++j) umma_bf16(tmem + buf * BN, da + 2 * j, db + 2 * j, idesc, (k > k0 || j) ? 1u : 0u);
                    umma_commit(sbase + S::EMPTY + 8 * s);
                }
                if (ok) umma_commit(sbase + S::ACC_FULL + 8 * buf);
            }
        }
    } else {
        pdl_wait();
        lt_count(g);
        uint32_t n = 0;
        for (uint32_t tile = blockIdx.x; tile < g.total; tile += gridDim.x, ++n) {
            const uint32_t buf = n % S::NBUF;
            uint32_t batch, rt, tt, t0, t_end;
            lt_tile(g, tile / g.splits, &batch, &rt, &tt);
            lt_rows(g, a.T, tt, &batch, &t0, &t_end);
            if (!mbar_wait(sbase + S::ACC_FULL + 8 * buf, (n / S::NBUF) & 1u, abort)) break;
            tc_fence_after();
            const uint32_t t = t0 + warp * 32 + lane;
#pragma unroll 1
            for (int c = 0; c < BN / 32; ++c) {
                uint32_t u[32];
                __syncwarp();
                tmem_ld32(tmem + ((uint32_t)(warp * 32) << 16) + buf * BN + c * 32, u);
                tmem_ld_wait();
                float v[32];
#pragma unroll
                for (int i = 0; i < 32; ++i) v[i] = __uint_as_float(u[i]);
                const uint32_t r = rt * BN + c * 32;
                if (t < t_end && r < a.n_rows) {
                    if (g.splits == 1) epilogue_store<__nv_bfloat16, 32>(a, batch, t, r, v);
                    else store_row<32>(g.part + ((uint64_t)tile * LT_SPLIT_TOKENS + t) * BN + c * 32, v, 32);
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(sbase + S::ACC_EMPTY + 8 * buf);
        }
    }
    __syncwarp();
    if (*abort) {  // let copies that are still in flight land before the shared memory goes away
        for (int i = 0; i < 200; ++i) __nanosleep(1000);
    }
    tc_fence_before();
    __syncthreads();
    if (warp == LT_MMA_WARP) tmem_dealloc(tmem, S::COLS);
}

// The splits of every (token, 4 weight rows) added up, then the epilogue.
template <int BN>
__global__ void __launch_bounds__(256) linear_finish_kernel(const __grid_constant__ LinArgs a, const LtTiles g) {
    pdl_release();
    pdl_wait();
    const uint32_t per = a.n_rows / 4, i = blockIdx.x * 256 + threadIdx.x;
    if (i >= per * a.T * a.n_batch) return;
    const uint32_t r = i % per * 4, t = i / per % a.T, batch = i / per / a.T, tile = batch * g.rows + r / BN;
    const float *p = g.part + ((uint64_t)tile * g.splits * LT_SPLIT_TOKENS + t) * BN + r % BN;
    float v[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll 4
    for (uint32_t k = 0; k < g.splits; ++k) {
        const float4 u = *reinterpret_cast<const float4 *>(p + (uint64_t)k * LT_SPLIT_TOKENS * BN);
        v[0] += u.x, v[1] += u.y, v[2] += u.z, v[3] += u.w;
    }
    epilogue_store<__nv_bfloat16, 4>(a, batch, t, r, v);
}

template <int BN, int AR>
cudaError_t configure_tc5() {
    return cudaFuncSetAttribute(linear_tc5_kernel<BN, AR>, cudaFuncAttributeMaxDynamicSharedMemorySize, LtSmem<BN, AR>::ALLOC);
}

template <int BN, int AR>
bool launch_tc5(const LinArgs &a, int sm_count, cudaStream_t st, uint32_t splits = 1) {
    CUtensorMap tm_x, tm_w;
    if (!make_map_2d(&tm_x, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.x, a.x_pitch, a.T, (uint64_t)a.x_pitch * 2, 64, AR, CU_TENSOR_MAP_SWIZZLE_128B)) return false;
    if (!make_map_2d(&tm_w, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.w, a.kp, (uint64_t)a.n_batch * a.n_rows, (uint64_t)a.kp * 2, 64, BN, CU_TENSOR_MAP_SWIZZLE_128B)) return false;
    LtTiles g{(a.n_rows + BN - 1) / BN, a.tiles ? a.max_tiles : (a.T + LT_M - 1) / LT_M, 0, splits, a.split_part, a.tiles, a.n_tiles};
    g.total = g.rows * g.toks * (a.tiles ? 1 : a.n_batch) * splits;
    const uint32_t ctas = BN == 256 ? std::min(g.total, (uint32_t)sm_count) : g.total;
    launch_pdl(linear_tc5_kernel<BN, AR>, ctas, LT_THREADS, LtSmem<BN, AR>::ALLOC, st, tm_x, tm_w, a, g);
    if (splits > 1) launch_pdl(linear_finish_kernel<BN>, (a.n_rows / 4 * a.T * a.n_batch + 255) / 256, 256, 0, st, a, g);
    g_tc5_launched.store(true, std::memory_order_relaxed);
    return true;
}

template <typename TA>
void launch_gemv_act(const LinArgs &a, int sm_count, cudaStream_t st) {
    // lanes per pair of rows: as many as have columns; then split the columns over warps while the GPU has room for them
    uint32_t G = 32;
    while (G > 4 && a.kp / 8 <= G / 2) G /= 2;
    uint32_t KS = 1;
    const uint32_t n_z = a.row_batch ? a.T : a.n_batch, pairs = a.n_rows / 2 * n_z;
    if (G == 32)
        while (KS < 8 && pairs * KS * 2 <= (uint32_t)sm_count * 64 && a.kp / 8 >= 32 * KS * 2) KS *= 2;
    const uint32_t units = KS > 1 ? 8 / KS : 8 * (32 / G);
    const dim3 grid((a.n_rows / 2 + units - 1) / units, 1, n_z);
    switch (a.row_batch ? 1 : a.T) {
    case 1: launch_pdl(gemv_act_kernel<TA, 1>, grid, GV_THREADS, 0, st, a, G, KS); break;
    case 2: launch_pdl(gemv_act_kernel<TA, 2>, grid, GV_THREADS, 0, st, a, G, KS); break;
    case 3: launch_pdl(gemv_act_kernel<TA, 3>, grid, GV_THREADS, 0, st, a, G, KS); break;
    default: launch_pdl(gemv_act_kernel<TA, 4>, grid, GV_THREADS, 0, st, a, G, KS); break;
    }
}
constexpr uint32_t GV_MAX_TOKENS = 4;
constexpr uint32_t LT_SPLIT_CTAS = 296;  // of a launch that splits K

}  // namespace

cudaError_t linear_configure() {
    static PerDeviceOnce once;
    return once.run([] {
        cudaError_t e = configure_tc5<256, 128>();
        for (cudaError_t (*f)() : {configure_tc5<128, 128>, configure_tc5<128, 64>, configure_tc5<128, 16>, configure_tc5<64, 128>, configure_tc5<32, 128>})
            if (e == cudaSuccess) e = f();
        return e;
    });
}

uint32_t launch_linear(const LinArgs &a, bool f32, int sm_count, cudaStream_t st) {
    if (!a.T || !a.n_rows) return 1;
    if (a.tiles) {
        if (f32) {
            launch_pdl(linear_simt_kernel<float>, dim3((a.n_rows + 63) / 64, a.max_tiles, 1), 256, 0, st, a);
            return 1;
        }
        if (a.tile_rows == 16) return launch_tc5<128, 16>(a, sm_count, st);
        if (a.tile_rows == 64) return launch_tc5<128, 64>(a, sm_count, st);
        // (the real number of tiles is near the lower bound when tiles are full)
        return (a.n_rows + 255) / 256 * (a.T / LT_M + 1) >= (uint32_t)sm_count ? launch_tc5<256, 128>(a, sm_count, st) : launch_tc5<128, 128>(a, sm_count, st);
    }
    if (a.T <= GV_MAX_TOKENS || a.row_batch) {
        if (f32) launch_gemv_act<float>(a, sm_count, st);
        else launch_gemv_act<__nv_bfloat16>(a, sm_count, st);
        return 1;
    }
    if (f32) {
        launch_pdl(linear_simt_kernel<float>, dim3((a.n_rows + 63) / 64, (a.T + 63) / 64, a.n_batch), 256, 0, st, a);
        return 1;
    }
    // the widest tile that still gives every SM a CTA
    const uint32_t tok_tiles = (a.T + LT_M - 1) / LT_M * a.n_batch;
    auto ctas = [&](uint32_t bn) { return (a.n_rows + bn - 1) / bn * tok_tiles; };
    const uint32_t sms = (uint32_t)sm_count;
    if (a.T <= LT_SPLIT_TOKENS) {
        const uint32_t tiles = ctas(128), steps = a.kp / 64;
        const uint32_t splits = std::max(1u, std::min({LT_SPLIT_CTAS / tiles, 2 * sms / tiles, steps / 4}));
        const bool ok = a.T <= 16 ? launch_tc5<128, 16>(a, sm_count, st, splits) : launch_tc5<128, 64>(a, sm_count, st, splits);
        return ok ? 1 + (splits > 1) : 0;
    }
    if (ctas(256) >= sms) return launch_tc5<256, 128>(a, sm_count, st);
    if (ctas(128) >= sms) return launch_tc5<128, 128>(a, sm_count, st);
    if (ctas(64) >= sms) return launch_tc5<64, 128>(a, sm_count, st);
    return launch_tc5<32, 128>(a, sm_count, st);
}

uint32_t linear_tile_rows(uint32_t rows, uint32_t batches, bool f32) {
    if (f32) return 64;
    return rows <= 12 * batches ? 16 : rows <= 48 * batches ? 64 : 128;
}

size_t linear_split_bytes() { return (size_t)LT_SPLIT_CTAS * LT_SPLIT_TOKENS * 128 * 4; }

int linear_take_status() { return tc5_take_status(); }
void linear_mark_launched() { g_tc5_launched.store(true, std::memory_order_relaxed); }

}  // namespace ob
