// Routing of a mixture of experts: scores, choice, and the order in which grouped products (linear.cu) take the pairs.
//
// A pair is a token and one of its chosen experts.  A few pairs stay in order and run row by row; more are brought into expert
// order, so that an expert's weights are read once per tile of its rows: the routing kernel counts every expert's pairs and gives
// each pair its place among them, the gathering kernel turns counts into offsets and copies the inputs.  Which place a pair gets
// depends on timing, what is computed for it does not.
#include "mixers_common.cuh"
#include "../../include/orangu_b200.h"

namespace ob {

namespace {

// Eight consecutive weights or activations.
__device__ __forceinline__ void eight(const bf16 *p, float (&f)[8]) {
    const uint4 w = *reinterpret_cast<const uint4 *>(p);
    const uint32_t u[4] = {w.x, w.y, w.z, w.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) f[2 * i] = __uint_as_float(u[i] << 16), f[2 * i + 1] = __uint_as_float(u[i] & 0xffff0000u);
}
__device__ __forceinline__ void eight(const float *p, float (&f)[8]) {
    const float4 a = reinterpret_cast<const float4 *>(p)[0], b = reinterpret_cast<const float4 *>(p)[1];
    f[0] = a.x, f[1] = a.y, f[2] = a.z, f[3] = a.w, f[4] = b.x, f[5] = b.y, f[6] = b.z, f[7] = b.w;
}

// One warp: the largest of the z[0 .. n) whose lane's bit (z[lane + 32 j]: bit j) is not set, the first of equals.  What is not a
// number counts as the smallest: whatever the logits are, the lanes agree on one that exists.
__device__ __forceinline__ void largest(const float *z, uint32_t n, uint32_t closed, float *value, uint32_t *place) {
    float best = -INFINITY;
    uint32_t at = 0xffffffffu;
    for (uint32_t e = threadIdx.x & 31, j = 0; e < n; e += 32, ++j)
        if (!(closed >> j & 1u) && (z[e] > best || at == 0xffffffffu)) best = fmaxf(z[e], -INFINITY), at = e;
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float v = __shfl_xor_sync(0xffffffffu, best, o);
        const uint32_t w = __shfl_xor_sync(0xffffffffu, at, o);
        if (w != 0xffffffffu && (at == 0xffffffffu || v > best || (v == best && w < at))) best = v, at = w;
    }
    *value = best, *place = at;
}

// One warp: the `top` largest of z[0 .. n) (the first of equals), best first.  Sigmoid and softmax are monotonic, so logits decide.
__device__ __forceinline__ void choose(const MoeArgs &a, uint32_t t, const float *z) {
    const uint32_t lane = threadIdx.x & 31;
    const uint32_t p0 = t * (a.top + a.n_shared);
    uint32_t taken = 0;  // of this lane's logits: bit j, as in largest()
    if (a.n_group > a.keep) {
        const uint32_t size = a.n_expert / a.n_group;
        uint32_t seen = 0;  // the best logit outside the groups found so far is in the next best group
        for (uint32_t i = 0; i < a.keep; ++i) {
            float best;
            uint32_t at;
            largest(z, a.n_expert, seen, &best, &at);
            const uint32_t lo = at / size * size;
            for (uint32_t e = lane, j = 0; e < a.n_expert; e += 32, ++j)
                if (e - lo < size) seen |= 1u << j;
        }
        taken = ~seen;
    }
    float first = 0.0f, sum = 0.0f;  // softmax: the largest logit, and the sum of exponentials below it
    for (uint32_t i = 0; i < a.top; ++i) {
        float best;
        uint32_t at;
        largest(z, a.n_expert, taken, &best, &at);
        if (at % 32 == lane) taken |= 1u << (at / 32);
        if (lane == 0) {
            const uint32_t p = p0 + i;
            a.expert[p] = at;
            if (i == 0) first = best;
            sum += expf(best - first);
            a.score[p] = a.score_of != OB_ROUTER_SIGMOID ? best : 1.0f / (1.0f + expf(-best));
            if (a.count) a.rank[p] = atomicAdd(a.count + at, 1u);
        }
    }
    if (a.score_of == OB_ROUTER_SOFTMAX_ALL) {  // (the largest logit of all has been chosen)
        first = __shfl_sync(0xffffffffu, first, 0);
        sum = 0.0f;
        for (uint32_t e = lane; e < a.n_expert; e += 32) sum += expf(z[e] - first);
        sum = warp_sum(sum);
    }
    if (a.score_of != OB_ROUTER_SIGMOID && lane == 0)
        for (uint32_t i = 0; i < a.top; ++i) a.score[p0 + i] = expf(a.score[p0 + i] - first) / sum * (a.score_of == OB_ROUTER_SOFTMAX_ALL ? a.scale : 1.0f);
    for (uint32_t i = lane; i < a.n_shared; i += 32) {
        const uint32_t p = p0 + a.top + i, e = a.n_expert + i;
        a.expert[p] = e;
        a.score[p] = 1.0f / (1.0f + expf(-z[a.n_expert]));
        if (a.count) {
            a.rank[p] = t;
            if (t == 0) a.count[e] = a.T;
        }
    }
}

// A CTA per token: logits, then the choice.
template <typename TA>
__global__ void __launch_bounds__(1024) moe_route_dot_kernel(MoeArgs a) {
    __shared__ float z[MOE_MAX_EXPERTS + 1];
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const TA *x = static_cast<const TA *>(a.x) + (uint64_t)t * a.x_pitch;
    for (uint32_t e = warp; e < a.n_expert + (a.n_shared > 0); e += blockDim.x / 32) {
        const bf16 *w = a.w + (uint64_t)e * a.x_pitch;
        float s = 0.0f;
#pragma unroll 4
        for (uint32_t c = 8 * lane; c < a.x_pitch; c += 256) {
            float wv[8], xv[8];
            eight(w + c, wv);
            eight(x + c, xv);
#pragma unroll
            for (int i = 0; i < 8; ++i) s = fmaf(wv[i], xv[i], s);
        }
        s = warp_sum(s);
        if (lane == 0) z[e] = s;
    }
    __syncthreads();
    if (warp == 0) choose(a, t, z);
}

// A warp per token: the logits are there.
__global__ void __launch_bounds__(256) moe_route_kernel(MoeArgs a) {
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x * 8 + (threadIdx.x >> 5);
    if (t < a.T) choose(a, t, a.logits + (uint64_t)t * a.logit_pitch);
}

// Offsets and numbers of tiles before every expert, then a warp per pair copies its token's input to the pair's row.
template <typename TA>
__global__ void __launch_bounds__(256) moe_gather_kernel(MoeArgs a) {
    __shared__ uint32_t first[MOE_MAX_EXPERTS], tile0[MOE_MAX_EXPERTS];
    pdl_release();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n_all = a.n_expert + a.n_shared, per = a.top + a.n_shared;
    if (warp == 0) {
        uint32_t rows = 0, tiles = 0;
        for (uint32_t e0 = 0; e0 < n_all; e0 += 32) {
            const uint32_t e = e0 + lane, n = e < n_all ? a.count[e] : 0, k = (n + a.tile_rows - 1) / a.tile_rows;
            uint32_t rs = n, ts = k;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const uint32_t ru = __shfl_up_sync(0xffffffffu, rs, o), tu = __shfl_up_sync(0xffffffffu, ts, o);
                if (lane >= o) rs += ru, ts += tu;
            }
            if (e < n_all) first[e] = rows + rs - n, tile0[e] = tiles + ts - k;
            rows += __shfl_sync(0xffffffffu, rs, 31), tiles += __shfl_sync(0xffffffffu, ts, 31);
        }
        if (blockIdx.x == 0 && lane == 0) *a.n_tiles = tiles;
    }
    __syncthreads();
    if (blockIdx.x == 0)
        for (uint32_t e = threadIdx.x; e < n_all; e += blockDim.x) {
            const uint32_t n = a.count[e];
            for (uint32_t r = 0, k = tile0[e]; r < n; r += a.tile_rows, ++k) a.tiles[k] = LinTile{e, first[e] + r, min(a.tile_rows, n - r)};
        }
    const uint32_t p = blockIdx.x * 8 + warp;
    if (p >= a.T * per) return;
    const uint32_t row = first[a.expert[p]] + a.rank[p];
    if (lane == 0) a.row[p] = row, a.row_score[row] = a.score[p];
    const uint4 *src = reinterpret_cast<const uint4 *>(static_cast<const TA *>(a.x) + (uint64_t)(p / per) * a.x_pitch);
    uint4 *dst = reinterpret_cast<uint4 *>(static_cast<TA *>(a.gathered) + (uint64_t)row * a.x_pitch);
    const uint32_t n = a.x_pitch * (uint32_t)sizeof(TA) / 16;
#pragma unroll 4
    for (uint32_t i = lane; i < n; i += 32) dst[i] = src[i];
}

template <typename TA>
uint32_t route(const MoeArgs &a, cudaStream_t st) {
    if (a.logits) launch_pdl(moe_route_kernel, (a.T + 7) / 8, 256, 0, st, a);
    else launch_pdl(moe_route_dot_kernel<TA>, a.T, a.n_expert + (a.n_shared > 0) > 16 ? 1024 : 512, 0, st, a);
    if (!a.count) return 1;
    launch_pdl(moe_gather_kernel<TA>, (a.T * (a.top + a.n_shared) + 7) / 8, 256, 0, st, a);
    return 2;
}

}  // namespace

uint32_t launch_moe_route(const MoeArgs &a, bool f32, cudaStream_t st) { return f32 ? route<float>(a, st) : route<bf16>(a, st); }

}  // namespace ob
