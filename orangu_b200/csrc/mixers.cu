// Kernels around the products of models given as a list of layers: embedding, norms with a scalar gain, the per-layer token
// input, latent attention over the paged latent cache, retention over the per-sequence state.
//
// Latent attention runs in the latent space: the query is multiplied by the key up-projection once per token and head (a batched
// product, linear.cu), so a cache row (latent | shared rotated key part) is key and, in its first part, value of every head; the
// value up-projection follows the attention.  Keys outside a row's window are never weighted, whole tiles outside are not read.
#include <math.h>

#include <algorithm>

#include "mixers_common.cuh"

namespace ob {

namespace {

// (No __restrict__ on what an earlier kernel writes: a load the compiler may take for invariant could move above pdl_wait.)
// ---- embedding, norms ------------------------------------------------------------------------------------------------------
// x = the token's embedding, h = x / rms(x) * gain (* w) or x.
template <typename TA, int NV>
__global__ void __launch_bounds__(1024) embed_kernel(const bf16 *table, uint32_t width, const uint32_t *tokens, float *x, bool normed, float eps, float gain, const float *w, TA *h,
                                                     uint32_t h_pitch) {
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    const bf16 *row = table + (uint64_t)tokens[blockIdx.x] * width;
    float *xr = x + (uint64_t)blockIdx.x * width;
    TA *hr = h + (uint64_t)blockIdx.x * h_pitch;
    float s = 0.0f;
    if constexpr (NV > 0) {
        float4 v[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            if (c >= width) continue;
            const uint2 u = *reinterpret_cast<const uint2 *>(row + c);
            v[i] = make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
            *reinterpret_cast<float4 *>(xr + c) = v[i];
            s += sq4(v[i]);
        }
        const float f = normed ? inv_rms(block_sum(s, red), width, eps) * gain : 1.0f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            if (c < width) store4<TA>(hr + c, w ? mul44(mul4(v[i], f), *reinterpret_cast<const float4 *>(w + c)) : mul4(v[i], f));
        }
    } else {
        for (uint32_t i = threadIdx.x; i < width; i += blockDim.x) {
            const float v = __bfloat162float(row[i]);
            xr[i] = v;
            s += v * v;
        }
        const float f = normed ? inv_rms(block_sum(s, red), width, eps) * gain : 1.0f;
        for (uint32_t i = threadIdx.x; i < width; i += blockDim.x) hr[i] = to_act<TA>(xr[i] * f * (w ? w[i] : 1.0f));
    }
}

template <typename TA, int NV>
__global__ void __launch_bounds__(1024) norm_kernel(const float *x, uint32_t width, const uint32_t *rows, float eps, float gain, const float *w, TA *h, uint32_t h_pitch) {
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    const float *row = x + (uint64_t)(rows ? rows[blockIdx.x] : blockIdx.x) * width;
    TA *hr = h + (uint64_t)blockIdx.x * h_pitch;
    float s = 0.0f;
    if constexpr (NV > 0) {
        float4 v[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            v[i] = c < width ? *reinterpret_cast<const float4 *>(row + c) : make_float4(0, 0, 0, 0);
            s += sq4(v[i]);
        }
        const float f = inv_rms(block_sum(s, red), width, eps) * gain;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            if (c >= width) continue;
            float4 o = mul4(v[i], f);
            if (w) o = mul44(o, *reinterpret_cast<const float4 *>(w + c));
            store4<TA>(hr + c, o);
        }
    } else {
        for (uint32_t i = threadIdx.x; i < width; i += blockDim.x) s += row[i] * row[i];
        const float f = inv_rms(block_sum(s, red), width, eps) * gain;
        for (uint32_t i = threadIdx.x; i < width; i += blockDim.x) hr[i] = to_act<TA>(row[i] * f * (w ? w[i] : 1.0f));
    }
}

template <typename TA, int NV>
__global__ void __launch_bounds__(1024) side_finish_kernel(float *x, const float *y, const float *w, uint32_t width, float eps, float gain, TA *h, uint32_t h_pitch) {
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    float *xr = x + (uint64_t)blockIdx.x * width;
    const float *yr = y + (uint64_t)blockIdx.x * width;
    TA *hr = h + (uint64_t)blockIdx.x * h_pitch;
    float s = 0.0f, s2 = 0.0f;
    if constexpr (NV > 0) {
        float4 v[NV], yv[NV], wv[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            const bool in = c < width;
            yv[i] = in ? *reinterpret_cast<const float4 *>(yr + c) : make_float4(0, 0, 0, 0);
            v[i] = in ? *reinterpret_cast<const float4 *>(xr + c) : make_float4(0, 0, 0, 0);
            wv[i] = in ? *reinterpret_cast<const float4 *>(w + c) : make_float4(0, 0, 0, 0);
            s += sq4(yv[i]);
        }
        const float f = inv_rms(block_sum(s, red), width, eps);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            v[i].x += yv[i].x * f * wv[i].x, v[i].y += yv[i].y * f * wv[i].y, v[i].z += yv[i].z * f * wv[i].z, v[i].w += yv[i].w * f * wv[i].w;
            if (c < width) *reinterpret_cast<float4 *>(xr + c) = v[i];
            s2 += sq4(v[i]);
        }
        if (!h) return;
        const float f2 = inv_rms(block_sum(s2, red), width, eps) * gain;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            if (c < width) store4<TA>(hr + c, mul4(v[i], f2));
        }
    } else {
        for (uint32_t i = threadIdx.x; i < width; i += blockDim.x) s += yr[i] * yr[i];
        const float f = inv_rms(block_sum(s, red), width, eps);
        for (uint32_t i = threadIdx.x; i < width; i += blockDim.x) {
            const float v = xr[i] + yr[i] * f * w[i];
            xr[i] = v;
            s2 += v * v;
        }
        if (!h) return;
        const float f2 = inv_rms(block_sum(s2, red), width, eps) * gain;
        for (uint32_t i = threadIdx.x; i < width; i += blockDim.x) hr[i] = to_act<TA>(xr[i] * f2);
    }
}

// x += mult * y / rms(y) * w, h = x or x / rms(x) * next_w; y is the sum of a token's `top` rows.
template <typename TA, int NV>
__global__ void __launch_bounds__(1024) post_norm_kernel(PostNormArgs a) {
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    float *xr = a.x + (uint64_t)blockIdx.x * a.width;
    TA *hr = a.h ? static_cast<TA *>(a.h) + (uint64_t)blockIdx.x * a.h_pitch : nullptr;
    auto row = [&](uint32_t i) {
        const uint32_t p = blockIdx.x * a.top + i;
        return a.y + (uint64_t)(a.rows ? a.rows[p] : p) * a.width;
    };
    if (a.zero && blockIdx.x == 0)
        for (uint32_t i = threadIdx.x; i < a.n_zero; i += blockDim.x) a.zero[i] = 0;
    float s = 0.0f;
    if constexpr (NV > 0) {
        float4 yv[NV], v[NV], wv[NV];
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            const bool in = c < a.width;
            yv[i] = in ? *reinterpret_cast<const float4 *>(row(0) + c) : make_float4(0, 0, 0, 0);
            v[i] = in ? *reinterpret_cast<const float4 *>(xr + c) : make_float4(0, 0, 0, 0);
            wv[i] = in ? *reinterpret_cast<const float4 *>(a.w + c) : make_float4(0, 0, 0, 0);
        }
        for (uint32_t k = 1; k < a.top; ++k) {
            const float *y = row(k);
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
                if (c >= a.width) continue;
                const float4 u = *reinterpret_cast<const float4 *>(y + c);
                yv[i].x += u.x, yv[i].y += u.y, yv[i].z += u.z, yv[i].w += u.w;
            }
        }
#pragma unroll
        for (int i = 0; i < NV; ++i) s += sq4(yv[i]);
        const float f = inv_rms(block_sum(s, red), a.width, a.eps) * a.mult;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            if (c >= a.width) continue;
            v[i].x += yv[i].x * f * wv[i].x, v[i].y += yv[i].y * f * wv[i].y, v[i].z += yv[i].z * f * wv[i].z, v[i].w += yv[i].w * f * wv[i].w;
            *reinterpret_cast<float4 *>(xr + c) = v[i];
            if (hr && !a.next_w) store4<TA>(hr + c, v[i]);
        }
        if (!hr || !a.next_w) return;
        float s2 = 0.0f;
#pragma unroll
        for (int i = 0; i < NV; ++i) s2 += sq4(v[i]);  // (zero past the end)
        const float f2 = inv_rms(block_sum(s2, red), a.width, a.eps);
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            if (c < a.width) store4<TA>(hr + c, mul44(mul4(v[i], f2), *reinterpret_cast<const float4 *>(a.next_w + c)));
        }
    } else {
        auto sum = [&](uint32_t c) {
            float v = row(0)[c];
            for (uint32_t k = 1; k < a.top; ++k) v += row(k)[c];
            return v;
        };
        for (uint32_t c = threadIdx.x; c < a.width; c += blockDim.x) {
            const float v = sum(c);
            s += v * v;
        }
        const float f = inv_rms(block_sum(s, red), a.width, a.eps) * a.mult;
        float s2 = 0.0f;
        for (uint32_t c = threadIdx.x; c < a.width; c += blockDim.x) {
            const float v = xr[c] + sum(c) * f * a.w[c];
            xr[c] = v;
            s2 += v * v;
            if (hr && !a.next_w) hr[c] = to_act<TA>(v);
        }
        if (!hr || !a.next_w) return;
        const float f2 = inv_rms(block_sum(s2, red), a.width, a.eps);
        for (uint32_t c = threadIdx.x; c < a.width; c += blockDim.x) hr[c] = to_act<TA>(xr[c] * f2 * a.next_w[c]);
    }
}

// ---- latent attention: what a token leaves in the cache, and its rotated query parts -----------------------------------------------
// A warp per token.  Part 0 is the token's cache row, every further part PREP_Q entries of its rotated query parts.
constexpr uint32_t PREP_Q = 256, PREP_TOKENS = 8;

// Entries [d, d + 4) of a rotated vector (rotated() has them one by one); d and half the rotated width are multiples of four.
__device__ __forceinline__ float4 rotated4(const float *v, uint32_t d, const Rot &r, const float2 *cs) {
    const float4 x = *reinterpret_cast<const float4 *>(v + d);
    if (d >= r.dims) return x;
    const uint32_t half = r.dims / 2;
    if (r.interleaved) {
        const float4 c = *reinterpret_cast<const float4 *>(cs + d / 2);
        return make_float4(x.x * c.x - x.y * c.y, x.y * c.x + x.x * c.y, x.z * c.z - x.w * c.w, x.w * c.z + x.z * c.w);
    }
    const bool low = d < half;
    const float2 *q = cs + (low ? d : d - half);
    const float4 y = *reinterpret_cast<const float4 *>(v + (low ? d + half : d - half)), c0 = *reinterpret_cast<const float4 *>(q), c1 = *reinterpret_cast<const float4 *>(q + 2);
    const float s = low ? -1.0f : 1.0f;
    return make_float4(x.x * c0.x + s * y.x * c0.y, x.y * c0.z + s * y.y * c0.w, x.z * c1.x + s * y.z * c1.y, x.w * c1.z + s * y.w * c1.w);
}

template <typename TA, bool FOURS>  // FOURS: all sizes and pitches are multiples of four, half the rotated width too
__global__ void __launch_bounds__(32 * PREP_TOKENS) latent_prep_kernel(LatentArgs a) {
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x * PREP_TOKENS + threadIdx.x / 32, lane = threadIdx.x & 31;
    if (t >= a.T) return;
    constexpr uint32_t V = FOURS ? 4 : 1;
    const uint32_t pos = a.positions[t];
    const float *y = a.y + (uint64_t)t * a.y_pitch;
    const float2 *cs = a.rot.table + (uint64_t)pos * (a.rot.dims / 2);
    auto turn = [&](TA *to, const float *v, uint32_t d) {
        if constexpr (FOURS) store4<TA>(to + d, rotated4(v, d, a.rot, cs));
        else to[d] = to_act<TA>(rotated(v, d, a.rot, cs));
    };
    if (blockIdx.y > 0) {
        TA *q = static_cast<TA *>(a.q) + (uint64_t)t * a.n_head * a.dq + a.kv_p;
        const uint32_t first = (blockIdx.y - 1) * PREP_Q, n = a.n_head * a.rot_dim;
#pragma unroll 4
        for (uint32_t u = V * lane; u < PREP_Q; u += 32 * V) {
            const uint32_t i = first + u;
            if (i >= n) break;
            const uint32_t h = i / a.rot_dim;
            turn(q + (uint64_t)h * a.dq, y + (uint64_t)h * a.rot_dim, i - h * a.rot_dim);
        }
        return;
    }
    const float *lat = y + (uint64_t)a.n_head * a.rot_dim;
    TA *row = static_cast<TA *>(a.cache) + ((uint64_t)a.tables[t][pos / KV_PAGE] * KV_PAGE + pos % KV_PAGE) * a.dq;
    for (uint32_t d = V * lane; d < a.rot_dim; d += 32 * V) turn(row + a.kv_p, lat + a.kv_rank, d);
    float s = 0.0f;
    if constexpr (FOURS) {
        constexpr uint32_t KEEP = 4;  // rows of up to 512 stay in registers
        float4 x[KEEP];
#pragma unroll
        for (uint32_t k = 0; k < KEEP; ++k) {
            const uint32_t i = 4 * lane + 128 * k;
            x[k] = i < a.kv_rank ? *reinterpret_cast<const float4 *>(lat + i) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            s += sq4(x[k]);
        }
        for (uint32_t i = 4 * lane + 128 * KEEP; i < a.kv_rank; i += 128) s += sq4(*reinterpret_cast<const float4 *>(lat + i));
        const float f = inv_rms(warp_sum(s), a.kv_rank, a.eps);
#pragma unroll
        for (uint32_t k = 0; k < KEEP; ++k) {
            const uint32_t i = 4 * lane + 128 * k;
            if (i < a.kv_rank) store4<TA>(row + i, mul44(mul4(x[k], f), *reinterpret_cast<const float4 *>(a.kv_norm + i)));
        }
        for (uint32_t i = 4 * lane + 128 * KEEP; i < a.kv_rank; i += 128) store4<TA>(row + i, mul44(mul4(*reinterpret_cast<const float4 *>(lat + i), f), *reinterpret_cast<const float4 *>(a.kv_norm + i)));
    } else {
        for (uint32_t i = lane; i < a.kv_rank; i += 32) s += lat[i] * lat[i];
        const float f = inv_rms(warp_sum(s), a.kv_rank, a.eps);
        for (uint32_t i = lane; i < a.kv_rank; i += 32) row[i] = to_act<TA>(lat[i] * f * a.kv_norm[i]);
    }
}

// ---- latent attention, plain form: one CTA per (token, head), any sizes; fp32 throughout when the cache is fp32 ---------------------
// Keys in blocks of 128: scores by the warps (lanes over the row), online softmax, then every thread adds up its own columns.
constexpr int LA_KEYS = 128, LA_THREADS = 128;
template <typename TA>
__global__ void __launch_bounds__(LA_THREADS) latent_attn_plain_kernel(LatentArgs a) {
    extern __shared__ float sm[];
    float *q = sm, *acc = q + a.dq, *p = acc + a.kv_p;  // [dq], [kv_p], [LA_KEYS]
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x / a.n_head, h = blockIdx.x % a.n_head, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t pos = a.positions[t], lo = first_seen(pos, a.window), hi = pos + 1;
    const int32_t *table = a.tables[t];
    const TA *qg = static_cast<const TA *>(a.q) + ((uint64_t)t * a.n_head + h) * a.dq, *cache = static_cast<const TA *>(a.cache);
    for (uint32_t i = threadIdx.x; i < a.dq; i += blockDim.x) q[i] = i < a.kv_rank || (i >= a.kv_p && i < a.kv_p + a.rot_dim) ? from_act(qg[i]) : 0.0f;
    for (uint32_t i = threadIdx.x; i < a.kv_p; i += blockDim.x) acc[i] = 0.0f;
    auto row_of = [&](uint32_t j) { return cache + ((uint64_t)table[j / KV_PAGE] * KV_PAGE + j % KV_PAGE) * a.dq; };
    float m = a.sink ? a.sink[h] : -INFINITY, l = a.sink ? 1.0f : 0.0f;  // a sink is a key seen before all others, without a value
    __syncthreads();
    for (uint32_t j0 = lo; j0 < hi; j0 += LA_KEYS) {
        const uint32_t n = min((uint32_t)LA_KEYS, hi - j0);
        for (uint32_t j = warp; j < n; j += LA_THREADS / 32) {
            const TA *k = row_of(j0 + j);
            float s = 0.0f;
            for (uint32_t i = lane; i < a.dq; i += 32) s = fmaf(q[i], from_act(k[i]), s);
            s = warp_sum(s);
            if (lane == 0) p[j] = s * a.scale;
        }
        __syncthreads();
        const float own = threadIdx.x < n ? p[threadIdx.x] : -INFINITY;
        float bm = warp_max(own);
        if (lane == 0) red[warp] = bm;
        __syncthreads();
        bm = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float m_new = fmaxf(m, bm), keep = expf(m - m_new), e = threadIdx.x < n ? expf(own - m_new) : 0.0f;
        p[threadIdx.x] = e;
        l = l * keep + block_sum(e, red);  // synchronises: p is complete
        m = m_new;
        for (uint32_t i = threadIdx.x; i < a.kv_rank; i += blockDim.x) {
            float v = acc[i] * keep;
            for (uint32_t j = 0; j < n; ++j) v = fmaf(p[j], from_act(row_of(j0 + j)[i]), v);
            acc[i] = v;
        }
        __syncthreads();
    }
    TA *o = static_cast<TA *>(a.o) + (uint64_t)t * a.n_head * a.o_head + (uint64_t)h * a.o_head;
    for (uint32_t i = threadIdx.x; i < a.kv_rank; i += blockDim.x) o[i] = to_act<TA>(acc[i] / l);
}

// ---- latent attention on the tensor cores (bf16 cache) ----------------------------------------------------------------------------
// A CTA takes 16 * MT consecutive (token, head) rows of one sequence -- all heads share the cache rows, so rows of several tokens
// and heads make one tile -- and walks the union of their windows in tiles of KT keys, two stages of cp.async.  Scores: a warp has
// 16 rows x 16 keys over the whole row width.  Softmax statistics, scores and weights are fp32; the weights enter the second
// product as value plus remainder, two bf16 rows each.  Output: a warp has all rows x its share of the latent columns (16 at a
// time, LM_PAIRS shares of them).  With fewer rows the warps also split the row width of the score product.  (mma.sync on purpose: with few tokens M is the number of heads, and 512 output columns for
// 128 rows would take all of tensor memory.)
constexpr int LM_THREADS = 256, LM_PAIRS = 4, LM_KEYS = 32;
__host__ __device__ constexpr uint32_t lm_part_row(uint32_t kv_p) { return kv_p + 4; }  // floats of one partial result: output, then maximum and sum
struct LmPlan {
    uint32_t q, k, stage, s, ph, pl, stat, bytes;  // byte offsets; stage: bytes of one key stage
    uint32_t stages;  // two, or one where that lets a second CTA onto the SM (its products then cover this one's loads)
    __host__ __device__ LmPlan(int mt, uint32_t dq) : LmPlan(mt, dq, 2) {
        if (mt < 4 && 2 * bytes > 224 * 1024) *this = LmPlan(mt, dq, 1);
    }
    __host__ __device__ LmPlan(int mt, uint32_t dq, uint32_t n_stage) : stages(n_stage) {
        const uint32_t M = 16 * mt, KT = LM_KEYS, row = (dq + 8) * 2, parts = 4 / mt;
        q = 0;
        k = q + M * row;
        stage = KT * row;
        s = k + stages * stage;
        ph = s + parts * M * (KT + 4) * 4;
        pl = ph + M * (KT + 8) * 2;
        stat = pl + M * (KT + 8) * 2;  // m, l, keep [M] f32, position [M]
        bytes = stat + 4 * M * 4;
    }
};

// How a warp copies rows of `chunks` 16-byte pieces: several short rows at a time, or one row in steps of 32 pieces.
struct RowCopy {
    uint32_t rows, row, chunk, chunks;  // rows per step of a warp, this lane's row among them and its first piece (chunks: none)
    __device__ explicit RowCopy(uint32_t n) : chunks(n) {
        const uint32_t lane = threadIdx.x & 31;
        rows = n >= 32 ? 1 : 32 / n;
        row = n >= 32 ? 0 : lane / n;
        chunk = n >= 32 ? lane : row < rows ? lane - row * n : n;
    }
};

// What a sink adds to a sum of powers of two below `top` (the largest scaled score times log2(e)).
__device__ __forceinline__ float sink_weight(float sink, float top) { return pow2(sink * 1.4426950408889634f - top); }

// NP: shares of sixteen latent columns per warp; a warp whose last share does not exist repeats another and drops it.
template <int MT, int NP>
__global__ void __launch_bounds__(LM_THREADS, MT == 4 ? 1 : 2) latent_attn_mma_kernel(LatentArgs a) {
    constexpr int M = 16 * MT, KT = LM_KEYS, SP = KT + 4, PP = KT + 8, PARTS = 4 / MT;  // MT row tiles x 2 key groups x PARTS of the row width = 8 warps
    extern __shared__ __align__(16) uint8_t smem[];
    const LmPlan pl(MT, a.dq);
    float *S = reinterpret_cast<float *>(smem + pl.s), *mx = reinterpret_cast<float *>(smem + pl.stat), *sum = mx + M, *keep = sum + M;
    int *rpos = reinterpret_cast<int *>(keep + M);
    bf16 *Ph = reinterpret_cast<bf16 *>(smem + pl.ph), *Pl = reinterpret_cast<bf16 *>(smem + pl.pl);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, row_bytes = (a.dq + 8) * 2, chunks = a.dq / 8;
    pdl_release();
    pdl_wait();
    __shared__ uint32_t tile_info[3];
    if (warp == 0) {
        RowSpan sp{blockIdx.x, 1};
        uint32_t f = 0;
        const uint32_t per = (a.n_head + M - 1) / M;
        if (a.single) sp.row0 = blockIdx.x / per, f = blockIdx.x % per * M;
        else find_tile(a.spans, a.n_seq, a.n_head, M, blockIdx.x, &sp, &f);
        if (lane == 0) tile_info[0] = sp.row0, tile_info[1] = sp.n, tile_info[2] = f;
    }
    __syncthreads();
    const uint32_t row0 = tile_info[0], f0 = tile_info[2], n_flat = tile_info[1] * a.n_head;
    if (f0 >= n_flat) return;
    const uint32_t n_here = min((uint32_t)M, n_flat - f0), pos0 = a.positions[row0];
    const uint32_t first_tok = f0 / a.n_head, last_tok = (f0 + n_here - 1) / a.n_head;
    const int32_t *table = a.tables[row0];
    // this CTA's keys
    uint32_t lo = first_seen(pos0 + first_tok, a.window), hi = pos0 + last_tok + 1;
    {
        const uint32_t per = ((hi - lo + gridDim.y - 1) / gridDim.y + KT - 1) / KT * KT;
        lo = min(hi, lo + blockIdx.y * per);
        hi = min(hi, lo + per);
    }
    const uint32_t n_tiles = (hi - lo + KT - 1) / KT;

    const RowCopy rc(chunks);
    auto load_keys = [&](uint32_t it) {
        const uint32_t base = smem_addr(smem + pl.k) + (pl.stages == 2 ? it & 1u : 0u) * pl.stage, step = LM_THREADS / 32 * rc.rows;
        constexpr uint32_t AT_ONCE = 4;  // rows whose pages are looked up together
        for (uint32_t r0 = warp * rc.rows + rc.row; r0 < KT; r0 += AT_ONCE * step) {
            int32_t page[AT_ONCE];
#pragma unroll
            for (uint32_t u = 0; u < AT_ONCE; ++u) {
                const uint32_t j = lo + it * KT + r0 + u * step;
                page[u] = r0 + u * step < KT && j < hi ? table[j / KV_PAGE] : -1;
            }
#pragma unroll
            for (uint32_t u = 0; u < AT_ONCE; ++u) {
                const uint32_t r = r0 + u * step, j = lo + it * KT + r;
                if (r >= KT) break;
                const bf16 *src = static_cast<const bf16 *>(a.cache) + (page[u] >= 0 ? ((uint64_t)page[u] * KV_PAGE + j % KV_PAGE) * a.dq : 0);
                for (uint32_t c = rc.chunk; c < chunks; c += 32) cp16(base + r * row_bytes + c * 16, src + 8 * c, page[u] >= 0);
            }
        }
    };
    {   // queries: consecutive flat rows are consecutive in memory
        const bf16 *q = static_cast<const bf16 *>(a.q) + ((uint64_t)row0 * a.n_head + f0) * a.dq;
        for (uint32_t i = threadIdx.x; i < M * chunks; i += LM_THREADS) {
            const uint32_t r = i / chunks, c = i - r * chunks;
            cp16(smem_addr(smem + pl.q) + r * row_bytes + c * 16, q + (r < n_here ? (uint64_t)r * a.dq + 8 * c : 0), r < n_here);
        }
    }
    if (n_tiles) load_keys(0);
    cp_commit();
    if (threadIdx.x < M) {
        mx[threadIdx.x] = -INFINITY;
        sum[threadIdx.x] = 0.0f;
        rpos[threadIdx.x] = threadIdx.x < n_here ? (int)(pos0 + (f0 + threadIdx.x) / a.n_head) : -1;
    }
    const float scale2 = a.scale * 1.4426950408889634f;  // weights are powers of two of the scaled score
    const uint32_t n_pair = a.kv_p / 16;
    float acc[MT][NP][2][4];
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int p = 0; p < NP; ++p)
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[i][p][n][e] = 0.0f;

    const uint32_t qs = smem_addr(smem + pl.q), mt_s = warp % MT, kg = warp / MT % 2, wp = warp / (2 * MT);
    const uint32_t k_steps = a.dq / 16, k_first = k_steps * wp / PARTS, k_end = k_steps * (wp + 1) / PARTS;
    const uint32_t a_off = (lane & 15) * row_bytes + (lane >> 4) * 16, b_off = ((lane & 7) + ((lane >> 4) << 3)) * row_bytes + ((lane >> 3) & 1) * 16;
    const uint32_t v_off = ((lane & 7) + (((lane >> 3) & 1) << 3)) * row_bytes + (lane >> 4) * 16, p_off = (lane & 15) * (PP * 2) + (lane >> 4) * 16;
    for (uint32_t it = 0; it < n_tiles; ++it) {
        if (pl.stages == 2) {
            if (it + 1 < n_tiles) load_keys(it + 1);
            cp_commit();
            cp_wait<1>();
        } else {
            if (it) load_keys(it);
            cp_commit();
            cp_wait<0>();
        }
        __syncthreads();
        const uint32_t ks = smem_addr(smem + pl.k) + (pl.stages == 2 ? it & 1u : 0u) * pl.stage;
        {
            float c[2][2][4] = {};  // even and odd steps have accumulators of their own: no product waits for the one before
            const uint32_t qa = qs + mt_s * 16 * row_bytes + a_off, kb = ks + kg * 16 * row_bytes + b_off;
            auto step = [&](uint32_t k, float (&d)[2][4]) {
                uint32_t fa[4], fb[4];
                ldsm4(fa, qa + k * 32);
                ldsm4(fb, kb + k * 32);
                mma_bf16(d[0], fa, fb[0], fb[1]);
                mma_bf16(d[1], fa, fb[2], fb[3]);
            };
            uint32_t k = k_first;
#pragma unroll 3
            for (; k + 1 < k_end; k += 2) {
                step(k, c[0]);
                step(k + 1, c[1]);
            }
            if (k < k_end) step(k, c[0]);
            float *s = S + (wp * M + mt_s * 16 + lane / 4) * SP + kg * 16 + 2 * (lane & 3);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                *reinterpret_cast<float2 *>(s + 8 * n) = make_float2(c[0][n][0] + c[1][n][0], c[0][n][1] + c[1][n][1]);
                *reinterpret_cast<float2 *>(s + 8 * SP + 8 * n) = make_float2(c[0][n][2] + c[1][n][2], c[0][n][3] + c[1][n][3]);
            }
        }
        __syncthreads();
        {   // online softmax: lane = key, the warp's rows side by side
            constexpr int R = M / 8;
            const int j = (int)(lo + it * KT) + (int)lane, r0 = warp * R;
            float v[R], m_old[R], m_new[R], l[R];
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int p = rpos[r0 + i];
                float sc = S[(r0 + i) * SP + lane];
#pragma unroll
                for (int w = 1; w < PARTS; ++w) sc += S[(w * M + r0 + i) * SP + lane];
                v[i] = j <= p && j < (int)hi && (a.window == 0 || p - j < (int)a.window) ? sc * scale2 : -INFINITY;
                m_new[i] = v[i];
                m_old[i] = mx[r0 + i];
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int i = 0; i < R; ++i) m_new[i] = fmaxf(m_new[i], __shfl_xor_sync(0xffffffffu, m_new[i], o));
#pragma unroll
            for (int i = 0; i < R; ++i) {
                m_new[i] = fmaxf(m_new[i], m_old[i]);
                const float e = m_new[i] == -INFINITY ? 0.0f : pow2(v[i] - m_new[i]);
                const bf16 h = __float2bfloat16_rn(e);
                Ph[(r0 + i) * PP + lane] = h;
                Pl[(r0 + i) * PP + lane] = __float2bfloat16_rn(e - __bfloat162float(h));
                l[i] = e;
            }
#pragma unroll
            for (int o = 16; o > 0; o >>= 1)
#pragma unroll
                for (int i = 0; i < R; ++i) l[i] += __shfl_xor_sync(0xffffffffu, l[i], o);
            __syncwarp();  // every lane has read the old maxima
#pragma unroll
            for (int i = 0; i < R; ++i)
                if (lane == i) {
                    const float f = m_new[i] == -INFINITY ? 1.0f : pow2(m_old[i] - m_new[i]);
                    keep[r0 + i] = f;
                    mx[r0 + i] = m_new[i];
                    sum[r0 + i] = sum[r0 + i] * f + l[i];
                }
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < MT; ++i) {
            const float f0r = keep[i * 16 + lane / 4], f1r = keep[i * 16 + lane / 4 + 8];
#pragma unroll
            for (int p = 0; p < NP; ++p)
#pragma unroll
                for (int n = 0; n < 2; ++n) acc[i][p][n][0] *= f0r, acc[i][p][n][1] *= f0r, acc[i][p][n][2] *= f1r, acc[i][p][n][3] *= f1r;
        }
#pragma unroll
        for (int kk = 0; kk < KT / 16; ++kk) {
            uint32_t fh[MT][4], fl[MT][4];
#pragma unroll
            for (int i = 0; i < MT; ++i) {
                ldsm4(fh[i], smem_addr(Ph) + (i * 16 * PP + kk * 16) * 2 + p_off);
                ldsm4(fl[i], smem_addr(Pl) + (i * 16 * PP + kk * 16) * 2 + p_off);
            }
            uint32_t fv[NP][4];
#pragma unroll
            for (int p = 0; p < NP; ++p) ldsm4t(fv[p], ks + kk * 16 * row_bytes + min(warp + 8 * p, n_pair - 1) * 32 + v_off);
#pragma unroll
            for (int part = 0; part < 2; ++part)
#pragma unroll
                for (int p = 0; p < NP; ++p)
#pragma unroll
                    for (int i = 0; i < MT; ++i) {
                        mma_bf16(acc[i][p][0], part ? fl[i] : fh[i], fv[p][0], fv[p][1]);
                        mma_bf16(acc[i][p][1], part ? fl[i] : fh[i], fv[p][2], fv[p][3]);
                    }
        }
        __syncthreads();
    }
    cp_wait<0>();
    __syncthreads();
    const bool whole = gridDim.y == 1;
#pragma unroll
    for (int i = 0; i < MT; ++i)
#pragma unroll
        for (int hf = 0; hf < 2; ++hf) {
            const uint32_t r = i * 16 + lane / 4 + 8 * hf;
            if (r >= n_here) continue;
            const uint64_t flat = (uint64_t)row0 * a.n_head + f0 + r;
            const float inv = whole ? 1.0f / (sum[r] + (a.sink ? sink_weight(a.sink[(f0 + r) % a.n_head], mx[r]) : 0.0f)) : 1.0f;
#pragma unroll
            for (int p = 0; p < NP; ++p) {
                if (warp + 8 * p >= n_pair) break;
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const uint32_t col = (warp + 8 * p) * 16 + n * 8 + 2 * (lane & 3);
                    const float v0 = acc[i][p][n][2 * hf] * inv, v1 = acc[i][p][n][2 * hf + 1] * inv;
                    if (whole) *reinterpret_cast<__nv_bfloat162 *>(static_cast<bf16 *>(a.o) + flat * a.o_head + col) = __floats2bfloat162_rn(v0, v1);
                    else *reinterpret_cast<float2 *>(a.part + ((uint64_t)blockIdx.y * a.T * a.n_head + flat) * lm_part_row(a.kv_p) + col) = make_float2(v0, v1);
                }
            }
            if (!whole && warp == 0 && (lane & 3) == 0)
                *reinterpret_cast<float2 *>(a.part + ((uint64_t)blockIdx.y * a.T * a.n_head + flat) * lm_part_row(a.kv_p) + a.kv_p) = make_float2(mx[r], sum[r]);
        }
}

// The splits of one (token, head) row put together, a CTA per row: `groups` groups of 128 threads take splits in turn, a thread four
// columns (and every 512th).  What the first splits hold is requested before their weights are known.
constexpr uint32_t MERGE_MAX = 256, MERGE_AT_ONCE = 8, MERGE_GROUPS = 8;  // splits; loads of a thread in flight
__global__ void __launch_bounds__(128 * MERGE_GROUPS) latent_merge_kernel(LatentArgs a, uint32_t n_splits) {
    extern __shared__ float sums[];  // [groups - 1][512]
    __shared__ float weight[MERGE_MAX], total;
    const uint32_t lane = threadIdx.x & 31, group = threadIdx.x / 128, groups = blockDim.x / 128;
    pdl_release();
    pdl_wait();
    uint64_t flat = blockIdx.x;
    if (!a.single) {  // only the rows of these spans have partial results
        RowSpan sp;
        uint32_t f;
        find_tile(a.spans, a.n_seq, a.n_head, 1, (uint32_t)flat, &sp, &f);
        flat = (uint64_t)sp.row0 * a.n_head + f;
    }
    const uint64_t stride = (uint64_t)a.T * a.n_head * lm_part_row(a.kv_p);
    const float *p = a.part + flat * lm_part_row(a.kv_p), *ml = p + a.kv_p;
    bf16 *o = static_cast<bf16 *>(a.o) + flat * a.o_head;
    const uint32_t steps = (a.kv_p + 511) / 512;
    for (uint32_t k = 0; k < steps; ++k) {
        const uint32_t c = 512 * k + 4 * (threadIdx.x % 128);
        const bool in = c < a.kv_p;
        float4 u[MERGE_AT_ONCE];
        auto request = [&](uint32_t s0) {
#pragma unroll
            for (uint32_t i = 0; i < MERGE_AT_ONCE; ++i) {
                const uint32_t s = s0 + i * groups;
                u[i] = in && s < n_splits ? *reinterpret_cast<const float4 *>(p + s * stride + c) : make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            }
        };
        request(group);
        if (k == 0) {
            if (threadIdx.x < 32) {
                float2 t[MERGE_MAX / 32];
                float m = -INFINITY, l = 0.0f;
#pragma unroll
                for (uint32_t i = 0; i < MERGE_MAX / 32; ++i) {
                    const uint32_t s = lane + 32 * i;
                    t[i] = s < n_splits ? *reinterpret_cast<const float2 *>(ml + s * stride) : make_float2(-INFINITY, 0.0f);
                    m = fmaxf(m, t[i].x);
                }
                m = warp_max(m);
#pragma unroll
                for (uint32_t i = 0; i < MERGE_MAX / 32; ++i) {
                    const float w = pow2(t[i].x - m);
                    weight[lane + 32 * i] = w;
                    l += w * t[i].y;
                }
                l = warp_sum(l);
                if (a.sink) l += sink_weight(a.sink[flat % a.n_head], m);
                if (lane == 0) total = l;
            }
            __syncthreads();
        }
        float4 v = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        for (uint32_t s0 = group; s0 < n_splits; s0 += MERGE_AT_ONCE * groups) {
            if (s0 != group) request(s0);
#pragma unroll
            for (uint32_t i = 0; i < MERGE_AT_ONCE; ++i) {
                const uint32_t s = s0 + i * groups;
                const float w = s < n_splits ? weight[s] : 0.0f;
                v.x = fmaf(w, u[i].x, v.x), v.y = fmaf(w, u[i].y, v.y), v.z = fmaf(w, u[i].z, v.z), v.w = fmaf(w, u[i].w, v.w);
            }
        }
        if (groups > 1) {
            if (k) __syncthreads();  // (the sums before have been read)
            float4 *mine = reinterpret_cast<float4 *>(sums) + threadIdx.x % 128;
            if (group) mine[(group - 1) * 128] = v;
            __syncthreads();
            if (group) continue;
            for (uint32_t g = 0; g + 1 < groups; ++g) {
                const float4 w = mine[g * 128];
                v.x += w.x, v.y += w.y, v.z += w.z, v.w += w.w;
            }
        }
        if (in) store4<bf16>(o + c, mul4(v, 1.0f / total));
    }
}

// ---- latent attention of prompts: keys and values rebuilt from the latent, bf16 -------------------------------------------------------
// With many tokens per sequence it is cheaper to multiply the window's latents out once (linear.cu) and attend per head: the score
// product is dim + rot_dim wide and the output vdim wide, against kv_rank each in the latent space.  A CTA takes one head and 64
// consecutive tokens of a sequence, a warp 16 of them; keys come in tiles of 64, the next keys while this tile is
// weighted, the next values during the next scores.  Scores, softmax
// and the weights' two bf16 parts (value and remainder) stay in registers.
constexpr int PF_TOKENS = 64, PF_KEYS = 64, PF_THREADS = 128;
struct PfPlan {
    uint32_t k, v, k_stage, v_stage, bytes;
    __host__ __device__ PfPlan(uint32_t dqk, uint32_t vd) {
        k = PF_TOKENS * (dqk + 8) * 2;
        k_stage = PF_KEYS * (dqk + 8) * 2;
        v = k + k_stage;
        v_stage = PF_KEYS * (vd + 8) * 2;
        bytes = v + v_stage + 128;  // a row's reads may go up to 64 columns past its end
    }
};

__global__ void __launch_bounds__(256) latent_gather_kernel(LatentPrefillArgs a) {
    pdl_release();
    pdl_wait();
    const uint32_t key = blockIdx.x * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (key >= a.n_keys) return;
    uint32_t s = 0;
    while (s + 1 < a.n_span && key >= a.span[s + 1].key0) ++s;
    const PrefillSpan sp = a.span[s];
    const uint32_t p = sp.pos0 - sp.hist + (key - sp.key0);
    const bool live = p < sp.pos0 + sp.n;
    const uint4 *src = reinterpret_cast<const uint4 *>(static_cast<const bf16 *>(a.cache) + (live ? ((uint64_t)a.tables[sp.row0][p / KV_PAGE] * KV_PAGE + p % KV_PAGE) * a.dq : 0));
    uint4 *dst = reinterpret_cast<uint4 *>(static_cast<bf16 *>(a.lat) + (uint64_t)key * a.dq);
    for (uint32_t i = lane; i < a.dq / 8; i += 32) dst[i] = live ? src[i] : make_uint4(0, 0, 0, 0);
    if (!a.pages) return;
    if (key == sp.key0 && lane == 0) a.page_tables[sp.row0] = a.numbers + ((int64_t)(sp.key0 / KV_PAGE) - (int64_t)(p / KV_PAGE));
    const uint32_t chunks = (a.dq - a.kv_p) / 8;  // of the rotated part, which every head's row gets
    if (!chunks) return;
    const RowCopy rc(chunks);
    bf16 *page = static_cast<bf16 *>(a.pages) + ((uint64_t)(key / KV_PAGE) * a.n_head * KV_PAGE + key % KV_PAGE) * a.page_row + a.page_rot0;
    for (uint32_t c = rc.chunk; c < chunks; c += 32) {
        const uint4 v = live ? src[a.kv_p / 8 + c] : make_uint4(0, 0, 0, 0);
        for (uint32_t h = rc.row; h < a.n_head; h += rc.rows) reinterpret_cast<uint4 *>(page + (uint64_t)h * KV_PAGE * a.page_row)[c] = v;
    }
}

template <int NV>  // columns of a value in sixteens; what goes past vdim_k is computed from whatever follows in shared memory and dropped
__global__ void __launch_bounds__(PF_THREADS, NV <= 8 ? 3 : 1) latent_prefill_kernel(LatentPrefillArgs a) {
    extern __shared__ __align__(16) uint8_t smem[];
    const uint32_t rot_p = a.dq - a.kv_p, dqk = a.dim_k + rot_p, qrow = (dqk + 8) * 2, vrow = (a.vdim_k + 8) * 2;
    const PfPlan pl(dqk, a.vdim_k);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y;
    pdl_release();
    pdl_wait();
    uint32_t s = 0;
    while (s + 1 < a.n_span && blockIdx.x >= a.span[s + 1].tile0) ++s;
    const PrefillSpan sp = a.span[s];
    const uint32_t t0 = (blockIdx.x - sp.tile0) * PF_TOKENS, n_tok = min((uint32_t)PF_TOKENS, sp.n - t0);
    const uint32_t lo = first_seen(sp.pos0 + t0, a.window), hi = sp.pos0 + t0 + n_tok, kbase = sp.pos0 - sp.hist;
    const uint32_t n_tiles = (hi - lo + PF_KEYS - 1) / PF_KEYS;
    const uint32_t qs = smem_addr(smem);

    {   // queries: unrotated and rotated parts side by side
        const uint32_t cn = a.dim_k / 8, cr = rot_p / 8, ct = cn + cr;
        for (uint32_t i = threadIdx.x; i < PF_TOKENS * ct; i += PF_THREADS) {
            const uint32_t r = i / ct, c = i - r * ct;
            const bool in = r < n_tok;
            const uint64_t t = sp.row0 + t0 + (in ? r : 0);
            const bf16 *src = c < cn ? static_cast<const bf16 *>(a.qn) + t * a.qn_pitch + (uint64_t)h * a.dim_p + 8 * c
                                     : static_cast<const bf16 *>(a.q) + (t * a.n_head + h) * a.dq + a.kv_p + 8 * (c - cn);
            cp16(qs + r * qrow + c * 16, src, in);
        }
    }
    auto load_k = [&](uint32_t it) {
        const uint32_t j0 = lo + it * PF_KEYS, cn = a.dim_k / 8, ct = cn + rot_p / 8;
        for (uint32_t i = threadIdx.x; i < PF_KEYS * ct; i += PF_THREADS) {
            const uint32_t r = i / ct, c = i - r * ct;
            const bool in = j0 + r < hi;
            const uint64_t key = sp.key0 + (in ? j0 + r - kbase : 0);
            const bf16 *src = c < cn ? static_cast<const bf16 *>(a.expanded) + key * a.ex_pitch + (uint64_t)h * a.dim_k + 8 * c
                                     : static_cast<const bf16 *>(a.lat) + key * a.dq + a.kv_p + 8 * (c - cn);
            cp16(qs + pl.k + r * qrow + c * 16, src, in);
        }
    };
    auto load_v = [&](uint32_t it) {
        const uint32_t j0 = lo + it * PF_KEYS, cv = a.vdim_k / 8;
        for (uint32_t i = threadIdx.x; i < PF_KEYS * cv; i += PF_THREADS) {
            const uint32_t r = i / cv, c = i - r * cv;
            const bool in = j0 + r < hi;
            const uint64_t key = sp.key0 + (in ? j0 + r - kbase : 0);
            cp16(qs + pl.v + r * vrow + c * 16, static_cast<const bf16 *>(a.expanded) + key * a.ex_pitch + a.ex_v0 + (uint64_t)h * a.vdim_k + 8 * c, in);
        }
    };
    load_k(0);
    cp_commit();
    load_v(0);
    cp_commit();
    const float scale2 = a.scale * 1.4426950408889634f;
    const int p0 = (int)(sp.pos0 + t0 + warp * 16 + lane / 4), p1 = p0 + 8;  // positions of this thread's two rows
    const int w_first = (int)(sp.pos0 + t0 + warp * 16), w_last = w_first + 15, win = a.window ? (int)a.window : 0x7fffffff;
    float o[NV][2][4], m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[v][n][e] = 0.0f;
    const uint32_t qa = qs + (warp * 16 + (lane & 15)) * qrow + (lane >> 4) * 16;
    const uint32_t b_off = ((lane & 7) + ((lane >> 4) << 3)) * qrow + ((lane >> 3) & 1) * 16, v_off = ((lane & 7) + (((lane >> 3) & 1) << 3)) * vrow + (lane >> 4) * 16;
    for (uint32_t it = 0; it < n_tiles; ++it) {
        cp_wait<1>();
        __syncthreads();  // this tile's keys are there
        const int j0 = (int)(lo + it * PF_KEYS);
        const bool any = j0 <= w_last && (long long)j0 + PF_KEYS - 1 > (long long)w_first - win;  // does one of the warp's tokens see one of these keys?
        const uint32_t kb = qs + pl.k, vb = qs + pl.v;
        float c[PF_KEYS / 8][4];
#pragma unroll
        for (int n = 0; n < PF_KEYS / 8; ++n) c[n][0] = c[n][1] = c[n][2] = c[n][3] = 0.0f;
        if (any) {
#pragma unroll 4
            for (uint32_t k = 0; k < dqk / 16; ++k) {
                uint32_t fa[4];
                ldsm4(fa, qa + k * 32);
#pragma unroll
                for (int g = 0; g < PF_KEYS / 16; ++g) {
                    uint32_t fb[4];
                    ldsm4(fb, kb + g * 16 * qrow + b_off + k * 32);
                    mma_bf16(c[2 * g], fa, fb[0], fb[1]);
                    mma_bf16(c[2 * g + 1], fa, fb[2], fb[3]);
                }
            }
        }
        __syncthreads();  // nobody reads them any more: the next tile's may come
        if (it + 1 < n_tiles) load_k(it + 1);
        cp_commit();
        if (any) {
            const bool inside = j0 + PF_KEYS - 1 <= w_first && (long long)w_last - j0 < win && j0 + PF_KEYS <= (int)hi;  // nothing to mask
            float b0 = -INFINITY, b1 = -INFINITY;
#pragma unroll
            for (int n = 0; n < PF_KEYS / 8; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int j = j0 + 8 * n + 2 * (int)(lane & 3) + e;
                    c[n][e] = inside || (j <= p0 && p0 - j < win) ? c[n][e] * scale2 : -INFINITY;
                    c[n][2 + e] = inside || (j <= p1 && p1 - j < win) ? c[n][2 + e] * scale2 : -INFINITY;
                    b0 = fmaxf(b0, c[n][e]);
                    b1 = fmaxf(b1, c[n][2 + e]);
                }
            b0 = fmaxf(b0, __shfl_xor_sync(0xffffffffu, b0, 1)), b0 = fmaxf(b0, __shfl_xor_sync(0xffffffffu, b0, 2));
            b1 = fmaxf(b1, __shfl_xor_sync(0xffffffffu, b1, 1)), b1 = fmaxf(b1, __shfl_xor_sync(0xffffffffu, b1, 2));
            const float n0 = fmaxf(m0, b0), n1 = fmaxf(m1, b1);
            const float s0 = n0 == -INFINITY ? 0.0f : n0, s1 = n1 == -INFINITY ? 0.0f : n1;  // a row that has seen nothing yet keeps weights of zero
            const float f0 = pow2(m0 - s0), f1 = pow2(m1 - s1);
            m0 = n0, m1 = n1;
            l0 *= f0, l1 *= f1;
#pragma unroll
            for (int v = 0; v < NV; ++v)
#pragma unroll
                for (int n = 0; n < 2; ++n) o[v][n][0] *= f0, o[v][n][1] *= f0, o[v][n][2] *= f1, o[v][n][3] *= f1;
        }
        cp_wait<1>();
        __syncthreads();  // and the values
        if (any) {
            const float s0 = m0 == -INFINITY ? 0.0f : m0, s1 = m1 == -INFINITY ? 0.0f : m1;
#pragma unroll
            for (int kk = 0; kk < PF_KEYS / 16; ++kk) {
                uint32_t ph[4], pr[4];
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int r = 0; r < 2; ++r) {  // fragment register 2n + r: row half r of key half n
                        const float mr = r ? s1 : s0;
                        const float e0 = pow2(c[2 * kk + n][2 * r] - mr), e1 = pow2(c[2 * kk + n][2 * r + 1] - mr);
                        if (r) l1 += e0 + e1;
                        else l0 += e0 + e1;
                        const __nv_bfloat162 hi2 = __floats2bfloat162_rn(e0, e1);
                        const __nv_bfloat162 lo2 = __floats2bfloat162_rn(e0 - __low2float(hi2), e1 - __high2float(hi2));
                        ph[2 * n + r] = *reinterpret_cast<const uint32_t *>(&hi2);
                        pr[2 * n + r] = *reinterpret_cast<const uint32_t *>(&lo2);
                    }
#pragma unroll
                for (int v = 0; v < NV; ++v) {
                    uint32_t fv[4];
                    ldsm4t(fv, vb + kk * 16 * vrow + v * 32 + v_off);
                    mma_bf16(o[v][0], ph, fv[0], fv[1]);
                    mma_bf16(o[v][1], ph, fv[2], fv[3]);
                    mma_bf16(o[v][0], pr, fv[0], fv[1]);
                    mma_bf16(o[v][1], pr, fv[2], fv[3]);
                }
            }
        }
        __syncthreads();
        if (it + 1 < n_tiles) load_v(it + 1);
        cp_commit();
    }
    cp_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1), l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1), l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const uint32_t tl = warp * 16 + lane / 4 + 8 * r;
        if (tl >= n_tok) continue;
        const uint64_t t = sp.row0 + t0 + tl;
        float sum = r ? l1 : l0;
        if (a.sink) sum += sink_weight(a.sink[h], r ? m1 : m0);
        if (a.gate) sum *= 1.0f + expf(-a.gate[t * a.gate_pitch + h]);
        const float f = 1.0f / sum;
        bf16 *out = static_cast<bf16 *>(a.out) + t * a.out_pitch + (uint64_t)h * a.vdim;
        const bf16 *gate = a.gate_act ? static_cast<const bf16 *>(a.gate_act) + t * a.gate_pitch + (uint64_t)h * a.vdim : nullptr;
#pragma unroll
        for (int v = 0; v < NV; ++v)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const uint32_t col = v * 16 + n * 8 + 2 * (lane & 3);
                if (col >= a.vdim) continue;
                float o0 = o[v][n][2 * r] * f, o1 = o[v][n][2 * r + 1] * f;
                if (gate) {
                    o0 /= 1.0f + expf(-__bfloat162float(gate[col]));
                    if (col + 1 < a.vdim) o1 /= 1.0f + expf(-__bfloat162float(gate[col + 1]));
                }
                if ((a.vdim & 1) == 0) *reinterpret_cast<__nv_bfloat162 *>(out + col) = __floats2bfloat162_rn(o0, o1);
                else {
                    out[col] = __float2bfloat16_rn(o0);
                    if (col + 1 < a.vdim) out[col + 1] = __float2bfloat16_rn(o1);
                }
            }
    }
}

// ---- retention -------------------------------------------------------------------------------------------------------------------
// q and k of a token rotated in place, k scaled.
__global__ void __launch_bounds__(256) retention_prep_kernel(RetentionArgs a) {
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x, half = a.rot.dims / 2, rest = a.dim - a.rot.dims, per = half + rest;
    const float2 *cs = a.rot.table + (uint64_t)a.positions[t] * half;
    float *y = a.y + (uint64_t)t * a.y_pitch;
    for (uint32_t i = threadIdx.x; i < 2 * a.n_head * per; i += blockDim.x) {
        const uint32_t v = i / per, e = i - v * per;  // vector (queries, then keys) and pair or unrotated entry within it
        float *p = y + (uint64_t)v * a.dim;
        const float s = v >= a.n_head ? a.k_scale : 1.0f;
        if (e < half) {
            const uint32_t iu = a.rot.interleaved ? 2 * e : e, iv = a.rot.interleaved ? 2 * e + 1 : e + half;
            const float u = p[iu], w = p[iv];
            p[iu] = (u * cs[e].x - w * cs[e].y) * s;
            p[iv] = (w * cs[e].x + u * cs[e].y) * s;
        } else {
            p[a.rot.dims + e - half] *= s;
        }
    }
}

// One CTA carries 32 columns of one head's state through the rows of one sequence, token by token: lane = column, warp = DW of
// the state's rows, kept in registers.  S = decay S + k v^T, o = S^T q; the warps' parts of o are added up once per block of tokens,
// while the next block's q, k and v are on their way to shared memory.
template <int DW>
struct RtPlan {
    static constexpr int D = 8 * DW, BLOCK = DW > 16 ? 8 : 16;
    static constexpr uint32_t Q = 0, K = Q + BLOCK * D, V = K + BLOCK * D, STAGE = V + BLOCK * 32, PART = 2 * STAGE, FLOATS = PART + 8 * BLOCK * 32;
};
__device__ __forceinline__ void cp4(float *dst, const float *src, bool in) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(in ? 4 : 0) : "memory");
}
template <int DW>
__global__ void __launch_bounds__(256) retention_kernel(RetentionArgs a) {
    using R = RtPlan<DW>;
    constexpr int D = R::D, BLOCK = R::BLOCK;
    extern __shared__ __align__(16) float sm[];
    float *part = sm + R::PART;  // [8][BLOCK][32]
    pdl_release();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, col = blockIdx.x * 32 + lane;
    const RowSpan sp = a.spans[blockIdx.z];
    const bool live = col < a.vdim;
    const float decay = a.decay[h];
    float *state = a.state + (((uint64_t)a.slots[sp.row0] * a.n_head + h) * a.dim) * a.vdim + col;
    const float *yq = a.y + (uint64_t)sp.row0 * a.y_pitch + (uint64_t)h * a.dim, *yk = yq + (uint64_t)a.n_head * a.dim;
    const float *yv = a.y + (uint64_t)sp.row0 * a.y_pitch + 2ull * a.n_head * a.dim + (uint64_t)h * a.vdim + col;
    auto load = [&](uint32_t t0, uint32_t stage) {
        float *s = sm + stage * R::STAGE;
        const uint32_t n = min((uint32_t)BLOCK, sp.n - t0);
        for (uint32_t i = threadIdx.x; i < n * D; i += 256) {
            const uint32_t t = i / D, d = i % D;
            const bool in = d < a.dim;
            const uint64_t o = (uint64_t)(t0 + t) * a.y_pitch + (in ? d : 0);
            cp4(s + R::Q + i, yq + o, in);
            cp4(s + R::K + i, yk + o, in);
        }
        for (uint32_t t = warp; t < n; t += 8) cp4(s + R::V + t * 32 + lane, live ? yv + (uint64_t)(t0 + t) * a.y_pitch : a.y, live);
    };
    load(0, 0);
    cp_commit();
    float S[DW];
    const bool fresh = a.positions[sp.row0] == 0;
#pragma unroll
    for (int i = 0; i < DW; ++i) {
        const uint32_t d = warp * DW + i;
        S[i] = !fresh && live && d < a.dim ? state[d * a.vdim] : 0.0f;
    }
    uint32_t stage = 0;
    for (uint32_t t0 = 0; t0 < sp.n; t0 += BLOCK, stage ^= 1u) {
        const uint32_t n = min((uint32_t)BLOCK, sp.n - t0);
        if (t0 + BLOCK < sp.n) load(t0 + BLOCK, stage ^ 1u);
        cp_commit();
        cp_wait<1>();
        __syncthreads();  // this block's operands are there, and everyone is done with the sums of the last one
        const float *q = sm + stage * R::STAGE + R::Q + warp * DW, *k = sm + stage * R::STAGE + R::K + warp * DW, *v = sm + stage * R::STAGE + R::V + lane;
        auto token = [&](uint32_t t) {
            const float vv = v[t * 32];
            float o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int i = 0; i < DW; i += 4) {
                const float4 kk = *reinterpret_cast<const float4 *>(k + t * D + i), qq = *reinterpret_cast<const float4 *>(q + t * D + i);
                S[i] = fmaf(kk.x, vv, decay * S[i]), o[0] = fmaf(qq.x, S[i], o[0]);
                S[i + 1] = fmaf(kk.y, vv, decay * S[i + 1]), o[1] = fmaf(qq.y, S[i + 1], o[1]);
                S[i + 2] = fmaf(kk.z, vv, decay * S[i + 2]), o[2] = fmaf(qq.z, S[i + 2], o[2]);
                S[i + 3] = fmaf(kk.w, vv, decay * S[i + 3]), o[3] = fmaf(qq.w, S[i + 3], o[3]);
            }
            part[(warp * BLOCK + t) * 32 + lane] = (o[0] + o[1]) + (o[2] + o[3]);
        };
        if (n == BLOCK) {
#pragma unroll 4
            for (uint32_t t = 0; t < BLOCK; ++t) token(t);
        } else {
            for (uint32_t t = 0; t < n; ++t) token(t);
        }
        __syncthreads();
        for (uint32_t t = warp; t < n; t += 8) {
            float o = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; ++w) o += part[(w * BLOCK + t) * 32 + lane];
            if (live) a.o[((uint64_t)(sp.row0 + t0 + t) * a.n_head + h) * a.vdim + col] = o;
        }
    }
    cp_wait<0>();
#pragma unroll
    for (int i = 0; i < DW; ++i) {
        const uint32_t d = warp * DW + i;
        if (live && d < a.dim) state[d * a.vdim] = S[i];
    }
}

// The same recurrence for long spans.  A thread has R of the state's rows x 2 columns, so that one read of q and k from shared
// memory serves both: lane = rows, warp = columns, 16 columns per CTA.  Over a block of eight tokens the state is kept without its
// decay (S' = decay^-t S, the values scaled instead, the outputs scaled back), and the 16 sums of a block (token, column) are added
// over the lanes by one exchange that leaves every other lane the sum it stores.
constexpr int RS_BLOCK = 8, RS_COLS = 16;
template <int R>
__global__ void __launch_bounds__(256, R <= 4 ? 2 : 1) retention_span_kernel(RetentionArgs a) {
    constexpr int D = 32 * R, V4 = R <= 4 ? 1 : R / 4, W = R / V4;  // a lane's rows: V4 groups of W neighbours
    constexpr uint32_t STAGES = R <= 4 ? 4 : 2;
    __shared__ __align__(16) float qs[STAGES][RS_BLOCK][D], ks[STAGES][RS_BLOCK][D], vs[STAGES][RS_BLOCK][RS_COLS];
    pdl_release();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, col0 = blockIdx.x * RS_COLS;
    const RowSpan sp = a.spans[a.first_long + blockIdx.z];
    const float *yq = a.y + (uint64_t)sp.row0 * a.y_pitch + (uint64_t)h * a.dim, *yk = yq + (uint64_t)a.n_head * a.dim;
    const float *yv = a.y + (uint64_t)sp.row0 * a.y_pitch + 2ull * a.n_head * a.dim + (uint64_t)h * a.vdim + col0;
    const bool quads = a.dim % 4 == 0;  // rows of y start at multiples of 16 bytes, so do the heads then
    auto load = [&](uint32_t t0, uint32_t stage) {
        const uint32_t n = min((uint32_t)RS_BLOCK, sp.n - t0), step = quads ? 4 : 1;
        for (uint32_t i = threadIdx.x * step; i < RS_BLOCK * D; i += 256 * step) {
            const uint32_t t = i / D, d = i % D;
            const bool in = t < n && d < a.dim;
            const uint64_t o = in ? (uint64_t)(t0 + t) * a.y_pitch + d : 0;
            if (quads) {
                cp16(smem_addr(&qs[stage][t][d]), yq + o, in);
                cp16(smem_addr(&ks[stage][t][d]), yk + o, in);
            } else {
                cp4(&qs[stage][t][d], yq + o, in);
                cp4(&ks[stage][t][d], yk + o, in);
            }
        }
        if (threadIdx.x < RS_BLOCK * RS_COLS) {
            const uint32_t t = threadIdx.x / RS_COLS, c = threadIdx.x % RS_COLS;
            const bool in = t < n && col0 + c < a.vdim;
            cp4(&vs[stage][t][c], in ? yv + (uint64_t)(t0 + t) * a.y_pitch + c : a.y, in);
        }
    };
#pragma unroll
    for (uint32_t s = 0; s + 1 < STAGES; ++s) {
        if (s * RS_BLOCK < sp.n) load(s * RS_BLOCK, s);
        cp_commit();
    }
    const float decay = a.decay[h];
    float up[RS_BLOCK];  // decay^-(t+1)
    up[0] = 1.0f / decay;
#pragma unroll
    for (int t = 1; t < RS_BLOCK; ++t) up[t] = up[t - 1] * up[0];
    float down = decay, block = decay;  // decay^(t+1) of the token this lane stores, decay^RS_BLOCK
    for (uint32_t t = 0; t < lane / 4; ++t) down *= decay;
    for (int t = 1; t < RS_BLOCK; ++t) block *= decay;
    float *state = a.state + (((uint64_t)a.slots[sp.row0] * a.n_head + h) * a.dim) * a.vdim + col0 + 2 * warp;
    const bool fresh = a.positions[sp.row0] == 0;
    float S[R][2];
    auto row_of = [&](int i) { return (uint32_t)(i / W) * (32 * W) + lane * W + i % W; };
    auto exists = [&](int i, int c) { return row_of(i) < a.dim && col0 + 2 * warp + c < a.vdim; };
#pragma unroll
    for (int i = 0; i < R; ++i)
#pragma unroll
        for (int c = 0; c < 2; ++c) S[i][c] = !fresh && exists(i, c) ? state[row_of(i) * a.vdim + c] : 0.0f;
    uint32_t stage = 0;
    for (uint32_t t0 = 0; t0 < sp.n; t0 += RS_BLOCK, stage = (stage + 1) % STAGES) {
        const uint32_t n = min((uint32_t)RS_BLOCK, sp.n - t0);
        cp_wait<STAGES - 2>();
        __syncthreads();  // this block's operands are there, and everyone has left the stage that is filled next
        if (t0 + (STAGES - 1) * RS_BLOCK < sp.n) load(t0 + (STAGES - 1) * RS_BLOCK, (stage + STAGES - 1) % STAGES);
        cp_commit();
        float x[RS_BLOCK * 2];
#pragma unroll
        for (int t = 0; t < RS_BLOCK; ++t) {  // tokens past the end are zero: they change nothing
            const float2 v = *reinterpret_cast<const float2 *>(&vs[stage][t][2 * warp]);
            const float v0 = v.x * up[t], v1 = v.y * up[t];
            float x0 = 0.0f, x1 = 0.0f;
#pragma unroll
            for (int g = 0; g < V4; ++g) {
                float kk[W], qq[W];
                const float *kp = &ks[stage][t][g * 32 * W + lane * W], *qp = &qs[stage][t][g * 32 * W + lane * W];
                if constexpr (W == 4) {
                    *reinterpret_cast<float4 *>(kk) = *reinterpret_cast<const float4 *>(kp);
                    *reinterpret_cast<float4 *>(qq) = *reinterpret_cast<const float4 *>(qp);
                } else {
                    *reinterpret_cast<float2 *>(kk) = *reinterpret_cast<const float2 *>(kp);
                    *reinterpret_cast<float2 *>(qq) = *reinterpret_cast<const float2 *>(qp);
                }
#pragma unroll
                for (int e = 0; e < W; ++e) {
                    float(&s)[2] = S[g * W + e];
                    s[0] = fmaf(kk[e], v0, s[0]), s[1] = fmaf(kk[e], v1, s[1]);
                    x0 = fmaf(qq[e], s[0], x0), x1 = fmaf(qq[e], s[1], x1);
                }
            }
            x[2 * t] = x0, x[2 * t + 1] = x1;
        }
        float back = block;
        if (n < RS_BLOCK) {
            back = 1.0f;
            for (uint32_t t = 0; t < n; ++t) back *= decay;
        }
#pragma unroll
        for (int i = 0; i < R; ++i) S[i][0] *= back, S[i][1] *= back;
#pragma unroll
        for (int o = 8; o > 0; o >>= 1)  // lanes 2 l and 2 l + 1 end with the halves of the sum of x[l] over the lanes
#pragma unroll
            for (int i = 0; i < o; ++i) {
                const bool hi = lane & (2 * o);
                const float give = hi ? x[i] : x[i + o], mine = hi ? x[i + o] : x[i];
                x[i] = mine + __shfl_xor_sync(0xffffffffu, give, 2 * o);
            }
        x[0] += __shfl_xor_sync(0xffffffffu, x[0], 1);
        const uint32_t t = lane / 4, col = col0 + 2 * warp + lane / 2 % 2;
        if ((lane & 1) == 0 && t < n && col < a.vdim) a.o[((uint64_t)(sp.row0 + t0 + t) * a.n_head + h) * a.vdim + col] = x[0] * down;
    }
    cp_wait<0>();
#pragma unroll
    for (int i = 0; i < R; ++i)
#pragma unroll
        for (int c = 0; c < 2; ++c)
            if (exists(i, c)) state[row_of(i) * a.vdim + c] = S[i][c];
}

// Every head's output over its root mean square, times silu of its gate.  A warp per (token, head).
constexpr int POST_VALUES = 8;  // per lane in registers; wider heads read the rest twice
template <typename TA>
__global__ void __launch_bounds__(256) retention_post_kernel(RetentionArgs a) {
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x, lane = threadIdx.x & 31, h = blockIdx.y * 8 + (threadIdx.x >> 5);
    if (h >= a.n_head) return;
    const float *g = a.y + (uint64_t)t * a.y_pitch + 2ull * a.n_head * a.dim + (uint64_t)(a.n_head + h) * a.vdim;
    const float *o = a.o + ((uint64_t)t * a.n_head + h) * a.vdim;
    TA *out = static_cast<TA *>(a.out) + (uint64_t)t * a.out_pitch + (uint64_t)h * a.vdim;
    float v[POST_VALUES], z[POST_VALUES], s = 0.0f;
#pragma unroll
    for (int u = 0; u < POST_VALUES; ++u) {
        const uint32_t i = lane + 32 * u;
        v[u] = i < a.vdim ? o[i] : 0.0f;
        z[u] = i < a.vdim ? g[i] : 0.0f;
        s += v[u] * v[u];
    }
    for (uint32_t i = lane + 32 * POST_VALUES; i < a.vdim; i += 32) s += o[i] * o[i];
    const float f = inv_rms(warp_sum(s), a.vdim, a.eps);
    auto gated = [&](float x, float zz) { return to_act<TA>(x * f * (zz / (1.0f + expf(-zz)))); };
#pragma unroll
    for (int u = 0; u < POST_VALUES; ++u)
        if (lane + 32 * u < a.vdim) out[lane + 32 * u] = gated(v[u], z[u]);
    for (uint32_t i = lane + 32 * POST_VALUES; i < a.vdim; i += 32) out[i] = gated(o[i], g[i]);
}

__global__ void __launch_bounds__(256) copy_pool_pages_kernel(uint4 *pool, uint64_t page_vecs, const int32_t *__restrict__ src, const int32_t *__restrict__ dst) {
    const uint4 *s = pool + (uint64_t)src[blockIdx.x] * page_vecs;
    uint4 *d = pool + (uint64_t)dst[blockIdx.x] * page_vecs;
    for (uint64_t i = threadIdx.x; i < page_vecs; i += blockDim.x) d[i] = s[i];
}

constexpr uint32_t MAX_SMEM = 227 * 1024;
using LmKernel = void (*)(LatentArgs);
const LmKernel LM_KERNELS[3][LM_PAIRS] = {{latent_attn_mma_kernel<1, 1>, latent_attn_mma_kernel<1, 2>, latent_attn_mma_kernel<1, 3>, latent_attn_mma_kernel<1, 4>},
                                          {latent_attn_mma_kernel<2, 1>, latent_attn_mma_kernel<2, 2>, latent_attn_mma_kernel<2, 3>, latent_attn_mma_kernel<2, 4>},
                                          {latent_attn_mma_kernel<4, 1>, latent_attn_mma_kernel<4, 2>, latent_attn_mma_kernel<4, 3>, latent_attn_mma_kernel<4, 4>}};
size_t plain_smem(const LatentArgs &a) { return (size_t)(a.dq + a.kv_p + LA_KEYS) * 4; }

}  // namespace

// ---- launchers ----------------------------------------------------------------------------------------------------------------------
cudaError_t mixers_configure() {
    static PerDeviceOnce once;
    return once.run([] {
        cudaError_t e = cudaSuccess;
        for (int mt = 0; mt < 3; ++mt)
            for (auto k : LM_KERNELS[mt])
                if (e == cudaSuccess) e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_SMEM - 64);
        for (auto k : {latent_prefill_kernel<2>, latent_prefill_kernel<4>, latent_prefill_kernel<6>, latent_prefill_kernel<8>, latent_prefill_kernel<12>, latent_prefill_kernel<16>})
            if (e == cudaSuccess) e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_SMEM - 64);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(retention_kernel<8>, cudaFuncAttributeMaxDynamicSharedMemorySize, RtPlan<8>::FLOATS * 4);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(retention_kernel<16>, cudaFuncAttributeMaxDynamicSharedMemorySize, RtPlan<16>::FLOATS * 4);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(retention_kernel<32>, cudaFuncAttributeMaxDynamicSharedMemorySize, RtPlan<32>::FLOATS * 4);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(latent_attn_plain_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        if (e == cudaSuccess) e = cudaFuncSetAttribute(latent_attn_plain_kernel<bf16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 128 * 1024);
        return e;
    });
}

template <typename TA>
static void embed(const bf16 *table, uint32_t width, const uint32_t *tokens, uint32_t T, float *x, bool normed, float eps, float gain, const float *w, void *h, uint32_t h_pitch,
                  cudaStream_t st) {
    const RowShape r(width, T);
    launch_pdl(r.vec ? embed_kernel<TA, ROW_VECS> : embed_kernel<TA, 0>, T, r.threads, 0, st, table, width, tokens, x, normed, eps, gain, w, static_cast<TA *>(h), h_pitch);
}
void launch_embed(const bf16 *table, uint32_t width, const uint32_t *tokens, uint32_t T, float *x, bool normed, float eps, float gain, const float *w, void *h,
                  uint32_t h_pitch, bool f32, cudaStream_t st) {
    if (f32) embed<float>(table, width, tokens, T, x, normed, eps, gain, w, h, h_pitch, st);
    else embed<bf16>(table, width, tokens, T, x, normed, eps, gain, w, h, h_pitch, st);
}
template <typename TA>
static void norm(const float *x, uint32_t width, const uint32_t *rows, uint32_t n, float eps, float gain, const float *w, void *h, uint32_t h_pitch, cudaStream_t st) {
    const RowShape r(width, n);
    launch_pdl(r.vec ? norm_kernel<TA, ROW_VECS> : norm_kernel<TA, 0>, n, r.threads, 0, st, x, width, rows, eps, gain, w, static_cast<TA *>(h), h_pitch);
}
void launch_norm(const float *x, uint32_t width, const uint32_t *rows, uint32_t n, float eps, float gain, const float *w, void *h, uint32_t h_pitch, bool f32, cudaStream_t st) {
    if (f32) norm<float>(x, width, rows, n, eps, gain, w, h, h_pitch, st);
    else norm<bf16>(x, width, rows, n, eps, gain, w, h, h_pitch, st);
}
void launch_post_norm(const PostNormArgs &a, bool f32, cudaStream_t st) {
    const RowShape r(a.width, a.T);
    if (f32) launch_pdl(r.vec ? post_norm_kernel<float, ROW_VECS> : post_norm_kernel<float, 0>, a.T, r.threads, 0, st, a);
    else launch_pdl(r.vec ? post_norm_kernel<bf16, ROW_VECS> : post_norm_kernel<bf16, 0>, a.T, r.threads, 0, st, a);
}
template <typename TA>
static void side_finish(float *x, const float *y, const float *w, uint32_t width, uint32_t T, float eps, float gain, void *h, uint32_t h_pitch, cudaStream_t st) {
    const RowShape r(width, T);
    if (r.vec) launch_pdl(side_finish_kernel<TA, ROW_VECS>, T, r.threads, 0, st, x, y, w, width, eps, gain, static_cast<TA *>(h), h_pitch);
    else launch_pdl(side_finish_kernel<TA, 0>, T, r.threads, 0, st, x, y, w, width, eps, gain, static_cast<TA *>(h), h_pitch);
}
void launch_side_finish(float *x, const float *y, const float *w, uint32_t width, uint32_t T, float eps, float gain, void *h, uint32_t h_pitch, bool f32, cudaStream_t st) {
    if (f32) side_finish<float>(x, y, w, width, T, eps, gain, h, h_pitch, st);
    else side_finish<bf16>(x, y, w, width, T, eps, gain, h, h_pitch, st);
}

void launch_latent_prep(const LatentArgs &a, bool f32, cudaStream_t st) {
    const dim3 grid((a.T + PREP_TOKENS - 1) / PREP_TOKENS, 1 + (a.n_head * a.rot_dim + PREP_Q - 1) / PREP_Q);
    const bool fours = a.y_pitch % 4 == 0 && a.kv_rank % 4 == 0 && a.rot_dim % 4 == 0 && a.rot.dims % (a.rot.interleaved ? 4 : 8) == 0;
    if (f32) launch_pdl(fours ? latent_prep_kernel<float, true> : latent_prep_kernel<float, false>, grid, 32 * PREP_TOKENS, 0, st, a);
    else launch_pdl(fours ? latent_prep_kernel<bf16, true> : latent_prep_kernel<bf16, false>, grid, 32 * PREP_TOKENS, 0, st, a);
}

uint32_t launch_latent_attention(const LatentArgs &a, bool f32, int sm_count, cudaStream_t st) {
    uint32_t longest = 1;
    if (!a.single)
        for (uint32_t s = 0; s < a.n_seq; ++s) longest = std::max(longest, a.h_spans[s].n);
    const uint64_t rows = (uint64_t)longest * a.n_head;
    const int mt = rows <= 16 ? 1 : rows <= 32 ? 2 : 4;
    const LmPlan plan(mt, a.dq);
    if (f32 || a.kv_p > 16 * 8 * LM_PAIRS || plan.bytes > MAX_SMEM - 64) {
        if (f32) launch_pdl(latent_attn_plain_kernel<float>, a.T * a.n_head, LA_THREADS, plain_smem(a), st, a);
        else launch_pdl(latent_attn_plain_kernel<bf16>, a.T * a.n_head, LA_THREADS, plain_smem(a), st, a);
        return 1;
    }
    const uint32_t M = 16 * mt, KT = LM_KEYS;
    uint32_t tiles = 0;
    if (a.single) tiles = a.n_seq * ((a.n_head + M - 1) / M);
    else
        for (uint32_t s = 0; s < a.n_seq; ++s) tiles += (a.h_spans[s].n * a.n_head + M - 1) / M;
    // few tiles: their keys are split over CTAs and put together afterwards
    const uint32_t span = M / a.n_head + 2, reach = a.window ? std::min<uint64_t>(a.max_pos, (uint64_t)a.window + span) : a.max_pos;
    const uint32_t slots = (uint32_t)sm_count * (mt == 4 || 2 * plan.bytes > 224 * 1024 ? 1 : 2);
    uint32_t splits = std::max(1u, std::min(std::min(slots, MERGE_MAX) / std::max(1u, tiles), (reach + KT - 1) / KT));
    while (splits > 1 && (uint64_t)splits * a.T * a.n_head * lm_part_row(a.kv_p) > a.part_cap) --splits;
    const dim3 grid(tiles, splits);
    launch_pdl(LM_KERNELS[mt == 4 ? 2 : mt - 1][(a.kv_p / 16 + 7) / 8 - 1], grid, LM_THREADS, plan.bytes, st, a);
    if (splits == 1) return 1;
    uint32_t merge_rows = a.single ? a.n_seq * a.n_head : 0;
    if (!a.single)
        for (uint32_t s = 0; s < a.n_seq; ++s) merge_rows += a.h_spans[s].n * a.n_head;
    const uint32_t groups = std::min(MERGE_GROUPS, (splits + MERGE_AT_ONCE - 1) / MERGE_AT_ONCE);
    launch_pdl(latent_merge_kernel, merge_rows, 128 * groups, (groups - 1) * 512 * sizeof(float), st, a, splits);
    return 2;
}

bool latent_prefill_supported(uint32_t dim_k, uint32_t rot_p, uint32_t vdim_k) {
    return vdim_k <= 256 && PfPlan(dim_k + rot_p, vdim_k).bytes <= MAX_SMEM - 64;
}
uint32_t latent_prefill_tiles(uint32_t n) { return (n + PF_TOKENS - 1) / PF_TOKENS; }
void launch_latent_gather(const LatentPrefillArgs &a, cudaStream_t st) { launch_pdl(latent_gather_kernel, (a.n_keys + 7) / 8, 256, 0, st, a); }
void launch_latent_prefill(const LatentPrefillArgs &a, cudaStream_t st) {
    const PfPlan pl(a.dim_k + a.dq - a.kv_p, a.vdim_k);
    const dim3 grid(a.n_tiles, a.n_head);
    const uint32_t nv = a.vdim_k / 16;
    auto run = [&](void (*k)(LatentPrefillArgs)) { launch_pdl(k, grid, PF_THREADS, pl.bytes, st, a); };
    if (nv <= 2) run(latent_prefill_kernel<2>);
    else if (nv <= 4) run(latent_prefill_kernel<4>);
    else if (nv <= 6) run(latent_prefill_kernel<6>);
    else if (nv <= 8) run(latent_prefill_kernel<8>);
    else if (nv <= 12) run(latent_prefill_kernel<12>);
    else run(latent_prefill_kernel<16>);
}

bool retention_supported(uint32_t dim) { return dim >= 1 && dim <= 256; }

uint32_t launch_retention(const RetentionArgs &a, bool f32, int sm_count, cudaStream_t st) {
    (void)sm_count;
    launch_pdl(retention_prep_kernel, a.T, 256, 0, st, a);
    // spans of a few tokens are bound by the state's traffic, long ones by the recurrence (and a block's decay must stay in range)
    const uint32_t n_long = a.decay_min >= 0.05f ? a.n_seq - a.first_long : 0, n_short = a.n_seq - n_long;
    const dim3 grid((a.vdim + 31) / 32, a.n_head, n_short), grid_long((a.vdim + RS_COLS - 1) / RS_COLS, a.n_head, n_long);
    if (n_short) {
        if (a.dim <= 64) launch_pdl(retention_kernel<8>, grid, 256, RtPlan<8>::FLOATS * 4, st, a);
        else if (a.dim <= 128) launch_pdl(retention_kernel<16>, grid, 256, RtPlan<16>::FLOATS * 4, st, a);
        else launch_pdl(retention_kernel<32>, grid, 256, RtPlan<32>::FLOATS * 4, st, a);
    }
    if (n_long) {
        if (a.dim <= 64) launch_pdl(retention_span_kernel<2>, grid_long, 256, 0, st, a);
        else if (a.dim <= 128) launch_pdl(retention_span_kernel<4>, grid_long, 256, 0, st, a);
        else launch_pdl(retention_span_kernel<8>, grid_long, 256, 0, st, a);
    }
    const dim3 post(a.T, (a.n_head + 7) / 8);
    if (f32) launch_pdl(retention_post_kernel<float>, post, 256, 0, st, a);
    else launch_pdl(retention_post_kernel<bf16>, post, 256, 0, st, a);
    return 2 + (n_short > 0) + (n_long > 0);
}

void launch_copy_pages(void *pool, uint64_t page_bytes, const int32_t *src, const int32_t *dst, uint32_t n_pages, cudaStream_t st) {
    if (n_pages) copy_pool_pages_kernel<<<n_pages, 256, 0, st>>>(static_cast<uint4 *>(pool), page_bytes / 16, src, dst);
}

}  // namespace ob
