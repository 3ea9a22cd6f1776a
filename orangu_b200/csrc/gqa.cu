// Softmax attention over paged keys and values, several query heads per key/value head, within a sliding window or without one.
//
// With two maps per head (differential attention) both maps have queries and keys of their own and share the values; the head's
// output is map 1 - map_weight * map 2, brought to unit root mean square and scaled.  An elementwise sigmoid gate may follow.
//
// With one map, the first positions may stay visible beyond the window, scores may be capped, a sink per head may enter the softmax's
// denominator, a gate may scale whole heads, and keys and values may be another layer's.
//
//   attention_prep_kernel    norms and rotates queries and keys, appends keys and values to the cache
//   attention_step_kernel    decoded tokens and short portions: every warp takes pages of its own, a cluster of CTAs shares the
//                            keys of one tile and adds up over distributed shared memory
//   attention_prompt_kernel  portions of prompts on tcgen05 (gqa_tc5.cu)
//   attention_span_kernel    portions of prompts whose values are wider than that takes: 64 or 128 (token, head) rows of one
//                            key/value head, keys in tiles of 64
//   attention_plain_kernel   any sizes, fp32 cache
//
// A page holds 16 positions of every key/value head next to one another.  A cache row is [keys of the maps | value | 8 entries of
// padding]: an odd number of 16-byte pieces, so that a page lands in shared memory with one straight copy and ldmatrix reads it
// without bank conflicts.
#include <algorithm>

#include "mixers_common.cuh"

namespace ob {

namespace {

constexpr float LOG2E = 1.4426950408889634f;
constexpr uint32_t MAX_SMEM = 225 * 1024;  // beside the static part

__device__ __forceinline__ uint64_t page_at(const AttentionArgs &a, int32_t page, uint32_t g) { return ((uint64_t)page * a.n_kv + g) * KV_PAGE * a.row; }

// ---- queries, keys, values of a token -------------------------------------------------------------------------------------------
// A warp per vector: queries [n_head][n_map], keys [n_kv][n_map], values [n_kv].
constexpr int PREP_WARPS = 8;
template <typename TA>
__global__ void __launch_bounds__(PREP_WARPS * 32) attention_prep_kernel(AttentionArgs a) {
    extern __shared__ float sm[];  // [PREP_WARPS][dim]
    pdl_release();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.x, i = blockIdx.y * PREP_WARPS + warp;
    const uint32_t n_q = a.n_head * a.n_map, n_k = a.own_kv ? a.n_kv * a.n_map : 0, n_v = a.own_kv ? a.n_kv : 0;
    if (i >= n_q + n_k + n_v) return;
    const uint32_t pos = a.positions[t];
    const float *y = a.y + (uint64_t)t * a.y_pitch;
    TA *cache = static_cast<TA *>(a.cache) + page_at(a, a.tables[t][pos / KV_PAGE], 0) + (uint64_t)(pos % KV_PAGE) * a.row;
    const uint64_t head = (uint64_t)KV_PAGE * a.row;  // from one key/value head to the next within a page
    if (i >= n_q + n_k) {
        const uint32_t g = i - n_q - n_k;
        TA *dst = cache + g * head + a.n_map * a.dim_p;
        if (a.has_v) {
            const TA *src = static_cast<const TA *>(a.va) + (uint64_t)t * a.va_pitch + (uint64_t)g * a.vdim;
            for (uint32_t d = lane; d < a.vdim; d += 32) dst[d] = src[d];
        } else {
            const float *src = y + (uint64_t)(n_q + g) * a.dim;
            for (uint32_t d = lane; d < a.vdim; d += 32) dst[d] = to_act<TA>(src[d]);
        }
        return;
    }
    const bool query = i < n_q;
    const uint32_t k = i - n_q;
    const float *src = y + (uint64_t)i * a.dim, *w = query ? a.q_norm : a.k_norm;
    TA *dst = query ? static_cast<TA *>(a.q) + ((uint64_t)t * n_q + i) * a.dim_p : cache + k / a.n_map * head + k % a.n_map * a.dim_p;
    float *v = sm + warp * a.dim, s = 0.0f;
    for (uint32_t d = lane; d < a.dim; d += 32) {
        const float e = src[d];
        v[d] = e;
        s += e * e;
    }
    if (w) {
        uint32_t n = a.dim;
        if (a.norm_whole) {  // every warp adds up the whole projection
            n *= query ? n_q : n_k;
            const float *all = query ? y : y + (uint64_t)n_q * a.dim;
            s = 0.0f;
            for (uint32_t d = lane; d < n; d += 32) s += all[d] * all[d];
            w += (uint64_t)(query ? i : k) * a.dim;
        }
        const float f = inv_rms(warp_sum(s), n, a.eps);
        for (uint32_t d = lane; d < a.dim; d += 32) v[d] *= f * w[d];
    }
    __syncwarp();
    const float2 *cs = a.rot.table + (uint64_t)pos * (a.rot.dims / 2);
    for (uint32_t d = lane; d < a.dim_p; d += 32) dst[d] = to_act<TA>(d < a.dim ? rotated(v, d, a.rot, cs) : 0.0f);
}

// The same for sizes in eights (head sizes, half of the rotated entries): `group` neighbouring lanes per vector, eight entries each.
// With norms over whole projections a CTA has all vectors of its token (gridDim.y 1) and goes over them twice.
constexpr int PREP_THREADS = 256;
__device__ __forceinline__ void load_eight(const float *p, float (&v)[8]) {
    const float4 a = reinterpret_cast<const float4 *>(p)[0], b = reinterpret_cast<const float4 *>(p)[1];
    v[0] = a.x, v[1] = a.y, v[2] = a.z, v[3] = a.w, v[4] = b.x, v[5] = b.y, v[6] = b.z, v[7] = b.w;
}
template <typename TA> __device__ __forceinline__ void store_eight(TA *p, const float (&v)[8]) {
    store4<TA>(p, make_float4(v[0], v[1], v[2], v[3]));
    store4<TA>(p + 4, make_float4(v[4], v[5], v[6], v[7]));
}
template <typename TA>
__global__ void __launch_bounds__(PREP_THREADS) attention_prep_vec_kernel(AttentionArgs a, uint32_t group) {
    pdl_release();
    pdl_wait();
    __shared__ float red[33];
    const uint32_t t = blockIdx.x, c = threadIdx.x & (group - 1);
    const uint32_t n_q = a.n_head * a.n_map, n_k = a.own_kv ? a.n_kv * a.n_map : 0, n = n_q + n_k + (a.own_kv ? a.n_kv : 0), d = 8 * c;
    const uint32_t pos = a.positions[t];
    const float *y = a.y + (uint64_t)t * a.y_pitch;
    TA *cache = static_cast<TA *>(a.cache) + page_at(a, a.tables[t][pos / KV_PAGE], 0) + (uint64_t)(pos % KV_PAGE) * a.row;
    const uint64_t head = (uint64_t)KV_PAGE * a.row;  // from one key/value head to the next within a page
    float f_q = 1.0f, f_k = 1.0f;
    if (a.norm_whole) {
        float s[2] = {0.0f, 0.0f};
#pragma unroll 4
        for (uint32_t e = 4 * threadIdx.x; e < (n_q + n_k) * a.dim; e += 4 * PREP_THREADS) s[e >= n_q * a.dim] += sq4(*reinterpret_cast<const float4 *>(y + e));
        f_q = inv_rms(block_sum(s[0], red), n_q * a.dim, a.eps);
        if (n_k) f_k = inv_rms(block_sum(s[1], red), n_k * a.dim, a.eps);
    }
    for (uint32_t i0 = blockIdx.y * (PREP_THREADS / group); i0 < n; i0 += gridDim.y * (PREP_THREADS / group)) {
        const uint32_t i = i0 + threadIdx.x / group;
        const bool exists = i < n, value = i >= n_q + n_k, query = i < n_q;
        if (exists && value) {
            const uint32_t g = i - n_q - n_k;
            TA *dst = cache + g * head + a.n_map * a.dim_p;
            for (uint32_t e = d; e < a.vdim; e += 8 * group) {
                float v[8];
                if (a.has_v) {
                    constexpr uint32_t P = 16 / sizeof(TA);
                    const TA *src = static_cast<const TA *>(a.va) + (uint64_t)t * a.va_pitch + (uint64_t)g * a.vdim + e;
#pragma unroll
                    for (uint32_t k = 0; k < 8; k += P) *reinterpret_cast<uint4 *>(dst + e + k) = *reinterpret_cast<const uint4 *>(src + k);
                } else {
                    load_eight(y + (uint64_t)(n_q + g) * a.dim + e, v);
                    store_eight<TA>(dst + e, v);
                }
            }
        }
        const bool mine = exists && !value && d < a.dim;
        float v[8] = {}, s = 0.0f;
        if (mine) load_eight(y + (uint64_t)i * a.dim + d, v);
        if (a.q_norm) {
            float f = query ? f_q : f_k;
            if (!a.norm_whole) {
#pragma unroll
                for (int e = 0; e < 8; ++e) s += v[e] * v[e];
                for (uint32_t o = group / 2; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
                f = inv_rms(s, a.dim, a.eps);
            }
            if (mine) {
                float w[8];
                const float *all = query ? a.q_norm : a.k_norm;
                load_eight(all + (a.norm_whole ? (uint64_t)(query ? i : i - n_q) * a.dim : 0) + d, w);
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] *= f * w[e];
            }
        }
        const uint32_t half = a.rot.dims / 2;
        const bool low = d < half, turns = d < a.rot.dims;
        if (a.rot.interleaved) {
            if (mine && turns) {
                const float2 *cs = a.rot.table + (uint64_t)pos * half + d / 2;
#pragma unroll
                for (int e = 0; e < 8; e += 2) {
                    const float2 r = cs[e / 2];
                    const float u = v[e], w = v[e + 1];
                    v[e] = u * r.x - w * r.y, v[e + 1] = w * r.x + u * r.y;
                }
            }
        } else {
            float other[8];  // the entries half of the rotated ones away
            const uint32_t lane = threadIdx.x & 31, from = turns ? (low ? lane + half / 8 : lane - half / 8) : lane;
#pragma unroll
            for (int e = 0; e < 8; ++e) other[e] = __shfl_sync(0xffffffffu, v[e], from);
            if (mine && turns) {
                const float2 *cs = a.rot.table + (uint64_t)pos * half + (low ? d : d - half);
#pragma unroll
                for (int e = 0; e < 8; ++e) {
                    const float2 r = cs[e];
                    v[e] = low ? v[e] * r.x - other[e] * r.y : v[e] * r.x + other[e] * r.y;
                }
            }
        }
        if (exists && !value && d < a.dim_p) {  // (zeros from dim on)
            const uint32_t k = i - n_q;
            store_eight<TA>((query ? static_cast<TA *>(a.q) + ((uint64_t)t * n_q + i) * a.dim_p : cache + k / a.n_map * head + k % a.n_map * a.dim_p) + d, v);
        }
    }
}

// ---- the end of a head: both maps put together, gates, store ----------------------------------------------------------------------
__device__ __forceinline__ float gate_of(const AttentionArgs &a, uint64_t t, uint32_t h, uint32_t c, bool f32) {
    const uint64_t at = t * a.va_pitch + a.gate0 + (uint64_t)h * a.vdim + c;
    const float z = f32 ? static_cast<const float *>(a.va)[at] : from_act(static_cast<const bf16 *>(a.va)[at]);
    return 1.0f / (1.0f + expf(-z));
}

// Factor of a whole head of token t (one map).
__device__ __forceinline__ float head_factor(const AttentionArgs &a, uint64_t t, uint32_t h) {
    return a.head_gain * (a.head_gate ? 1.0f / (1.0f + expf(-a.head_gate[t * a.y_pitch + h])) : 1.0f);
}

// ---- plain form: one CTA per (token, head) --------------------------------------------------------------------------------------
// Keys in blocks of 128: scores by the warps (lanes over the row), online softmax, then every thread adds up its own columns.
constexpr int AP_KEYS = 128, AP_THREADS = 128;
template <typename TA>
__global__ void __launch_bounds__(AP_THREADS) attention_plain_kernel(AttentionArgs a) {
    extern __shared__ float sm[];
    float *q = sm, *acc = q + a.dim, *p = acc + a.n_map * a.vdim;  // [dim], [n_map][vdim], [AP_KEYS]
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x / a.n_head, h = blockIdx.x % a.n_head, g = h / (a.n_head / a.n_kv), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const uint32_t pos = a.positions[t], lo = first_seen(pos, a.window), kept = min(a.keep, lo), hi = kept + pos + 1 - lo;
    const int32_t *table = a.tables[t];
    auto row_of = [&](uint32_t i) {  // of the i'th visible position
        const uint32_t j = i < kept ? i : lo + i - kept;
        return static_cast<const TA *>(a.cache) + page_at(a, table[j / KV_PAGE], g) + (uint64_t)(j % KV_PAGE) * a.row;
    };
    for (uint32_t map = 0; map < a.n_map; ++map) {
        const TA *qg = static_cast<const TA *>(a.q) + (((uint64_t)t * a.n_head + h) * a.n_map + map) * a.dim_p;
        float *o = acc + map * a.vdim;
        __syncthreads();
        for (uint32_t i = threadIdx.x; i < a.dim; i += blockDim.x) q[i] = from_act(qg[i]);
        for (uint32_t i = threadIdx.x; i < a.vdim; i += blockDim.x) o[i] = 0.0f;
        float m = -INFINITY, l = 0.0f;
        __syncthreads();
        for (uint32_t j0 = 0; j0 < hi; j0 += AP_KEYS) {
            const uint32_t n = min((uint32_t)AP_KEYS, hi - j0);
            for (uint32_t j = warp; j < n; j += AP_THREADS / 32) {
                const TA *k = row_of(j0 + j) + map * a.dim_p;
                float s = 0.0f;
                for (uint32_t i = lane; i < a.dim; i += 32) s = fmaf(q[i], from_act(k[i]), s);
                s = warp_sum(s);
                s *= a.scale;
                if (lane == 0) p[j] = a.softcap > 0.0f ? a.softcap * tanhf(s / a.softcap) : s;
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
            for (uint32_t i = threadIdx.x; i < a.vdim; i += blockDim.x) {
                float v = o[i] * keep;
                for (uint32_t j = 0; j < n; ++j) v = fmaf(p[j], from_act(row_of(j0 + j)[a.n_map * a.dim_p + i]), v);
                o[i] = v;
            }
            __syncthreads();
        }
        if (a.sink) {
            const float top = fmaxf(m, a.sink[h]), keep = expf(m - top);
            l = l * keep + expf(a.sink[h] - top);
            for (uint32_t i = threadIdx.x; i < a.vdim; i += blockDim.x) o[i] *= keep;
        }
        for (uint32_t i = threadIdx.x; i < a.vdim; i += blockDim.x) o[i] /= l;
    }
    float f = a.n_map == 1 ? head_factor(a, t, h) : 1.0f;
    if (a.n_map == 2) {
        float s = 0.0f;
        for (uint32_t i = threadIdx.x; i < a.vdim; i += blockDim.x) {
            acc[i] -= a.map_weight * acc[a.vdim + i];
            s += acc[i] * acc[i];
        }
        f = inv_rms(block_sum(s, red), a.vdim, a.eps) * a.head_gain;
    }
    TA *out = static_cast<TA *>(a.out) + (uint64_t)t * a.out_pitch + (uint64_t)h * a.vdim;
    for (uint32_t i = threadIdx.x; i < a.vdim; i += blockDim.x) {
        float v = acc[i] * f;
        if (a.has_gate) v *= gate_of(a, t, h, i, sizeof(TA) == 4);
        out[i] = to_act<TA>(v);
    }
}

// ---- decoded tokens and short portions (bf16 cache) --------------------------------------------------------------------------------
// A tile is 16 consecutive (token, head) rows of one key/value head.  The tile's pages are dealt out over the warps of a cluster;
// a warp copies its pages to a ring of its own, keeps maximum, sum and output of its keys, and never waits for another one until
// all meet at the end.  Weights enter the second product as value plus remainder, two bf16 operands.
constexpr int ST_WARPS = 4, ST_THREADS = ST_WARPS * 32, ST_ROWS = 16, ST_MAX_CLUSTER = 8;
struct StPlan {
    uint32_t stages, ring, q_row, o_row, bytes;  // ring: bytes of one warp's region; q_row bytes; o_row floats
    __host__ __device__ StPlan(uint32_t n_map, uint32_t dim_p, uint32_t vdim_p, uint32_t row, uint32_t n) : stages(n) {
        const uint32_t page = KV_PAGE * row * 2, maps = n_map == 2 && vdim_p > 128 ? 1 : n_map;
        q_row = (n_map * dim_p + 8) * 2;
        o_row = vdim_p + 8;
        const uint32_t o = maps * ST_ROWS * o_row * 4;
        ring = stages * page > o ? stages * page : o;
        bytes = ST_ROWS * q_row + ST_WARPS * ring + 256 * 2 + 128;  // a page's last row is read up to 256 columns past its values
    }
    static uint32_t best_stages(uint32_t n_map, uint32_t dim_p, uint32_t vdim_p, uint32_t row) {
        // two CTAs per SM, else one (three with fewer stages, or more splits of a tile, are slower: a CTA's start and end cost)
        for (uint32_t s = 4; s >= 2; --s) {
            const uint32_t b = StPlan(n_map, dim_p, vdim_p, row, s).bytes;
            if (2 * (b + 2048) <= 227 * 1024 || (s == 2 && b <= MAX_SMEM)) return s;
        }
        return 0;
    }
};

__device__ __forceinline__ uint32_t cluster_rank() {
    uint32_t r;
    asm volatile("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}
__device__ __forceinline__ void cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n\tbarrier.cluster.wait.acquire.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t peer_addr(uint32_t addr, uint32_t rank) {  // the same shared-memory address in another CTA of the cluster
    uint32_t r;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(r) : "r"(addr), "r"(rank));
    return r;
}
__device__ __forceinline__ float4 peer_load4(uint32_t addr) {
    float4 v;
    asm volatile("ld.shared::cluster.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(v.x), "=f"(v.y), "=f"(v.z), "=f"(v.w) : "r"(addr) : "memory");
    return v;
}
__device__ __forceinline__ float2 peer_load2(uint32_t addr) {
    float2 v;
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(addr) : "memory");
    return v;
}

// NV: columns of a value in sixteens (what goes past vdim_p is computed from whatever follows in shared memory and dropped).
template <int NM, int NV, bool CAP>
__global__ void __launch_bounds__(ST_THREADS) attention_step_kernel(AttentionArgs a, uint32_t splits, uint32_t stages) {
    constexpr bool APART = NM == 2 && NV > 8;  // the maps of wide values are different warps' business: two accumulators would not fit
    constexpr int LM = APART ? 1 : NM;         // maps per warp
    constexpr uint32_t UNITS = APART ? ST_WARPS / 2 : ST_WARPS;  // warps that share the pages of one map
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ float2 stat[ST_WARPS][LM][ST_ROWS];  // maximum and sum
    __shared__ uint32_t tile_info[3];
    const StPlan pl(NM, a.dim_p, a.vdim_p, a.row, stages);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = blockIdx.y, rank = cluster_rank(), per = a.n_head / a.n_kv;
    pdl_release();
    pdl_wait();
    if (warp == 0) {
        const uint32_t tile = blockIdx.x / splits, each = (per + ST_ROWS - 1) / ST_ROWS;
        RowSpan sp{tile, 1};
        uint32_t f = 0;
        if (a.single) sp.row0 = tile / each, f = tile % each * ST_ROWS;
        else find_tile(a.spans, a.n_short, per, ST_ROWS, tile, &sp, &f);
        if (lane == 0) tile_info[0] = sp.row0, tile_info[1] = sp.n, tile_info[2] = f;
    }
    __syncthreads();
    const uint32_t row0 = tile_info[0], f0 = tile_info[2], n_flat = tile_info[1] * per;
    if (f0 >= n_flat) return;  // (the same for the whole cluster)
    const uint32_t n_here = min((uint32_t)ST_ROWS, n_flat - f0), pos0 = a.positions[row0];
    const int32_t *table = a.tables[row0];
    const PageList pages = page_list(pos0 + f0 / per, pos0 + (f0 + n_here - 1) / per, a.window, a.keep, 1);
    const uint32_t n_page = pages.n;
    const uint32_t unit = rank * UNITS + (APART ? warp >> 1 : warp), n_unit = splits * UNITS, map0 = APART ? warp & 1u : 0u;
    const uint32_t pieces = KV_PAGE * a.row / 8, qs = smem_addr(smem), ring = qs + ST_ROWS * pl.q_row + warp * pl.ring, page_bytes = KV_PAGE * a.row * 2;

    {   // queries
        const uint32_t per_map = a.dim_p / 8, per_row = NM * per_map;
        for (uint32_t i = threadIdx.x; i < ST_ROWS * per_row; i += ST_THREADS) {
            const uint32_t r = i / per_row, c = i - r * per_row, f = f0 + (r < n_here ? r : 0);
            const bf16 *src = static_cast<const bf16 *>(a.q) + ((uint64_t)(row0 + f / per) * a.n_head + g * per + f % per) * (NM * a.dim_p) + 8 * c;
            cp16(qs + r * pl.q_row + c * 16, src, r < n_here);
        }
    }
    const uint32_t ring_end = ring + stages * page_bytes;
    uint32_t next_page = unit, next_stage = ring;  // of the next load
    auto load = [&] {  // this warp's next page
        if (next_page < n_page) {
            const bf16 *src = static_cast<const bf16 *>(a.cache) + page_at(a, table[pages[next_page]], g) + 8 * lane;
            uint32_t dst = next_stage + 16 * lane, i = lane;
            for (; i + 96 < pieces; i += 128, src += 1024, dst += 2048)
#pragma unroll
                for (int k = 0; k < 4; ++k) cp16(dst + 512 * k, src + 256 * k, true);
            for (; i < pieces; i += 32, src += 256, dst += 512) cp16(dst, src, true);
        }
        cp_commit();
        next_page += n_unit;
        next_stage = next_stage + page_bytes == ring_end ? ring : next_stage + page_bytes;
    };
    // (the first group also holds the queries; with fewer than four stages empty groups keep the count)
    load();
    if (stages > 2) load();
    if (stages > 3) load();
    if (stages == 4) cp_wait<2>();
    else if (stages == 3) cp_wait<1>();
    else cp_wait<0>();
    __syncthreads();

    const float scale2 = a.scale * LOG2E, cap = a.softcap * LOG2E, cap_in = CAP ? 2.0f * scale2 / a.softcap : 0.0f;
    const int win = a.window ? (int)a.window : 0x7fffffff, keep = (int)a.keep;
    const int r0 = (int)(lane / 4), p0 = r0 < (int)n_here ? (int)(pos0 + (f0 + r0) / per) : -1, p1 = r0 + 8 < (int)n_here ? (int)(pos0 + (f0 + r0 + 8) / per) : -1;
    float o[LM][NV][2][4], m0[LM], m1[LM], l0[LM], l1[LM];
#pragma unroll
    for (int m = 0; m < LM; ++m) {
        m0[m] = m1[m] = -INFINITY, l0[m] = l1[m] = 0.0f;
#pragma unroll
        for (int v = 0; v < NV; ++v)
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[m][v][n][e] = 0.0f;
    }
    const uint32_t row_bytes = a.row * 2, k_steps = a.dim_p / 16;
    const uint32_t qa = qs + (lane & 15) * pl.q_row + (lane >> 4) * 16;
    const uint32_t b_off = ((lane & 7) + ((lane >> 4) << 3)) * row_bytes + ((lane >> 3) & 1) * 16;
    const uint32_t v_off = ((lane & 7) + (((lane >> 3) & 1) << 3)) * row_bytes + (lane >> 4) * 16 + NM * a.dim_p * 2;
    uint32_t kb = ring;
    for (uint32_t page = unit; page < n_page; page += n_unit, kb = kb + page_bytes == ring_end ? ring : kb + page_bytes) {
        load();
        if (stages == 4) cp_wait<3>();
        else if (stages == 3) cp_wait<2>();
        else cp_wait<1>();
        __syncwarp();
        const int j0 = (int)(pages[page] * KV_PAGE);
        uint32_t ph[LM][4], pr[LM][4];
#pragma unroll
        for (int m = 0; m < LM; ++m) {
            float c[2][4] = {}, d[2][4] = {};
            const uint32_t at = (map0 + m) * a.dim_p * 2, qm = qa + at, km = kb + b_off + at;
            auto step = [&](uint32_t k, float (&x)[2][4]) {
                uint32_t fa[4], fb[4];
                ldsm4(fa, qm + k * 32);
                ldsm4(fb, km + k * 32);
                mma_bf16(x[0], fa, fb[0], fb[1]);
                mma_bf16(x[1], fa, fb[2], fb[3]);
            };
            uint32_t k = 0;
#pragma unroll 2
            for (; k + 1 < k_steps; k += 2) {
                step(k, c);
                step(k + 1, d);
            }
            if (k < k_steps) step(k, c);
            float b0 = -INFINITY, b1 = -INFINITY;
#pragma unroll
            for (int h = 0; h < 2; ++h)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int j = j0 + 8 * h + 2 * (int)(lane & 3) + e;
                    float s0 = c[h][e] + d[h][e], s1 = c[h][2 + e] + d[h][2 + e];
                    if constexpr (CAP) s0 = soft_cap(s0, cap_in, cap), s1 = soft_cap(s1, cap_in, cap);
                    else s0 *= scale2, s1 *= scale2;
                    c[h][e] = j <= p0 && (p0 - j < win || j < keep) ? s0 : -INFINITY;
                    c[h][2 + e] = j <= p1 && (p1 - j < win || j < keep) ? s1 : -INFINITY;
                    b0 = fmaxf(b0, c[h][e]);
                    b1 = fmaxf(b1, c[h][2 + e]);
                }
            b0 = fmaxf(b0, __shfl_xor_sync(0xffffffffu, b0, 1)), b0 = fmaxf(b0, __shfl_xor_sync(0xffffffffu, b0, 2));
            b1 = fmaxf(b1, __shfl_xor_sync(0xffffffffu, b1, 1)), b1 = fmaxf(b1, __shfl_xor_sync(0xffffffffu, b1, 2));
            // (rescaling only when the maximum has grown much puts a branch between the maps' products: slower)
            const float n0 = fmaxf(m0[m], b0), n1 = fmaxf(m1[m], b1);
            const float s0 = n0 == -INFINITY ? 0.0f : n0, s1 = n1 == -INFINITY ? 0.0f : n1;  // a row that has seen nothing yet keeps weights of zero
            const float g0 = pow2(m0[m] - s0), g1 = pow2(m1[m] - s1);
            m0[m] = n0, m1[m] = n1;
            l0[m] *= g0, l1[m] *= g1;
#pragma unroll
            for (int v = 0; v < NV; ++v)
#pragma unroll
                for (int h = 0; h < 2; ++h) o[m][v][h][0] *= g0, o[m][v][h][1] *= g0, o[m][v][h][2] *= g1, o[m][v][h][3] *= g1;
#pragma unroll
            for (int h = 0; h < 2; ++h)
#pragma unroll
                for (int r = 0; r < 2; ++r) {  // fragment register 2 h + r: row half r of key half h
                    const float e0 = pow2(c[h][2 * r] - (r ? s1 : s0)), e1 = pow2(c[h][2 * r + 1] - (r ? s1 : s0));
                    if (r) l1[m] += e0 + e1;
                    else l0[m] += e0 + e1;
                    const __nv_bfloat162 hi2 = __floats2bfloat162_rn(e0, e1);
                    const __nv_bfloat162 lo2 = __floats2bfloat162_rn(e0 - __low2float(hi2), e1 - __high2float(hi2));
                    ph[m][2 * h + r] = *reinterpret_cast<const uint32_t *>(&hi2);
                    pr[m][2 * h + r] = *reinterpret_cast<const uint32_t *>(&lo2);
                }
        }
#pragma unroll
        for (int v = 0; v < NV; ++v) {
            uint32_t fv[4];
            ldsm4t(fv, kb + v_off + v * 32);
#pragma unroll
            for (int m = 0; m < LM; ++m) {
                mma_bf16(o[m][v][0], ph[m], fv[0], fv[1]);
                mma_bf16(o[m][v][1], ph[m], fv[2], fv[3]);
                mma_bf16(o[m][v][0], pr[m], fv[0], fv[1]);
                mma_bf16(o[m][v][1], pr[m], fv[2], fv[3]);
            }
        }
        __syncwarp();  // everyone has read the page before its stage is filled again
    }
    cp_wait<0>();
    __syncwarp();
    // every warp leaves its part in its ring
    float *mine = reinterpret_cast<float *>(smem + ST_ROWS * pl.q_row + warp * pl.ring);
#pragma unroll
    for (int m = 0; m < LM; ++m) {
        l0[m] += __shfl_xor_sync(0xffffffffu, l0[m], 1), l0[m] += __shfl_xor_sync(0xffffffffu, l0[m], 2);
        l1[m] += __shfl_xor_sync(0xffffffffu, l1[m], 1), l1[m] += __shfl_xor_sync(0xffffffffu, l1[m], 2);
        if ((lane & 3) == 0) stat[warp][m][r0] = make_float2(m0[m], l0[m]), stat[warp][m][r0 + 8] = make_float2(m1[m], l1[m]);
#pragma unroll
        for (int v = 0; v < NV; ++v)
#pragma unroll
            for (int h = 0; h < 2; ++h) {
                const uint32_t col = v * 16 + h * 8 + 2 * (lane & 3);
                if (v * 16 >= (int)a.vdim_p) continue;
                *reinterpret_cast<float2 *>(mine + (m * ST_ROWS + r0) * pl.o_row + col) = make_float2(o[m][v][h][0], o[m][v][h][1]);
                *reinterpret_cast<float2 *>(mine + (m * ST_ROWS + r0 + 8) * pl.o_row + col) = make_float2(o[m][v][h][2], o[m][v][h][3]);
            }
    }
    cluster_sync();
    // a warp per row: the parts of all warps of the cluster added up
    constexpr int NC = (NV + 7) / 8;  // columns of a lane in fours
    for (uint32_t r = rank + splits * warp; r < n_here; r += splits * ST_WARPS) {
        float4 sum[NM][NC];
#pragma unroll
        for (int m = 0; m < NM; ++m) {
            // lane = part: its CTA and warp
            const uint32_t part_rank = lane / UNITS, part_warp = APART ? 2 * (lane % UNITS) + m : lane % UNITS;
            const bool part = lane < n_unit;
            float2 ml = make_float2(-INFINITY, 0.0f);
            if (part) ml = peer_load2(peer_addr(smem_addr(&stat[part_warp][APART ? 0 : m][r]), part_rank));
            const float top = warp_max(ml.x), w = part && ml.x > -INFINITY ? pow2(ml.x - top) : 0.0f;
            float sum_w = warp_sum(w * ml.y);
            if (a.sink) sum_w += pow2(a.sink[g * per + (f0 + r) % per] * LOG2E - top);
            const float inv = 1.0f / sum_w;
            const uint32_t base = peer_addr(qs + ST_ROWS * pl.q_row + part_warp * pl.ring + (uint32_t)((APART ? 0 : m) * ST_ROWS + r) * pl.o_row * 4, part ? part_rank : 0);
#pragma unroll
            for (int i = 0; i < NC; ++i) sum[m][i] = make_float4(0, 0, 0, 0);
#pragma unroll 4
            for (uint32_t p = 0; p < n_unit; ++p) {
                const float f = __shfl_sync(0xffffffffu, w, p) * inv;
                const uint32_t from = __shfl_sync(0xffffffffu, base, p);
#pragma unroll
                for (int i = 0; i < NC; ++i) {
                    const uint32_t c = 4 * lane + 128 * i;
                    if (f == 0.0f || c >= a.vdim_p) continue;
                    const float4 u = peer_load4(from + c * 4);
                    sum[m][i].x = fmaf(f, u.x, sum[m][i].x), sum[m][i].y = fmaf(f, u.y, sum[m][i].y);
                    sum[m][i].z = fmaf(f, u.z, sum[m][i].z), sum[m][i].w = fmaf(f, u.w, sum[m][i].w);
                }
            }
        }
        const uint64_t t = row0 + (f0 + r) / per;
        const uint32_t h = g * per + (f0 + r) % per;
        float f = NM == 1 ? head_factor(a, t, h) : 1.0f;
        if constexpr (NM == 2) {
            float s = 0.0f;
#pragma unroll
            for (int i = 0; i < NC; ++i) {
                float4 &x = sum[0][i];
                const float4 z = sum[1][i];
                x.x -= a.map_weight * z.x, x.y -= a.map_weight * z.y, x.z -= a.map_weight * z.z, x.w -= a.map_weight * z.w;
                s += sq4(x);  // columns past vdim are zero: so are the values there
            }
            f = inv_rms(warp_sum(s), a.vdim, a.eps) * a.head_gain;
        }
        bf16 *out = static_cast<bf16 *>(a.out) + t * a.out_pitch + (uint64_t)h * a.vdim;
#pragma unroll
        for (int i = 0; i < NC; ++i) {
            const float x[4] = {sum[0][i].x, sum[0][i].y, sum[0][i].z, sum[0][i].w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const uint32_t c = 4 * lane + 128 * i + e;
                if (c < a.vdim) out[c] = to_act<bf16>(x[e] * f * (a.has_gate ? gate_of(a, t, h, c, false) : 1.0f));
            }
        }
    }
    cluster_sync();  // nobody leaves while another CTA still reads its shared memory
}

// ---- portions of prompts (bf16 cache) ------------------------------------------------------------------------------------------------
// 256 threads: with one map eight warps of 16 rows each, with two maps four warps per map over the same rows.  Keys come in tiles
// of 64, two stages.  Scores, softmax and the weights' two bf16 parts (value and remainder) stay in registers.
constexpr int SP_THREADS = 256, SP_KEYS = 64, SP_PAGES = SP_KEYS / KV_PAGE;
struct SpPlan {
    uint32_t rows, q_row, stage, k, bytes;
    __host__ __device__ SpPlan(uint32_t n_map, uint32_t dim_p, uint32_t vdim_p, uint32_t row) {
        rows = n_map == 2 ? 64 : 128;
        q_row = (n_map * dim_p + 8) * 2;
        stage = SP_KEYS * row * 2;
        k = rows * q_row;
        bytes = k + 2 * stage + 256 * 2 + 128;  // a row's values are read up to 256 columns past their end
    }
};

template <int NM, int NV, bool CAP>
__global__ void __launch_bounds__(SP_THREADS, NV <= 8 ? 2 : 1) attention_span_kernel(AttentionArgs a) {
    constexpr int RW = SP_THREADS / 32 / NM, M = 16 * RW;  // warps over the rows
    extern __shared__ __align__(16) uint8_t smem[];
    __shared__ uint32_t tile_info[3];
    const SpPlan pl(NM, a.dim_p, a.vdim_p, a.row);
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = blockIdx.y, per = a.n_head / a.n_kv, rw = warp % RW, map = warp / RW;
    pdl_release();
    pdl_wait();
    if (warp == 0) {
        RowSpan sp;
        uint32_t f;
        // (the last rows of a span see the most keys: they start first)
        find_tile(a.spans + a.n_short, a.n_seq - a.n_short, per, M, gridDim.x - 1 - blockIdx.x, &sp, &f);
        if (lane == 0) tile_info[0] = sp.row0, tile_info[1] = sp.n, tile_info[2] = f;
    }
    __syncthreads();
    const uint32_t row0 = tile_info[0], f0 = tile_info[2], n_flat = tile_info[1] * per;
    if (f0 >= n_flat) return;
    const uint32_t n_here = min((uint32_t)M, n_flat - f0), pos0 = a.positions[row0];
    const int32_t *table = a.tables[row0];
    const PageList pages = page_list(pos0 + f0 / per, pos0 + (f0 + n_here - 1) / per, a.window, a.keep, SP_PAGES);
    const uint32_t n_page = pages.n, n_tiles = (n_page + SP_PAGES - 1) / SP_PAGES;
    const uint32_t qs = smem_addr(smem), pieces = KV_PAGE * a.row / 8;
    {   // queries
        const uint32_t per_row = NM * a.dim_p / 8;
        for (uint32_t i = threadIdx.x; i < M * per_row; i += SP_THREADS) {
            const uint32_t r = i / per_row, c = i - r * per_row, f = f0 + (r < n_here ? r : 0);
            const bf16 *src = static_cast<const bf16 *>(a.q) + ((uint64_t)(row0 + f / per) * a.n_head + g * per + f % per) * (NM * a.dim_p) + 8 * c;
            cp16(qs + r * pl.q_row + c * 16, src, r < n_here);
        }
    }
    auto load = [&](uint32_t it) {
        const uint32_t dst = qs + pl.k + (it & 1u) * pl.stage;
#pragma unroll
        for (uint32_t p = 0; p < SP_PAGES; ++p) {  // past the last page: the last one again, which nobody sees there
            const bf16 *src = static_cast<const bf16 *>(a.cache) + page_at(a, table[pages[min(it * SP_PAGES + p, n_page - 1)]], g);
            for (uint32_t i = threadIdx.x; i < pieces; i += SP_THREADS) cp16(dst + (p * pieces + i) * 16, src + 8 * i, true);
        }
    };
    load(0);
    cp_commit();
    const float scale2 = a.scale * LOG2E, cap = a.softcap * LOG2E, cap_in = CAP ? 2.0f * scale2 / a.softcap : 0.0f;
    const int win = a.window ? (int)a.window : 0x7fffffff, keep = (int)a.keep;
    const uint32_t wr = rw * 16, ra = wr + lane / 4;
    const int p0 = ra < n_here ? (int)(pos0 + (f0 + ra) / per) : -1, p1 = ra + 8 < n_here ? (int)(pos0 + (f0 + ra + 8) / per) : -1;
    const bool live = wr < n_here;
    const int w_first = (int)(pos0 + (f0 + wr) / per), w_last = (int)(pos0 + (f0 + min(wr + 15, n_here - 1)) / per);  // of a live warp
    const bool full = wr + 16 <= n_here;
    float o[NV][2][4], m0 = -INFINITY, m1 = -INFINITY, l0 = 0.0f, l1 = 0.0f;
#pragma unroll
    for (int v = 0; v < NV; ++v)
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) o[v][n][e] = 0.0f;
    const uint32_t row_bytes = a.row * 2, at = map * a.dim_p * 2, k_steps = a.dim_p / 16;
    const uint32_t qa = qs + (wr + (lane & 15)) * pl.q_row + (lane >> 4) * 16 + at;
    const uint32_t b_off = ((lane & 7) + ((lane >> 4) << 3)) * row_bytes + ((lane >> 3) & 1) * 16 + at;
    const uint32_t v_off = ((lane & 7) + (((lane >> 3) & 1) << 3)) * row_bytes + (lane >> 4) * 16 + NM * a.dim_p * 2;
    for (uint32_t it = 0; it < n_tiles; ++it) {
        if (it + 1 < n_tiles) load(it + 1);
        cp_commit();
        cp_wait<1>();
        __syncthreads();  // this tile is there
        const int j0 = (int)(pages[it * SP_PAGES] * KV_PAGE);
        const uint32_t kb = qs + pl.k + (it & 1u) * pl.stage;
        if (live && j0 <= w_last && (j0 < keep || (long long)j0 + SP_KEYS - 1 > (long long)w_first - win)) {  // one of the warp's rows sees one of these keys
            float c[SP_KEYS / 8][4];
#pragma unroll
            for (int n = 0; n < SP_KEYS / 8; ++n) c[n][0] = c[n][1] = c[n][2] = c[n][3] = 0.0f;
#pragma unroll 2
            for (uint32_t k = 0; k < k_steps; ++k) {
                uint32_t fa[4];
                ldsm4(fa, qa + k * 32);
#pragma unroll
                for (int n = 0; n < SP_KEYS / 16; ++n) {
                    uint32_t fb[4];
                    ldsm4(fb, kb + n * 16 * row_bytes + b_off + k * 32);
                    mma_bf16(c[2 * n], fa, fb[0], fb[1]);
                    mma_bf16(c[2 * n + 1], fa, fb[2], fb[3]);
                }
            }
            const bool inside = full && j0 + SP_KEYS - 1 <= w_first && (long long)w_last - j0 < win;  // nothing to mask
            float b0 = -INFINITY, b1 = -INFINITY;
#pragma unroll
            for (int n = 0; n < SP_KEYS / 8; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int j = j0 + 8 * n + 2 * (int)(lane & 3) + e;
                    float s0 = c[n][e], s1 = c[n][2 + e];
                    if constexpr (CAP) s0 = soft_cap(s0, cap_in, cap), s1 = soft_cap(s1, cap_in, cap);
                    else s0 *= scale2, s1 *= scale2;
                    c[n][e] = inside || (j <= p0 && (p0 - j < win || j < keep)) ? s0 : -INFINITY;
                    c[n][2 + e] = inside || (j <= p1 && (p1 - j < win || j < keep)) ? s1 : -INFINITY;
                    b0 = fmaxf(b0, c[n][e]);
                    b1 = fmaxf(b1, c[n][2 + e]);
                }
            b0 = fmaxf(b0, __shfl_xor_sync(0xffffffffu, b0, 1)), b0 = fmaxf(b0, __shfl_xor_sync(0xffffffffu, b0, 2));
            b1 = fmaxf(b1, __shfl_xor_sync(0xffffffffu, b1, 1)), b1 = fmaxf(b1, __shfl_xor_sync(0xffffffffu, b1, 2));
            const float n0 = fmaxf(m0, b0), n1 = fmaxf(m1, b1);
            const float s0 = n0 == -INFINITY ? 0.0f : n0, s1 = n1 == -INFINITY ? 0.0f : n1;  // a row that has seen nothing yet keeps weights of zero
            const float g0 = pow2(m0 - s0), g1 = pow2(m1 - s1);
            m0 = n0, m1 = n1;
            l0 *= g0, l1 *= g1;
#pragma unroll
            for (int v = 0; v < NV; ++v)
#pragma unroll
                for (int n = 0; n < 2; ++n) o[v][n][0] *= g0, o[v][n][1] *= g0, o[v][n][2] *= g1, o[v][n][3] *= g1;
#pragma unroll
            for (int kk = 0; kk < SP_KEYS / 16; ++kk) {
                uint32_t ph[4], pr[4];
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int r = 0; r < 2; ++r) {  // fragment register 2 n + r: row half r of key half n
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
                    ldsm4t(fv, kb + kk * 16 * row_bytes + v * 32 + v_off);
                    mma_bf16(o[v][0], ph, fv[0], fv[1]);
                    mma_bf16(o[v][1], ph, fv[2], fv[3]);
                    mma_bf16(o[v][0], pr, fv[0], fv[1]);
                    mma_bf16(o[v][1], pr, fv[2], fv[3]);
                }
            }
        }
        __syncthreads();  // nobody reads this stage any more
    }
    cp_wait<0>();
    l0 += __shfl_xor_sync(0xffffffffu, l0, 1), l0 += __shfl_xor_sync(0xffffffffu, l0, 2);
    l1 += __shfl_xor_sync(0xffffffffu, l1, 1), l1 += __shfl_xor_sync(0xffffffffu, l1, 2);
    float f[2];
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const uint32_t i = min(ra + 8 * r, n_here - 1), h = g * per + (f0 + i) % per;
        float l = r ? l1 : l0;
        if (a.sink) l += pow2(a.sink[h] * LOG2E - (r ? m1 : m0));
        f[r] = (NM == 1 ? head_factor(a, row0 + (f0 + i) / per, h) : 1.0f) / l;
    }
    if constexpr (NM == 2) {  // the second map's rows go to the first map's warps through shared memory
        const uint32_t o_row = a.vdim_p + 8;
        float *ex = reinterpret_cast<float *>(smem + pl.k);
        if (map == 1) {
#pragma unroll
            for (int v = 0; v < NV; ++v)
#pragma unroll
                for (int n = 0; n < 2; ++n)
#pragma unroll
                    for (int r = 0; r < 2; ++r) {
                        if (v * 16 >= (int)a.vdim_p) continue;
                        const float w = f[r] * a.map_weight;
                        *reinterpret_cast<float2 *>(ex + (ra + 8 * r) * o_row + v * 16 + n * 8 + 2 * (lane & 3)) = make_float2(o[v][n][2 * r] * w, o[v][n][2 * r + 1] * w);
                    }
        }
        __syncthreads();
        if (map == 1) return;
        float s[2] = {0.0f, 0.0f};
#pragma unroll
        for (int v = 0; v < NV; ++v)
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int r = 0; r < 2; ++r) {
                    if (v * 16 >= (int)a.vdim_p) continue;
                    const float2 z = *reinterpret_cast<const float2 *>(ex + (ra + 8 * r) * o_row + v * 16 + n * 8 + 2 * (lane & 3));
                    const float x0 = o[v][n][2 * r] * f[r] - z.x, x1 = o[v][n][2 * r + 1] * f[r] - z.y;  // columns past vdim are zero: so are the values there
                    o[v][n][2 * r] = x0, o[v][n][2 * r + 1] = x1;
                    s[r] += x0 * x0 + x1 * x1;
                }
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            s[r] += __shfl_xor_sync(0xffffffffu, s[r], 1), s[r] += __shfl_xor_sync(0xffffffffu, s[r], 2);
            f[r] = inv_rms(s[r], a.vdim, a.eps) * a.head_gain;
        }
    }
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const uint32_t i = ra + 8 * r;
        if (i >= n_here) continue;
        const uint64_t t = row0 + (f0 + i) / per;
        const uint32_t h = g * per + (f0 + i) % per;
        bf16 *out = static_cast<bf16 *>(a.out) + t * a.out_pitch + (uint64_t)h * a.vdim;
        const bf16 *gate = static_cast<const bf16 *>(a.va) + t * a.va_pitch + a.gate0 + (uint64_t)h * a.vdim;
#pragma unroll
        for (int v = 0; v < NV; ++v)
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const uint32_t col = v * 16 + n * 8 + 2 * (lane & 3);
                if (col >= a.vdim) continue;
                float x0 = o[v][n][2 * r] * f[r], x1 = o[v][n][2 * r + 1] * f[r];
                if ((a.vdim & 1) == 0) {
                    if (a.has_gate) {
                        const __nv_bfloat162 z = *reinterpret_cast<const __nv_bfloat162 *>(gate + col);
                        x0 /= 1.0f + expf(-__low2float(z)), x1 /= 1.0f + expf(-__high2float(z));
                    }
                    *reinterpret_cast<__nv_bfloat162 *>(out + col) = __floats2bfloat162_rn(x0, x1);
                } else {
                    if (a.has_gate) x0 /= 1.0f + expf(-from_act(gate[col]));
                    out[col] = __float2bfloat16_rn(x0);
                    if (col + 1 < a.vdim) {
                        if (a.has_gate) x1 /= 1.0f + expf(-from_act(gate[col + 1]));
                        out[col + 1] = __float2bfloat16_rn(x1);
                    }
                }
            }
    }
}

using StKernel = void (*)(AttentionArgs, uint32_t, uint32_t);
using SpKernel = void (*)(AttentionArgs);
constexpr int N_FORM = 6;
const uint32_t FORMS[N_FORM] = {2, 4, 6, 8, 12, 16};  // columns of a value in sixteens
#define OB_FORMS(KERNEL, NM, CAP) {KERNEL<NM, 2, CAP>, KERNEL<NM, 4, CAP>, KERNEL<NM, 6, CAP>, KERNEL<NM, 8, CAP>, KERNEL<NM, 12, CAP>, KERNEL<NM, 16, CAP>}
constexpr int N_KIND = 3;  // one map, two maps, one map with a soft cap
const StKernel ST_KERNELS[N_KIND][N_FORM] = {OB_FORMS(attention_step_kernel, 1, false), OB_FORMS(attention_step_kernel, 2, false), OB_FORMS(attention_step_kernel, 1, true)};
const SpKernel SP_KERNELS[N_KIND][N_FORM] = {OB_FORMS(attention_span_kernel, 1, false), OB_FORMS(attention_span_kernel, 2, false), OB_FORMS(attention_span_kernel, 1, true)};
#undef OB_FORMS
int kind_of(const AttentionArgs &a) { return a.n_map == 2 ? 1 : a.softcap > 0.0f ? 2 : 0; }
int form_of(uint32_t vdim_p) {
    int f = 0;
    while (f < N_FORM && 16 * FORMS[f] < vdim_p) ++f;
    return f;
}
size_t plain_smem(const AttentionArgs &a) { return (size_t)(a.dim + a.n_map * a.vdim + AP_KEYS) * 4; }

}  // namespace

// ---- launchers ----------------------------------------------------------------------------------------------------------------------
cudaError_t attention_configure() {
    static PerDeviceOnce once;
    return once.run([] {
        cudaError_t e = cudaSuccess;
        auto set = [&](auto k) {
            if (e == cudaSuccess) e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, MAX_SMEM);
        };
        for (int m = 0; m < N_KIND; ++m)
            for (int f = 0; f < N_FORM; ++f) set(ST_KERNELS[m][f]), set(SP_KERNELS[m][f]);
        set(attention_plain_kernel<float>), set(attention_plain_kernel<bf16>);
        set(attention_prep_kernel<float>), set(attention_prep_kernel<bf16>);
        return e != cudaSuccess ? e : attention_prompt_configure();
    });
}

uint32_t attention_cache_row(uint32_t n_map, uint32_t dim_p, uint32_t vdim_p) { return n_map * dim_p + vdim_p + 8; }

bool attention_supported(uint32_t dim, uint32_t vdim) { return (uint64_t)PREP_WARPS * dim * 4 <= MAX_SMEM && (uint64_t)(dim + 2 * vdim + AP_KEYS) * 4 <= MAX_SMEM; }

void launch_attention_prep(const AttentionArgs &a, bool f32, cudaStream_t st) {
    const uint32_t n = a.n_head * a.n_map + (a.own_kv ? a.n_kv * (a.n_map + 1) : 0);
    if (a.dim % 8 == 0 && a.vdim % 8 == 0 && a.rot.dims % (a.rot.interleaved ? 8 : 16) == 0 && a.dim_p <= 256) {
        uint32_t group = 1;
        while (8 * group < a.dim_p) group *= 2;
        const uint32_t each = PREP_THREADS / group;
        launch_pdl(f32 ? attention_prep_vec_kernel<float> : attention_prep_vec_kernel<bf16>, dim3(a.T, a.norm_whole ? 1 : (n + each - 1) / each), PREP_THREADS, 0, st, a, group);
        return;
    }
    const dim3 grid(a.T, (n + PREP_WARPS - 1) / PREP_WARPS);
    launch_pdl(f32 ? attention_prep_kernel<float> : attention_prep_kernel<bf16>, grid, PREP_WARPS * 32, (size_t)PREP_WARPS * a.dim * 4, st, a);
}

uint32_t launch_attention(const AttentionArgs &in, bool f32, int sm_count, cudaStream_t st) {
    AttentionArgs a = in;
    const int form = form_of(a.vdim_p);
    const uint32_t stages = StPlan::best_stages(a.n_map, a.dim_p, a.vdim_p, a.row), per = a.n_head / a.n_kv;
    if (f32 || form == N_FORM || !stages) {
        launch_pdl(f32 ? attention_plain_kernel<float> : attention_plain_kernel<bf16>, a.T * a.n_head, AP_THREADS, plain_smem(a), st, a);
        return 1;
    }
    const SpPlan sp(a.n_map, a.dim_p, a.vdim_p, a.row);
    const bool tc5 = attention_prompt_supported(a.n_map, a.dim_p, a.vdim_p);
    if (!tc5 && sp.bytes > MAX_SMEM) a.n_short = a.n_seq;
    uint32_t launched = 0;
    if (a.n_short) {
        uint32_t tiles = 0;
        if (a.single) tiles = a.n_seq * ((per + ST_ROWS - 1) / ST_ROWS);
        else
            for (uint32_t s = 0; s < a.n_short; ++s) tiles += (a.h_spans[s].n * per + ST_ROWS - 1) / ST_ROWS;
        // few tiles: clusters share their keys, down to two pages per warp
        const uint32_t units = ST_WARPS, reach = (a.window ? std::min(a.max_pos, a.window + a.keep) : a.max_pos) / KV_PAGE + 1;
        uint32_t splits = 1;
        while (splits < ST_MAX_CLUSTER && (uint64_t)tiles * a.n_kv * splits * 2 <= 2ull * sm_count && reach > units * splits * 2) splits *= 2;
        cudaLaunchAttribute at[2];
        at[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
        at[0].val.programmaticStreamSerializationAllowed = 1;
        at[1].id = cudaLaunchAttributeClusterDimension;
        at[1].val.clusterDim.x = splits, at[1].val.clusterDim.y = 1, at[1].val.clusterDim.z = 1;
        cudaLaunchConfig_t cfg{};
        cfg.gridDim = dim3(tiles * splits, a.n_kv);
        cfg.blockDim = ST_THREADS;
        cfg.dynamicSmemBytes = StPlan(a.n_map, a.dim_p, a.vdim_p, a.row, stages).bytes;
        cfg.stream = st;
        cfg.attrs = at;
        cfg.numAttrs = splits > 1 ? 2 : 1;
        cudaLaunchKernelEx(&cfg, ST_KERNELS[kind_of(a)][form], a, splits, stages);
        ++launched;
    }
    if (a.n_short < a.n_seq && tc5) {
        if (!launch_attention_prompt(a, sm_count, st)) return 0;
        ++launched;
    } else if (a.n_short < a.n_seq) {
        uint32_t tiles = 0;
        for (uint32_t s = a.n_short; s < a.n_seq; ++s) tiles += (a.h_spans[s].n * per + sp.rows - 1) / sp.rows;
        launch_pdl(SP_KERNELS[kind_of(a)][form], dim3(tiles, a.n_kv), SP_THREADS, sp.bytes, st, a);
        ++launched;
    }
    return launched;
}

}  // namespace ob
