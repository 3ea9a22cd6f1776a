// Device helpers shared by the kernels around the products (mixers.cu, gqa.cu, moe.cu): activations in either precision, sums,
// rotation, shared-memory copies and mma.sync fragments, tiles of (token, head) rows.
#pragma once

#include <math.h>

#include <algorithm>

#include "layered.h"
#include "pdl.cuh"

namespace ob {

using bf16 = __nv_bfloat16;

template <typename TA> __device__ __forceinline__ TA to_act(float v);
template <> __device__ __forceinline__ float to_act<float>(float v) { return v; }
template <> __device__ __forceinline__ bf16 to_act<bf16>(float v) { return __float2bfloat16_rn(v); }
__device__ __forceinline__ float from_act(float v) { return v; }
__device__ __forceinline__ float from_act(bf16 v) { return __bfloat162float(v); }

// Sum over the CTA; every thread gets it.  red: 33 floats.
__device__ __forceinline__ float block_sum(float v, float *red) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    if (threadIdx.x < 32) {
        float s = threadIdx.x < blockDim.x / 32 ? red[threadIdx.x] : 0.0f;
        s = warp_sum(s);
        if (threadIdx.x == 0) red[32] = s;
    }
    __syncthreads();
    return red[32];
}

__device__ __forceinline__ float inv_rms(float sum_sq, uint32_t n, float eps) { return 1.0f / sqrtf(sum_sq / (float)n + eps); }

// A row in registers: element group i of a thread is columns 4 (threadIdx + i blockDim) .. + 3; NV = 0: any width, one column
// at a time through memory.
constexpr int ROW_VECS = 4;

// Kernel form and threads for rows of `width`: in registers when the columns come in fours and fit, few rows on wide CTAs.
struct RowShape {
    bool vec;
    uint32_t threads;
    RowShape(uint32_t width, uint32_t rows, int sm_rows = 296) {
        const uint32_t want = (width / 4 + 31) / 32 * 32;
        threads = rows <= (uint32_t)sm_rows ? std::min(1024u, std::max(128u, want)) : std::min(1024u, std::max(128u, (want / ROW_VECS + 31) / 32 * 32));
        vec = width % 4 == 0 && (uint64_t)threads * 4 * ROW_VECS >= width;
    }
};

// A row of activations from four fp32 values per thread and step.
template <typename TA> __device__ __forceinline__ void store4(TA *p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float *p, float4 v) { *reinterpret_cast<float4 *>(p) = v; }
template <> __device__ __forceinline__ void store4<bf16>(bf16 *p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2 *>(p) = make_uint2(*reinterpret_cast<const uint32_t *>(&lo), *reinterpret_cast<const uint32_t *>(&hi));
}
__device__ __forceinline__ float sq4(float4 v) { return v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w; }
__device__ __forceinline__ float4 mul4(float4 v, float f) { return make_float4(v.x * f, v.y * f, v.z * f, v.w * f); }
__device__ __forceinline__ float4 mul44(float4 a, float4 b) { return make_float4(a.x * b.x, a.y * b.y, a.z * b.z, a.w * b.w); }

// Value d of the rotated vector whose unrotated values are v[0..]; cs: this position's (cos, sin) row.
__device__ __forceinline__ float rotated(const float *v, uint32_t d, const Rot &r, const float2 *cs) {
    if (d >= r.dims) return v[d];
    const uint32_t half = r.dims / 2;
    if (r.interleaved) {
        const float2 c = cs[d >> 1];
        return d & 1 ? v[d] * c.x + v[d - 1] * c.y : v[d] * c.x - v[d + 1] * c.y;
    }
    const float2 c = cs[d < half ? d : d - half];
    return d < half ? v[d] * c.x - v[d + half] * c.y : v[d] * c.x + v[d - half] * c.y;
}

// First position row t of a sequence sees.
__device__ __forceinline__ uint32_t first_seen(uint32_t pos, uint32_t window) { return window && pos + 1 > window ? pos + 1 - window : 0u; }

// Pages a group of rows of one sequence reads: the kept first ones, then those from the window's start on.  Counted from 0 to `n`.
struct PageList {
    uint32_t kept, gap, n;  // page i < kept is page i, the others page i + gap
    __device__ __forceinline__ uint32_t operator[](uint32_t i) const { return i < kept ? i : i + gap; }
};
// Rows at positions [first, last]; the kept pages come in multiples of `unit`.
__device__ __forceinline__ PageList page_list(uint32_t first, uint32_t last, uint32_t window, uint32_t keep, uint32_t unit) {
    const uint32_t from = first_seen(first, window) / KV_PAGE, end = last / KV_PAGE + 1;
    const uint32_t kept = (keep + KV_PAGE - 1) / KV_PAGE, whole = (kept + unit - 1) / unit * unit;
    if (from <= whole && keep) return PageList{0, 0, end};  // nothing between them
    return PageList{whole, from - whole, whole + end - from};
}

// softcap tanh(s / softcap) with c = 2 log2(e) / softcap times s's factor: exact to fp32 where it counts, absolutely.
__device__ __forceinline__ float soft_cap(float s, float c, float cap) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(s * c));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(e + 1.0f));
    return fmaf(-2.0f * cap, r, cap);
}

__device__ __forceinline__ uint32_t smem_addr(const void *p) { return (uint32_t)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp16(uint32_t dst, const void *src, bool in) {  // 16 bytes, or zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(in ? 16 : 0) : "memory");
}
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void cp_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ void ldsm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldsm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void mma_bf16(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

__device__ __forceinline__ float pow2(float x) {  // relative error below 2^-22; 0 for -inf
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}

// The tile'th group of `rows` (token, head) rows: its span and first row within the span.  One warp; every lane gets the answer.
__device__ __forceinline__ void find_tile(const RowSpan *spans, uint32_t n_seq, uint32_t n_head, uint32_t rows, uint32_t tile, RowSpan *span, uint32_t *first) {
    const uint32_t lane = threadIdx.x & 31;
    for (uint32_t s0 = 0;; s0 += 32) {
        const RowSpan sp = s0 + lane < n_seq ? spans[s0 + lane] : RowSpan{0, 0};
        const uint32_t n = (sp.n * n_head + rows - 1) / rows;
        uint32_t sum = n;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const uint32_t up = __shfl_up_sync(0xffffffffu, sum, o);
            if (lane >= o) sum += up;
        }
        const uint32_t hit = __ballot_sync(0xffffffffu, tile < sum);
        if (hit || s0 + 32 >= n_seq) {
            const int src = hit ? __ffs(hit) - 1 : 31;
            span->row0 = __shfl_sync(0xffffffffu, sp.row0, src);
            span->n = hit ? __shfl_sync(0xffffffffu, sp.n, src) : 0;
            *first = (tile - __shfl_sync(0xffffffffu, sum - n, src)) * rows;
            return;
        }
        tile -= __shfl_sync(0xffffffffu, sum, 31);
    }
}

}  // namespace ob
