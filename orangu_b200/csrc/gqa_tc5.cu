// Attention of prompts on the fifth-generation tensor cores (gqa.cu has the other forms; bf16 cache, values of at most 128).
//
// A CTA is persistent; each of its items is two streams of 128 (token, head) rows of one key/value head: with one map two
// neighbouring tiles of rows that share keys and values, with two maps the maps of the same rows, which share the values.  While one
// stream's scores go through the softmax, the tensor core works for the other; the next item's keys, values, queries and first
// scores come under the end of the present one.
//
//   warps 0-15 softmax: eight warps per stream, two threads per row with 64 keys each.  Scores come from tensor memory, weights go
//              back into the same columns as value plus remainder, two bf16 operands, so that they are not rounded to 8 bits.
//   warp 16    issues the products: scores = queries (shared memory) x keys, output += weights (tensor memory) x values
//   warp 17    issues the TMA loads of pages: 16 rows x 64 columns each, straight from the cache into the swizzled operand tiles
//
// Tensor memory: scores / weights of the streams 2 x 128 columns, outputs 2 x 128.  The output is only rescaled when a row's maximum
// has grown by more than 2^8 since the last time; until then weights are relative to the older maximum.  All waits are bounded.
#include <algorithm>

#include "mixers_common.cuh"
#include "tc5_common.cuh"

namespace ob {

namespace {

constexpr uint32_t PT_ROWS = 128, PT_KEYS = 128, PT_PAGES = PT_KEYS / KV_PAGE, PT_BLOCK = PT_KEYS * 128;  // block: 128 rows of 64 columns
constexpr int PT_MMA_WARP = 16, PT_TMA_WARP = 17, PT_THREADS = 18 * 32;
constexpr uint32_t PT_TMEM_S = 0, PT_TMEM_O = 256, PT_TMEM_COLS = 512;
constexpr float PT_SLACK = 8.0f;  // growth of the maximum (powers of two) that is put up with

constexpr uint32_t PT_STAGE = 1024;  // of a warp: 32 rows x 16 columns of output on their way from a thread per row to whole sectors
constexpr uint32_t PT_SHARED = 320 + 2 * 2 * PT_ROWS * 4 + 48 + 16 * PT_STAGE;  // mbarriers, items, a number per stream, half and row, stages
struct PtPlan {
    uint32_t nb, nbv, k_bytes, v_bytes, stages, k, v, bar, bytes;  // blocks of 64 columns of a map's keys and of a value; operands of one stage
    __host__ __device__ PtPlan(uint32_t n_map, uint32_t dim_p, uint32_t vdim_p) {
        nb = (dim_p + 63) / 64, nbv = (vdim_p + 63) / 64;
        k_bytes = n_map * nb * PT_BLOCK, v_bytes = nbv * PT_BLOCK;
        const uint32_t q = 2 * nb * PT_BLOCK, room = 225 * 1024 - PT_SHARED;
        stages = q + 2 * (k_bytes + v_bytes) <= room ? 2 : q + k_bytes + v_bytes <= room ? 1 : 0;
        k = q;
        v = k + stages * k_bytes;
        bar = v + stages * v_bytes;
        bytes = bar + PT_SHARED + 1024;
    }
};
// mbarriers, byte offsets from PtPlan::bar
constexpr uint32_t PT_K_FULL = 0, PT_K_EMPTY = 16, PT_V_FULL = 32, PT_V_EMPTY = 48, PT_S_FULL = 64, PT_P_FULL = 80, PT_O_FULL = 96, PT_Q_FULL = 112, PT_SLOT = 128, PT_ABORT = 132,
                   PT_ITEMS = 160, PT_ITEM_FULL = 288, PT_EXCHANGE = 320, PT_STAGES = PT_EXCHANGE + 2 * 2 * PT_ROWS * 4 + 48;

// Two fp32 multiply-adds in one instruction.
__device__ __forceinline__ void fma2(float &d0, float &d1, float a0, float a1, float b, float c) {
    asm("{\n\t.reg .b64 x, y, z;\n\tmov.b64 x, {%2, %3};\n\tmov.b64 y, {%4, %4};\n\tmov.b64 z, {%5, %5};\n\tfma.rn.f32x2 x, x, y, z;\n\tmov.b64 {%0, %1}, x;\n\t}"
        : "=f"(d0), "=f"(d1)
        : "f"(a0), "f"(a1), "f"(b), "f"(c));
}
__device__ __forceinline__ void add2(float &d0, float &d1, float a0, float a1) {
    asm("{\n\t.reg .b64 x, y;\n\tmov.b64 x, {%0, %1};\n\tmov.b64 y, {%2, %3};\n\tadd.rn.f32x2 x, x, y;\n\tmov.b64 {%0, %1}, x;\n\t}" : "+f"(d0), "+f"(d1) : "f"(a0), "f"(a1));
}
__device__ __forceinline__ void pair_sync(uint32_t id) { asm volatile("bar.sync %0, 64;" ::"r"(id) : "memory"); }
__device__ __forceinline__ void quad_sync(uint32_t id) { asm volatile("bar.sync %0, 128;" ::"r"(id) : "memory"); }

// Sigmoid to a few units in the last place.
__device__ __forceinline__ float gate_factor(float z) { return __fdividef(1.0f, 1.0f + pow2(z * -1.4426950408889634f)); }

// A CTA's piece of work: 128 (two maps) or 256 (one map) consecutive (token, head) rows of one key/value head.  The TMA warp looks
// it up and leaves it in a ring of four with an mbarrier each (it is never more than three items ahead).
struct PtItem {
    uint32_t row0, f0, n_here, pos0, g;
    PageList pages;  // the kept ones fill whole tiles
    __device__ __forceinline__ uint32_t n_tiles() const { return (pages.n + PT_PAGES - 1) / PT_PAGES; }
};
__device__ __forceinline__ PtItem pt_read(const uint8_t *smem, uint32_t turn) {
    const volatile uint32_t *p = reinterpret_cast<const volatile uint32_t *>(smem + PT_ITEMS) + turn % 4 * 8;
    return PtItem{p[0], p[1], p[2], p[3], p[4], PageList{p[5], p[6], p[7]}};
}
__device__ __forceinline__ void pt_write(uint8_t *smem, uint32_t turn, const PtItem &w) {
    volatile uint32_t *p = reinterpret_cast<volatile uint32_t *>(smem + PT_ITEMS) + turn % 4 * 8;
    p[0] = w.row0, p[1] = w.f0, p[2] = w.n_here, p[3] = w.pos0, p[4] = w.g, p[5] = w.pages.kept, p[6] = w.pages.gap, p[7] = w.pages.n;
}
template <int NM>
__device__ __forceinline__ PtItem pt_item(const AttentionArgs &a, uint32_t item, uint32_t n_row_tiles) {  // one warp; every lane gets the answer
    constexpr uint32_t M = NM == 2 ? PT_ROWS : 2 * PT_ROWS;
    const uint32_t per = a.n_head / a.n_kv;
    PtItem w;
    RowSpan sp;
    // (the last rows of a span see the most keys: they come first)
    find_tile(a.spans + a.n_short, a.n_seq - a.n_short, per, M, n_row_tiles - 1 - item / a.n_kv, &sp, &w.f0);
    w.row0 = sp.row0, w.g = item % a.n_kv;
    w.n_here = min(M, sp.n * per - w.f0);
    w.pos0 = a.positions[w.row0];
    w.pages = page_list(w.pos0 + w.f0 / per, w.pos0 + (w.f0 + w.n_here - 1) / per, a.window, a.keep, PT_PAGES);
    return w;
}
// The output of a warp's 32 rows, 16 columns at a time: gates come and activations go by way of the warp's stage, where two lanes
// share a row.
struct RowOut {
    uint64_t at[2];     // this lane's two rows (lane / 2, and 16 on): first entry of their head in the output ...
    uint64_t gate[2];   // ... and of their gates
    bool live[2];
    bool wide;          // entries come in eights
};
__device__ __forceinline__ RowOut row_out(const AttentionArgs &a, const PtItem &w, uint32_t warp_row0) {
    RowOut ro;
    const uint32_t per = a.n_head / a.n_kv, lane = threadIdx.x & 31;
#pragma unroll
    for (uint32_t k = 0; k < 2; ++k) {
        const uint32_t i = warp_row0 + 16 * k + lane / 2, f = w.f0 + min(i, w.n_here - 1);
        const uint64_t t = w.row0 + f / per, h = w.g * per + f % per;
        ro.live[k] = i < w.n_here;
        ro.at[k] = t * a.out_pitch + h * a.vdim;
        ro.gate[k] = t * a.va_pitch + a.gate0 + h * a.vdim;
    }
    ro.wide = a.vdim % 8 == 0;
    return ro;
}
// Gates of columns [c, c + 16): a lane's eight of either row.
__device__ __forceinline__ void load_gates(const AttentionArgs &a, const RowOut &ro, uint32_t c, uint4 (&z)[2]) {
    const uint32_t e = c + 8 * (threadIdx.x & 1);
#pragma unroll
    for (uint32_t k = 0; k < 2; ++k) {
        const bf16 *p = static_cast<const bf16 *>(a.va) + ro.gate[k] + e;
        z[k] = make_uint4(0, 0, 0, 0);
        if (ro.wide && ro.live[k] && e < a.vdim) z[k] = *reinterpret_cast<const uint4 *>(p);
        if (ro.wide) continue;
        uint32_t u[4] = {0, 0, 0, 0};
#pragma unroll
        for (uint32_t i = 0; i < 8; ++i)
            if (ro.live[k] && e + i < a.vdim) u[i / 2] |= (uint32_t)__bfloat16_as_ushort(p[i]) << (i % 2 * 16);
        z[k] = make_uint4(u[0], u[1], u[2], u[3]);
    }
}
// x: columns [c, c + 16) of this lane's own row (row `lane` of the warp), z: load_gates of the same columns.
__device__ __forceinline__ void store_rows(const AttentionArgs &a, const RowOut &ro, uint8_t *stage, uint32_t c, float (&x)[16], const uint4 (&z)[2]) {
    const uint32_t lane = threadIdx.x & 31;
    auto place = [&](uint32_t row, uint32_t half) { return reinterpret_cast<uint4 *>(stage + row * 32 + ((half ^ (row >> 2 & 1)) << 4)); };  // (no bank conflicts either way)
    if (a.has_gate) {
#pragma unroll
        for (uint32_t k = 0; k < 2; ++k) *place(16 * k + lane / 2, lane & 1) = z[k];
        __syncwarp();
#pragma unroll
        for (uint32_t b = 0; b < 2; ++b) {
            const uint4 g = *place(lane, b);
            const uint32_t gw[4] = {g.x, g.y, g.z, g.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                x[8 * b + 2 * e] *= gate_factor(__uint_as_float(gw[e] << 16));
                x[8 * b + 2 * e + 1] *= gate_factor(__uint_as_float(gw[e] & 0xffff0000u));
            }
        }
    }
#pragma unroll
    for (uint32_t b = 0; b < 2; ++b) {
        uint32_t o[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const __nv_bfloat162 v = __floats2bfloat162_rn(x[8 * b + 2 * e], x[8 * b + 2 * e + 1]);
            o[e] = *reinterpret_cast<const uint32_t *>(&v);
        }
        *place(lane, b) = make_uint4(o[0], o[1], o[2], o[3]);
    }
    __syncwarp();
    const uint32_t e = c + 8 * (lane & 1);
#pragma unroll
    for (uint32_t k = 0; k < 2; ++k) {
        const uint4 v = *place(16 * k + lane / 2, lane & 1);
        bf16 *p = static_cast<bf16 *>(a.out) + ro.at[k] + e;
        if (!ro.live[k] || e >= a.vdim) continue;
        if (ro.wide) {
            *reinterpret_cast<uint4 *>(p) = v;
        } else {
            const uint32_t u[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
            for (uint32_t i = 0; i < 8; ++i)
                if (e + i < a.vdim) p[i] = __ushort_as_bfloat16((unsigned short)(u[i / 2] >> (i % 2 * 16)));
        }
    }
    __syncwarp();
}
// Tiles of keys that a stream's rows see: [first, end).  Only with one map may the second stream have no rows.
template <int NM>
__device__ __forceinline__ uint32_t pt_first(const AttentionArgs &a, const PtItem &w, uint32_t s) {
    if (NM == 2 || s == 0 || w.n_here <= PT_ROWS || a.keep) return 0;
    return (first_seen(w.pos0 + (w.f0 + PT_ROWS) / (a.n_head / a.n_kv), a.window) / KV_PAGE - w.pages.gap) / PT_PAGES;
}
template <int NM>
__device__ __forceinline__ uint32_t pt_end(const AttentionArgs &a, const PtItem &w, uint32_t s) {
    if (NM == 2) return w.n_tiles();
    if (s == 1) return w.n_here > PT_ROWS ? w.n_tiles() : 0;
    return ((w.pos0 + (w.f0 + min(w.n_here, PT_ROWS) - 1) / (a.n_head / a.n_kv)) / KV_PAGE - w.pages.gap) / PT_PAGES + 1;
}

template <int NM, bool CAP>
__global__ void __launch_bounds__(PT_THREADS, 1)
attention_prompt_kernel(const __grid_constant__ CUtensorMap tm, const __grid_constant__ AttentionArgs a, uint32_t n_row_tiles) {
    extern __shared__ uint8_t smem_raw[];
    const uint32_t sbase = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t *smem = smem_raw + (sbase - smem_u32(smem_raw));
    const PtPlan pl(NM, a.dim_p, a.vdim_p);
    const uint32_t bar = sbase + pl.bar, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, per = a.n_head / a.n_kv, n_items = n_row_tiles * a.n_kv;
    volatile uint32_t *abort = reinterpret_cast<volatile uint32_t *>(smem + pl.bar + PT_ABORT);
    if (threadIdx.x == 0) {
        for (uint32_t s = 0; s < 2; ++s) {
            mbar_init(bar + PT_K_FULL + 8 * s, 1);
            mbar_init(bar + PT_K_EMPTY + 8 * s, 1);
            mbar_init(bar + PT_V_FULL + 8 * s, 1);
            mbar_init(bar + PT_V_EMPTY + 8 * s, 1);
            mbar_init(bar + PT_S_FULL + 8 * s, 1);
            mbar_init(bar + PT_P_FULL + 8 * s, 8);
            mbar_init(bar + PT_O_FULL + 8 * s, 1);
            mbar_init(bar + PT_Q_FULL + 8 * s, 8);
        }
        for (uint32_t i = 0; i < 4; ++i) mbar_init(bar + PT_ITEM_FULL + 8 * i, 1);
        *abort = 0u;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == PT_MMA_WARP) tmem_alloc(bar + PT_SLOT, PT_TMEM_COLS);
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    pdl_release();  // (only now: a CTA of the next kernel must not take the tensor memory first, it would keep it until this grid is done)
    pdl_wait();
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t *>(smem + pl.bar + PT_SLOT);

    if (warp == PT_TMA_WARP) {
        uint32_t n = 0, turn = 0;  // tiles and items so far
        bool ok = true;
        for (uint32_t item = blockIdx.x; item < n_items; item += gridDim.x, ++turn) {
            const PtItem w = pt_item<NM>(a, item, n_row_tiles);
            if (lane == 0) {
                const int32_t *table = a.tables[w.row0];
                pt_write(smem + pl.bar, turn, w);
                mbar_arrive(bar + PT_ITEM_FULL + 8 * (turn % 4));
                for (uint32_t i = 0; i < w.n_tiles() && ok; ++i, ++n) {
                    const uint32_t st = n % pl.stages, par = ((n / pl.stages) & 1u) ^ 1u;
                    int32_t y[PT_PAGES];
#pragma unroll
                    for (uint32_t p = 0; p < PT_PAGES; ++p)  // past the last page: the last one again, which nobody sees there
                        y[p] = (int32_t)((table[w.pages[min(i * PT_PAGES + p, w.pages.n - 1)]] * a.n_kv + w.g) * KV_PAGE);
                    if (n >= pl.stages && !(ok = mbar_wait(bar + PT_K_EMPTY + 8 * st, par, abort))) break;
                    mbar_expect_tx(bar + PT_K_FULL + 8 * st, pl.k_bytes);
                    for (uint32_t b = 0; b < NM * pl.nb; ++b) {
                        const int32_t x = (int32_t)(b / pl.nb * a.dim_p + b % pl.nb * 64);
#pragma unroll
                        for (uint32_t p = 0; p < PT_PAGES; ++p)
                            tma_load_2d(sbase + pl.k + st * pl.k_bytes + b * PT_BLOCK + p * (KV_PAGE * 128), &tm, x, y[p], bar + PT_K_FULL + 8 * st);
                    }
                    if (n >= pl.stages && !(ok = mbar_wait(bar + PT_V_EMPTY + 8 * st, par, abort))) break;
                    mbar_expect_tx(bar + PT_V_FULL + 8 * st, pl.v_bytes);
                    for (uint32_t b = 0; b < pl.nbv; ++b) {
                        const int32_t x = (int32_t)(NM * a.dim_p + b * 64);
#pragma unroll
                        for (uint32_t p = 0; p < PT_PAGES; ++p)
                            tma_load_2d(sbase + pl.v + st * pl.v_bytes + b * PT_BLOCK + p * (KV_PAGE * 128), &tm, x, y[p], bar + PT_V_FULL + 8 * st);
                    }
                }
            }
            __syncwarp();
        }
    } else if (warp == PT_MMA_WARP) {
        const uint32_t id_s = umma_idesc_bf16(PT_KEYS), id_o = umma_idesc_bf16(a.vdim_p) | UMMA_B_MN_MAJOR, k_steps = a.dim_p / 16;
        uint32_t n = 0, turn = 0, used0 = 0, used1 = 0;  // tiles and items so far, weights taken from each stream so far
        bool ok = true;
        const uint64_t q_desc = umma_desc_sw128(sbase), k_desc = umma_desc_sw128(sbase + pl.k), v_desc = umma_desc_sw128_mn(sbase + pl.v, PT_BLOCK);
        auto scores = [&](uint32_t s, uint32_t at) {
            const uint32_t st = at % pl.stages;
            if (!mbar_wait_warp(bar + PT_K_FULL + 8 * st, (at / pl.stages) & 1u, abort)) return false;
            tc_fence_after();
            uint64_t qd = q_desc + (s * pl.nb * PT_BLOCK >> 4), kd = k_desc + (st * pl.k_bytes + (NM == 2 ? s * pl.nb * PT_BLOCK : 0) >> 4);
            for (uint32_t b = 0; b < k_steps; b += 4, qd += PT_BLOCK >> 4, kd += PT_BLOCK >> 4)
#pragma unroll
                for (uint32_t j = 0; j < 4; ++j)
                    if (b + j < k_steps) umma_bf16_warp(tmem + PT_TMEM_S + s * PT_KEYS, qd + 2 * j, kd + 2 * j, id_s, b + j ? 1u : 0u);
            umma_commit_warp(bar + PT_S_FULL + 8 * s);
            return true;
        };
        for (uint32_t item = blockIdx.x; item < n_items && ok; item += gridDim.x, ++turn) {
            ok = mbar_wait_warp(bar + PT_K_FULL + 8 * (n % pl.stages), (n / pl.stages) & 1u, abort);
            if (!ok) break;
            const PtItem w = pt_read(smem + pl.bar, turn);
            auto uniform = [](uint32_t v) { return __shfl_sync(0xffffffffu, v, 0); };
            const uint32_t first0 = uniform(pt_first<NM>(a, w, 0)), first1 = uniform(pt_first<NM>(a, w, 1)), end0 = uniform(pt_end<NM>(a, w, 0)), end1 = uniform(pt_end<NM>(a, w, 1));
            const uint32_t n_tiles = uniform(w.n_tiles());
            ok = mbar_wait_warp(bar + PT_Q_FULL, turn & 1u, abort) && mbar_wait_warp(bar + PT_Q_FULL + 8, turn & 1u, abort);
#pragma unroll
            for (uint32_t s = 0; s < 2; ++s)
                if (ok && (s ? first1 : first0) == 0 && (s ? end1 : end0) > 0) ok = scores(s, n);
            if (ok) umma_commit_warp(bar + PT_K_EMPTY + 8 * (n % pl.stages));
            for (uint32_t i = 0; i < n_tiles && ok; ++i) {
                const uint32_t st = (n + i) % pl.stages;
#pragma unroll
                for (uint32_t s = 0; s < 2; ++s) {
                    const uint32_t first = s ? first1 : first0, end = s ? end1 : end0;
                    if (ok && i >= first && i < end) {
                        uint32_t &used = s ? used1 : used0;
                        ok = mbar_wait_warp(bar + PT_P_FULL + 8 * s, used & 1u, abort) && mbar_wait_warp(bar + PT_V_FULL + 8 * st, ((n + i) / pl.stages) & 1u, abort);
                        ++used;
                        if (ok) {
                            tc_fence_after();
                            const uint32_t p = tmem + PT_TMEM_S + s * PT_KEYS, d = tmem + PT_TMEM_O + s * 128;
                            const uint64_t vd = v_desc + (st * pl.v_bytes >> 4);
#pragma unroll
                            for (uint32_t kk = 0; kk < PT_KEYS / 16; ++kk) {  // 16 keys: value, then remainder
                                umma_bf16_ta_warp(d, p + kk * 16, vd + kk * 128, id_o, i > first || kk ? 1u : 0u);
                                umma_bf16_ta_warp(d, p + kk * 16 + 8, vd + kk * 128, id_o, 1u);
                            }
                            if (i + 1 == end) umma_commit_warp(bar + PT_O_FULL + 8 * s);
                        }
                    }
                    if (ok && i + 1 >= first && i + 1 < end) ok = scores(s, n + i + 1);
                }
                if (!ok) break;
                umma_commit_warp(bar + PT_V_EMPTY + 8 * st);
                if (i + 1 < n_tiles) umma_commit_warp(bar + PT_K_EMPTY + 8 * ((n + i + 1) % pl.stages));
            }
            if (ok && end1 == 0) umma_commit_warp(bar + PT_O_FULL + 8);  // a stream without rows keeps in step
            n += n_tiles;
        }
    } else {
        const uint32_t s = warp / 8, part = warp / 4 % 2, quad = warp % 4, r = quad * 32 + lane, pair = 1 + s * 4 + quad;
        const int win = a.window ? (int)min(a.window, 0x3fffffffu) : 0x3fffffff;
        constexpr float LOG2E = 1.4426950408889634f;  // weights are powers of two of the scaled score
        const float scale2 = CAP ? 1.0f : a.scale * LOG2E, cap = a.softcap * LOG2E, cap_in = CAP ? 2.0f * LOG2E * a.scale / a.softcap : 0.0f;
        const uint32_t lanes = tmem + ((quad * 32) << 16), ts = lanes + PT_TMEM_S + s * PT_KEYS + part * 64, to = lanes + PT_TMEM_O;
        volatile float *xchg = reinterpret_cast<volatile float *>(smem + pl.bar + PT_EXCHANGE) + r;  // a number per stream, half and row
        const uint32_t own = (2 * s + part) * PT_ROWS, other = (2 * s + (part ^ 1u)) * PT_ROWS;
        bool ok = true;
        auto load_query = [&](const PtItem &w) {  // the row's query (this half of it) into the swizzled operand tile
            const uint32_t i = (NM == 2 ? 0 : s * PT_ROWS) + r, f = w.f0 + min(i, w.n_here - 1);
            const uint64_t t = w.row0 + f / per, h = w.g * per + f % per;
            const bool two = NM == 1 && a.q2;
            const bf16 *q = static_cast<const bf16 *>(a.q) + (two ? t * a.q_pitch + h * a.q_head : ((t * a.n_head + h) * NM + (NM == 2 ? s : 0)) * a.dim_p);
            const bf16 *q2 = two ? static_cast<const bf16 *>(a.q2) + t * a.q2_pitch + h * a.q2_head - a.q_split : q;
            const uint32_t split = two ? a.q_split / 8 : 0;
            uint8_t *dst = smem + s * pl.nb * PT_BLOCK + r * 128;
            for (uint32_t c0 = part; c0 < a.dim_p / 8; c0 += 8) {
                uint4 v[4];
#pragma unroll
                for (uint32_t k = 0; k < 4; ++k) {
                    const uint32_t c = c0 + 2 * k;
                    v[k] = i < w.n_here && c < a.dim_p / 8 ? *reinterpret_cast<const uint4 *>((c < split ? q : q2) + 8 * c) : make_uint4(0, 0, 0, 0);
                }
#pragma unroll
                for (uint32_t k = 0; k < 4; ++k) {
                    const uint32_t c = c0 + 2 * k;
                    if (c < a.dim_p / 8) *reinterpret_cast<uint4 *>(dst + c / 8 * PT_BLOCK + (((c & 7) ^ (r & 7)) << 4)) = v[k];
                }
            }
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(bar + PT_Q_FULL + 8 * s);
        };
        uint32_t turn = 0, used = 0;  // items and tiles of scores so far
        // The item of turn `at`.  (Not by its first keys' barrier: a stream that is done with the item before while that one's last
        // keys are still to come would, with one stage, take the keys two tiles back for them.)
        auto item_at = [&](uint32_t at, uint32_t item) {
            ok = ok && mbar_wait_warp(bar + PT_ITEM_FULL + 8 * (at % 4), (at / 4) & 1u, abort);
            return ok ? pt_read(smem + pl.bar, at) : pt_item<NM>(a, item, n_row_tiles);
        };
        PtItem w{};
        if (blockIdx.x < n_items) {
            w = item_at(0, blockIdx.x);
            load_query(w);
        }
        for (uint32_t item = blockIdx.x; item < n_items; item += gridDim.x, ++turn) {
            const uint32_t i_row = (NM == 2 ? 0 : s * PT_ROWS) + r, w0 = (NM == 2 ? 0 : s * PT_ROWS) + quad * 32, first = pt_first<NM>(a, w, s), end = pt_end<NM>(a, w, s);
            const bool live = i_row < w.n_here, whole = w0 + 32 <= w.n_here;
            const int pos = live ? (int)(w.pos0 + (w.f0 + i_row) / per) : -1;
            const int w_first = (int)(w.pos0 + (w.f0 + w0) / per), w_last = (int)(w.pos0 + (w.f0 + w0 + 31) / per);  // positions of the warp's rows
            float m = -INFINITY, l = 0.0f;
            for (uint32_t i = first; i < end; ++i, ++used) {
                ok = ok && mbar_wait_warp(bar + PT_S_FULL + 8 * s, used & 1u, abort);
                if (!ok) {  // a wait was given up: nothing more is computed, but the other warps' barriers are kept company
                    pair_sync(pair);
                    continue;
                }
                tc_fence_after();
                const int j0 = (int)(w.pages[i * PT_PAGES] * KV_PAGE + part * 64);
                uint32_t u[2][32];
                tmem_ld32(ts, u[0]);
                tmem_ld32(ts + 32, u[1]);
                tmem_ld_wait();
                if constexpr (CAP) {
#pragma unroll
                    for (int c = 0; c < 2; ++c)
#pragma unroll
                        for (int e = 0; e < 32; ++e) u[c][e] = __float_as_uint(soft_cap(__uint_as_float(u[c][e]), cap_in, cap));
                }
                const int hi = pos - j0, lo = hi - win + 1, kept = (int)a.keep - j0;  // visible columns of the row: [lo, hi] and below kept (pos -1: none)
                if (!whole || j0 + 63 > w_first) {           // keys after some row
#pragma unroll
                    for (int c = 0; c < 2; ++c)
#pragma unroll
                        for (int e = 0; e < 32; ++e)
                            if (c * 32 + e > hi) u[c][e] = 0xff800000u;
                }
                if (w_last - j0 >= win) {  // keys before some row's window
#pragma unroll
                    for (int c = 0; c < 2; ++c)
#pragma unroll
                        for (int e = 0; e < 32; ++e)
                            if (c * 32 + e < lo && c * 32 + e >= kept) u[c][e] = 0xff800000u;
                }
                float top[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int e = 0; e < 32; ++e) top[e % 4] = fmaxf(top[e % 4], __uint_as_float(u[c][e]));
                const float mine = fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])) * scale2;
                xchg[own] = mine;
                pair_sync(pair);
                const float now = fmaxf(mine, xchg[other]);
                const bool grown = m > -INFINITY && now > m + PT_SLACK;
                if (__any_sync(0xffffffffu, grown)) {  // the product before this tile's scores is done: the output may be rescaled
                    const float keep = grown ? pow2(m - now) : 1.0f;
                    if (grown) m = now, l *= keep;
                    for (uint32_t c = 16 * part; c < a.vdim_p; c += 32) {
                        uint32_t o[16];
                        tmem_ld16(to + s * 128 + c, o);
                        tmem_ld_wait();
#pragma unroll
                        for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * keep);
                        tmem_st16(to + s * 128 + c, o);
                    }
                }
                if (m == -INFINITY) m = now;
                const float base = m == -INFINITY ? 0.0f : -m;  // a row that has seen nothing yet keeps weights of zero
                float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
                for (int c = 0; c < 4; ++c) {  // 16 keys: eight columns of values, eight of remainders
                    uint32_t v[16];
#pragma unroll
                    for (int e = 0; e < 8; ++e) {
                        const uint32_t(&x)[32] = u[c / 2];
                        float e0, e1;
                        fma2(e0, e1, __uint_as_float(x[c % 2 * 16 + 2 * e]), __uint_as_float(x[c % 2 * 16 + 2 * e + 1]), scale2, base);
                        e0 = pow2(e0), e1 = pow2(e1);
                        add2(sum0, sum1, e0, e1);
                        const __nv_bfloat162 hi2 = __floats2bfloat162_rn(e0, e1);
                        const uint32_t hw = *reinterpret_cast<const uint32_t *>(&hi2);
                        const __nv_bfloat162 lo2 = __floats2bfloat162_rn(e0 - __uint_as_float(hw << 16), e1 - __uint_as_float(hw & 0xffff0000u));
                        v[e] = hw, v[8 + e] = *reinterpret_cast<const uint32_t *>(&lo2);
                    }
                    tmem_st16(ts + 16 * c, v);
                }
                l += sum0 + sum1;
                tmem_st_wait();
                tc_fence_before();
                __syncwarp();
                if (lane == 0) mbar_arrive(bar + PT_P_FULL + 8 * s);
            }
            // the next item's queries while the last product runs: nobody reads the present ones any more.  A stream without rows
            // learns that from the end of the item.
            const bool more = item + gridDim.x < n_items;
            PtItem next{};
            if (more) next = item_at(turn + 1, item + gridDim.x);
            const bool idle = end == first;
            const RowOut ro = row_out(a, w, w0);
            uint8_t *stage = smem + pl.bar + PT_STAGES + warp * PT_STAGE;
            const uint32_t c_first = 16 * (NM == 1 ? part : warp / 4), c_step = NM == 1 ? 32 : 64;  // columns of this warp
            uint4 gates[2][2] = {};
            if (a.has_gate) {
                load_gates(a, ro, c_first, gates[0]);
                load_gates(a, ro, c_first + c_step, gates[1]);
            }
            if (idle) ok = ok && mbar_wait_warp(bar + PT_O_FULL + 8 * s, turn & 1u, abort);
            if (more) load_query(next);
            if (!idle) ok = ok && mbar_wait_warp(bar + PT_O_FULL + 8 * s, turn & 1u, abort);
            tc_fence_after();

            pair_sync(pair);  // (the last maxima have been read)
            float gain = 1.0f;  // of the row's head
            if constexpr (NM == 1) {
                const uint32_t f = w.f0 + min(i_row, w.n_here - 1), h = w.g * per + f % per;
                if (a.sink && part == 0) l += pow2(a.sink[h] * LOG2E - m);
                gain = a.head_gain;
                if (a.head_gate) gain *= gate_factor(a.head_gate[(uint64_t)(w.row0 + f / per) * a.y_pitch + h]);
            }
            xchg[own] = l;
            auto put = [&](uint32_t c, float (&x)[16], uint32_t turn) {
                store_rows(a, ro, stage, c, x, gates[turn]);
                if (a.has_gate && c + 2 * c_step < a.vdim_p) load_gates(a, ro, c + 2 * c_step, gates[turn]);
            };
            if constexpr (NM == 1) {
                pair_sync(pair);
                const float fac = gain / (l + xchg[other]);
                if (ok && !idle)
#pragma unroll
                    for (uint32_t k = 0; k < 4; ++k) {
                        const uint32_t c = c_first + k * c_step;
                        if (c >= a.vdim_p) break;
                        uint32_t o[16];
                        tmem_ld16(to + s * 128 + c, o);
                        tmem_ld_wait();
                        float x[16];
#pragma unroll
                        for (int e = 0; e < 16; ++e) x[e] = __uint_as_float(o[e]) * fac;
                        put(c, x, k % 2);
                    }
                pair_sync(pair);  // (the sums have been read)
            } else {  // four warps share 32 rows: both maps' outputs are in the same lanes of tensor memory
                quad_sync(9 + quad);
                const float fac0 = 1.0f / (xchg[0] + xchg[PT_ROWS]), fac1 = a.map_weight / (xchg[2 * PT_ROWS] + xchg[3 * PT_ROWS]);
                float q = 0.0f, x[2][16];
                if (ok)
#pragma unroll
                    for (uint32_t k = 0; k < 2; ++k) {
                        const uint32_t c = c_first + k * c_step;
                        if (c >= a.vdim_p) break;
                        uint32_t o0[16], o1[16];
                        tmem_ld16(to + c, o0);
                        tmem_ld16(to + 128 + c, o1);
                        tmem_ld_wait();
#pragma unroll
                        for (int e = 0; e < 16; ++e) {  // columns past vdim are zero: so are the values there
                            x[k][e] = __uint_as_float(o0[e]) * fac0 - __uint_as_float(o1[e]) * fac1;
                            q += x[k][e] * x[k][e];
                        }
                    }
                tc_fence_before();
                quad_sync(9 + quad);  // the sums and the outputs have been read: the next weights may come
                xchg[own] = q;
                quad_sync(9 + quad);
                gain = inv_rms((xchg[0] + xchg[PT_ROWS]) + (xchg[2 * PT_ROWS] + xchg[3 * PT_ROWS]), a.vdim, a.eps) * a.head_gain;
                if (ok)
#pragma unroll
                    for (uint32_t k = 0; k < 2; ++k) {
                        const uint32_t c = c_first + k * c_step;
                        if (c >= a.vdim_p) break;
#pragma unroll
                        for (int e = 0; e < 16; ++e) x[k][e] *= gain;
                        put(c, x[k], k);
                    }
                quad_sync(9 + quad);  // (the squares have been read)
            }
            tc_fence_before();
            w = next;
        }
    }
    __syncwarp();
    if (*abort) {  // let copies that are still in flight land before the shared memory goes away
        for (int i = 0; i < 200; ++i) __nanosleep(1000);
    }
    tc_fence_before();
    __syncthreads();
    if (warp == PT_MMA_WARP) tmem_dealloc(tmem, PT_TMEM_COLS);
}

}  // namespace

cudaError_t attention_prompt_configure() {
    static PerDeviceOnce once;
    return once.run([] {
        cudaError_t e = cudaSuccess;
        for (auto k : {attention_prompt_kernel<1, false>, attention_prompt_kernel<2, false>, attention_prompt_kernel<1, true>})
            if (e == cudaSuccess) e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
        return e;
    });
}

bool attention_prompt_supported(uint32_t n_map, uint32_t dim_p, uint32_t vdim_p) { return vdim_p <= 128 && PtPlan(n_map, dim_p, vdim_p).stages > 0; }

bool launch_attention_prompt(const AttentionArgs &a, int sm_count, cudaStream_t st) {
    const uint32_t per = a.n_head / a.n_kv, M = a.n_map == 2 ? PT_ROWS : 2 * PT_ROWS;
    uint32_t tiles = 0;
    for (uint32_t s = a.n_short; s < a.n_seq; ++s) tiles += (a.h_spans[s].n * per + M - 1) / M;
    CUtensorMap tm;
    if (!make_map_2d(&tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.cache, a.row, (uint64_t)a.n_pages * a.n_kv * KV_PAGE, (uint64_t)a.row * 2, 64, KV_PAGE, CU_TENSOR_MAP_SWIZZLE_128B)) return false;
    const PtPlan pl(a.n_map, a.dim_p, a.vdim_p);
    launch_pdl(a.n_map == 2 ? attention_prompt_kernel<2, false> : a.softcap > 0.0f ? attention_prompt_kernel<1, true> : attention_prompt_kernel<1, false>, std::min(tiles * a.n_kv, (uint32_t)sm_count), PT_THREADS, pl.bytes, st, tm, a, tiles);
    g_tc5_launched.store(true, std::memory_order_relaxed);
    return true;
}

int attention_take_status() { return tc5_take_status(); }

}  // namespace ob
