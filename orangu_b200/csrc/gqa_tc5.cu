// Attention of prompts on the fifth-generation tensor cores (gqa.cu has the other forms; bf16 cache, values of at most 128).
//
// A CTA runs two streams of 128 (token, head) rows of one key/value head: with one map two neighbouring tiles of rows that share
// keys and values, with two maps the maps of the same rows, which share the values.  While one stream's scores go through the
// softmax, the tensor core works for the other.
//
//   warps 0-15 softmax: eight warps per stream, two threads per row with 64 keys each.  Scores come from tensor memory, weights go
//              back into the same columns as value plus remainder, two bf16 operands, so that they are not rounded to 8 bits.
//   warp 16    issues the products: scores = queries (shared memory) x keys, output += weights (tensor memory) x values
//   warp 17    issues the TMA loads of pages: 16 rows x 64 columns each, straight from the cache into the swizzled operand tiles
//
// Tensor memory: scores / weights of the streams 2 x 128 columns, outputs 2 x 128.  The output is only rescaled when a row's maximum
// has grown by more than 2^8 since the last time; until then weights are relative to the older maximum.  All waits are bounded.
#include "mixers_common.cuh"
#include "tc5_common.cuh"

namespace ob {

namespace {

constexpr uint32_t PT_ROWS = 128, PT_KEYS = 128, PT_PAGES = PT_KEYS / KV_PAGE, PT_BLOCK = PT_KEYS * 128;  // block: 128 rows of 64 columns
constexpr int PT_SOFTMAX_WARPS = 16, PT_MMA_WARP = 16, PT_TMA_WARP = 17, PT_THREADS = 18 * 32;
constexpr uint32_t PT_TMEM_S = 0, PT_TMEM_O = 256, PT_TMEM_COLS = 512;
constexpr float PT_SLACK = 8.0f;  // growth of the maximum (powers of two) that is put up with

constexpr uint32_t PT_SHARED = 256 + 2 * 2 * PT_ROWS * 4;  // mbarriers, then a number per stream, half and row
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
constexpr uint32_t PT_K_FULL = 0, PT_K_EMPTY = 16, PT_V_FULL = 32, PT_V_EMPTY = 48, PT_S_FULL = 64, PT_P_FULL = 80, PT_O_FULL = 96, PT_Q_FULL = 112, PT_SLOT = 120, PT_ABORT = 124,
                   PT_INFO = 128, PT_EXCHANGE = 256;

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

// Entries [c, c + 16) of a head's output, gated, as activations.
__device__ __forceinline__ void store_head(const AttentionArgs &a, uint64_t t, uint32_t h, uint32_t c, float (&x)[16]) {
    bf16 *out = static_cast<bf16 *>(a.out) + t * a.out_pitch + (uint64_t)h * a.vdim + c;
    const bf16 *gate = static_cast<const bf16 *>(a.va) + t * a.va_pitch + a.gate0 + (uint64_t)h * a.vdim + c;
#pragma unroll
    for (uint32_t b = 0; b < 2; ++b) {
        float(&v)[8] = *reinterpret_cast<float(*)[8]>(x + 8 * b);
        if (a.vdim % 8 == 0) {
            if (c + 8 * b >= a.vdim) return;
            if (a.has_gate) {
                const uint4 z = *reinterpret_cast<const uint4 *>(gate + 8 * b);
                const uint32_t zw[4] = {z.x, z.y, z.z, z.w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    v[2 * e] /= 1.0f + expf(-__uint_as_float(zw[e] << 16));
                    v[2 * e + 1] /= 1.0f + expf(-__uint_as_float(zw[e] & 0xffff0000u));
                }
            }
            store4<bf16>(out + 8 * b, make_float4(v[0], v[1], v[2], v[3]));
            store4<bf16>(out + 8 * b + 4, make_float4(v[4], v[5], v[6], v[7]));
        } else {
#pragma unroll
            for (uint32_t e = 0; e < 8; ++e)
                if (c + 8 * b + e < a.vdim) out[8 * b + e] = __float2bfloat16_rn(a.has_gate ? v[e] / (1.0f + expf(-from_act(gate[8 * b + e]))) : v[e]);
        }
    }
}

template <int NM>
__global__ void __launch_bounds__(PT_THREADS, 1) attention_prompt_kernel(const __grid_constant__ CUtensorMap tm, const __grid_constant__ AttentionArgs a) {
    constexpr uint32_t M = NM == 2 ? PT_ROWS : 2 * PT_ROWS;  // rows of the CTA
    extern __shared__ uint8_t smem_raw[];
    const uint32_t sbase = (smem_u32(smem_raw) + 1023u) & ~1023u;
    uint8_t *smem = smem_raw + (sbase - smem_u32(smem_raw));
    const PtPlan pl(NM, a.dim_p, a.vdim_p);
    const uint32_t bar = sbase + pl.bar, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = blockIdx.y, per = a.n_head / a.n_kv;
    volatile uint32_t *abort = reinterpret_cast<volatile uint32_t *>(smem + pl.bar + PT_ABORT);
    volatile uint32_t *info = reinterpret_cast<volatile uint32_t *>(smem + pl.bar + PT_INFO);
    if (threadIdx.x == 0) {
        for (uint32_t s = 0; s < 2; ++s) {
            mbar_init(bar + PT_K_FULL + 8 * s, 1);
            mbar_init(bar + PT_K_EMPTY + 8 * s, 1);
            mbar_init(bar + PT_V_FULL + 8 * s, 1);
            mbar_init(bar + PT_V_EMPTY + 8 * s, 1);
            mbar_init(bar + PT_S_FULL + 8 * s, 1);
            mbar_init(bar + PT_P_FULL + 8 * s, 8);
            mbar_init(bar + PT_O_FULL + 8 * s, 1);
        }
        mbar_init(bar + PT_Q_FULL, PT_SOFTMAX_WARPS);
        *abort = 0u;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
        asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
    }
    if (warp == PT_MMA_WARP) tmem_alloc(bar + PT_SLOT, PT_TMEM_COLS);
    pdl_wait();
    if (warp == 0) {
        RowSpan sp;
        uint32_t f;
        // (the last rows of a span see the most keys: they start first)
        find_tile(a.spans + a.n_short, a.n_seq - a.n_short, per, M, gridDim.x - 1 - blockIdx.x, &sp, &f);
        if (lane == 0) info[0] = sp.row0, info[1] = sp.n, info[2] = f;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    pdl_release();  // (only now: a CTA of the next kernel must not take the tensor memory first, it would keep it until this grid is done)
    const uint32_t tmem = *reinterpret_cast<volatile uint32_t *>(smem + pl.bar + PT_SLOT);
    const uint32_t row0 = info[0], f0 = info[2], n_flat = info[1] * per;
    const uint32_t n_here = f0 < n_flat ? min(M, n_flat - f0) : 0, pos0 = a.positions[row0];
    const int32_t *table = a.tables[row0];
    const uint32_t lo = first_seen(pos0 + f0 / per, a.window), hi = pos0 + (f0 + max(n_here, 1u) - 1) / per + 1;
    const uint32_t page0 = lo / KV_PAGE, n_page = (hi + KV_PAGE - 1) / KV_PAGE - page0, n_tiles = n_here ? (n_page + PT_PAGES - 1) / PT_PAGES : 0;
    // tiles of keys that a stream's rows see: [first_tile, end_tile)
    auto first_tile = [&](uint32_t s) {
        return NM == 2 || s == 0 || s * PT_ROWS >= n_here ? 0u : (first_seen(pos0 + (f0 + s * PT_ROWS) / per, a.window) / KV_PAGE - page0) / PT_PAGES;
    };
    auto end_tile = [&](uint32_t s) {
        if (NM == 2 || s == 1) return s * PT_ROWS * (NM == 1) < n_here ? n_tiles : 0u;
        return n_here ? ((pos0 + (f0 + min(n_here, PT_ROWS) - 1) / per) / KV_PAGE - page0) / PT_PAGES + 1 : 0u;
    };

    if (warp == PT_TMA_WARP) {
        if (lane == 0) {
            for (uint32_t i = 0; i < n_tiles; ++i) {
                const uint32_t st = i % pl.stages, par = ((i / pl.stages) & 1u) ^ 1u;
                int32_t y[PT_PAGES];
#pragma unroll
                for (uint32_t p = 0; p < PT_PAGES; ++p)  // past the last page: the last one again, which nobody sees there
                    y[p] = (int32_t)((table[page0 + min(i * PT_PAGES + p, n_page - 1)] * a.n_kv + g) * KV_PAGE);
                if (i >= pl.stages && !mbar_wait(bar + PT_K_EMPTY + 8 * st, par, abort)) break;
                mbar_expect_tx(bar + PT_K_FULL + 8 * st, pl.k_bytes);
                for (uint32_t b = 0; b < NM * pl.nb; ++b) {
                    const int32_t x = (int32_t)(b / pl.nb * a.dim_p + b % pl.nb * 64);
#pragma unroll
                    for (uint32_t p = 0; p < PT_PAGES; ++p)
                        tma_load_2d(sbase + pl.k + st * pl.k_bytes + b * PT_BLOCK + p * (KV_PAGE * 128), &tm, x, y[p], bar + PT_K_FULL + 8 * st);
                }
                if (i >= pl.stages && !mbar_wait(bar + PT_V_EMPTY + 8 * st, par, abort)) break;
                mbar_expect_tx(bar + PT_V_FULL + 8 * st, pl.v_bytes);
                for (uint32_t b = 0; b < pl.nbv; ++b) {
                    const int32_t x = (int32_t)(NM * a.dim_p + b * 64);
#pragma unroll
                    for (uint32_t p = 0; p < PT_PAGES; ++p)
                        tma_load_2d(sbase + pl.v + st * pl.v_bytes + b * PT_BLOCK + p * (KV_PAGE * 128), &tm, x, y[p], bar + PT_V_FULL + 8 * st);
                }
            }
        }
    } else if (warp == PT_MMA_WARP) {
        const uint32_t t0_0 = first_tile(0), t0_1 = first_tile(1), t1_0 = end_tile(0), t1_1 = end_tile(1);
        if (lane == 0 && n_tiles && mbar_wait(bar + PT_Q_FULL, 0, abort)) {
            const uint32_t id_s = umma_idesc_bf16(PT_KEYS), id_o = umma_idesc_bf16(a.vdim_p) | UMMA_B_MN_MAJOR, k_steps = a.dim_p / 16;
            auto scores = [&](uint32_t s, uint32_t i) {
                const uint32_t st = i % pl.stages;
                if (!mbar_wait(bar + PT_K_FULL + 8 * st, (i / pl.stages) & 1u, abort)) return false;
                tc_fence_after();
                const uint32_t qa = sbase + s * pl.nb * PT_BLOCK, ka = sbase + pl.k + st * pl.k_bytes + (NM == 2 ? s * pl.nb * PT_BLOCK : 0);
                for (uint32_t k = 0; k < k_steps; ++k)
                    umma_bf16(tmem + PT_TMEM_S + s * PT_KEYS, umma_desc_sw128(qa + k / 4 * PT_BLOCK) + 2 * (k % 4), umma_desc_sw128(ka + k / 4 * PT_BLOCK) + 2 * (k % 4), id_s, k ? 1u : 0u);
                umma_commit(bar + PT_S_FULL + 8 * s);
                return true;
            };
            bool ok = true;
            for (uint32_t s = 0; s < 2 && ok; ++s)
                if ((s ? t0_1 : t0_0) == 0 && (s ? t1_1 : t1_0) > 0) ok = scores(s, 0);
            if (ok) umma_commit(bar + PT_K_EMPTY);
            for (uint32_t i = 0; i < n_tiles && ok; ++i) {
                const uint32_t st = i % pl.stages;
#pragma unroll 1
                for (uint32_t s = 0; s < 2 && ok; ++s) {
                    const uint32_t t0 = s ? t0_1 : t0_0, t1 = s ? t1_1 : t1_0;
                    if (i >= t0 && i < t1) {
                        if (!(ok = mbar_wait(bar + PT_P_FULL + 8 * s, (i - t0) & 1u, abort) && mbar_wait(bar + PT_V_FULL + 8 * st, (i / pl.stages) & 1u, abort))) break;
                        tc_fence_after();
                        const uint32_t p = tmem + PT_TMEM_S + s * PT_KEYS, d = tmem + PT_TMEM_O + s * 128;
                        const uint64_t vd = umma_desc_sw128_mn(sbase + pl.v + st * pl.v_bytes, PT_BLOCK);
#pragma unroll
                        for (uint32_t kk = 0; kk < PT_KEYS / 16; ++kk) {  // 16 keys: value, then remainder
                            umma_bf16_ta(d, p + kk * 16, vd + kk * 128, id_o, i > t0 || kk ? 1u : 0u);
                            umma_bf16_ta(d, p + kk * 16 + 8, vd + kk * 128, id_o, 1u);
                        }
                        if (i + 1 == t1) umma_commit(bar + PT_O_FULL + 8 * s);
                    }
                    if (i + 1 >= t0 && i + 1 < t1) ok = scores(s, i + 1);
                }
                if (!ok) break;
                umma_commit(bar + PT_V_EMPTY + 8 * st);
                if (i + 1 < n_tiles) umma_commit(bar + PT_K_EMPTY + 8 * ((i + 1) % pl.stages));
            }
        }
    } else {
        const uint32_t s = warp / 8, part = warp / 4 % 2, quad = warp % 4, r = quad * 32 + lane, i_row = (NM == 2 ? 0 : s * PT_ROWS) + r;  // row within the CTA
        const bool live = i_row < n_here;
        const uint32_t t0 = first_tile(s), t1 = end_tile(s), pair = 1 + s * 4 + quad;
        const uint32_t f = f0 + (live ? i_row : 0), h = g * per + f % per;
        const uint64_t t = row0 + f / per;
        const int pos = live ? (int)(pos0 + f / per) : -1, win = a.window ? (int)min(a.window, 0x3fffffffu) : 0x3fffffff;
        volatile float *xchg = reinterpret_cast<volatile float *>(smem + pl.bar + PT_EXCHANGE) + s * 2 * PT_ROWS + r;  // own half at part * PT_ROWS, the other's beside it
        {   // the row's query into the swizzled operand tile
            const bf16 *q = static_cast<const bf16 *>(a.q) + ((t * a.n_head + h) * NM + (NM == 2 ? s : 0)) * a.dim_p;
            uint8_t *dst = smem + s * pl.nb * PT_BLOCK + r * 128;
            for (uint32_t c = part; c < a.dim_p / 8; c += 2)
                *reinterpret_cast<uint4 *>(dst + c / 8 * PT_BLOCK + (((c & 7) ^ (r & 7)) << 4)) = live ? *reinterpret_cast<const uint4 *>(q + 8 * c) : make_uint4(0, 0, 0, 0);
            asm volatile("fence.proxy.async.shared::cta;" ::: "memory");
            __syncwarp();
            if (lane == 0) mbar_arrive(bar + PT_Q_FULL);
        }
        const float scale2 = a.scale * 1.4426950408889634f;  // weights are powers of two of the scaled score
        const uint32_t lanes = tmem + ((quad * 32) << 16), ts = lanes + PT_TMEM_S + s * PT_KEYS + part * 64, to = lanes + PT_TMEM_O + s * 128;
        // first and last position of the warp's rows (dead rows do not count)
        const uint32_t w0 = (NM == 2 ? 0 : s * PT_ROWS) + quad * 32;
        const bool whole = w0 + 32 <= n_here;
        const int w_first = (int)(pos0 + (f0 + w0) / per), w_last = (int)(pos0 + (f0 + w0 + 31) / per);
        float m = -INFINITY, l = 0.0f;
        bool ok = true;
        for (uint32_t i = t0; i < t1; ++i) {
            ok = ok && __all_sync(0xffffffffu, mbar_wait(bar + PT_S_FULL + 8 * s, (i - t0) & 1u, abort));
            if (!ok) {  // a wait was given up: nothing more is computed, but the other half's barriers are kept company
                pair_sync(pair);
                continue;
            }
            tc_fence_after();
            const int j0 = (int)((page0 + i * PT_PAGES) * KV_PAGE + part * 64);
            const bool masked = !(whole && j0 + 63 <= w_first && w_last - j0 < win);  // keys outside the window of some row
            const int last = pos - j0, first = last - win + 1;                        // visible columns (pos -1: none)
            uint32_t u[2][32];
            tmem_ld32(ts, u[0]);
            tmem_ld32(ts + 32, u[1]);
            tmem_ld_wait();
            if (masked) {
#pragma unroll
                for (int c = 0; c < 2; ++c)
#pragma unroll
                    for (int e = 0; e < 32; ++e)
                        if (c * 32 + e > last || c * 32 + e < first) u[c][e] = 0xff800000u;
            }
            float top[4] = {-INFINITY, -INFINITY, -INFINITY, -INFINITY};
#pragma unroll
            for (int c = 0; c < 2; ++c)
#pragma unroll
                for (int e = 0; e < 32; ++e) top[e % 4] = fmaxf(top[e % 4], __uint_as_float(u[c][e]));
            const float own = fmaxf(fmaxf(top[0], top[1]), fmaxf(top[2], top[3])) * scale2;
            xchg[part * PT_ROWS] = own;
            pair_sync(pair);
            const float now = fmaxf(own, xchg[(part ^ 1u) * PT_ROWS]);
            const bool grown = m > -INFINITY && now > m + PT_SLACK;
            if (__any_sync(0xffffffffu, grown)) {  // the product before this tile's scores is done: the output may be rescaled
                const float keep = grown ? pow2(m - now) : 1.0f;
                if (grown) m = now, l *= keep;
                for (uint32_t c = 16 * part; c < a.vdim_p; c += 32) {
                    uint32_t o[16];
                    tmem_ld16(to + c, o);
                    tmem_ld_wait();
#pragma unroll
                    for (int e = 0; e < 16; ++e) o[e] = __float_as_uint(__uint_as_float(o[e]) * keep);
                    tmem_st16(to + c, o);
                }
            }
            if (m == -INFINITY) m = now;
            const float base = m == -INFINITY ? 0.0f : -m;  // a row that has seen nothing yet keeps weights of zero
            float sum0 = 0.0f, sum1 = 0.0f;
#pragma unroll
            for (int c = 0; c < 4; ++c) {  // 16 keys: eight columns of values, eight of remainders
                uint32_t w[16];
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
                    w[e] = hw, w[8 + e] = *reinterpret_cast<const uint32_t *>(&lo2);
                }
                tmem_st16(ts + 16 * c, w);
            }
            l += sum0 + sum1;
            tmem_st_wait();
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(bar + PT_P_FULL + 8 * s);
        }
        if (ok && t1 > t0) ok = mbar_wait(bar + PT_O_FULL + 8 * s, 0, abort);
        tc_fence_after();
        ok = __all_sync(0xffffffffu, ok) && t1 > t0;
        pair_sync(pair);
        xchg[part * PT_ROWS] = l;
        pair_sync(pair);
        const float fac = 1.0f / (l + xchg[(part ^ 1u) * PT_ROWS]);
        float gain = fac;
        float *ex = reinterpret_cast<float *>(smem + pl.k) + r * (a.vdim_p + 4);  // [128 rows]: the second map's share
        auto output = [&](uint32_t c, float (&x)[16]) {  // entries [c, c + 16) of the row's output
            uint32_t o[16];
            tmem_ld16(to + c, o);
            tmem_ld_wait();
#pragma unroll
            for (int e = 0; e < 16; ++e) x[e] = __uint_as_float(o[e]) * fac;
        };
        if constexpr (NM == 2) {
            if (s == 1 && ok) {
                for (uint32_t c = 16 * part; c < a.vdim_p; c += 32) {
                    float x[16];
                    output(c, x);
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        *reinterpret_cast<float4 *>(ex + c + 4 * e) = mul4(make_float4(x[4 * e], x[4 * e + 1], x[4 * e + 2], x[4 * e + 3]), a.map_weight);
                }
            }
            asm volatile("bar.sync 9, 512;" ::: "memory");
            float q = 0.0f;
            if (s == 0 && ok) {
                for (uint32_t c = 16 * part; c < a.vdim_p; c += 32) {
                    float x[16];
                    output(c, x);
#pragma unroll
                    for (int e = 0; e < 16; ++e) {  // columns past vdim are zero: so are the values there
                        const float d = x[e] - ex[c + e];
                        q += d * d;
                    }
                }
            }
            xchg[part * PT_ROWS] = q;  // (both have read the sums: the barrier above)
            pair_sync(pair);
            gain = inv_rms(q + xchg[(part ^ 1u) * PT_ROWS], a.vdim, a.eps) * a.head_gain;
        }
        if (ok && (NM == 1 || s == 0)) {
            for (uint32_t c = 16 * part; c < a.vdim_p; c += 32) {
                float x[16];
                output(c, x);
                if constexpr (NM == 2) {
#pragma unroll
                    for (int e = 0; e < 16; ++e) x[e] = (x[e] - ex[c + e]) * gain;
                }
                if (live) store_head(a, t, h, c, x);
            }
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
        cudaError_t e = cudaFuncSetAttribute(attention_prompt_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
        return e != cudaSuccess ? e : cudaFuncSetAttribute(attention_prompt_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024);
    });
}

bool attention_prompt_supported(uint32_t n_map, uint32_t dim_p, uint32_t vdim_p) { return vdim_p <= 128 && PtPlan(n_map, dim_p, vdim_p).stages > 0; }

bool launch_attention_prompt(const AttentionArgs &a, cudaStream_t st) {
    const uint32_t per = a.n_head / a.n_kv, M = a.n_map == 2 ? PT_ROWS : 2 * PT_ROWS;
    uint32_t tiles = 0;
    for (uint32_t s = a.n_short; s < a.n_seq; ++s) tiles += (a.h_spans[s].n * per + M - 1) / M;
    CUtensorMap tm;
    if (!make_map_2d(&tm, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, a.cache, a.row, (uint64_t)a.n_pages * a.n_kv * KV_PAGE, (uint64_t)a.row * 2, 64, KV_PAGE, CU_TENSOR_MAP_SWIZZLE_128B)) return false;
    const PtPlan pl(a.n_map, a.dim_p, a.vdim_p);
    launch_pdl(a.n_map == 2 ? attention_prompt_kernel<2> : attention_prompt_kernel<1>, dim3(tiles, a.n_kv), PT_THREADS, pl.bytes, st, tm, a);
    g_tc5_launched.store(true, std::memory_order_relaxed);
    return true;
}

int attention_take_status() { return tc5_take_status(); }

}  // namespace ob
