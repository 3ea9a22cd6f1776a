// Between two sublayers of a block that adds their outputs as they are: the output joins the residual, a layer's result is averaged
// with the results of the layers before it, the sum is normed in groups, and a short causal convolution over time is added to it.
// One kernel makes all of it, so what the next sublayer reads is written once:
//   s = x + mult * (rows of y of the token)        or the token's embedding
//   v = depth[n] s + sum_j depth[j] history[j]     or s
//   n = v over the root mean square of its group, times the norm's factors
//   h = n + sum_k conv[k] n of the token taps - 1 - k before
// The last taps - 1 rows n of a sequence are its state.
//
// residual_run_kernel   a CTA takes consecutive tokens of a span with the rows n the convolution reaches back to in registers; it
//                       makes the ones before its first token again (nothing it reads is overwritten: sums go elsewhere)
// residual_row_kernel   any width, group and number of taps: a CTA per token up to n, then the convolution (recurrence.cu)
#include <algorithm>

#include "mixers_common.cuh"

namespace ob {

namespace {

__device__ __forceinline__ float4 add4(float4 a, float4 b) { return make_float4(a.x + b.x, a.y + b.y, a.z + b.z, a.w + b.w); }
__device__ __forceinline__ float4 fma4(float f, float4 a, float4 b) { return make_float4(fmaf(f, a.x, b.x), fmaf(f, a.y, b.y), fmaf(f, a.z, b.z), fmaf(f, a.w, b.w)); }
__device__ __forceinline__ float4 fma44(float4 a, float4 b, float4 c) { return make_float4(fmaf(a.x, b.x, c.x), fmaf(a.y, b.y, c.y), fmaf(a.z, b.z, c.z), fmaf(a.w, b.w, c.w)); }
__device__ __forceinline__ float4 bf16x4(const bf16 *p) {
    const uint2 u = *reinterpret_cast<const uint2 *>(p);
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16), __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ float4 f4(const float *p) { return *reinterpret_cast<const float4 *>(p); }

// Squares are summed in units: a warp's 128 columns when groups consist of such, else a thread's four.
__host__ __device__ constexpr uint32_t unit_columns(uint32_t group) { return group % 128 ? 4 : 128; }

// NV: float4 of a thread; TAPS: of the convolution, 0: none.
template <typename TA, int NV, int TAPS>
__global__ void __launch_bounds__(1024) residual_run_kernel(ResidualArgs a, uint32_t run) {
    extern __shared__ float sm[];
    constexpr int BACK = TAPS > 1 ? TAPS - 1 : 0;
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5;
    const uint32_t group = a.width / a.n_group, unit = unit_columns(group), per_group = group / unit;
    float *units = sm, *inv = sm + a.width / unit;
    pdl_release();
    pdl_wait();
    RowSpan sp{blockIdx.x, 1};
    uint32_t f0 = 0;
    if (run > 1) find_tile(a.spans, a.n_seq, 1, run, blockIdx.x, &sp, &f0);
    if (f0 >= sp.n) return;
    if (a.zero && blockIdx.x == 0)
        for (uint32_t i = threadIdx.x; i < a.n_zero; i += blockDim.x) a.zero[i] = 0;
    const int n = (int)sp.n, first = (int)f0, last = min(first + (int)run, n);
    float *state = nullptr;
    bool fresh = true;
    if (BACK) {
        state = a.state + (uint64_t)a.slots[sp.row0] * BACK * a.width;
        fresh = a.positions[sp.row0] == 0;
    }
    auto col = [&](int i) { return 4 * (threadIdx.x + i * blockDim.x); };
    // The row before the norm; stored where the token is this CTA's own.
    auto value = [&](uint32_t t, bool own, float4 (&v)[NV]) {
        const uint64_t at = (uint64_t)t * a.width;
        const float *x = a.x ? a.x + (uint64_t)(a.x_rows ? a.x_rows[t] : t) * a.width : nullptr;
        const bf16 *e = a.x ? nullptr : a.table + (uint64_t)a.tokens[t] * a.width;
        const float last_weight = a.depth ? a.depth[a.n_history] : 1.0f;
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = col(i);
            v[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
            if (c >= a.width) continue;
            v[i] = x ? f4(x + c) : bf16x4(e + c);
            if (a.y) {
                float4 y = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
#pragma unroll 4
                for (uint32_t k = 0; k < a.top; ++k) {
                    const uint32_t p = t * a.top + k;
                    y = add4(y, f4(a.y + (uint64_t)(a.rows ? a.rows[p] : p) * a.width + c));
                }
                v[i] = fma4(a.mult, y, v[i]);
            }
            if (own && a.sum) *reinterpret_cast<float4 *>(a.sum + at + c) = v[i];
            if (a.depth) {
                float4 s = mul4(v[i], last_weight);
#pragma unroll 8
                for (uint32_t j = 0; j < a.n_history; ++j) s = fma4(a.depth[j], f4(a.history + j * a.history_step + at + c), s);
                v[i] = s;
                if (own && a.average) *reinterpret_cast<float4 *>(a.average + at + c) = s;
            }
        }
    };
    auto normed = [&](float4 (&v)[NV]) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = col(i);
            const float s = sq4(v[i]);
            if (unit == 128) {
                const float w = warp_sum(s);
                if (lane == 0 && c < a.width) units[c / 128] = w;
            } else if (c < a.width) {
                units[c / 4] = s;
            }
        }
        __syncthreads();
        for (uint32_t g = warp; g < a.n_group; g += warps) {
            float s = 0.0f;
            for (uint32_t u = lane; u < per_group; u += 32) s += units[g * per_group + u];
            s = warp_sum(s);
            if (lane == 0) inv[g] = inv_rms(s, group, a.eps);
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = col(i);
            if (c < a.width) v[i] = mul44(mul4(v[i], inv[c / group]), f4(a.norm + c));
        }
    };
    float4 ring[BACK > 0 ? BACK : 1][NV];  // the rows n before the current one, the oldest first
    auto push = [&](const float4 (&v)[NV]) {
        if constexpr (BACK > 0) {
#pragma unroll
            for (int i = 0; i < NV; ++i) {
#pragma unroll
                for (int k = 0; k + 1 < BACK; ++k) ring[k][i] = ring[k + 1][i];
                ring[BACK - 1][i] = v[i];
            }
        }
    };
    TA *h = static_cast<TA *>(a.h);
    for (int t = first - BACK; t < last; ++t) {
        float4 v[NV];
        if (t < 0) {
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const uint32_t c = col(i);
                v[i] = fresh || c >= a.width ? make_float4(0.0f, 0.0f, 0.0f, 0.0f) : f4(state + (uint64_t)(t + BACK) * a.width + c);
            }
        } else {
            value(sp.row0 + t, t >= first, v);
            if (!a.norm) continue;
            normed(v);
        }
        if (t >= first) {
#pragma unroll
            for (int i = 0; i < NV; ++i) {
                const uint32_t c = col(i);
                if (c >= a.width) continue;
                float4 o = v[i];
                if constexpr (TAPS > 0) {
                    const float *w = a.conv + c;  // [taps][width]
                    o = fma44(f4(w + (uint64_t)BACK * a.width), v[i], o);
#pragma unroll
                    for (int k = 0; k < BACK; ++k) o = fma44(f4(w + (uint64_t)k * a.width), ring[k][i], o);
                }
                store4<TA>(h + (uint64_t)(sp.row0 + t) * a.h_pitch + c, o);
            }
        }
        push(v);
    }
    if constexpr (BACK > 0) {
        if (first > 0) return;  // the CTA that has read the state replaces it
        if (n > last)           // (a run is not shorter than the convolution reaches back)
            for (int t = n - BACK; t < n; ++t) {
                float4 v[NV];
                value(sp.row0 + t, false, v);
                normed(v);
                push(v);
            }
#pragma unroll
        for (int i = 0; i < NV; ++i)
            if (col(i) < a.width)
#pragma unroll
                for (int k = 0; k < BACK; ++k) *reinterpret_cast<float4 *>(state + (uint64_t)k * a.width + col(i)) = ring[k][i];
    }
}

template <typename TA>
__global__ void __launch_bounds__(512) residual_row_kernel(ResidualArgs a) {
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    if (a.zero && blockIdx.x == 0)
        for (uint32_t i = threadIdx.x; i < a.n_zero; i += blockDim.x) a.zero[i] = 0;
    const uint32_t t = blockIdx.x, group = a.width / a.n_group;
    const uint64_t at = (uint64_t)t * a.width;
    auto value = [&](uint32_t c, bool store) {
        float v = a.x ? a.x[(uint64_t)(a.x_rows ? a.x_rows[t] : t) * a.width + c] : __bfloat162float(a.table[(uint64_t)a.tokens[t] * a.width + c]);
        if (a.y) {
            float y = 0.0f;
            for (uint32_t k = 0; k < a.top; ++k) {
                const uint32_t p = t * a.top + k;
                y += a.y[(uint64_t)(a.rows ? a.rows[p] : p) * a.width + c];
            }
            v = fmaf(a.mult, y, v);
        }
        float s = v;
        if (a.depth) {
            s = v * a.depth[a.n_history];
            for (uint32_t j = 0; j < a.n_history; ++j) s = fmaf(a.depth[j], a.history[j * a.history_step + at + c], s);
        }
        if (store) {
            if (a.sum) a.sum[at + c] = v;
            if (a.depth && a.average) a.average[at + c] = s;
        }
        return s;
    };
    for (uint32_t g = 0; g < a.n_group; ++g) {
        float s = 0.0f;
        for (uint32_t c = g * group + threadIdx.x; a.norm && c < (g + 1) * group; c += blockDim.x) {
            const float v = value(c, false);
            s += v * v;
        }
        const float f = a.norm ? inv_rms(block_sum(s, red), group, a.eps) : 0.0f;
        for (uint32_t c = g * group + threadIdx.x; c < (g + 1) * group; c += blockDim.x) {  // (a sum may replace its own x)
            const float v = value(c, true);
            if (!a.norm) continue;
            if (a.taps) a.normed[at + c] = v * f * a.norm[c];
            else static_cast<TA *>(a.h)[(uint64_t)t * a.h_pitch + c] = to_act<TA>(v * f * a.norm[c]);
        }
    }
}

constexpr uint32_t RUN_MAX_TAPS = 4, RUN_MAX = 32;

template <typename TA, int NV>
void run_form(const ResidualArgs &a, uint32_t grid, uint32_t threads, uint32_t run, size_t smem, cudaStream_t st) {
    auto launch = [&](void (*k)(ResidualArgs, uint32_t)) { launch_pdl(k, grid, threads, smem, st, a, run); };
    switch (a.norm ? a.taps : 0) {
    case 0: launch(residual_run_kernel<TA, NV, 0>); break;
    case 1: launch(residual_run_kernel<TA, NV, 1>); break;
    case 2: launch(residual_run_kernel<TA, NV, 2>); break;
    case 3: launch(residual_run_kernel<TA, NV, 3>); break;
    default: launch(residual_run_kernel<TA, NV, 4>); break;
    }
}

template <typename TA>
uint32_t residual(const ResidualArgs &a, bool f32, int sm_count, cudaStream_t st) {
    const uint32_t group = a.width / a.n_group, taps = a.norm ? a.taps : 0;
    if (a.width % 4 == 0 && group % 4 == 0 && a.width <= 8192 && taps <= RUN_MAX_TAPS) {
        // as many tokens per CTA as give every SM two CTAs
        uint32_t run = 1, grid = a.T;
        if (!a.single && taps > 1) {
            run = std::min(RUN_MAX, std::max(RUN_MAX_TAPS, (a.T + 2 * (uint32_t)sm_count - 1) / (2 * (uint32_t)sm_count)));
            grid = 0;
            for (uint32_t s = 0; s < a.n_seq; ++s) grid += (a.h_spans[s].n + run - 1) / run;
        }
        const uint32_t nv = a.width > 4096 ? 2 : 1, threads = (a.width / 4 / nv + 31) / 32 * 32;
        const size_t smem = (a.width / unit_columns(group) + a.n_group) * sizeof(float);
        if (nv == 1) run_form<TA, 1>(a, grid, threads, run, smem, st);
        else run_form<TA, 2>(a, grid, threads, run, smem, st);
        return 1;
    }
    launch_pdl(residual_row_kernel<TA>, a.T, 512, 0, st, a);
    if (!taps) return 1;
    ConvArgs c{};
    c.y = a.normed;
    c.y_pitch = c.n_channel = a.width;
    c.taps = taps;
    c.w = a.conv;
    c.tap_step = a.width;
    c.state = a.state;
    c.h = a.h;
    c.h_pitch = a.h_pitch;
    c.T = a.T;
    c.n_seq = a.n_seq;
    c.spans = a.spans;
    c.h_spans = a.h_spans;
    c.single = a.single;
    c.positions = a.positions;
    c.slots = a.slots;
    launch_conv(c, f32, st);
    return 2;
}

}  // namespace

uint32_t launch_residual(const ResidualArgs &a, bool f32, int sm_count, cudaStream_t st) {
    return f32 ? residual<float>(a, f32, sm_count, st) : residual<bf16>(a, f32, sm_count, st);
}

}  // namespace ob
