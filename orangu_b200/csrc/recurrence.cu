// Recurrent layers with data-dependent decay: the state recurrence itself, the short convolution and step sizes of a state-space
// layer, the token shift of a time-mixing layer, and what follows the recurrence in either.
//
//   recurrence_kernel       decoded tokens and short spans, bound by the state's traffic: a warp has a few rows of the state, a lane a column
//   recurrence_span_kernel  long spans, bound by fp32 arithmetic: a lane has neighbouring rows, two of them per packed instruction
// Everything is fp32; the state goes token by token, so a result does not depend on how a sequence was cut.
#include <algorithm>

#include "mixers_common.cuh"

namespace ob {

namespace {

__device__ __forceinline__ void cp4(float *dst, const float *src, bool in) {  // 4 bytes, or zero
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(in ? 4 : 0) : "memory");
}
__device__ __forceinline__ void cp8(void *dst, const void *src, bool in) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(smem_addr(dst)), "l"(src), "r"(in ? 8 : 0) : "memory");
}
__device__ __forceinline__ float silu(float z) { return z / (1.0f + expf(-z)); }

// ---- decoded tokens and short spans ---------------------------------------------------------------------------------------------
// One CTA carries 32 columns of one head's state through the rows of one sequence: lane = column, warp = DW of the state's rows,
// kept in registers.  The warps' parts of the outputs are added up once per block of tokens, while the next block's operands are on
// their way to shared memory.
template <int DW, bool KEYED>  // KEYED: a decay per key entry, outputs before the update
struct RcPlan {
    static constexpr int D = 8 * DW, BLOCK = DW > 16 ? 8 : 16;
    static constexpr uint32_t Q = 0, K = Q + BLOCK * D, W = K + BLOCK * D, V = W + (KEYED ? BLOCK * D : 0), A = V + BLOCK * 32, STAGE = A + 2 * BLOCK,
                              PART = 2 * STAGE, FLOATS = PART + 8 * BLOCK * 32;
};
template <int DW, bool KEYED>
__global__ void __launch_bounds__(256) recurrence_kernel(RecurrenceArgs a) {
    using R = RcPlan<DW, KEYED>;
    constexpr int D = R::D, BLOCK = R::BLOCK;
    extern __shared__ __align__(16) float sm[];
    float *part = sm + R::PART;  // [8][BLOCK][32]
    pdl_release();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, col = blockIdx.x * 32 + lane;
    const RowSpan sp = a.spans[blockIdx.z];
    const bool live = col < a.vdim;
    float *state = a.state + (((uint64_t)a.slots[sp.row0] * a.n_head + h) * a.dim) * a.vdim + col;
    const uint64_t row0 = (uint64_t)sp.row0 * a.pitch;
    const float *gq = a.q + row0 + (uint64_t)(h / a.share) * a.dim, *gk = a.k + row0 + (uint64_t)(h / a.share) * a.dim;
    const float *gv = a.v + row0 + (uint64_t)h * a.vdim + col, *gw = KEYED ? a.w + (uint64_t)sp.row0 * a.w_pitch + (uint64_t)h * a.dim : nullptr;
    const float2 *ga = KEYED ? nullptr : a.step + (uint64_t)sp.row0 * a.n_head + h;
    auto load = [&](uint32_t t0, uint32_t stage) {
        float *s = sm + stage * R::STAGE;
        const uint32_t n = min((uint32_t)BLOCK, sp.n - t0);
        for (uint32_t i = threadIdx.x; i < n * D; i += 256) {
            const uint32_t t = i / D, d = i % D;
            const bool in = d < a.dim;
            const uint64_t o = (uint64_t)(t0 + t) * a.pitch + (in ? d : 0);
            cp4(s + R::Q + i, gq + o, in);
            cp4(s + R::K + i, gk + o, in);
            if constexpr (KEYED) cp4(s + R::W + i, gw + (uint64_t)(t0 + t) * a.w_pitch + (in ? d : 0), in);
        }
        for (uint32_t t = warp; t < n; t += 8) cp4(s + R::V + t * 32 + lane, live ? gv + (uint64_t)(t0 + t) * a.pitch : a.v, live);
        if constexpr (!KEYED)
            if (threadIdx.x < n) cp8(s + R::A + 2 * threadIdx.x, ga + (uint64_t)(t0 + threadIdx.x) * a.n_head, true);
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
        const float *base = sm + stage * R::STAGE, *q = base + R::Q + warp * DW, *k = base + R::K + warp * DW, *w = base + R::W + warp * DW, *v = base + R::V + lane;
        for (uint32_t t = 0; t < n; ++t) {
            float vv = v[t * 32], decay = 0.0f;
            if constexpr (!KEYED) {
                const float2 st = *reinterpret_cast<const float2 *>(base + R::A + 2 * t);
                decay = st.x;
                vv *= st.y;
            }
            float o[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
            for (int i = 0; i < DW; i += 4) {
                const float4 k4 = *reinterpret_cast<const float4 *>(k + t * D + i), q4 = *reinterpret_cast<const float4 *>(q + t * D + i);
                const float kk[4] = {k4.x, k4.y, k4.z, k4.w}, qq[4] = {q4.x, q4.y, q4.z, q4.w};
                float ww[4] = {decay, decay, decay, decay};
                if constexpr (KEYED) {
                    const float4 w4 = *reinterpret_cast<const float4 *>(w + t * D + i);
                    ww[0] = w4.x, ww[1] = w4.y, ww[2] = w4.z, ww[3] = w4.w;
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    if constexpr (KEYED) o[e] = fmaf(qq[e], S[i + e], o[e]);
                    S[i + e] = fmaf(kk[e], vv, ww[e] * S[i + e]);
                    if constexpr (!KEYED) o[e] = fmaf(qq[e], S[i + e], o[e]);
                }
            }
            part[(warp * BLOCK + t) * 32 + lane] = (o[0] + o[1]) + (o[2] + o[3]);
        }
        __syncthreads();
        for (uint32_t t = warp; t < n; t += 8) {
            float o = 0.0f;
#pragma unroll
            for (int x = 0; x < 8; ++x) o += part[(x * BLOCK + t) * 32 + lane];
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

// ---- long spans -------------------------------------------------------------------------------------------------------------------
// Two fp32 values in one register pair, and instructions that work on both.
__device__ __forceinline__ uint64_t pair(float a, float b) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpair(uint64_t p) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(p));
    return r;
}
__device__ __forceinline__ uint64_t mul2(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
__device__ __forceinline__ uint64_t fma2(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}

// A lane has R neighbouring rows of the state (two groups of four when R is 8) x C columns, a warp C columns of all rows.  The sums
// of a block of eight tokens are added over the lanes by one exchange, after which a lane or a few neighbours have the sum they store.
constexpr int RS_BLOCK = 8;
template <int R, int C, bool KEYED>
struct RsPlan {
    static constexpr int D = 32 * R, COLS = 8 * C, STAGES = R <= 4 ? 4 : 3;
    static constexpr uint32_t Q = 0, K = Q + RS_BLOCK * D, W = K + RS_BLOCK * D, V = W + (KEYED ? RS_BLOCK * D : 0), A = V + RS_BLOCK * COLS, STAGE = A + 2 * RS_BLOCK,
                              FLOATS = STAGES * STAGE;
};
template <int R, int C, bool KEYED>
__global__ void __launch_bounds__(256, R * C <= 16 ? 2 : 1) recurrence_span_kernel(RecurrenceArgs a) {
    using P = RsPlan<R, C, KEYED>;
    constexpr int D = P::D, V4 = R <= 4 ? 1 : R / 4, W = R / V4;  // a lane's rows: V4 groups of W neighbours
    constexpr uint32_t STAGES = P::STAGES;
    extern __shared__ __align__(16) float sm[];
    pdl_release();
    pdl_wait();
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y, col0 = blockIdx.x * P::COLS;
    const RowSpan sp = a.spans[a.first_long + blockIdx.z];
    const uint64_t row0 = (uint64_t)sp.row0 * a.pitch;
    const float *gq = a.q + row0 + (uint64_t)(h / a.share) * a.dim, *gk = a.k + row0 + (uint64_t)(h / a.share) * a.dim;
    const float *gv = a.v + row0 + (uint64_t)h * a.vdim + col0, *gw = KEYED ? a.w + (uint64_t)sp.row0 * a.w_pitch + (uint64_t)h * a.dim : nullptr;
    const float2 *ga = KEYED ? nullptr : a.step + (uint64_t)sp.row0 * a.n_head + h;
    auto aligned = [](const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool quads = a.dim % 4 == 0 && a.pitch % 4 == 0 && aligned(gq) && aligned(gk) && (!KEYED || (a.w_pitch % 4 == 0 && aligned(gw)));
    auto load = [&](uint32_t t0, uint32_t stage) {
        float *s = sm + stage * P::STAGE;
        const uint32_t n = min((uint32_t)RS_BLOCK, sp.n - t0), step = quads ? 4 : 1;
        for (uint32_t i = threadIdx.x * step; i < RS_BLOCK * D; i += 256 * step) {
            const uint32_t t = i / D, d = i % D;
            const bool in = t < n && d < a.dim;
            const uint64_t o = in ? (uint64_t)(t0 + t) * a.pitch + d : 0, ow = KEYED && in ? (uint64_t)(t0 + t) * a.w_pitch + d : 0;
            if (quads) {
                cp16(smem_addr(s + P::Q + i), gq + o, in);
                cp16(smem_addr(s + P::K + i), gk + o, in);
                if constexpr (KEYED) cp16(smem_addr(s + P::W + i), gw + ow, in);
            } else {
                cp4(s + P::Q + i, gq + o, in);
                cp4(s + P::K + i, gk + o, in);
                if constexpr (KEYED) cp4(s + P::W + i, gw + ow, in);
            }
        }
        for (uint32_t i = threadIdx.x; i < RS_BLOCK * P::COLS; i += 256) {
            const uint32_t t = i / P::COLS, c = i % P::COLS;
            const bool in = t < n && col0 + c < a.vdim;
            cp4(s + P::V + i, in ? gv + (uint64_t)(t0 + t) * a.pitch + c : a.v, in);
        }
        if constexpr (!KEYED)
            if (threadIdx.x < RS_BLOCK) cp8(s + P::A + 2 * threadIdx.x, ga + (threadIdx.x < n ? (uint64_t)(t0 + threadIdx.x) * a.n_head : 0), threadIdx.x < n);
    };
#pragma unroll
    for (uint32_t s = 0; s + 1 < STAGES; ++s) {
        if (s * RS_BLOCK < sp.n) load(s * RS_BLOCK, s);
        cp_commit();
    }
    float *state = a.state + (((uint64_t)a.slots[sp.row0] * a.n_head + h) * a.dim) * a.vdim + col0 + C * warp;
    const bool fresh = a.positions[sp.row0] == 0;
    uint64_t S[R / 2][C];  // rows in pairs
    auto row_of = [&](int i) { return (uint32_t)(i / W) * (32 * W) + lane * W + i % W; };
    auto exists = [&](int i, int c) { return row_of(i) < a.dim && col0 + C * warp + c < a.vdim; };
#pragma unroll
    for (int i = 0; i < R; i += 2)
#pragma unroll
        for (int c = 0; c < C; ++c)
            S[i / 2][c] = pair(!fresh && exists(i, c) ? state[row_of(i) * a.vdim + c] : 0.0f, !fresh && exists(i + 1, c) ? state[row_of(i + 1) * a.vdim + c] : 0.0f);
    uint32_t stage = 0;
    for (uint32_t t0 = 0; t0 < sp.n; t0 += RS_BLOCK, stage = (stage + 1) % STAGES) {
        const uint32_t n = min((uint32_t)RS_BLOCK, sp.n - t0);
        cp_wait<STAGES - 2>();
        __syncthreads();  // this block's operands are there, and everyone has left the stage that is filled next
        if (t0 + (STAGES - 1) * RS_BLOCK < sp.n) load(t0 + (STAGES - 1) * RS_BLOCK, (stage + STAGES - 1) % STAGES);
        cp_commit();
        const float *base = sm + stage * P::STAGE;
        float x[RS_BLOCK * C];
        auto token = [&](int t) {
            uint64_t v[C], o[C], decay = 0;
            float s = 1.0f;
            if constexpr (!KEYED) {
                const float2 st = *reinterpret_cast<const float2 *>(base + P::A + 2 * t);
                decay = pair(st.x, st.x);
                s = st.y;
            }
#pragma unroll
            for (int c = 0; c < C; ++c) {
                const float f = base[P::V + t * P::COLS + C * warp + c] * s;
                v[c] = pair(f, f);
                o[c] = 0;
            }
#pragma unroll
            for (int g = 0; g < V4; ++g) {
                const uint32_t at = t * D + g * 32 * W + lane * W;
                uint64_t kk[W / 2], qq[W / 2], ww[W / 2];
                if constexpr (W == 4) {
                    const ulonglong2 k2 = *reinterpret_cast<const ulonglong2 *>(base + P::K + at), q2 = *reinterpret_cast<const ulonglong2 *>(base + P::Q + at);
                    kk[0] = k2.x, kk[1] = k2.y, qq[0] = q2.x, qq[1] = q2.y;
                    if constexpr (KEYED) {
                        const ulonglong2 w2 = *reinterpret_cast<const ulonglong2 *>(base + P::W + at);
                        ww[0] = w2.x, ww[1] = w2.y;
                    }
                } else {
                    kk[0] = *reinterpret_cast<const uint64_t *>(base + P::K + at), qq[0] = *reinterpret_cast<const uint64_t *>(base + P::Q + at);
                    if constexpr (KEYED) ww[0] = *reinterpret_cast<const uint64_t *>(base + P::W + at);
                }
#pragma unroll
                for (int e = 0; e < W / 2; ++e)
#pragma unroll
                    for (int c = 0; c < C; ++c) {
                        uint64_t &st = S[g * W / 2 + e][c];
                        if constexpr (KEYED) {
                            o[c] = fma2(qq[e], st, o[c]);
                            st = fma2(ww[e], st, mul2(kk[e], v[c]));
                        } else {
                            st = fma2(kk[e], v[c], mul2(decay, st));
                            o[c] = fma2(qq[e], st, o[c]);
                        }
                    }
            }
#pragma unroll
            for (int c = 0; c < C; ++c) {
                const float2 u = unpair(o[c]);
                x[C * t + c] = u.x + u.y;
            }
        };
        if (n == RS_BLOCK) {
#pragma unroll
            for (int t = 0; t < RS_BLOCK; ++t) token(t);
        } else {  // the last block: tokens past the end would decay the state
#pragma unroll
            for (int t = 0; t < RS_BLOCK; ++t) {
                if (t < (int)n) token(t);
                else
#pragma unroll
                    for (int c = 0; c < C; ++c) x[C * t + c] = 0.0f;
            }
        }
        // sums over the lanes: halves of the values go to the lane that differs in one bit, until one value is left
        constexpr int N = RS_BLOCK * C, REST = 32 / N;  // REST neighbouring lanes end with the same value
#pragma unroll
        for (int o = N / 2, bit = 16; o > 0; o >>= 1, bit >>= 1)
#pragma unroll
            for (int i = 0; i < o; ++i) {
                const bool hi = lane & bit;
                const float give = hi ? x[i] : x[i + o], mine = hi ? x[i + o] : x[i];
                x[i] = mine + __shfl_xor_sync(0xffffffffu, give, bit);
            }
#pragma unroll
        for (int bit = REST / 2; bit > 0; bit >>= 1) x[0] += __shfl_xor_sync(0xffffffffu, x[0], bit);
        const uint32_t i = lane / REST, t = i / C, col = col0 + C * warp + i % C;
        if (lane % REST == 0 && t < n && col < a.vdim) a.o[((uint64_t)(sp.row0 + t0 + t) * a.n_head + h) * a.vdim + col] = x[0];
    }
    cp_wait<0>();
#pragma unroll
    for (int i = 0; i < R; i += 2)
#pragma unroll
        for (int c = 0; c < C; ++c) {
            const float2 u = unpair(S[i / 2][c]);
            if (exists(i, c)) state[row_of(i) * a.vdim + c] = u.x;
            if (exists(i + 1, c)) state[row_of(i + 1) * a.vdim + c] = u.y;
        }
}

// ---- state space: convolution and steps ---------------------------------------------------------------------------------------------
// A thread has one channel of CV_TOKENS consecutive tokens of a span; threads past the channels have a head's step sizes.  The
// thread with the first tokens of a span is the only one that reads the state, and replaces it when it has.
constexpr int CV_THREADS = 128, CV_TOKENS = 16;
template <int K>  // taps; 0: a.taps
__global__ void __launch_bounds__(CV_THREADS) conv_kernel(ConvArgs a) {
    pdl_release();
    pdl_wait();
    RowSpan sp{blockIdx.x, 1};
    uint32_t f0 = 0;
    if (!a.single) find_tile(a.spans, a.n_seq, 1, CV_TOKENS, blockIdx.x, &sp, &f0);
    const uint32_t c = blockIdx.y * CV_THREADS + threadIdx.x;
    if (f0 >= sp.n || c >= a.n_channel + a.n_head) return;
    const int n = (int)sp.n, first = (int)f0, last = min(first + CV_TOKENS, n);
    const float *y = a.y + (uint64_t)sp.row0 * a.y_pitch + c;
    if (c >= a.n_channel) {
        const uint32_t h = c - a.n_channel;
        const float bias = a.dt_bias[h], rate = -expf(a.a_log[h]);
        for (int t = first; t < last; ++t) {
            const float z = y[(uint64_t)t * a.y_pitch] + bias, dt = fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z)));
            a.step[(uint64_t)(sp.row0 + t) * a.n_head + h] = make_float2(expf(rate * dt), dt);
        }
        return;
    }
    const int taps = K ? K : (int)a.taps, back = taps - 1;
    float *state = a.state + (uint64_t)a.slots[sp.row0] * back * a.n_channel + c;
    const bool fresh = a.positions[sp.row0] == 0;
    auto input = [&](int t) { return t >= 0 ? y[(uint64_t)t * a.y_pitch] : fresh ? 0.0f : state[(uint64_t)(t + back) * a.n_channel]; };
    const float *w = a.w + (uint64_t)c * taps;
    const float bias = a.b[c];
    float *u = a.u + (uint64_t)sp.row0 * a.n_channel + c;
    if constexpr (K > 0) {
        float wk[K], x[K];
#pragma unroll
        for (int i = 0; i < K; ++i) wk[i] = w[i];
#pragma unroll
        for (int i = 0; i + 1 < K; ++i) x[i + 1] = input(first - back + i);
#pragma unroll 4
        for (int t = first; t < last; ++t) {
#pragma unroll
            for (int i = 0; i + 1 < K; ++i) x[i] = x[i + 1];
            x[K - 1] = y[(uint64_t)t * a.y_pitch];
            float s = bias;
#pragma unroll
            for (int i = 0; i < K; ++i) s = fmaf(wk[i], x[i], s);
            u[(uint64_t)t * a.n_channel] = silu(s);
        }
    } else {
        for (int t = first; t < last; ++t) {
            float s = bias;
            for (int i = 0; i < taps; ++i) s = fmaf(w[i], input(t - back + i), s);
            u[(uint64_t)t * a.n_channel] = silu(s);
        }
    }
    if (first == 0)  // (an entry that is read here has a higher number than the one it goes to: it has not been replaced yet)
        for (int i = 0; i < back; ++i) state[(uint64_t)i * a.n_channel] = input(n - back + i);
}

// A CTA per token and part.
template <typename TA>
__global__ void __launch_bounds__(256) state_space_out_kernel(StateSpaceOutArgs a) {
    extern __shared__ float sm[];
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x, n = a.inner / a.n_part, c0 = blockIdx.y * n;
    const float *o = a.o + (uint64_t)t * a.inner + c0, *x = a.x + (uint64_t)t * a.x_pitch + c0;
    const TA *z = static_cast<const TA *>(a.z) + (uint64_t)t * a.z_pitch + c0;
    float s = 0.0f;
#pragma unroll 4
    for (uint32_t i = threadIdx.x; i < n; i += 256) {
        const float v = fmaf(a.skip[(c0 + i) / a.vdim], x[i], o[i]) * silu(from_act(z[i]));
        sm[i] = v;
        s += v * v;
    }
    const float f = inv_rms(block_sum(s, red), n, a.eps);
    TA *out = static_cast<TA *>(a.out) + (uint64_t)t * a.out_pitch + c0;
#pragma unroll 4
    for (uint32_t i = threadIdx.x; i < n; i += 256) out[i] = to_act<TA>(sm[i] * f * a.norm[c0 + i]);
}

// ---- time mixing: token shift --------------------------------------------------------------------------------------------------------
// A CTA per row.  The CTA of a span's first row is the only one that reads the state, and replaces it when it has.
template <int V> struct Vals { float v[V]; };
template <int V>
__device__ __forceinline__ Vals<V> load_vals(const float *p) {
    Vals<V> r;
    if constexpr (V == 4) {
        const float4 u = *reinterpret_cast<const float4 *>(p);
        r.v[0] = u.x, r.v[1] = u.y, r.v[2] = u.z, r.v[3] = u.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <typename TA, int V>
__global__ void __launch_bounds__(512) shift_mix_kernel(ShiftMixArgs a) {
    __shared__ float red[33];
    __shared__ uint32_t span_rows;
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x;
    const int32_t slot = a.slots[t];
    const bool first = a.single || t == 0 || a.slots[t - 1] != slot, fresh = first && a.positions[t] == 0;
    if (threadIdx.x == 0) span_rows = 1;
    __syncthreads();
    if (first && !a.single)
        for (uint32_t s = threadIdx.x; s < a.n_seq; s += blockDim.x)
            if (a.spans[s].row0 == t) span_rows = a.spans[s].n;
    auto scale = [&](const float *x) {
        if (!a.norm) return 1.0f;
        float s = 0.0f;
        for (uint32_t c = V * threadIdx.x; c < a.width; c += V * blockDim.x) {
            const Vals<V> u = load_vals<V>(x + c);
#pragma unroll
            for (int e = 0; e < V; ++e) s += u.v[e] * u.v[e];
        }
        return inv_rms(block_sum(s, red), a.width, a.eps);
    };
    const float *x = a.x + (uint64_t)t * a.width, *before = x - a.width;
    float *state = a.state + (uint64_t)slot * a.width;
    const float f = scale(x), fb = first ? 1.0f : scale(before);
    TA *mix = static_cast<TA *>(a.mix) + (uint64_t)t * SHIFT_MIXES * a.pitch;
    __syncthreads();
    const uint32_t n = span_rows;
    const float *last = x + (uint64_t)(n - 1) * a.width;
    const float fl = first ? (n > 1 ? scale(last) : f) : 0.0f;
    for (uint32_t c = V * threadIdx.x; c < a.width; c += V * blockDim.x) {
        Vals<V> g, h = load_vals<V>(x + c), p;
        if (a.norm) g = load_vals<V>(a.norm + c);
        else
#pragma unroll
            for (int e = 0; e < V; ++e) g.v[e] = 1.0f;
        if (fresh)
#pragma unroll
            for (int e = 0; e < V; ++e) p.v[e] = 0.0f;
        else p = load_vals<V>((first ? state : before) + c);
#pragma unroll
        for (int e = 0; e < V; ++e) {
            h.v[e] *= f * g.v[e];
            if (!first) p.v[e] *= fb * g.v[e];
        }
#pragma unroll
        for (uint32_t i = 0; i < SHIFT_MIXES; ++i) {
            const Vals<V> mu = load_vals<V>(a.mu[i] + c);
            float m[V];
#pragma unroll
            for (int e = 0; e < V; ++e) m[e] = fmaf(p.v[e] - h.v[e], mu.v[e], h.v[e]);
            TA *dst = mix + (uint64_t)i * a.pitch + c;
            if constexpr (V == 4) store4<TA>(dst, make_float4(m[0], m[1], m[2], m[3]));
            else *dst = to_act<TA>(m[0]);
        }
        if (first) {
            if (n > 1) {
                h = load_vals<V>(last + c);
#pragma unroll
                for (int e = 0; e < V; ++e) h.v[e] *= fl * g.v[e];
            }
            if constexpr (V == 4) *reinterpret_cast<float4 *>(state + c) = make_float4(h.v[0], h.v[1], h.v[2], h.v[3]);
            else state[c] = h.v[0];
        }
    }
}

// ---- time mixing: what follows the recurrence ------------------------------------------------------------------------------------------
// A warp per (token, head).
constexpr int TM_VALUES = 4;  // per lane in registers; wider heads read the rest twice
template <typename TA>
__global__ void __launch_bounds__(256) time_mix_out_kernel(TimeMixOutArgs a) {
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x, lane = threadIdx.x & 31, h = blockIdx.y * 8 + (threadIdx.x >> 5), c0 = h * a.dim;
    if (h >= a.n_head) return;
    const uint64_t at = (uint64_t)t * a.pitch + c0;
    const float *r = a.r + at, *k = a.k + at, *v = a.v + at, *gate = a.gate + at, *o = a.o + (uint64_t)t * a.n_head * a.dim + c0;
    TA *out = static_cast<TA *>(a.out) + (uint64_t)t * a.out_pitch + c0;
    float x[TM_VALUES], vv[TM_VALUES], z[TM_VALUES], b = 0.0f;
#pragma unroll
    for (int u = 0; u < TM_VALUES; ++u) {
        const uint32_t i = lane + 32 * u;
        const bool in = i < a.dim;
        x[u] = in ? o[i] : 0.0f, vv[u] = in ? v[i] : 0.0f, z[u] = in ? gate[i] : 0.0f;
        if (in) b = fmaf(r[i] * a.bonus[c0 + i], k[i], b);
    }
    for (uint32_t i = lane + 32 * TM_VALUES; i < a.dim; i += 32) b = fmaf(r[i] * a.bonus[c0 + i], k[i], b);
    b = warp_sum(b);
    float s = 0.0f;
#pragma unroll
    for (int u = 0; u < TM_VALUES; ++u) {
        x[u] = fmaf(b, vv[u], x[u]);
        s += x[u] * x[u];
    }
    for (uint32_t i = lane + 32 * TM_VALUES; i < a.dim; i += 32) {
        const float e = fmaf(b, v[i], o[i]);
        s += e * e;
    }
    const float f = inv_rms(warp_sum(s), a.dim, a.eps);
#pragma unroll
    for (int u = 0; u < TM_VALUES; ++u) {
        const uint32_t i = lane + 32 * u;
        if (i < a.dim) out[i] = to_act<TA>(x[u] * f * a.norm[c0 + i] * silu(z[u]));
    }
    for (uint32_t i = lane + 32 * TM_VALUES; i < a.dim; i += 32) out[i] = to_act<TA>(fmaf(b, v[i], o[i]) * f * a.norm[c0 + i] * silu(gate[i]));
}

constexpr uint32_t OUT_SMEM = 200 * 1024;
template <int DW, bool KEYED>
cudaError_t configure_short() {
    return cudaFuncSetAttribute(recurrence_kernel<DW, KEYED>, cudaFuncAttributeMaxDynamicSharedMemorySize, RcPlan<DW, KEYED>::FLOATS * 4);
}
template <int R, int C, bool KEYED>
cudaError_t configure_span() {
    return cudaFuncSetAttribute(recurrence_span_kernel<R, C, KEYED>, cudaFuncAttributeMaxDynamicSharedMemorySize, RsPlan<R, C, KEYED>::FLOATS * 4);
}
template <int DW, bool KEYED>
void run_short(const RecurrenceArgs &a, uint32_t n, cudaStream_t st) {
    launch_pdl(recurrence_kernel<DW, KEYED>, dim3((a.vdim + 31) / 32, a.n_head, n), 256, RcPlan<DW, KEYED>::FLOATS * 4, st, a);
}
template <int R, int C, bool KEYED>
void run_span(const RecurrenceArgs &a, uint32_t n, cudaStream_t st) {
    using P = RsPlan<R, C, KEYED>;
    launch_pdl(recurrence_span_kernel<R, C, KEYED>, dim3((a.vdim + P::COLS - 1) / P::COLS, a.n_head, n), 256, P::FLOATS * 4, st, a);
}
template <bool KEYED>
uint32_t run(const RecurrenceArgs &a, cudaStream_t st) {
    const uint32_t n_long = a.n_seq - a.first_long, n_short = a.first_long;
    if (n_short) {
        if (a.dim <= 64) run_short<8, KEYED>(a, n_short, st);
        else if (a.dim <= 128) run_short<16, KEYED>(a, n_short, st);
        else run_short<32, KEYED>(a, n_short, st);
    }
    if (n_long) {
        if (a.dim <= 64) run_span<2, 2, KEYED>(a, n_long, st);
        else if (a.dim <= 128) run_span<4, 2, KEYED>(a, n_long, st);
        else run_span<8, 2, KEYED>(a, n_long, st);
    }
    return (n_short > 0) + (n_long > 0);
}

}  // namespace

// ---- launchers ----------------------------------------------------------------------------------------------------------------------
cudaError_t recurrence_configure() {
    static PerDeviceOnce once;
    return once.run([] {
        cudaError_t e = cudaSuccess;
        for (cudaError_t (*f)() : {configure_short<8, false>, configure_short<16, false>, configure_short<32, false>, configure_short<8, true>, configure_short<16, true>,
                                   configure_short<32, true>, configure_span<2, 2, false>, configure_span<4, 2, false>, configure_span<8, 2, false>, configure_span<2, 2, true>,
                                   configure_span<4, 2, true>, configure_span<8, 2, true>})
            if (e == cudaSuccess) e = f();
        for (auto k : {state_space_out_kernel<float>, state_space_out_kernel<bf16>})
            if (e == cudaSuccess) e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, OUT_SMEM);
        return e;
    });
}

bool recurrence_supported(uint32_t dim) { return dim >= 1 && dim <= 256; }

uint32_t launch_recurrence(const RecurrenceArgs &a, int sm_count, cudaStream_t st) {
    (void)sm_count;
    return a.step ? run<false>(a, st) : run<true>(a, st);
}

void launch_conv(const ConvArgs &a, cudaStream_t st) {
    uint32_t tiles = a.T;
    if (!a.single) {
        tiles = 0;
        for (uint32_t s = 0; s < a.n_seq; ++s) tiles += (a.h_spans[s].n + CV_TOKENS - 1) / CV_TOKENS;
    }
    const dim3 grid(tiles, (a.n_channel + a.n_head + CV_THREADS - 1) / CV_THREADS);
    launch_pdl(a.taps == 4 ? conv_kernel<4> : a.taps == 3 ? conv_kernel<3> : a.taps == 2 ? conv_kernel<2> : conv_kernel<0>, grid, CV_THREADS, 0, st, a);
}

bool state_space_out_supported(uint32_t part) { return (uint64_t)part * 4 <= OUT_SMEM; }

void launch_state_space_out(const StateSpaceOutArgs &a, bool f32, cudaStream_t st) {
    launch_pdl(f32 ? state_space_out_kernel<float> : state_space_out_kernel<bf16>, dim3(a.T, a.n_part), 256, (size_t)(a.inner / a.n_part) * 4, st, a);
}

void launch_shift_mix(const ShiftMixArgs &a, bool f32, cudaStream_t st) {
    const uint32_t threads = std::min(512u, std::max(64u, (a.width / 4 + 31) / 32 * 32));
    if (a.width % 4 == 0) launch_pdl(f32 ? shift_mix_kernel<float, 4> : shift_mix_kernel<bf16, 4>, a.T, threads, 0, st, a);
    else launch_pdl(f32 ? shift_mix_kernel<float, 1> : shift_mix_kernel<bf16, 1>, a.T, threads, 0, st, a);
}

void launch_time_mix_out(const TimeMixOutArgs &a, bool f32, cudaStream_t st) {
    launch_pdl(f32 ? time_mix_out_kernel<float> : time_mix_out_kernel<bf16>, dim3(a.T, (a.n_head + 7) / 8), 256, 0, st, a);
}

}  // namespace ob
