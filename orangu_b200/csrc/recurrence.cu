// Recurrent layers with data-dependent decay: the state recurrence itself, the short convolution and step sizes of a state-space
// layer, the token shift of a time-mixing layer, and what follows the recurrence in either.
//
//   recurrence_kernel       decoded tokens and short spans, bound by the state's traffic: a warp has a few rows of the state, a lane a column
//   recurrence_span_kernel  long spans, bound by fp32 arithmetic: a lane has neighbouring rows, two of them per packed instruction
// Everything is fp32; the state goes token by token, so a result does not depend on how a sequence was cut.
#include <algorithm>
#include <type_traits>

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

// A lane has R rows of the state (groups of four neighbours) x C columns; LG lanes have all rows, so a warp has 32 / LG groups of C
// columns.  The sums of a block of eight tokens are added over the LG lanes by one exchange, after which every lane has the sums it
// stores.  With one decay per token the state is kept without its decay over a block (S' = S / a_1 .. a_t, the values scaled instead,
// the outputs scaled back) unless it decays by more than RS_FOLD within the block.
constexpr int RS_BLOCK = 8;
constexpr float RS_FOLD = 1e-18f;
template <int D, int R, int C, int NW, bool KEYED>
struct RsPlan {
    static constexpr int LG = D / R, COLS = NW * (32 / LG) * C, STAGES = 4, ARRAYS = KEYED ? 3 : 2;
    static constexpr uint32_t Q = 0, K = Q + RS_BLOCK * D, W = K + RS_BLOCK * D, V = ARRAYS * RS_BLOCK * D, A = V + RS_BLOCK * COLS, STAGE = A + 2 * RS_BLOCK, FLOATS = STAGES * STAGE;
    static_assert(LG <= 32 && R % 4 == 0 && (C == 2 || C == 4), "");
};
template <int D, int R, int C, int NW, bool KEYED>
__global__ void __launch_bounds__(32 * NW) recurrence_span_kernel(RecurrenceArgs a) {
    using P = RsPlan<D, R, C, NW, KEYED>;
    constexpr int LG = P::LG, THREADS = 32 * NW, COLS = P::COLS;
    constexpr uint32_t STAGES = P::STAGES;
    extern __shared__ __align__(16) float sm[];
    pdl_release();
    pdl_wait();
    const uint32_t lane = threadIdx.x & 31, lg = lane % LG, h = blockIdx.y, col0 = blockIdx.x * COLS, my_col = (threadIdx.x / LG) * C;
    const RowSpan sp = a.spans[a.first_long + blockIdx.z];
    const uint64_t row0 = (uint64_t)sp.row0 * a.pitch;
    const float *gq = a.q + row0 + (uint64_t)(h / a.share) * a.dim, *gk = a.k + row0 + (uint64_t)(h / a.share) * a.dim;
    const float *gv = a.v + row0 + (uint64_t)h * a.vdim + col0, *gw = KEYED ? a.w + (uint64_t)sp.row0 * a.w_pitch + (uint64_t)h * a.dim : nullptr;
    const float2 *ga = KEYED ? nullptr : a.step + (uint64_t)sp.row0 * a.n_head + h;
    auto aligned = [](const void *p) { return (reinterpret_cast<uintptr_t>(p) & 15) == 0; };
    const bool quads = a.dim % 4 == 0 && a.vdim % 4 == 0 && a.pitch % 4 == 0 && aligned(gq) && aligned(gk) && aligned(gv) && (!KEYED || (a.w_pitch % 4 == 0 && aligned(gw)));
    auto load = [&](uint32_t t0, uint32_t stage) {
        float *s = sm + stage * P::STAGE;
        const uint32_t n = min((uint32_t)RS_BLOCK, sp.n - t0);
        if (quads) {
            constexpr uint32_t N = RS_BLOCK * D / 4;
#pragma unroll
            for (uint32_t k = 0; k < (P::ARRAYS * N + THREADS - 1) / THREADS; ++k) {
                const uint32_t i = threadIdx.x + k * THREADS, t = i / (D / 4) % RS_BLOCK, d = i % (D / 4) * 4;
                if (P::ARRAYS * N % THREADS && i >= P::ARRAYS * N) break;
                const float *base = i < N ? gq : i < 2 * N ? gk : gw;
                const bool in = t < n && d < a.dim;
                cp16(smem_addr(s + 4 * i), base + (in ? (uint64_t)(t0 + t) * (KEYED && i >= 2 * N ? a.w_pitch : a.pitch) + d : 0), in);
            }
            for (uint32_t i = threadIdx.x; i < RS_BLOCK * COLS / 4; i += THREADS) {
                const uint32_t t = i / (COLS / 4), c = i % (COLS / 4) * 4;
                const bool in = t < n && col0 + c < a.vdim;
                cp16(smem_addr(s + P::V + 4 * i), in ? gv + (uint64_t)(t0 + t) * a.pitch + c : a.v, in);
            }
        } else {
            for (uint32_t i = threadIdx.x; i < RS_BLOCK * D; i += THREADS) {
                const uint32_t t = i / D, d = i % D;
                const bool in = t < n && d < a.dim;
                const uint64_t o = in ? (uint64_t)(t0 + t) * a.pitch + d : 0;
                cp4(s + P::Q + i, gq + o, in);
                cp4(s + P::K + i, gk + o, in);
                if constexpr (KEYED) cp4(s + P::W + i, gw + (in ? (uint64_t)(t0 + t) * a.w_pitch + d : 0), in);
            }
            for (uint32_t i = threadIdx.x; i < RS_BLOCK * COLS; i += THREADS) {
                const uint32_t t = i / COLS, c = i % COLS;
                const bool in = t < n && col0 + c < a.vdim;
                cp4(s + P::V + i, in ? gv + (uint64_t)(t0 + t) * a.pitch + c : a.v, in);
            }
        }
        if constexpr (!KEYED)
            if (threadIdx.x < RS_BLOCK) cp8(s + P::A + 2 * threadIdx.x, ga + (threadIdx.x < n ? (uint64_t)(t0 + threadIdx.x) * a.n_head : 0), threadIdx.x < n);
    };
#pragma unroll
    for (uint32_t s = 0; s + 1 < STAGES; ++s) {
        if (s * RS_BLOCK < sp.n) load(s * RS_BLOCK, s);
        cp_commit();
    }
    float *state = a.state + (((uint64_t)a.slots[sp.row0] * a.n_head + h) * a.dim) * a.vdim + col0 + my_col;
    const bool fresh = a.positions[sp.row0] == 0;
    uint64_t S[R / 2][C];  // rows in pairs
    auto row_of = [&](int i) { return (uint32_t)(i / 4) * (4 * LG) + lg * 4 + i % 4; };
    auto exists = [&](int i, int c) { return row_of(i) < a.dim && col0 + my_col + c < a.vdim; };
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
        const float *base = sm + stage * P::STAGE, *vs = base + P::V + my_col;
        constexpr int N = RS_BLOCK * C;  // sums of a block
        float x[N];
        float2 own = make_float2(1.0f, 0.0f);  // decay and factor of token lane % 8; tokens past the end change nothing
        float since = 1.0f;                    // decay from the block's start through that token
        if constexpr (!KEYED) {
            if (lane % RS_BLOCK < n) own = *reinterpret_cast<const float2 *>(base + P::A + 2 * (lane % RS_BLOCK));
            since = own.x;
#pragma unroll
            for (int o = 1; o < RS_BLOCK; o <<= 1) {
                const float up = __shfl_up_sync(0xffffffffu, since, o, RS_BLOCK);
                if (lane % RS_BLOCK >= o) since *= up;
            }
        }
        const float whole = KEYED ? 1.0f : __shfl_sync(0xffffffffu, since, RS_BLOCK - 1);
        const bool fold = !KEYED && whole > RS_FOLD;
        const float factor = fold ? own.y / since : own.y;
        struct Operands {
            uint64_t k[R / 2], q[R / 2], w[R / 2];
            float v[C];
        };
        auto fetch = [&](int t, Operands &x) {
#pragma unroll
            for (int g = 0; g < R / 4; ++g) {
                const float *at = base + t * D + g * 4 * LG + lg * 4;
                *reinterpret_cast<ulonglong2 *>(x.k + 2 * g) = *reinterpret_cast<const ulonglong2 *>(at + P::K);
                *reinterpret_cast<ulonglong2 *>(x.q + 2 * g) = *reinterpret_cast<const ulonglong2 *>(at + P::Q);
                if constexpr (KEYED) *reinterpret_cast<ulonglong2 *>(x.w + 2 * g) = *reinterpret_cast<const ulonglong2 *>(at + P::W);
            }
            if constexpr (C == 4) *reinterpret_cast<float4 *>(x.v) = *reinterpret_cast<const float4 *>(vs + t * COLS);
            else *reinterpret_cast<float2 *>(x.v) = *reinterpret_cast<const float2 *>(vs + t * COLS);
        };
        Operands ops[2];
        fetch(0, ops[0]);
        auto token = [&](int t, auto folded) {
            [[maybe_unused]] constexpr bool FOLDED = decltype(folded)::value;
            uint64_t v[C], o[C];
            [[maybe_unused]] uint64_t decay = 0;
            if (t + 1 < RS_BLOCK) fetch(t + 1, ops[(t + 1) % 2]);  // on its way while this token is computed
            const Operands &in = ops[t % 2];
            float f[C];
#pragma unroll
            for (int c = 0; c < C; ++c) f[c] = in.v[c];
            if constexpr (!KEYED) {
                const float s = __shfl_sync(0xffffffffu, factor, t);
#pragma unroll
                for (int c = 0; c < C; ++c) f[c] *= s;
                if constexpr (!FOLDED) {
                    const float d = __shfl_sync(0xffffffffu, own.x, t);
                    decay = pair(d, d);
                }
            }
#pragma unroll
            for (int c = 0; c < C; ++c) v[c] = pair(f[c], f[c]), o[c] = 0;
#pragma unroll
            for (int e = 0; e < R / 2; ++e)
#pragma unroll
                for (int c = 0; c < C; ++c) {
                    uint64_t &st = S[e][c];
                    if constexpr (KEYED) {
                        o[c] = fma2(in.q[e], st, o[c]);
                        st = fma2(in.w[e], st, mul2(in.k[e], v[c]));
                    } else {
                        st = fma2(in.k[e], v[c], FOLDED ? st : mul2(decay, st));
                        o[c] = fma2(in.q[e], st, o[c]);
                    }
                }
#pragma unroll
            for (int c = 0; c < C; ++c) {
                const float2 u = unpair(o[c]);
                x[C * t + c] = u.x + u.y;
            }
        };
        if (fold) {
#pragma unroll
            for (int t = 0; t < RS_BLOCK; ++t) token(t, std::true_type{});
            const uint64_t w2 = pair(whole, whole);
#pragma unroll
            for (int i = 0; i < R / 2; ++i)
#pragma unroll
                for (int c = 0; c < C; ++c) S[i][c] = mul2(w2, S[i][c]);
        } else if (!KEYED || n == RS_BLOCK) {
#pragma unroll
            for (int t = 0; t < RS_BLOCK; ++t) token(t, std::false_type{});
        } else {  // (decays of tokens past the end are not there)
#pragma unroll
            for (int t = 0; t < RS_BLOCK; ++t) {
                if (t < (int)n) token(t, std::false_type{});
                else
#pragma unroll
                    for (int c = 0; c < C; ++c) x[C * t + c] = 0.0f;
            }
        }
        // sums over the LG lanes: half of the values go to the lane that differs in one bit, until one is left
        constexpr int LEFT = N > LG ? N / LG : 1, SAME = LG > N ? LG / N : 1;  // values a lane ends with; neighbours that end with the same
#pragma unroll
        for (int o = N / 2, bit = LG / 2; bit > 0; o >>= 1, bit >>= 1) {
            if (o > 0) {
                const bool hi = lane & bit;
#pragma unroll
                for (int i = 0; i < o; ++i) {
                    const float give = hi ? x[i] : x[i + o], mine = hi ? x[i + o] : x[i];
                    x[i] = mine + __shfl_xor_sync(0xffffffffu, give, bit);
                }
            } else {
                x[0] += __shfl_xor_sync(0xffffffffu, x[0], bit);
            }
        }
        const uint32_t i = lg / SAME * LEFT, t = i / C, c = i % C;
        const float back = fold ? __shfl_sync(0xffffffffu, since, t) : 1.0f;
        if (lg % SAME == 0 && t < n) {
            float *o = a.o + ((uint64_t)(sp.row0 + t0 + t) * a.n_head + h) * a.vdim + col0 + my_col + c;
#pragma unroll
            for (int e = 0; e < LEFT; ++e)
                if (col0 + my_col + c + e < a.vdim) o[e] = x[e] * back;
        }
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
constexpr int CV_THREADS = 128, CV_TOKENS = 16;  // (a decoded token: one)
template <int K, int TOKENS>  // taps (0: a.taps), tokens of a thread
__global__ void __launch_bounds__(CV_THREADS) conv_kernel(ConvArgs a) {
    pdl_release();
    pdl_wait();
    RowSpan sp{blockIdx.x, 1};
    uint32_t f0 = 0;
    if (!a.single) find_tile(a.spans, a.n_seq, 1, TOKENS, blockIdx.x, &sp, &f0);
    const uint32_t c = blockIdx.y * CV_THREADS + threadIdx.x;
    if (f0 >= sp.n || c >= a.n_channel + a.n_head) return;
    const int n = (int)sp.n, first = (int)f0, last = min(first + TOKENS, n);
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
        float wk[K], x[K - 1 + TOKENS];  // all inputs are requested before the first is used
#pragma unroll
        for (int i = 0; i < K; ++i) wk[i] = w[i];
#pragma unroll
        for (int i = 0; i + 1 < K; ++i) x[i] = input(first - back + i);
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) x[K - 1 + i] = first + i < last ? y[(uint64_t)(first + i) * a.y_pitch] : 0.0f;
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) {
            float s = bias;
#pragma unroll
            for (int k = 0; k < K; ++k) s = fmaf(wk[k], x[i + k], s);
            if (first + i < last) u[(uint64_t)(first + i) * a.n_channel] = silu(s);
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

// A CTA per token and part; V: entries of a thread side by side.
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
template <int V>
__device__ __forceinline__ Vals<V> load_vals(const bf16 *p) {
    Vals<V> r;
    if constexpr (V == 4) {
        const uint2 u = *reinterpret_cast<const uint2 *>(p);
        r.v[0] = __uint_as_float(u.x << 16), r.v[1] = __uint_as_float(u.x & 0xffff0000u), r.v[2] = __uint_as_float(u.y << 16), r.v[3] = __uint_as_float(u.y & 0xffff0000u);
    } else {
        r.v[0] = from_act(*p);
    }
    return r;
}
template <typename TA, int V>
__device__ __forceinline__ void store_vals(TA *p, const Vals<V> &x) {
    if constexpr (V == 4) store4<TA>(p, make_float4(x.v[0], x.v[1], x.v[2], x.v[3]));
    else *p = to_act<TA>(x.v[0]);
}
// Gate of the outputs: silu, its quotient within two units in the last place.
__device__ __forceinline__ float fast_silu(float z) { return __fdividef(z, 1.0f + expf(-fmaxf(z, -80.0f))); }

template <typename TA, int V>
__global__ void __launch_bounds__(256) state_space_out_kernel(StateSpaceOutArgs a) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    const uint32_t t = blockIdx.x, n = a.inner / a.n_part, c0 = blockIdx.y * n;
    const float *o = a.o + (uint64_t)t * a.inner + c0, *x = a.x + (uint64_t)t * a.x_pitch + c0;
    const TA *z = static_cast<const TA *>(a.z) + (uint64_t)t * a.z_pitch + c0;
    float s = 0.0f;
#pragma unroll 2
    for (uint32_t i = V * threadIdx.x; i < n; i += V * 256) {  // (V entries are of one head)
        const Vals<V> ov = load_vals<V>(o + i), xv = load_vals<V>(x + i), zv = load_vals<V>(z + i);
        const float skip = a.skip[(c0 + i) / a.vdim];
        Vals<V> v;
#pragma unroll
        for (int e = 0; e < V; ++e) {
            v.v[e] = fmaf(skip, xv.v[e], ov.v[e]) * fast_silu(zv.v[e]);
            s += v.v[e] * v.v[e];
        }
        store_vals<float, V>(sm + i, v);
    }
    const float f = inv_rms(block_sum(s, red), n, a.eps);
    TA *out = static_cast<TA *>(a.out) + (uint64_t)t * a.out_pitch + c0;
#pragma unroll 2
    for (uint32_t i = V * threadIdx.x; i < n; i += V * 256) {
        Vals<V> v = load_vals<V>(sm + i);
        const Vals<V> g = load_vals<V>(a.norm + c0 + i);
#pragma unroll
        for (int e = 0; e < V; ++e) v.v[e] *= f * g.v[e];
        store_vals<TA, V>(out + i, v);
    }
}

// ---- time mixing: token shift --------------------------------------------------------------------------------------------------------
// A CTA per row.  The CTA of a span's first row is the only one that reads the state, and replaces it when it has.
template <typename TA, int V>
__global__ void __launch_bounds__(1024) shift_mix_kernel(ShiftMixArgs a) {
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
            Vals<V> m;
#pragma unroll
            for (int e = 0; e < V; ++e) m.v[e] = fmaf(p.v[e] - h.v[e], mu.v[e], h.v[e]);
            store_vals<TA, V>(mix + (uint64_t)i * a.pitch + c, m);
        }
        if (first) {
            if (n > 1) {
                h = load_vals<V>(last + c);
#pragma unroll
                for (int e = 0; e < V; ++e) h.v[e] *= fl * g.v[e];
            }
            store_vals<float, V>(state + c, h);
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
template <int D, int R, int C, int NW, bool KEYED>
cudaError_t configure_span() {
    return cudaFuncSetAttribute(recurrence_span_kernel<D, R, C, NW, KEYED>, cudaFuncAttributeMaxDynamicSharedMemorySize, RsPlan<D, R, C, NW, KEYED>::FLOATS * 4);
}
template <int DW, bool KEYED>
void run_short(const RecurrenceArgs &a, uint32_t n, cudaStream_t st) {
    launch_pdl(recurrence_kernel<DW, KEYED>, dim3((a.vdim + 31) / 32, a.n_head, n), 256, RcPlan<DW, KEYED>::FLOATS * 4, st, a);
}
template <int D, int R, int C, int NW, bool KEYED>
void run_span(const RecurrenceArgs &a, uint32_t n, cudaStream_t st) {
    using P = RsPlan<D, R, C, NW, KEYED>;
    launch_pdl(recurrence_span_kernel<D, R, C, NW, KEYED>, dim3((a.vdim + P::COLS - 1) / P::COLS, a.n_head, n), 32 * NW, P::FLOATS * 4, st, a);
}
template <bool KEYED>
uint32_t run(const RecurrenceArgs &a, int sm_count, cudaStream_t st) {
    const uint32_t n_long = a.n_seq - a.first_long, n_short = a.first_long;
    if (n_short) {
        if (a.dim <= 64) run_short<8, KEYED>(a, n_short, st);
        else if (a.dim <= 128) run_short<16, KEYED>(a, n_short, st);
        else run_short<32, KEYED>(a, n_short, st);
    }
    if (n_long) {
        const uint32_t ctas = (a.vdim + 63) / 64 * a.n_head * n_long;  // with 64 columns each
        if (a.dim <= 64) run_span<64, 4, 4, 4, KEYED>(a, n_long, st);
        else if (a.dim > 128) run_span<256, 8, 4, 8, KEYED>(a, n_long, st);
        else if (KEYED) run_span<128, 4, 4, 4, true>(a, n_long, st);
        else if (ctas >= (uint32_t)sm_count * 3 / 4) run_span<128, 8, 4, 8, false>(a, n_long, st);
        else run_span<128, 8, 4, 4, false>(a, n_long, st);
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
                                   configure_short<32, true>, configure_span<64, 4, 4, 4, false>, configure_span<128, 8, 4, 8, false>, configure_span<128, 8, 4, 4, false>,
                                   configure_span<256, 8, 4, 8, false>, configure_span<64, 4, 4, 4, true>, configure_span<128, 4, 4, 4, true>, configure_span<256, 8, 4, 8, true>})
            if (e == cudaSuccess) e = f();
        for (auto k : {state_space_out_kernel<float, 4>, state_space_out_kernel<bf16, 4>, state_space_out_kernel<float, 1>, state_space_out_kernel<bf16, 1>})
            if (e == cudaSuccess) e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, OUT_SMEM);
        return e;
    });
}

bool recurrence_supported(uint32_t dim) { return dim >= 1 && dim <= 256; }

uint32_t launch_recurrence(const RecurrenceArgs &a, int sm_count, cudaStream_t st) {
    return a.step ? run<false>(a, sm_count, st) : run<true>(a, sm_count, st);
}

void launch_conv(const ConvArgs &a, cudaStream_t st) {
    uint32_t tiles = a.T;
    if (!a.single) {
        tiles = 0;
        for (uint32_t s = 0; s < a.n_seq; ++s) tiles += (a.h_spans[s].n + CV_TOKENS - 1) / CV_TOKENS;
    }
    const dim3 grid(tiles, (a.n_channel + a.n_head + CV_THREADS - 1) / CV_THREADS);
    auto run = [&](auto tokens) {
        constexpr int N = decltype(tokens)::value;
        launch_pdl(a.taps == 4 ? conv_kernel<4, N> : a.taps == 3 ? conv_kernel<3, N> : a.taps == 2 ? conv_kernel<2, N> : conv_kernel<0, N>, grid, CV_THREADS, 0, st, a);
    };
    if (a.single) run(std::integral_constant<int, 1>{});
    else run(std::integral_constant<int, CV_TOKENS>{});
}

bool state_space_out_supported(uint32_t part) { return (uint64_t)part * 4 <= OUT_SMEM; }

void launch_state_space_out(const StateSpaceOutArgs &a, bool f32, cudaStream_t st) {
    const bool fours = a.vdim % 4 == 0 && a.inner / a.n_part % 4 == 0 && a.x_pitch % 4 == 0;
    const dim3 grid(a.T, a.n_part);
    const size_t smem = (size_t)(a.inner / a.n_part) * 4;
    if (fours) launch_pdl(f32 ? state_space_out_kernel<float, 4> : state_space_out_kernel<bf16, 4>, grid, 256, smem, st, a);
    else launch_pdl(f32 ? state_space_out_kernel<float, 1> : state_space_out_kernel<bf16, 1>, grid, 256, smem, st, a);
}

void launch_shift_mix(const ShiftMixArgs &a, bool f32, cudaStream_t st) {
    const uint32_t threads = std::min(a.T <= 296 ? 1024u : 512u, std::max(64u, (a.width / 4 + 31) / 32 * 32));
    if (a.width % 4 == 0) launch_pdl(f32 ? shift_mix_kernel<float, 4> : shift_mix_kernel<bf16, 4>, a.T, threads, 0, st, a);
    else launch_pdl(f32 ? shift_mix_kernel<float, 1> : shift_mix_kernel<bf16, 1>, a.T, threads, 0, st, a);
}

void launch_time_mix_out(const TimeMixOutArgs &a, bool f32, cudaStream_t st) {
    launch_pdl(f32 ? time_mix_out_kernel<float> : time_mix_out_kernel<bf16>, dim3(a.T, (a.n_head + 7) / 8), 256, 0, st, a);
}

}  // namespace ob
