// Between two sublayers of a block that adds their outputs as they are: the output joins the residual, a layer's result is averaged
// with the results of the layers before it, the sum is normed in groups, and a short causal convolution over time is added to it.
//   s = x + mult * (rows of y of the token)        or the token's embedding
//   v = depth[n] s + sum_j depth[j] history[j]     or s
//   n = v over the root mean square of its group, times the norm's factors
//   h = n + sum_k conv[k] n of the token taps - 1 - k before
// The last taps - 1 rows n of a sequence are its state.
//
// residual_kernel     a CTA per token: s, v, and n or (every token from another sequence) h.  For spans it leaves the inverse root mean
//                     squares instead: n is then a product of three numbers, and is made where it is used
// input_conv_kernel   h of spans: a few channels of several tokens per thread, no exchange between threads
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

enum Leave { LEAVE_INPUT = 0, LEAVE_INVERSE = 1 };  // h; the inverse root mean squares

// Conv of one token alone: n of the tokens before it are the state, which moves on by one.
template <int V, typename F>
__device__ __forceinline__ void conv_step(const ResidualArgs &a, float *state, bool fresh, uint32_t c, const float (&n)[V], F store) {
    float o[V];
    const uint32_t back = a.taps - 1;
#pragma unroll
    for (int e = 0; e < V; ++e) o[e] = fmaf(a.conv[(uint64_t)back * a.width + c + e], n[e], n[e]);
    for (uint32_t k = 0; k < back; ++k) {
        float *p = state + (uint64_t)k * a.width + c;
#pragma unroll
        for (int e = 0; e < V; ++e) {
            const float before = fresh ? 0.0f : p[e];
            o[e] = fmaf(a.conv[(uint64_t)k * a.width + c + e], before, o[e]);
            if (k) p[e - (int)a.width] = before;
            if (k + 1 == back) p[e] = n[e];
        }
    }
    store(o);
}

template <typename TA, int NV, Leave LEAVE>
__global__ void __launch_bounds__(1024) residual_kernel(ResidualArgs a) {
    extern __shared__ float sm[];
    const uint32_t warp = threadIdx.x >> 5, lane = threadIdx.x & 31, warps = blockDim.x >> 5, t = blockIdx.x;
    const uint32_t group = a.width / a.n_group, unit = unit_columns(group), per_group = group / unit;
    float *units = sm, *inv = sm + a.width / unit;
    pdl_release();
    pdl_wait();
    if (a.zero && t == 0)
        for (uint32_t i = threadIdx.x; i < a.n_zero; i += blockDim.x) a.zero[i] = 0;
    const uint64_t at = (uint64_t)t * a.width;
    const float *x = a.x ? a.x + (uint64_t)(a.x_rows ? a.x_rows[t] : t) * a.width : nullptr;
    const bf16 *embedding = a.x ? nullptr : a.table + (uint64_t)a.tokens[t] * a.width;
    float4 v[NV];
    auto each = [&](auto f) {
#pragma unroll
        for (int i = 0; i < NV; ++i) {
            const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
            if (c < a.width) f(i, c);
        }
    };
#pragma unroll
    for (int i = 0; i < NV; ++i) v[i] = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
    each([&](int i, uint32_t c) { v[i] = x ? f4(x + c) : bf16x4(embedding + c); });
    if (a.y) {
        float4 y[NV];
        const float *row = a.y + (uint64_t)(a.rows ? a.rows[t * a.top] : t * a.top) * a.width;
        each([&](int i, uint32_t c) { y[i] = f4(row + c); });
        for (uint32_t k = 1; k < a.top; ++k) {
            const float *more = a.y + (uint64_t)(a.rows ? a.rows[t * a.top + k] : t * a.top + k) * a.width;
            each([&](int i, uint32_t c) { y[i] = add4(y[i], f4(more + c)); });
        }
        each([&](int i, uint32_t c) { v[i] = fma4(a.mult, y[i], v[i]); });
    }
    if (a.sum) each([&](int i, uint32_t c) { *reinterpret_cast<float4 *>(a.sum + at + c) = v[i]; });
    if (a.depth) {
        const float own = a.depth[a.n_history];
        each([&](int i, uint32_t) { v[i] = mul4(v[i], own); });
#pragma unroll 2
        for (uint32_t j = 0; j < a.n_history; ++j) {
            const float f = a.depth[j];
            const float *past = a.history + j * a.history_step + at;
            each([&](int i, uint32_t c) { v[i] = fma4(f, f4(past + c), v[i]); });
        }
        if (a.average) each([&](int i, uint32_t c) { *reinterpret_cast<float4 *>(a.average + at + c) = v[i]; });
    }
    if (!a.norm) return;
#pragma unroll
    for (int i = 0; i < NV; ++i) {
        const uint32_t c = 4 * (threadIdx.x + i * blockDim.x);
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
        if (lane == 0) (LEAVE == LEAVE_INVERSE ? a.inverse + (uint64_t)t * a.n_group : inv)[g] = inv_rms(s, group, a.eps);
    }
    if constexpr (LEAVE == LEAVE_INPUT) {
        __syncthreads();
        TA *h = static_cast<TA *>(a.h) + (uint64_t)t * a.h_pitch;
        float *state = a.taps > 1 ? a.state + (uint64_t)a.slots[t] * (a.taps - 1) * a.width : nullptr;
        const bool fresh = a.taps > 1 && a.positions[t] == 0;
        each([&](int i, uint32_t c) {
            const float4 n = mul44(mul4(v[i], inv[c / group]), f4(a.norm + c));
            if (!a.taps) {
                store4<TA>(h + c, n);
            } else if (a.taps == 4) {  // all of the state is requested at once
                float *p = state + c;
                const uint32_t w = a.width;
                float4 b[3] = {};
                if (!fresh) b[0] = f4(p), b[1] = f4(p + w), b[2] = f4(p + 2 * w);
                float4 o = fma44(f4(a.conv + 3 * w + c), n, n);
#pragma unroll
                for (int k = 0; k < 3; ++k) o = fma44(f4(a.conv + k * w + c), b[k], o);
                *reinterpret_cast<float4 *>(p) = b[1], *reinterpret_cast<float4 *>(p + w) = b[2], *reinterpret_cast<float4 *>(p + 2 * w) = n;
                store4<TA>(h + c, o);
            } else {
                const float e[4] = {n.x, n.y, n.z, n.w};
                conv_step<4>(a, state, fresh, c, e, [&](const float(&o)[4]) { store4<TA>(h + c, make_float4(o[0], o[1], o[2], o[3])); });
            }
        });
    }
}

// Any width and groups: columns one at a time through memory.
template <typename TA, Leave LEAVE>
__global__ void __launch_bounds__(512) residual_any_kernel(ResidualArgs a) {
    __shared__ float red[33];
    pdl_release();
    pdl_wait();
    if (a.zero && blockIdx.x == 0)
        for (uint32_t i = threadIdx.x; i < a.n_zero; i += blockDim.x) a.zero[i] = 0;
    const uint32_t t = blockIdx.x, group = a.width / a.n_group;
    const uint64_t at = (uint64_t)t * a.width;
    auto sum = [&](uint32_t c) {
        float v = a.x ? a.x[(uint64_t)(a.x_rows ? a.x_rows[t] : t) * a.width + c] : __bfloat162float(a.table[(uint64_t)a.tokens[t] * a.width + c]);
        if (!a.y) return v;
        float y = 0.0f;
        for (uint32_t k = 0; k < a.top; ++k) {
            const uint32_t p = t * a.top + k;
            y += a.y[(uint64_t)(a.rows ? a.rows[p] : p) * a.width + c];
        }
        return fmaf(a.mult, y, v);
    };
    auto averaged = [&](uint32_t c, float s) {
        if (!a.depth) return s;
        float v = s * a.depth[a.n_history];
        for (uint32_t j = 0; j < a.n_history; ++j) v = fmaf(a.depth[j], a.history[j * a.history_step + at + c], v);
        return v;
    };
    float *state = LEAVE == LEAVE_INPUT && a.norm && a.taps > 1 ? a.state + (uint64_t)a.slots[t] * (a.taps - 1) * a.width : nullptr;
    const bool fresh = state && a.positions[t] == 0;
    TA *h = static_cast<TA *>(a.h) + (uint64_t)t * a.h_pitch;
    for (uint32_t g = 0; g < a.n_group; ++g) {
        const uint32_t c0 = g * group + threadIdx.x, c1 = (g + 1) * group;
        float q = 0.0f;
        for (uint32_t c = c0; a.norm && c < c1; c += blockDim.x) {
            const float v = averaged(c, sum(c));
            q += v * v;
        }
        const float f = a.norm ? inv_rms(block_sum(q, red), group, a.eps) : 0.0f;
        if (LEAVE == LEAVE_INVERSE && threadIdx.x == 0) a.inverse[(uint64_t)t * a.n_group + g] = f;
        for (uint32_t c = c0; c < c1; c += blockDim.x) {  // (each x is read before it is replaced)
            const float s = sum(c), v = averaged(c, s);
            if (a.sum) a.sum[at + c] = s;
            if (a.depth && a.average) a.average[at + c] = v;
            if (LEAVE == LEAVE_INVERSE || !a.norm) continue;
            const float n[1] = {v * f * a.norm[c]};
            if (!a.taps) h[c] = to_act<TA>(n[0]);
            else conv_step<1>(a, state, fresh, c, n, [&](const float(&o)[1]) { h[c] = to_act<TA>(o[0]); });
        }
    }
}

// A thread has V channels of TOKENS consecutive tokens of a span.  The thread with a span's first tokens is the only one that reads
// the state (a thread's tokens are not fewer than the convolution reaches back), and replaces it when it has.
template <int V> struct Channels { float v[V]; };
template <int V>
__device__ __forceinline__ Channels<V> channels(const float *p) {
    Channels<V> r;
    if constexpr (V == 4) {
        const float4 u = f4(p);
        r.v[0] = u.x, r.v[1] = u.y, r.v[2] = u.z, r.v[3] = u.w;
    } else {
        r.v[0] = *p;
    }
    return r;
}
template <typename TA, int V>
__device__ __forceinline__ void put(TA *p, const Channels<V> &x) {
    if constexpr (V == 4) store4<TA>(p, make_float4(x.v[0], x.v[1], x.v[2], x.v[3]));
    else *p = to_act<TA>(x.v[0]);
}
constexpr int IC_THREADS = 128;
template <int K> constexpr int IC_TOKENS = K ? 8 : 16;
static_assert(IC_TOKENS<0> >= (int)CONV_MAX_TAPS - 1, "a thread's tokens reach over the state");

template <typename TA, int K, int V>  // taps (0: a.taps)
__global__ void __launch_bounds__(IC_THREADS) input_conv_kernel(ResidualArgs a, const float *v) {
    constexpr int TOKENS = IC_TOKENS<K>;
    const uint32_t c = V * (blockIdx.y * IC_THREADS + threadIdx.x), c_in = min(c, a.width - V);
    const Channels<V> factor = channels<V>(a.norm + c_in);
    Channels<V> w[K > 0 ? K : 1];
#pragma unroll
    for (int k = 0; k < K; ++k) w[k] = channels<V>(a.conv + (uint64_t)k * a.width + c_in);
    pdl_release();
    pdl_wait();
    RowSpan sp;
    uint32_t f0;
    find_tile(a.spans, a.n_seq, 1, TOKENS, blockIdx.x, &sp, &f0);
    if (f0 >= sp.n || c >= a.width) return;
    const int n = (int)sp.n, first = (int)f0, last = min(first + TOKENS, n), taps = K ? K : (int)a.taps, back = taps - 1;
    const uint32_t g = c / (a.width / a.n_group);
    const float *x = v + (uint64_t)sp.row0 * a.width + c, *inv = a.inverse + (uint64_t)sp.row0 * a.n_group + g;
    float *state = back ? a.state + (uint64_t)a.slots[sp.row0] * back * a.width + c : nullptr;
    const bool fresh = a.positions[sp.row0] == 0;
    auto scaled = [&](Channels<V> &r, float f) {
#pragma unroll
        for (int e = 0; e < V; ++e) r.v[e] = r.v[e] * f * factor.v[e];
    };
    auto normed = [&](int t) {
        Channels<V> r = channels<V>(x + (uint64_t)t * a.width);
        scaled(r, inv[(uint64_t)t * a.n_group]);
        return r;
    };
    auto input = [&](int t) {
        if (t >= 0) return normed(t);
        return fresh ? Channels<V>{} : channels<V>(state + (uint64_t)(t + back) * a.width);
    };
    TA *h = static_cast<TA *>(a.h) + (uint64_t)sp.row0 * a.h_pitch + c;
    auto add = [&](Channels<V> &o, const Channels<V> &tap, const Channels<V> &before) {
#pragma unroll
        for (int e = 0; e < V; ++e) o.v[e] = fmaf(tap.v[e], before.v[e], o.v[e]);
    };
    if constexpr (K > 0) {
        Channels<V> in[K - 1 + TOKENS];  // all of them are requested before the first is used (past the ends: the last one and the first again)
        float f[K - 1 + TOKENS];
#pragma unroll
        for (int i = 0; i < K - 1 + TOKENS; ++i) {
            const int t = max(min(first - back + i, last - 1), 0);
            in[i] = channels<V>(x + (uint64_t)t * a.width);
            f[i] = inv[(uint64_t)t * a.n_group];
        }
#pragma unroll
        for (int i = 0; i < K - 1 + TOKENS; ++i) scaled(in[i], f[i]);
        if (first == 0) {
#pragma unroll
            for (int i = 0; i + 1 < K; ++i) in[i] = input(i - back);
        }
#pragma unroll
        for (int i = 0; i < TOKENS; ++i) {
            Channels<V> o = in[K - 1 + i];
#pragma unroll
            for (int k = 0; k < K; ++k) add(o, w[k], in[i + k]);
            if (first + i < last) put<TA, V>(h + (uint64_t)(first + i) * a.h_pitch, o);
        }
    } else {
        for (int t = first; t < last; ++t) {
            Channels<V> o = normed(t);
            for (int k = 0; k < taps; ++k) add(o, channels<V>(a.conv + (uint64_t)k * a.width + c), input(t - back + k));
            put<TA, V>(h + (uint64_t)t * a.h_pitch, o);
        }
    }
    if (first == 0)  // (an entry that is read here has a higher number than the one it goes to: it has not been replaced yet)
        for (int i = 0; i < back; ++i) put<float, V>(state + (uint64_t)i * a.width, input(n - back + i));
}

template <typename TA, int V>
void input_conv(const ResidualArgs &a, const float *v, cudaStream_t st) {
    auto run = [&](void (*k)(ResidualArgs, const float *), uint32_t tokens) {
        uint32_t tiles = 0;
        for (uint32_t s = 0; s < a.n_seq; ++s) tiles += (a.h_spans[s].n + tokens - 1) / tokens;
        launch_pdl(k, dim3(tiles, (a.width / V + IC_THREADS - 1) / IC_THREADS), IC_THREADS, 0, st, a, v);
    };
    switch (a.taps) {
    case 2: return run(input_conv_kernel<TA, 2, V>, IC_TOKENS<2>);
    case 3: return run(input_conv_kernel<TA, 3, V>, IC_TOKENS<3>);
    case 4: return run(input_conv_kernel<TA, 4, V>, IC_TOKENS<4>);
    default: return run(input_conv_kernel<TA, 0, V>, IC_TOKENS<0>);
    }
}

template <typename TA>
uint32_t residual(const ResidualArgs &a, cudaStream_t st) {
    const uint32_t group = a.width / a.n_group;
    const RowShape r(a.width, a.T);
    const bool conv = a.norm && a.taps > 1 && !a.single;  // else a token's convolution needs its own row and the state
    if (r.vec && group % 4 == 0) {
        const size_t smem = (a.width / unit_columns(group) + a.n_group) * sizeof(float);
        launch_pdl(conv ? residual_kernel<TA, ROW_VECS, LEAVE_INVERSE> : residual_kernel<TA, ROW_VECS, LEAVE_INPUT>, a.T, r.threads, smem, st, a);
    } else {
        launch_pdl(conv ? residual_any_kernel<TA, LEAVE_INVERSE> : residual_any_kernel<TA, LEAVE_INPUT>, a.T, 512, 0, st, a);
    }
    if (!conv) return 1;
    const float *v = a.depth ? a.average : a.sum;
    if (a.width % 4 == 0 && group % 4 == 0) input_conv<TA, 4>(a, v, st);
    else input_conv<TA, 1>(a, v, st);
    return 2;
}

}  // namespace

uint32_t launch_residual(const ResidualArgs &a, bool f32, cudaStream_t st) { return f32 ? residual<float>(a, st) : residual<bf16>(a, st); }

}  // namespace ob
