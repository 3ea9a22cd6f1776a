// Models given as a list of layers (ob_layered_desc): weights as padded bfloat16 matrices, a cache pool per attention layer (latents,
// or keys and values) on the model's pages, a state pool per recurrent layer on the model's slots, and the step.
//
// A layer is a short chain of launches.  In a parallel block all products that read the normed input are one matrix, its feed-forward rows
// interleaved (gate, up) so that the activation is the epilogue; the mixer's output and the feed-forward's activations sit side
// by side in one row, so the two output products and the residual addition are one product too.
//   in      [mixer projections | gate/up]  <- h
//   mixer   latent attention: prep (norm, rotate, append), absorbed query (per head), attention, value up-projection with gate
//           retention: rotate, recurrence, norm with gate
//   out     x += [W_o | W_down] [mixer | ff]
//   side    gate (gelu, token entry), proj, then norm + residual + the next layer's norm in one kernel
// A sequential block reads the residual itself (h: its activation form) or its norm, and norms what it adds or adds it as it is:
//   in      mixer projections <- h
//   mixer   attention: prep, attention with the heads' epilogue
//           state space: convolution and steps, recurrence, gate and norm
//           time mixing: token shift, projections of the mixes, recurrence, norm and gate
//           a second mixer leaves its output beside the first one's, so that one product adds up both
//   out     product, bias as epilogue
//   post    x += mult norm(out), h = x or norm(x) in one kernel; plain sums: x += mult out, average over depth, grouped norm and
//           convolution over time in one kernel (residual.cu)
//   ff      dense: up (activation as epilogue), down; experts: routing, grouped gate/up and down (moe.cu); post as above
#include <math.h>
#include <string.h>

#include <algorithm>
#include <cmath>
#include <memory>

#include "model.h"

namespace {

constexpr uint32_t MOE_ROWS_IN_ORDER = 8;  // so many (token, expert) pairs run row by row, more are grouped by expert

constexpr uint32_t round_up(uint32_t v, uint32_t m) { return (v + m - 1) / m * m; }
constexpr bool recurrent_kind(uint32_t kind) { return kind == OB_MIXER_RETENTION || kind == OB_MIXER_STATE_SPACE || kind == OB_MIXER_TIME_MIXING; }

struct Dense {  // rows x kp bfloat16 on the device
    __nv_bfloat16 *w = nullptr;
    uint32_t rows = 0, kp = 0;
};

struct MixerPlan {
    ob_mixer_desc mx{};  // sizes and constants only
    float scale = 1.0f;  // of its output
    Dense in;            // projections of the block's input
    float *in_bias = nullptr;
    Rot rot{};
    // rows of `in`: [activations (unrotated queries; values, gates; the state space's gate) | f32 projections]
    uint32_t act_rows = 0, f32_row0 = 0, f32_rows = 0;
    uint32_t cols = 0, col0 = 0;  // columns of its output in the out product's input, and the first of them
    uint32_t out_width = 0;       // of its output
    // attention
    float *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr;
    uint32_t vdim_p = 0, row = 0, gate0 = 0;  // row: elements of a cache row per key/value head
    bool has_v = false, has_gate = false, head_gate = false, own_kv = true;  // gates: of every output, or of whole heads
    // latent attention
    Dense uk, uv;        // per head [kv_rank <- dim], [vdim <- kv_rank]
    Dense expand;        // latent -> keys [H][dim_k], then (from row ex_v0) values [H][vdim_k]; no rows: prompts attend in the latent space too
    bool paged = false;  // prompts' keys and values go into pages, per head (keys, from row ex_v0 values)
    uint32_t dim_p = 0, kv_p = 0, dq = 0, kv_w = 0, dim_k = 0, vdim_k = 0, ex_v0 = 0;
    float *kv_norm = nullptr;
    void *pool = nullptr;
    // recurrent layers: the state, and the last inputs of the convolution or of the token shift
    float *state = nullptr, *tail = nullptr;
    uint32_t tail_elems = 0;  // per slot
    // retention
    float *decay = nullptr;
    float decay_min = 0.0f;
    // state space
    float *conv_w = nullptr, *conv_b = nullptr, *dt_bias = nullptr, *a_log = nullptr, *skip = nullptr, *out_norm = nullptr;
    // time mixing: r, k, v and gate one after the other, equally many rows each
    Dense rkvg, decay1, decay2;
    float *mu[SHIFT_MIXES] = {}, *decay0 = nullptr, *bonus = nullptr;

    uint32_t channels() const { return mx.n_head * mx.vdim + 2 * mx.n_group * mx.dim; }  // of the convolution
};

struct LayerPlan : MixerPlan {
    std::unique_ptr<MixerPlan> second;
    float norm_gain = 0.0f, glu_limit = 0.0f, glu_alpha = 0.0f;
    uint32_t n_ff = 0, glu_row0 = 0;  // parallel blocks: gate/up rows of `in`, after the mixer's
    Dense out, side_gate, side_proj;
    bool sequential = false;
    float *out_bias = nullptr, *pre1 = nullptr, *pre2 = nullptr, *post1 = nullptr, *post2 = nullptr;
    // plain sums: convolution of the two sublayers' inputs [taps][width] and its last inputs per slot; factors of the average over depth
    float *conv_in[2] = {}, *tail_in[2] = {}, *depth = nullptr;
    uint32_t ff_kind = 0, n_expert = 0, top = 1;
    uint32_t n_shared = 0;  // pieces of the shared expert, each of an expert's size
    Dense up, down, router;  // feed-forward of a sequential block, one after the other for every expert (gate and up rows interleaved)
    uint32_t score_of = 0, n_group = 1, keep_group = 1;
    float router_scale = 1.0f;
    float *side_norm = nullptr;

    uint32_t pairs() const { return top + n_shared; }  // experts of a token
};

// A zero-padded bfloat16 matrix put together on the host from parts of others.
struct HostDense {
    uint32_t rows, kp;
    std::vector<uint16_t> v;
    HostDense(uint32_t r, uint32_t k) : rows(r), kp(k), v((size_t)r * k, 0) {}
    void copy(uint32_t row, uint32_t col, const ob_matrix_desc &src, uint32_t src_row) { copy(row, col, src, src_row, 0, src.in_dim); }
    void copy(uint32_t row, uint32_t col, const ob_matrix_desc &src, uint32_t src_row, uint32_t src_col, uint32_t n) {
        memcpy(v.data() + (size_t)row * kp + col, src.data + ((size_t)src_row * src.in_dim + src_col) * 2, (size_t)n * 2);
    }
};

struct LayeredGraph : StepGraph {
    ob_model *m = nullptr;
    bool f32 = false, has_state = false;
    uint32_t width = 0, h_pitch = 0, side_dim = 0, side_p = 0, y_pitch = 0, cat_pitch = 0;
    float eps = 0.0f, final_gain = 0.0f, residual_mult = 1.0f;
    // plain sums: embeddings and results of the layers, inverse root mean squares of groups
    bool plain = false;
    uint32_t n_group = 1, taps = 0;
    float *history = nullptr, *inverse = nullptr;
    float *final_norm = nullptr;
    std::vector<LayerPlan> L;
    __nv_bfloat16 *embd = nullptr, *side_embd = nullptr;
    Dense output;
    void *mix = nullptr;                    // time mixing: the mixes of every row, and the low-rank half of the decay
    void *low = nullptr;
    float *conv = nullptr, *decays = nullptr;
    float2 *steps = nullptr;
    uint32_t low_p = 0;
    void *h = nullptr, *xb = nullptr, *qn = nullptr, *q = nullptr, *o_lat = nullptr, *cat = nullptr, *sg = nullptr;
    float *y = nullptr, *o_ret = nullptr, *sy = nullptr, *part = nullptr;
    void *lat = nullptr, *expanded = nullptr;  // gathered latents of prompts, their keys and values: key_cap rows
    uint32_t key_cap = 0;
    int32_t *numbers = nullptr;                // tables of pages that lie in order
    const int32_t **page_tables = nullptr;
    void *ffa = nullptr;      // feed-forward activations of sequential blocks, a row per token or (token, expert) pair
    float *yo = nullptr;      // their outputs, and the mixers'
    MoeArgs moe{};            // routing buffers
    float *router_logits = nullptr;
    uint64_t part_cap = 0;
    float *split_part = nullptr;
    bool failed = false;  // a product could not be launched

    size_t es() const { return f32 ? 4 : 2; }
    void *column(uint32_t c) const { return static_cast<uint8_t *>(cat) + c * es(); }  // of the out product's input
    bool recurrent() const override { return has_state; }
    bool take_failure() override {
        const bool f = failed;
        failed = false;
        return f;
    }

    void linear(const LinArgs &a, cudaStream_t st) {
        const uint32_t n = launch_linear(a, f32, m->ctx->sm_count, st);
        if (!n) failed = true;
        m->ctx->launches += n;
    }
    LinArgs product(const Dense &w, const void *x, uint32_t x_pitch, uint32_t T) const {
        LinArgs a{};
        a.w = w.w;
        a.n_rows = w.rows;
        a.kp = w.kp;
        a.x = x;
        a.x_pitch = x_pitch;
        a.T = T;
        a.n_batch = 1;
        a.split_part = split_part;
        return a;
    }
    static void segment(LinArgs &a, uint32_t row0, uint32_t n, int epi, void *out, uint32_t pitch, uint32_t col0 = 0, uint32_t batch_cols = 0) {
        if (n) a.seg[a.n_seg++] = LinSegment{row0, n, epi, out, pitch, col0, batch_cols};
    }

    void layers(uint32_t T, uint32_t n_seq, const RowSpan *spans, uint32_t max_pos, cudaStream_t st) override;
    void head(const uint32_t *d_rows, uint32_t n, cudaStream_t st) override;
    void latent(const MixerPlan &P, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, uint32_t max_pos, cudaStream_t st);
    void prompt_in_pages(const MixerPlan &P, const float *head_gate, const LatentArgs &l, uint32_t n_keys, uint32_t s0, uint32_t s1, cudaStream_t st);
    void retention(const MixerPlan &P, uint32_t T, uint32_t n_seq, const RowSpan *spans, cudaStream_t st);
    void state_space(const MixerPlan &P, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, cudaStream_t st);
    void time_mixing(const MixerPlan &P, const float *norm, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, cudaStream_t st);
    void recurrence(const MixerPlan &P, RecurrenceArgs a, uint32_t n_seq, const RowSpan *spans, cudaStream_t st);
    void attention(const MixerPlan &P, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, uint32_t max_pos, cudaStream_t st);
    void project(const MixerPlan &P, uint32_t T, cudaStream_t st);
    void mixer(const MixerPlan &P, const float *norm, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, uint32_t max_pos, cudaStream_t st);
    void sequential(const LayerPlan &P, const LayerPlan *next, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, uint32_t max_pos, cudaStream_t st);
    struct Added {  // what a sublayer leaves in yo: `top` rows per token
        uint32_t top = 1;
        const uint32_t *rows = nullptr;  // where they are; null: in order
        uint32_t n_zero = 0;             // of moe.count, to be zeroed
    };
    struct Step {
        uint32_t T, n_seq;
        const RowSpan *spans;
        bool single;
    };
    Added feed_forward(const LayerPlan &P, uint32_t T, cudaStream_t st);
    void post(const float *w, uint32_t T, bool last, const float *next, const Added &y, cudaStream_t st);
    ResidualArgs residual_step(const Step &s) const;
    void read_by(ResidualArgs &r, const LayerPlan &P, int sublayer) const;
    void add(const LayerPlan &P, const LayerPlan *next, int sublayer, const Added &y, const Step &s, cudaStream_t st);
    void residual(const ResidualArgs &r, cudaStream_t st) { m->ctx->launches += launch_residual(r, f32, st); }
    float *result(size_t i) const { return history + i * (size_t)m->T * width; }  // embeddings, then the results of the layers
    uint32_t in_state() const { return taps > 1 ? (taps - 1) * width : 0; }         // of one input's convolution, per slot
    uint32_t cache_elems(const MixerPlan &P) const { return P.mx.kind == OB_MIXER_ATTENTION ? P.mx.n_kv_head * P.row : P.dq; }  // per position
    int copy_prefix(ob_kv *dst, const ob_kv *src, uint32_t n) override;
    int read_pages(const ob_kv *kv, uint32_t layer, uint32_t pos0, uint32_t n, float *k_out, float *v_out) override;
    int read_state(const ob_kv *kv, uint32_t layer, float *out) override;
    size_t state_elems(const MixerPlan &P) const { return (size_t)P.mx.n_head * P.mx.dim * P.mx.vdim; }
    // The mixers of all layers.
    template <typename F> void each_mixer(F f) {
        for (LayerPlan &P : L) {
            f(static_cast<MixerPlan &>(P));
            if (P.second) f(*P.second);
        }
    }

    int upload(const HostDense &src, Dense *out) {
        int rc = dev_alloc(m, &out->w, src.v.size());
        if (rc) return rc;
        out->rows = src.rows;
        out->kp = src.kp;
        OB_CUDA(m->ctx, cudaMemcpy(out->w, src.v.data(), src.v.size() * 2, cudaMemcpyHostToDevice));
        return OB_OK;
    }
    int scratch(void **p, size_t elems, size_t elem_bytes) {  // zeroed: padding columns stay finite
        uint8_t *b = nullptr;
        int rc = dev_alloc(m, &b, elems * elem_bytes);
        if (rc) return rc;
        OB_CUDA(m->ctx, cudaMemset(b, 0, std::max<size_t>(elems * elem_bytes, 16)));
        *p = b;
        return OB_OK;
    }
    int scratch_f32(float **p, size_t elems) {
        void *v = nullptr;
        int rc = scratch(&v, elems, 4);
        *p = static_cast<float *>(v);
        return rc;
    }
    int build(const ob_layered_desc &c);
    int build_layer(const ob_block_desc &b, LayerPlan &P);
    void size_mixer(const ob_mixer_desc &x, MixerPlan &P) const;
    int fill_in(const ob_mixer_desc &x, MixerPlan &P, HostDense &in);
    int build_mixer(const ob_mixer_desc &x, MixerPlan &P);
    int build_ff(const ob_block_desc &b, LayerPlan &P);
    int rotation(MixerPlan &P, std::map<std::pair<std::vector<double>, float>, float2 *> &tables);
    int upload_now(const float *src, size_t n, float **out, float gain = 1.0f) {  // the source may end with the caller
        std::vector<float> scaled(src, src + n);
        for (float &v : scaled) v *= gain;
        int rc = dev_alloc(m, out, n);
        if (rc) return rc;
        OB_CUDA(m->ctx, cudaMemcpy(*out, scaled.data(), n * 4, cudaMemcpyHostToDevice));
        return OB_OK;
    }
};

// Spans of a step come with the long ones last (forward_spans).
uint32_t first_long(const RowSpan *spans, uint32_t n_seq) {
    while (n_seq && spans[n_seq - 1].n >= PREFILL_SPAN) --n_seq;
    return n_seq;
}

void LayeredGraph::latent(const MixerPlan &P, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, uint32_t max_pos, cudaStream_t st) {
    const MetaLayout ml(m->T);
    const uint32_t H = P.mx.n_head;
    LatentArgs a{};
    a.y = y;
    a.y_pitch = y_pitch;
    a.n_head = H;
    a.kv_rank = P.mx.kv_rank;
    a.rot_dim = P.mx.rot_dim;
    a.window = P.mx.window;
    a.kv_p = P.kv_p;
    a.dq = P.dq;
    a.eps = eps;
    a.scale = P.mx.scale;
    a.sink = P.sink;
    a.kv_norm = P.kv_norm;
    a.rot = P.rot;
    a.q = q;
    a.cache = P.pool;
    a.o = o_lat;
    a.o_head = P.kv_w;
    a.part = part;
    a.part_cap = part_cap;
    a.T = T;
    a.n_seq = n_seq;
    a.spans = reinterpret_cast<const RowSpan *>(m->d_meta + ml.off_spans);
    a.h_spans = spans;
    a.single = single;
    a.positions = reinterpret_cast<const uint32_t *>(m->d_meta + ml.off_positions);
    a.tables = reinterpret_cast<const int32_t *const *>(m->d_meta + ml.off_tables);
    a.max_pos = max_pos;
    launch_latent_prep(a, f32, st);
    m->ctx->launches++;
    const uint32_t n_short = P.expand.rows ? first_long(spans, n_seq) : n_seq;  // spans that attend in the latent space
    const float *gate = P.head_gate ? y + (size_t)H * P.mx.rot_dim + P.mx.kv_rank + P.mx.rot_dim : nullptr;
    const void *gate_act = P.has_gate ? static_cast<const uint8_t *>(qn) + P.gate0 * es() : nullptr;
    const uint32_t gate_pitch = P.has_gate ? P.act_rows : y_pitch;
    if (n_short) {
        a.n_seq = n_short;
        LinArgs uk = product(P.uk, qn, P.act_rows, T);  // head h: its unrotated query through the key up-projection
        uk.n_rows = P.uk.rows / H;
        uk.n_batch = H;
        uk.x_step = P.dim_p;
        segment(uk, 0, P.mx.kv_rank, LE_ACT, q, H * P.dq, 0, P.dq);
        linear(uk, st);
        m->ctx->launches += launch_latent_attention(a, f32, m->ctx->sm_count, st);
        LinArgs uv = product(P.uv, o_lat, H * P.kv_w, T);
        uv.n_rows = P.uv.rows / H;
        uv.n_batch = H;
        uv.x_step = P.kv_w;
        uv.gate = gate;
        uv.gate_act = gate_act;
        uv.gate_pitch = gate_pitch;
        segment(uv, 0, P.mx.vdim, gate ? LE_GATED : gate_act ? LE_GATED_EACH : LE_ACT, cat, cat_pitch, 0, P.mx.vdim);
        linear(uv, st);
    }
    LatentPrefillArgs p{};
    p.n_head = H;
    p.vdim = P.mx.vdim;
    p.window = P.mx.window;
    p.dim_k = P.dim_k;
    p.vdim_k = P.vdim_k;
    p.kv_p = P.kv_p;
    p.dq = P.dq;
    p.dim_p = P.dim_p;
    p.scale = P.mx.scale;
    p.tables = a.tables;
    p.cache = P.pool;
    p.lat = lat;
    p.expanded = expanded;
    p.ex_pitch = P.expand.rows;
    p.ex_v0 = P.ex_v0;
    p.qn = qn;
    p.qn_pitch = P.act_rows;
    p.q = q;
    p.gate = gate;
    p.gate_act = gate_act;
    p.gate_pitch = gate_pitch;
    p.sink = P.sink;
    p.out = cat;
    p.out_pitch = cat_pitch;
    const uint32_t *h_pos = reinterpret_cast<const uint32_t *>(m->h_meta + ml.off_positions);
    if (P.paged) {
        p.pages = expanded;
        p.page_row = P.row;
        p.page_rot0 = P.dim_k;
        p.numbers = numbers;
        p.page_tables = page_tables;
    }
    const uint32_t unit = P.paged ? KV_PAGE : 1;
    for (uint32_t s = n_short; s < n_seq;) {  // as many spans at a time as the buffers hold
        const uint32_t s0 = s;
        p.n_span = p.n_keys = p.n_tiles = 0;
        for (; s < n_seq && p.n_span < PREFILL_GROUP; ++s) {
            const uint32_t pos0 = h_pos[spans[s].row0], from = P.mx.window && pos0 >= P.mx.window ? pos0 - P.mx.window + 1 : 0, hist = pos0 - from / unit * unit;
            const uint32_t keys = round_up(hist + spans[s].n, unit);
            if (p.n_span && p.n_keys + keys > key_cap) break;
            p.span[p.n_span++] = PrefillSpan{spans[s].row0, spans[s].n, pos0, hist, p.n_keys, p.n_tiles};
            p.n_keys += keys;
            p.n_tiles += latent_prefill_tiles(spans[s].n);
        }
        launch_latent_gather(p, st);
        if (P.paged) {
            prompt_in_pages(P, gate, a, p.n_keys, s0, s, st);
            continue;
        }
        LinArgs ex = product(P.expand, lat, P.dq, p.n_keys);
        segment(ex, 0, P.expand.rows, LE_ACT, expanded, P.expand.rows);
        linear(ex, st);
        launch_latent_prefill(p, st);
        m->ctx->launches += 2;
    }
}

// Latent attention of spans [s0, s1): the gathered latents become pages of one key/value head per head, which are attended as such.
void LayeredGraph::prompt_in_pages(const MixerPlan &P, const float *head_gate, const LatentArgs &l, uint32_t n_keys, uint32_t s0, uint32_t s1, cudaStream_t st) {
    const uint32_t H = P.mx.n_head;
    LinArgs ex = product(P.expand, lat, P.dq, n_keys);
    ex.n_rows = P.expand.rows / H;
    ex.n_batch = H;
    segment(ex, 0, P.dim_k, LE_ACT, expanded, P.row, 0, KV_PAGE * P.row);
    segment(ex, P.ex_v0, P.vdim_k, LE_ACT, expanded, P.row, P.dim_k + P.dq - P.kv_p, KV_PAGE * P.row);
    for (int i = 0; i < 2; ++i) ex.seg[i].page_pitch = H * KV_PAGE * P.row;
    linear(ex, st);
    AttentionArgs a{};
    a.y_pitch = y_pitch;
    a.va = qn;
    a.va_pitch = P.act_rows;
    a.gate0 = P.gate0;
    a.has_gate = P.has_gate;
    a.n_head = a.n_kv = H;
    a.n_map = 1;
    a.vdim = P.mx.vdim;
    a.window = P.mx.window;
    a.dim_p = P.dim_k + P.dq - P.kv_p;
    a.vdim_p = P.vdim_k;
    a.row = P.row;
    a.scale = P.mx.scale;
    a.head_gain = 1.0f;
    a.sink = P.sink;
    a.head_gate = head_gate;
    a.q = qn;
    a.q2 = static_cast<uint8_t *>(q) + P.kv_p * es();
    a.q_split = P.dim_k;
    a.q_pitch = P.act_rows;
    a.q_head = P.dim_p;
    a.q2_pitch = H * P.dq;
    a.q2_head = P.dq;
    a.cache = expanded;
    a.n_pages = key_cap / KV_PAGE;
    a.out = cat;
    a.out_pitch = cat_pitch;
    a.T = l.T;
    a.n_seq = s1;
    a.n_short = s0;
    a.spans = l.spans;
    a.h_spans = l.h_spans;
    a.positions = l.positions;
    a.tables = page_tables;
    a.max_pos = l.max_pos;
    if (!launch_attention_prompt(a, m->ctx->sm_count, st)) failed = true;
    m->ctx->launches += 2;
}

void LayeredGraph::retention(const MixerPlan &P, uint32_t T, uint32_t n_seq, const RowSpan *spans, cudaStream_t st) {
    const MetaLayout ml(m->T);
    RetentionArgs a{};
    a.y = y;
    a.y_pitch = y_pitch;
    a.n_head = P.mx.n_head;
    a.dim = P.mx.dim;
    a.vdim = P.mx.vdim;
    a.eps = eps;
    a.k_scale = 1.0f / sqrtf((float)P.mx.dim);
    a.decay = P.decay;
    a.rot = P.rot;
    a.state = P.state;
    a.o = o_ret;
    a.out = cat;
    a.out_pitch = cat_pitch;
    a.T = T;
    a.n_seq = n_seq;
    a.spans = reinterpret_cast<const RowSpan *>(m->d_meta + ml.off_spans);
    a.positions = reinterpret_cast<const uint32_t *>(m->d_meta + ml.off_positions);
    a.slots = reinterpret_cast<const int32_t *>(m->d_meta + ml.off_slots);
    a.first_long = first_long(spans, n_seq);
    a.decay_min = P.decay_min;
    m->ctx->launches += launch_retention(a, f32, m->ctx->sm_count, st);
}

void LayeredGraph::attention(const MixerPlan &P, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, uint32_t max_pos, cudaStream_t st) {
    const MetaLayout ml(m->T);
    AttentionArgs a{};
    a.y = y;
    a.y_pitch = y_pitch;
    a.va = qn;
    a.va_pitch = P.act_rows;
    a.gate0 = P.gate0;
    a.has_v = P.has_v;
    a.has_gate = P.has_gate;
    a.n_head = P.mx.n_head;
    a.n_kv = P.mx.n_kv_head;
    a.n_map = P.mx.n_map;
    a.dim = P.mx.dim;
    a.vdim = P.mx.vdim;
    a.window = P.mx.window;
    a.dim_p = P.dim_p;
    a.vdim_p = P.vdim_p;
    a.row = P.row;
    a.eps = eps;
    a.scale = P.mx.scale;
    a.map_weight = P.mx.map_weight;
    a.head_gain = P.mx.n_map == 2 ? P.mx.head_gain : P.scale;
    a.norm_whole = P.mx.qk_norm_whole != 0;
    a.own_kv = P.own_kv;
    a.keep = P.mx.window ? P.mx.keep_first : 0;
    a.softcap = P.mx.softcap;
    a.sink = P.sink;
    a.head_gate = P.head_gate ? y + P.f32_rows - P.mx.n_head : nullptr;
    a.q_norm = P.q_norm;
    a.k_norm = P.k_norm;
    a.rot = P.rot;
    a.q = q;
    a.cache = P.pool;
    a.n_pages = m->pool_pages;
    a.out = column(P.col0);
    a.out_pitch = cat_pitch;
    a.T = T;
    a.n_seq = n_seq;
    a.n_short = first_long(spans, n_seq);
    a.spans = reinterpret_cast<const RowSpan *>(m->d_meta + ml.off_spans);
    a.h_spans = spans;
    a.single = single;
    a.positions = reinterpret_cast<const uint32_t *>(m->d_meta + ml.off_positions);
    a.tables = reinterpret_cast<const int32_t *const *>(m->d_meta + ml.off_tables);
    a.max_pos = max_pos;
    launch_attention_prep(a, f32, st);
    const uint32_t n = launch_attention(a, f32, m->ctx->sm_count, st);
    if (!n) failed = true;
    m->ctx->launches += 1 + n;
}

void LayeredGraph::recurrence(const MixerPlan &P, RecurrenceArgs a, uint32_t n_seq, const RowSpan *spans, cudaStream_t st) {
    const MetaLayout ml(m->T);
    a.n_head = P.mx.n_head;
    a.dim = P.mx.dim;
    a.vdim = P.mx.vdim;
    a.state = P.state;
    a.o = o_ret;
    a.n_seq = n_seq;
    a.first_long = first_long(spans, n_seq);
    a.spans = reinterpret_cast<const RowSpan *>(m->d_meta + ml.off_spans);
    a.positions = reinterpret_cast<const uint32_t *>(m->d_meta + ml.off_positions);
    a.slots = reinterpret_cast<const int32_t *>(m->d_meta + ml.off_slots);
    m->ctx->launches += launch_recurrence(a, m->ctx->sm_count, st);
}

// Rows of `in`: gate as activations; channels of the convolution and raw steps in y.
void LayeredGraph::state_space(const MixerPlan &P, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, cudaStream_t st) {
    const MetaLayout ml(m->T);
    const uint32_t inner = P.mx.n_head * P.mx.vdim, n = P.channels();
    ConvArgs c{};
    c.y = y;
    c.y_pitch = y_pitch;
    c.n_channel = n;
    c.taps = P.mx.conv_taps;
    c.n_head = P.mx.n_head;
    c.w = P.conv_w;
    c.b = P.conv_b;
    c.state = P.tail;
    c.u = conv;
    c.dt_bias = P.dt_bias;
    c.a_log = P.a_log;
    c.step = steps;
    c.T = T;
    c.n_seq = n_seq;
    c.spans = reinterpret_cast<const RowSpan *>(m->d_meta + ml.off_spans);
    c.h_spans = spans;
    c.single = single;
    c.positions = reinterpret_cast<const uint32_t *>(m->d_meta + ml.off_positions);
    c.slots = reinterpret_cast<const int32_t *>(m->d_meta + ml.off_slots);
    launch_conv(c, st);
    RecurrenceArgs r{};
    r.v = conv;
    r.k = conv + inner;
    r.q = conv + inner + (size_t)P.mx.n_group * P.mx.dim;
    r.pitch = n;
    r.share = P.mx.n_head / P.mx.n_group;
    r.step = steps;
    recurrence(P, r, n_seq, spans, st);
    StateSpaceOutArgs o{};
    o.o = o_ret;
    o.x = conv;
    o.x_pitch = n;
    o.z = qn;
    o.z_pitch = P.act_rows;
    o.inner = inner;
    o.vdim = P.mx.vdim;
    o.n_part = P.mx.n_norm_group;
    o.T = T;
    o.skip = P.skip;
    o.norm = P.out_norm;
    o.eps = eps;
    o.out = column(P.col0);
    o.out_pitch = cat_pitch;
    launch_state_space_out(o, f32, st);
    m->ctx->launches += 2;
}

void LayeredGraph::time_mixing(const MixerPlan &P, const float *norm, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, cudaStream_t st) {
    const MetaLayout ml(m->T);
    const uint32_t n = P.mx.n_head * P.mx.dim;
    ShiftMixArgs s{};
    s.x = m->x;
    s.norm = norm;
    for (uint32_t i = 0; i < SHIFT_MIXES; ++i) s.mu[i] = P.mu[i];
    s.state = P.tail;
    s.mix = mix;
    s.width = width;
    s.pitch = h_pitch;
    s.T = T;
    s.n_seq = n_seq;
    s.eps = eps;
    s.spans = reinterpret_cast<const RowSpan *>(m->d_meta + ml.off_spans);
    s.single = single;
    s.positions = reinterpret_cast<const uint32_t *>(m->d_meta + ml.off_positions);
    s.slots = reinterpret_cast<const int32_t *>(m->d_meta + ml.off_slots);
    launch_shift_mix(s, f32, st);
    LinArgs p = product(P.rkvg, mix, SHIFT_MIXES * h_pitch, T);  // mixes of r, k, v, gate with a matrix each
    p.n_rows = P.rkvg.rows / 4;
    p.n_batch = 4;
    p.x_step = h_pitch;
    segment(p, 0, n, LE_F32, y, y_pitch, 0, n);
    linear(p, st);
    LinArgs d1 = product(P.decay1, static_cast<uint8_t *>(mix) + 4 * h_pitch * es(), SHIFT_MIXES * h_pitch, T);
    segment(d1, 0, P.mx.w_decay1.out_dim, LE_TANH, low, P.decay2.kp);
    linear(d1, st);
    LinArgs d2 = product(P.decay2, low, P.decay2.kp, T);
    d2.bias = P.decay0;
    segment(d2, 0, n, LE_DECAY, decays, n);
    linear(d2, st);
    RecurrenceArgs r{};
    r.q = y;
    r.k = y + n;
    r.v = y + 2 * n;
    r.pitch = y_pitch;
    r.share = 1;
    r.w = decays;
    r.w_pitch = n;
    recurrence(P, r, n_seq, spans, st);
    TimeMixOutArgs o{};
    o.o = o_ret;
    o.r = y;
    o.k = y + n;
    o.v = y + 2 * n;
    o.gate = y + 3 * n;
    o.pitch = y_pitch;
    o.n_head = P.mx.n_head;
    o.dim = P.mx.dim;
    o.T = T;
    o.bonus = P.bonus;
    o.norm = P.out_norm;
    o.eps = eps;
    o.out = column(P.col0);
    o.out_pitch = cat_pitch;
    launch_time_mix_out(o, f32, st);
    m->ctx->launches += 2;
}

// The projections of a sequential block's input.
void LayeredGraph::project(const MixerPlan &P, uint32_t T, cudaStream_t st) {
    if (!P.in.rows) return;
    LinArgs in = product(P.in, h, h_pitch, T);
    in.bias = P.in_bias;
    segment(in, 0, P.act_rows, LE_ACT, qn, P.act_rows);
    segment(in, P.f32_row0, P.f32_rows, LE_F32, y, y_pitch);
    linear(in, st);
}

// norm: of the block's input h, which a time-mixing layer makes itself.
void LayeredGraph::mixer(const MixerPlan &P, const float *norm, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, uint32_t max_pos, cudaStream_t st) {
    switch (P.mx.kind) {
    case OB_MIXER_LATENT_ATTENTION: return latent(P, T, n_seq, spans, single, max_pos, st);
    case OB_MIXER_ATTENTION: return attention(P, T, n_seq, spans, single, max_pos, st);
    case OB_MIXER_STATE_SPACE: return state_space(P, T, n_seq, spans, single, st);
    case OB_MIXER_TIME_MIXING: return time_mixing(P, norm, T, n_seq, spans, single, st);
    default: return retention(P, T, n_seq, spans, st);
    }
}

void LayeredGraph::post(const float *w, uint32_t T, bool last, const float *next, const Added &y, cudaStream_t st) {
    PostNormArgs p{};
    p.x = m->x;
    p.y = yo;
    p.rows = y.rows;
    p.top = y.top;
    p.w = w;
    p.width = width;
    p.T = T;
    p.eps = eps;
    p.mult = residual_mult;
    p.h = last ? nullptr : h;
    p.h_pitch = h_pitch;
    p.next_w = next;
    p.zero = y.n_zero ? moe.count : nullptr;
    p.n_zero = y.n_zero;
    launch_post_norm(p, f32, st);
    m->ctx->launches++;
}

ResidualArgs LayeredGraph::residual_step(const Step &s) const {
    const MetaLayout ml(m->T);
    ResidualArgs r{};
    r.mult = residual_mult;
    r.n_group = n_group;
    r.eps = eps;
    r.inverse = inverse;
    r.h = h;
    r.h_pitch = h_pitch;
    r.width = width;
    r.T = s.T;
    r.n_seq = s.n_seq;
    r.spans = reinterpret_cast<const RowSpan *>(m->d_meta + ml.off_spans);
    r.h_spans = s.spans;
    r.single = s.single;
    r.positions = reinterpret_cast<const uint32_t *>(m->d_meta + ml.off_positions);
    r.slots = reinterpret_cast<const int32_t *>(m->d_meta + ml.off_slots);
    return r;
}

// The input of a sublayer: 0 the mixer, 1 the feed-forward.
void LayeredGraph::read_by(ResidualArgs &r, const LayerPlan &P, int sublayer) const {
    r.norm = sublayer ? P.pre2 : P.pre1;
    r.conv = P.conv_in[sublayer];
    r.taps = taps;
    r.state = P.tail_in[sublayer];
}

// Plain sums: a sublayer's output joins the residual, which becomes the input of the next one.
void LayeredGraph::add(const LayerPlan &P, const LayerPlan *next, int sublayer, const Added &y, const Step &s, cudaStream_t st) {
    const bool end = sublayer == 1 || !P.n_ff;
    ResidualArgs r = residual_step(s);
    const size_t i = &P - L.data();
    r.x = i == 0 && sublayer == 0 && history ? history : m->x;
    r.y = yo;
    r.top = y.top;
    r.rows = y.rows;
    r.zero = y.n_zero ? moe.count : nullptr;
    r.n_zero = y.n_zero;
    if (end && P.depth) {
        r.depth = P.depth;
        r.history = history;
        r.history_step = (uint64_t)m->T * width;
        r.n_history = (uint32_t)i + 1;
        r.sum = next ? result(i + 1) : nullptr;
        r.average = m->x;
    } else {
        r.sum = m->x;
    }
    if (!end) read_by(r, P, 1);
    else if (next) read_by(r, *next, 0);
    residual(r, st);
}

// next: the block that follows, null after the last one.
void LayeredGraph::sequential(const LayerPlan &P, const LayerPlan *next, uint32_t T, uint32_t n_seq, const RowSpan *spans, bool single, uint32_t max_pos, cudaStream_t st) {
    const float *next_pre = next ? next->pre1 : nullptr;
    const Step step{T, n_seq, spans, single};
    project(P, T, st);
    mixer(P, P.pre1, T, n_seq, spans, single, max_pos, st);
    if (P.second) {
        project(*P.second, T, st);
        mixer(*P.second, P.pre1, T, n_seq, spans, single, max_pos, st);
    }
    LinArgs out = product(P.out, cat, cat_pitch, T);
    out.bias = P.out_bias;
    segment(out, 0, width, LE_F32, yo, width);
    linear(out, st);
    if (plain) add(P, next, 0, Added{}, step, st);
    else post(P.post1, T, !next && !P.n_ff, P.n_ff ? P.pre2 : next_pre, Added{}, st);
    if (!P.n_ff) return;
    const Added y = feed_forward(P, T, st);
    if (plain) add(P, next, 1, y, step, st);
    else post(P.post2, T, !next, next_pre, y, st);
}

// h through the feed-forward of a sequential block.
LayeredGraph::Added LayeredGraph::feed_forward(const LayerPlan &P, uint32_t T, cudaStream_t st) {
    if (P.ff_kind != OB_FF_EXPERTS) {
        LinArgs up = product(P.up, h, h_pitch, T);
        if (P.ff_kind == OB_FF_GELU_GLU) segment(up, 0, 2 * P.n_ff, LE_GELU_GLU, ffa, P.down.kp);
        else segment(up, 0, P.n_ff, LE_RELU2, ffa, P.down.kp);
        linear(up, st);
        LinArgs down = product(P.down, ffa, P.down.kp, T);
        segment(down, 0, width, LE_F32, yo, width);
        linear(down, st);
        return Added{};
    }
    const uint32_t R = T * P.pairs(), E = P.n_expert + P.n_shared, n_logit = P.n_expert + (P.n_shared > 0);
    const bool in_order = T == 1 || R <= MOE_ROWS_IN_ORDER;
    MoeArgs r = moe;
    r.x = h;
    r.x_pitch = h_pitch;
    r.w = P.router.w;
    r.n_expert = P.n_expert;
    r.top = P.top;
    r.n_shared = P.n_shared;
    r.score_of = P.score_of;
    r.scale = P.router_scale;
    r.n_group = P.n_group;
    r.keep = P.keep_group;
    r.T = T;
    r.tile_rows = linear_tile_rows(R, E, f32);
    if (in_order) r.count = nullptr;
    if (T > MOE_DOT_TOKENS) {
        LinArgs z = product(P.router, h, h_pitch, T);
        segment(z, 0, n_logit, LE_F32, router_logits, n_logit);
        linear(z, st);
        r.logits = router_logits;
        r.logit_pitch = n_logit;
    }
    m->ctx->launches += launch_moe_route(r, f32, st);
    auto grouped = [&](const Dense &w, const void *x, uint32_t x_div) {
        LinArgs a = product(w, x, w.kp, R);
        a.n_rows = w.rows / E;
        a.n_batch = E;
        if (in_order) {
            a.row_batch = r.expert;
            a.x_div = x_div;
        } else {
            a.tiles = r.tiles;
            a.n_tiles = r.n_tiles;
            a.tile_rows = r.tile_rows;
            a.max_tiles = R / r.tile_rows + std::min(R, E);
        }
        return a;
    };
    LinArgs up = grouped(P.up, in_order ? h : r.gathered, P.pairs());
    (P.score_of != OB_ROUTER_SIGMOID ? up.out_scale : up.row_scale) = in_order ? r.score : r.row_score;
    segment(up, 0, 2 * P.n_ff, LE_SWIGLU, ffa, P.down.kp);
    linear(up, st);
    LinArgs down = grouped(P.down, ffa, 1);
    segment(down, 0, width, LE_F32, yo, width);
    linear(down, st);
    return Added{P.pairs(), in_order ? nullptr : r.row, in_order ? 0 : E};
}

void LayeredGraph::layers(uint32_t T, uint32_t n_seq, const RowSpan *spans, uint32_t max_pos, cudaStream_t st) {
    const MetaLayout ml(m->T);
    const uint32_t *tokens = reinterpret_cast<const uint32_t *>(m->d_meta + ml.off_tokens);
    const bool single = n_seq == T;
    if (plain) {
        ResidualArgs r = residual_step(Step{T, n_seq, spans, single});
        r.table = embd;
        r.tokens = tokens;
        r.sum = history ? history : m->x;
        read_by(r, L[0], 0);
        residual(r, st);
    } else {
        launch_embed(embd, width, tokens, T, m->x, !L[0].sequential || L[0].pre1, eps, L[0].sequential ? 1.0f : L[0].norm_gain, L[0].pre1, h, h_pitch, f32, st);
        m->ctx->launches++;
    }
    for (size_t li = 0; li < L.size(); ++li) {
        const LayerPlan &P = L[li];
        const bool last = li + 1 == L.size();
        if (P.sequential) {
            sequential(P, last ? nullptr : &L[li + 1], T, n_seq, spans, single, max_pos, st);
            continue;
        }
        LinArgs in = product(P.in, h, h_pitch, T);
        segment(in, 0, P.act_rows, LE_ACT, qn, P.act_rows);
        segment(in, P.f32_row0, P.f32_rows, LE_F32, y, y_pitch);
        in.bias = P.in_bias;
        segment(in, P.glu_row0, 2 * P.n_ff, LE_GLU, cat, cat_pitch, P.cols);
        in.glu_limit = P.glu_limit;
        in.glu_alpha = P.glu_alpha;
        linear(in, st);

        mixer(P, nullptr, T, n_seq, spans, single, max_pos, st);

        LinArgs out = product(P.out, cat, cat_pitch, T);
        segment(out, 0, width, LE_RESIDUAL, m->x, width);
        out.bias = P.out_bias;
        if (side_dim) {
            out.out2 = xb;
            out.out2_pitch = h_pitch;
        }
        linear(out, st);

        const float gain = last ? 0.0f : L[li + 1].norm_gain;
        if (side_dim) {
            LinArgs g = product(P.side_gate, xb, h_pitch, T);
            segment(g, 0, side_dim, LE_GELU_EMB, sg, side_p);
            g.tokens = tokens;
            g.emb = side_embd;
            g.emb_pitch = (uint32_t)L.size() * side_dim;
            g.emb_col0 = (uint32_t)li * side_dim;
            linear(g, st);
            LinArgs pr = product(P.side_proj, sg, side_p, T);
            segment(pr, 0, width, LE_F32, sy, width);
            linear(pr, st);
            launch_side_finish(m->x, sy, P.side_norm, width, T, eps, gain, last ? nullptr : h, h_pitch, f32, st);
            m->ctx->launches++;
        } else if (!last) {
            launch_norm(m->x, width, nullptr, T, eps, gain, nullptr, h, h_pitch, f32, st);
            m->ctx->launches++;
        }
    }
}

void LayeredGraph::head(const uint32_t *d_rows, uint32_t n, cudaStream_t st) {
    if (plain) {
        ResidualArgs r = residual_step(Step{n, n, nullptr, true});
        r.x = m->x;
        r.x_rows = d_rows;
        r.norm = final_norm;
        residual(r, st);
    } else {
        launch_norm(m->x, width, d_rows, n, eps, final_gain, final_norm, h, h_pitch, f32, st);
        m->ctx->launches++;
    }
    LinArgs a = product(output, h, h_pitch, n);
    segment(a, 0, m->cfg.n_vocab, LE_F32, m->logits, m->cfg.n_vocab);
    linear(a, st);
}

int LayeredGraph::copy_prefix(ob_kv *dst, const ob_kv *src, uint32_t n) {
    cudaStream_t st = m->ctx->stream;
    int rc = OB_OK;
    auto copy = [&](float *p, size_t e) -> int {  // of one slot
        if (p && e && src->slot >= 0 && dst->slot >= 0)
            OB_CUDA(m->ctx, cudaMemcpyAsync(p + (size_t)dst->slot * e, p + (size_t)src->slot * e, e * 4, cudaMemcpyDeviceToDevice, st));
        return OB_OK;
    };
    each_mixer([&](MixerPlan &P) {
        if (P.pool && P.own_kv) {
            launch_copy_pages(P.pool, (uint64_t)KV_PAGE * cache_elems(P) * es(), src->d_table, dst->d_table, (n + KV_PAGE - 1) / KV_PAGE, st);
            m->ctx->launches++;
        } else if (!rc) {
            rc = copy(P.state, state_elems(P));
            if (!rc) rc = copy(P.tail, P.tail_elems);
        }
    });
    for (LayerPlan &P : L)
        for (float *tail : P.tail_in)
            if (!rc) rc = copy(tail, in_state());
    return rc;
}

int LayeredGraph::read_pages(const ob_kv *kv, uint32_t layer, uint32_t pos0, uint32_t n, float *k_out, float *v_out) {
    const MixerPlan &P = L[layer].pool || !L[layer].second ? L[layer] : *L[layer].second;
    if (!P.pool) return fail(m->ctx, OB_ERR_INVALID, "kv_read: the layer caches no positions");
    const bool latent = P.mx.kind == OB_MIXER_LATENT_ATTENTION;
    std::vector<uint8_t> row((latent ? P.dq : P.row) * es());
    const uint32_t heads = latent ? 1 : P.mx.n_kv_head;  // of a page, KV_PAGE rows each
    for (uint32_t i = 0; i < n; ++i)
        for (uint32_t g = 0; g < heads; ++g) {
            const uint32_t p = pos0 + i;
            const uint8_t *src = static_cast<const uint8_t *>(P.pool) + (((size_t)kv->pages[p / KV_PAGE] * heads + g) * KV_PAGE + p % KV_PAGE) * row.size();
            OB_CUDA(m->ctx, cudaMemcpy(row.data(), src, row.size(), cudaMemcpyDeviceToHost));
            auto copy = [&](float *dst, uint32_t col, uint32_t count) {
                for (uint32_t c = 0; c < count; ++c) {
                    if (f32) {
                        memcpy(dst + c, row.data() + 4 * (col + c), 4);
                    } else {
                        uint16_t b;
                        memcpy(&b, row.data() + 2 * (col + c), 2);
                        const uint32_t u = (uint32_t)b << 16;
                        memcpy(dst + c, &u, 4);
                    }
                }
            };
            if (latent) {
                copy(k_out + (size_t)i * P.mx.kv_rank, 0, P.mx.kv_rank);
                copy(v_out + (size_t)i * P.mx.rot_dim, P.kv_p, P.mx.rot_dim);
            } else {
                for (uint32_t map = 0; map < P.mx.n_map; ++map) copy(k_out + (((size_t)i * heads + g) * P.mx.n_map + map) * P.mx.dim, map * P.dim_p, P.mx.dim);
                copy(v_out + ((size_t)i * heads + g) * P.mx.vdim, P.mx.n_map * P.dim_p, P.mx.vdim);
            }
        }
    return OB_OK;
}

int LayeredGraph::read_state(const ob_kv *kv, uint32_t layer, float *out) {
    const MixerPlan *P = layer < L.size() ? &L[layer] : nullptr;
    if (P && !P->state) P = L[layer].second.get();
    if (!P && layer < L.size() && L[layer].tail_in[0]) {  // the last inputs of both sublayers
        const size_t e = in_state();
        for (int k = 0; k < 2 && L[layer].tail_in[k]; ++k) OB_CUDA(m->ctx, cudaMemcpy(out + k * e, L[layer].tail_in[k] + (size_t)kv->slot * e, e * 4, cudaMemcpyDeviceToHost));
        return OB_OK;
    }
    if (!P || !P->state) return fail(m->ctx, OB_ERR_INVALID, "state_read: the layer has no recurrent state");
    const size_t e = state_elems(*P);
    OB_CUDA(m->ctx, cudaMemcpy(out, P->state + (size_t)kv->slot * e, e * 4, cudaMemcpyDeviceToHost));
    return OB_OK;
}

// Sizes of a mixer's parts; nothing is allocated.
void LayeredGraph::size_mixer(const ob_mixer_desc &x, MixerPlan &P) const {
    const uint32_t H = x.n_head, G = x.n_kv_head;
    P.mx = x;
    switch (x.kind) {
    case OB_MIXER_LATENT_ATTENTION:
        P.dim_p = round_up(x.dim, LIN_K_ALIGN);
        P.kv_p = round_up(x.kv_rank, 16);
        P.dq = P.kv_p + round_up(x.rot_dim, 16);
        P.kv_w = round_up(x.kv_rank, LIN_K_ALIGN);
        P.head_gate = x.w_gate.data && x.w_gate.out_dim == H && x.vdim != 1;
        P.has_gate = x.w_gate.data && !P.head_gate;
        P.gate0 = H * P.dim_p;
        P.act_rows = P.gate0 + (P.has_gate ? round_up(H * x.vdim, LIN_ROW_ALIGN) : 0);
        P.f32_rows = H * x.rot_dim + x.kv_rank + x.rot_dim + (P.head_gate ? H : 0);
        break;
    case OB_MIXER_ATTENTION:
        P.own_kv = !x.kv_layer;
        P.has_v = x.wv.data != nullptr;
        P.head_gate = x.w_gate.data && x.w_gate.out_dim == H && x.vdim != 1;
        P.has_gate = x.w_gate.data && !P.head_gate;
        P.dim_p = round_up(x.dim, 16);
        P.vdim_p = round_up(x.vdim, 16);
        P.row = attention_cache_row(x.n_map, P.dim_p, P.vdim_p);
        P.gate0 = P.has_v ? G * x.vdim : 0;
        P.act_rows = round_up(P.gate0 + (P.has_gate ? H * x.vdim : 0), LIN_ROW_ALIGN);
        P.f32_rows = (H + (P.own_kv ? G : 0)) * x.n_map * x.dim + (P.head_gate ? H : 0);
        break;
    case OB_MIXER_STATE_SPACE:
        P.act_rows = round_up(H * x.vdim, LIN_ROW_ALIGN);
        P.f32_rows = P.channels() + H;
        P.tail_elems = (x.conv_taps - 1) * P.channels();
        break;
    case OB_MIXER_TIME_MIXING:
        P.f32_rows = 4 * H * x.dim;
        P.tail_elems = width;
        break;
    default: P.f32_rows = H * (2 * x.dim + 2 * x.vdim);
    }
    P.f32_row0 = P.act_rows;
    P.out_width = H * x.vdim;
    P.cols = round_up(P.out_width, LIN_K_ALIGN);
}

// The projections of the block's input.
int LayeredGraph::fill_in(const ob_mixer_desc &x, MixerPlan &P, HostDense &in) {
    const uint32_t H = x.n_head, G = x.n_kv_head, inner = H * x.vdim;
    uint32_t r = P.f32_row0;
    auto rows = [&](const ob_matrix_desc &d) {
        for (uint32_t i = 0; i < d.out_dim; ++i) in.copy(r++, 0, d, i);
    };
    if (x.kind == OB_MIXER_LATENT_ATTENTION) {
        for (uint32_t hd = 0; hd < H; ++hd) {
            for (uint32_t i = 0; i < x.dim; ++i) in.copy(hd * P.dim_p + i, 0, x.wq, hd * (x.dim + x.rot_dim) + i);
            for (uint32_t i = 0; i < x.rot_dim; ++i) in.copy(r++, 0, x.wq, hd * (x.dim + x.rot_dim) + x.dim + i);
        }
        rows(x.w_dkv);
        if (P.has_gate) r = P.gate0;
        if (x.w_gate.data) rows(x.w_gate);
    } else if (x.kind == OB_MIXER_ATTENTION) {
        r = 0;
        if (P.has_v) rows(x.wv);
        if (P.has_gate) rows(x.w_gate);
        r = P.f32_row0;
        rows(x.wq);
        if (P.own_kv) rows(x.wk);
        if (P.head_gate) rows(x.w_gate);
        if (x.q_bias || x.k_bias || x.v_bias) {
            std::vector<float> bias(in.rows, 0.0f);
            if (x.v_bias) std::copy(x.v_bias, x.v_bias + G * x.vdim, bias.begin());
            if (x.q_bias) std::copy(x.q_bias, x.q_bias + H * x.n_map * x.dim, bias.begin() + P.f32_row0);
            if (x.k_bias) std::copy(x.k_bias, x.k_bias + G * x.n_map * x.dim, bias.begin() + P.f32_row0 + H * x.n_map * x.dim);
            if (int rc = upload_now(bias.data(), bias.size(), &P.in_bias)) return rc;
        }
    } else if (x.kind == OB_MIXER_STATE_SPACE) {  // gate | channels, steps
        for (uint32_t i = 0; i < inner; ++i) in.copy(i, 0, x.w_in, i);
        for (uint32_t i = 0; i < P.f32_rows; ++i) in.copy(r++, 0, x.w_in, inner + i);
    } else if (x.kind == OB_MIXER_RETENTION) {
        rows(x.wq);
        rows(x.wk);
        rows(x.wv);
        rows(x.w_gate);
    }
    return OB_OK;
}

int LayeredGraph::build_layer(const ob_block_desc &b, LayerPlan &P) {
    const ob_mixer_desc &x = b.mixer;
    int rc;
    size_mixer(x, P);
    P.sequential = b.post_norm1 || b.pre_norm1;
    P.ff_kind = b.ff_kind;
    const uint32_t glu = P.sequential ? 0 : b.n_ff;  // feed-forward inside the mixer's products
    P.norm_gain = b.norm_gain;
    P.n_ff = b.n_ff;
    P.glu_limit = b.glu_limit;
    P.glu_alpha = b.glu_alpha;
    if (b.mixer2.kind) {
        P.second = std::make_unique<MixerPlan>();
        size_mixer(b.mixer2, *P.second);
        P.scale = b.mixer_scale;
        P.second->scale = b.mixer2_scale;
        P.second->col0 = P.cols;
    }
    // ---- everything that reads the normed input
    P.glu_row0 = P.f32_row0 + round_up(P.f32_rows, LIN_ROW_ALIGN);
    for (MixerPlan *q : {static_cast<MixerPlan *>(&P), P.second.get()}) {
        if (!q || q->mx.kind == OB_MIXER_TIME_MIXING) continue;
        HostDense in(q->f32_row0 + round_up(q->f32_rows, LIN_ROW_ALIGN) + (q == &P ? round_up(2 * glu, LIN_ROW_ALIGN) : 0), h_pitch);
        if ((rc = fill_in(q == &P ? x : b.mixer2, *q, in))) return rc;
        for (uint32_t i = 0; q == &P && i < glu; ++i) {
            in.copy(P.glu_row0 + 2 * i, 0, b.w_gate, i);
            in.copy(P.glu_row0 + 2 * i + 1, 0, b.w_up, i);
        }
        if ((rc = upload(in, &q->in))) return rc;
    }
    // ---- output products side by side
    const uint32_t mix_cols = P.cols + (P.second ? P.second->cols : 0);
    HostDense out(round_up(width, LIN_ROW_ALIGN), mix_cols + round_up(glu, LIN_K_ALIGN));
    for (uint32_t i = 0; i < width; ++i) {
        out.copy(i, 0, x.wo, i);
        if (P.second) out.copy(i, P.cols, b.mixer2.wo, i);
        if (glu) out.copy(i, P.cols, b.w_down, i);
    }
    if ((rc = upload(out, &P.out))) return rc;
    if (x.o_bias) {
        std::vector<float> bias(out.rows, 0.0f);
        std::copy(x.o_bias, x.o_bias + width, bias.begin());
        if ((rc = upload_now(bias.data(), bias.size(), &P.out_bias))) return rc;
    }
    if (b.post_norm1 && (rc = upload_now(b.post_norm1, width, &P.post1))) return rc;
    if (P.sequential && (rc = build_ff(b, P))) return rc;
    if (b.pre_norm1 && (rc = upload_now(b.pre_norm1, width, &P.pre1))) return rc;
    const float *conv[2] = {b.conv1, P.n_ff ? b.conv2 : nullptr};
    for (int k = 0; taps && k < 2; ++k) {
        if (!conv[k]) continue;
        std::vector<float> w((size_t)taps * width);
        for (uint32_t c = 0; c < width; ++c)
            for (uint32_t i = 0; i < taps; ++i) w[(size_t)i * width + c] = conv[k][(size_t)c * taps + i];
        if ((rc = upload_now(w.data(), w.size(), &P.conv_in[k]))) return rc;
        if (in_state() && (rc = scratch_f32(&P.tail_in[k], (size_t)m->n_state_slots * in_state()))) return rc;
    }
    if (b.depth && (rc = upload_now(b.depth, &P - L.data() + 2, &P.depth))) return rc;
    if (side_dim) {
        HostDense g(round_up(side_dim, LIN_ROW_ALIGN), h_pitch), pr(round_up(width, LIN_ROW_ALIGN), side_p);
        for (uint32_t i = 0; i < side_dim; ++i) g.copy(i, 0, b.side_gate, i);
        for (uint32_t i = 0; i < width; ++i) pr.copy(i, 0, b.side_proj, i);
        if ((rc = upload(g, &P.side_gate)) || (rc = upload(pr, &P.side_proj))) return rc;
        if ((rc = upload_f32(m, b.side_norm, width, &P.side_norm))) return rc;
    }
    if ((rc = build_mixer(x, P)) || (P.second && (rc = build_mixer(b.mixer2, *P.second)))) return rc;
    OB_CUDA(m->ctx, cudaStreamSynchronize(m->ctx->stream));  // the host matrices end here
    return OB_OK;
}

// The mixer's own tensors, cache and state.
int LayeredGraph::build_mixer(const ob_mixer_desc &x, MixerPlan &P) {
    const uint32_t H = x.n_head, G = x.n_kv_head;
    int rc;
    if (x.kind == OB_MIXER_LATENT_ATTENTION) {
        const uint32_t kr = round_up(x.kv_rank, LIN_ROW_ALIGN), vr = round_up(x.vdim, LIN_ROW_ALIGN);
        HostDense uk(H * kr, P.dim_p), uv(H * vr, P.kv_w);
        const uint16_t *src = reinterpret_cast<const uint16_t *>(x.w_uk.data);
        for (uint32_t hd = 0; hd < H; ++hd) {
            for (uint32_t d = 0; d < x.dim; ++d)  // transposed: the query goes through it
                for (uint32_t c = 0; c < x.kv_rank; ++c) uk.v[(size_t)(hd * kr + c) * P.dim_p + d] = src[(size_t)(hd * x.dim + d) * x.kv_rank + c];
            for (uint32_t i = 0; i < x.vdim; ++i) uv.copy(hd * vr + i, 0, x.w_uv, hd * x.vdim + i);
        }
        if ((rc = upload(uk, &P.uk)) || (rc = upload(uv, &P.uv))) return rc;
        P.dim_k = round_up(x.dim, 16);
        P.vdim_k = round_up(x.vdim, 16);
        P.paged = !f32 && x.scale > 0 && attention_prompt_supported(1, P.dim_k + P.dq - P.kv_p, P.vdim_k);
        if (P.paged) {
            P.row = P.dim_k + P.dq - P.kv_p + P.vdim_k;
            P.ex_v0 = round_up(P.dim_k, LIN_ROW_ALIGN);
            const uint32_t per = P.ex_v0 + round_up(P.vdim_k, LIN_ROW_ALIGN);
            HostDense ex(H * per, P.kv_w);
            for (uint32_t hd = 0; hd < H; ++hd) {
                for (uint32_t d = 0; d < x.dim; ++d) ex.copy(hd * per + d, 0, x.w_uk, hd * x.dim + d);
                for (uint32_t d = 0; d < x.vdim; ++d) ex.copy(hd * per + P.ex_v0 + d, 0, x.w_uv, hd * x.vdim + d);
            }
            if ((rc = upload(ex, &P.expand))) return rc;
        } else if (!f32 && latent_prefill_supported(P.dim_k, P.dq - P.kv_p, P.vdim_k)) {
            P.ex_v0 = round_up(H * P.dim_k, LIN_ROW_ALIGN);
            HostDense ex(P.ex_v0 + round_up(H * P.vdim_k, LIN_ROW_ALIGN), P.kv_w);
            for (uint32_t hd = 0; hd < H; ++hd) {
                for (uint32_t d = 0; d < x.dim; ++d) ex.copy(hd * P.dim_k + d, 0, x.w_uk, hd * x.dim + d);
                for (uint32_t d = 0; d < x.vdim; ++d) ex.copy(P.ex_v0 + hd * P.vdim_k + d, 0, x.w_uv, hd * x.vdim + d);
            }
            if ((rc = upload(ex, &P.expand))) return rc;
        }
        if ((rc = upload_f32(m, x.kv_norm, x.kv_rank, &P.kv_norm))) return rc;
        if (x.sink && (rc = upload_now(x.sink, H, &P.sink))) return rc;
        if ((rc = scratch(&P.pool, (size_t)m->pool_pages * KV_PAGE * P.dq, es()))) return rc;
    } else if (x.kind == OB_MIXER_ATTENTION) {
        const uint32_t whole_q = x.qk_norm_whole ? H : 1, whole_k = x.qk_norm_whole ? G : 1;
        if (x.q_norm && (rc = upload_now(x.q_norm, whole_q * x.dim, &P.q_norm))) return rc;
        if (x.k_norm && (rc = upload_now(x.k_norm, whole_k * x.dim, &P.k_norm))) return rc;
        if (x.sink && (rc = upload_now(x.sink, H, &P.sink))) return rc;
        if (!P.own_kv) P.pool = L[x.kv_layer - 1].pool;
        else if ((rc = scratch(&P.pool, (size_t)m->pool_pages * KV_PAGE * cache_elems(P), es()))) return rc;
    } else if (x.kind == OB_MIXER_STATE_SPACE) {
        const uint32_t n = P.channels(), inner = H * x.vdim;
        if ((rc = upload_now(x.conv_w, (size_t)n * x.conv_taps, &P.conv_w)) || (rc = upload_now(x.conv_b, n, &P.conv_b))) return rc;
        if ((rc = upload_now(x.dt_bias, H, &P.dt_bias)) || (rc = upload_now(x.a_log, H, &P.a_log)) || (rc = upload_now(x.d_skip, H, &P.skip))) return rc;
        if ((rc = upload_now(x.out_norm, inner, &P.out_norm, P.scale))) return rc;
    } else if (x.kind == OB_MIXER_TIME_MIXING) {
        const uint32_t n = H * x.dim, np = round_up(n, LIN_ROW_ALIGN), rank = x.w_decay1.out_dim;
        HostDense rkvg(4 * np, h_pitch), d1(round_up(rank, LIN_ROW_ALIGN), h_pitch), d2(np, round_up(rank, LIN_K_ALIGN));
        const ob_matrix_desc *each[4] = {&x.wq, &x.wk, &x.wv, &x.w_gate};
        for (uint32_t k = 0; k < 4; ++k)
            for (uint32_t i = 0; i < n; ++i) rkvg.copy(k * np + i, 0, *each[k], i);
        for (uint32_t i = 0; i < rank; ++i) d1.copy(i, 0, x.w_decay1, i);
        for (uint32_t i = 0; i < n; ++i) d2.copy(i, 0, x.w_decay2, i);
        if ((rc = upload(rkvg, &P.rkvg)) || (rc = upload(d1, &P.decay1)) || (rc = upload(d2, &P.decay2))) return rc;
        std::vector<float> d0(np, 0.0f);
        std::copy(x.decay0, x.decay0 + n, d0.begin());
        const float *mu[SHIFT_MIXES] = {x.mu_r, x.mu_k, x.mu_v, x.mu_g, x.mu_w};
        for (uint32_t i = 0; i < SHIFT_MIXES; ++i)
            if ((rc = upload_now(mu[i], width, &P.mu[i]))) return rc;
        if ((rc = upload_now(d0.data(), np, &P.decay0)) || (rc = upload_now(x.bonus, n, &P.bonus)) || (rc = upload_now(x.out_norm, n, &P.out_norm, P.scale))) return rc;
    } else {
        if ((rc = upload_f32(m, x.decay, H, &P.decay))) return rc;
        P.decay_min = *std::min_element(x.decay, x.decay + H);
    }
    if (recurrent_kind(x.kind)) {
        if ((rc = scratch_f32(&P.state, (size_t)m->n_state_slots * state_elems(P)))) return rc;
        if (P.tail_elems && (rc = scratch_f32(&P.tail, (size_t)m->n_state_slots * P.tail_elems))) return rc;
        has_state = true;
    }
    OB_CUDA(m->ctx, cudaStreamSynchronize(m->ctx->stream));
    P.mx.decay = nullptr;
    P.mx.kv_norm = P.mx.q_norm = P.mx.k_norm = P.mx.q_bias = P.mx.k_bias = P.mx.v_bias = P.mx.o_bias = P.mx.sink = nullptr;
    P.mx.conv_w = P.mx.conv_b = P.mx.dt_bias = P.mx.a_log = P.mx.d_skip = P.mx.out_norm = P.mx.decay0 = P.mx.bonus = nullptr;
    P.mx.mu_r = P.mx.mu_k = P.mx.mu_v = P.mx.mu_g = P.mx.mu_w = nullptr;
    return OB_OK;
}

// Feed-forward of a sequential block.
int LayeredGraph::build_ff(const ob_block_desc &b, LayerPlan &P) {
    int rc;
    if (!b.n_ff) return OB_OK;
    const bool experts = b.ff_kind == OB_FF_EXPERTS, gated = experts || b.ff_kind == OB_FF_GELU_GLU;
    P.n_expert = experts ? b.n_expert : 0;
    P.top = experts ? b.n_expert_used : 1;
    P.score_of = b.router_softmax;
    P.router_scale = b.router_scale;
    if (b.n_expert_group) P.n_group = b.n_expert_group, P.keep_group = b.n_group_used;
    // A shared expert in pieces of an expert's size: a gated feed-forward is the sum of its parts.
    P.n_shared = experts ? (b.shared_ff + b.n_ff - 1) / b.n_ff : 0;
    const uint32_t E = experts ? P.n_expert + P.n_shared : 1, up_rows = round_up((gated ? 2 : 1) * b.n_ff, LIN_ROW_ALIGN), down_rows = round_up(width, LIN_ROW_ALIGN),
                   kp = round_up(b.n_ff, LIN_K_ALIGN);
    if (b.post_norm2 && (rc = upload_now(b.post_norm2, width, &P.post2))) return rc;
    if (b.pre_norm2 && (rc = upload_now(b.pre_norm2, width, &P.pre2))) return rc;
    HostDense up(E * up_rows, h_pitch), down(E * down_rows, kp);
    for (uint32_t e = 0; e < E; ++e) {
        const bool shared = experts && e >= P.n_expert;
        const uint32_t c0 = shared ? (e - P.n_expert) * b.n_ff : 0, n = shared ? std::min(b.n_ff, b.shared_ff - c0) : b.n_ff;
        const ob_matrix_desc &g = !experts ? b.w_gate : shared ? b.shared_gate : b.expert_gate[e], &u = !experts ? b.w_up : shared ? b.shared_up : b.expert_up[e],
                             &d = !experts ? b.w_down : shared ? b.shared_down : b.expert_down[e];
        for (uint32_t i = 0; i < n; ++i) {
            if (gated) up.copy(e * up_rows + 2 * i, 0, g, c0 + i);
            up.copy(e * up_rows + (gated ? 2 * i + 1 : i), 0, u, c0 + i);
        }
        for (uint32_t i = 0; i < width; ++i) down.copy(e * down_rows + i, 0, d, i, c0, n);
    }
    if ((rc = upload(up, &P.up)) || (rc = upload(down, &P.down))) return rc;
    if (experts) {
        HostDense z(round_up(P.n_expert + 1, LIN_ROW_ALIGN), h_pitch);
        for (uint32_t e = 0; e < P.n_expert; ++e) z.copy(e, 0, b.w_router, e);
        if (P.n_shared) z.copy(P.n_expert, 0, b.w_shared_scale, 0);
        if ((rc = upload(z, &P.router))) return rc;
    }
    return OB_OK;
}

// The mixer's (cos, sin) by position.  Angles in double on the host: the table is exact to fp32 at any position.
int LayeredGraph::rotation(MixerPlan &P, std::map<std::pair<std::vector<double>, float>, float2 *> &tables) {
    const uint32_t half = P.mx.rot_dims / 2;
    const float gain = P.mx.rot_gain != 0.0f ? P.mx.rot_gain : 1.0f;
    std::vector<double> f(half);
    for (uint32_t k = 0; k < half; ++k) f[k] = P.mx.rot_freqs ? P.mx.rot_freqs[k] : pow(P.mx.rot_base, -2.0 * k / P.mx.rot_dims);
    P.mx.rot_freqs = nullptr;
    float2 *&tab = tables[{f, gain}];
    if (!tab) {
        std::vector<float2> t((size_t)m->cfg.max_seq_len * half);
        for (uint32_t p = 0; p < m->cfg.max_seq_len; ++p)
            for (uint32_t k = 0; k < half; ++k) t[(size_t)p * half + k] = make_float2((float)(gain * cos(p * f[k])), (float)(gain * sin(p * f[k])));
        int rc = dev_alloc(m, &tab, t.size());
        if (rc) return rc;
        OB_CUDA(m->ctx, cudaMemcpy(tab, t.data(), t.size() * sizeof(float2), cudaMemcpyHostToDevice));
    }
    P.rot = Rot{tab, P.mx.rot_dims, P.mx.rot_interleaved != 0};
    return OB_OK;
}

int LayeredGraph::build(const ob_layered_desc &c) {
    int rc = OB_OK;
    const size_t T = m->T;
    f32 = c.compute_f32 != 0;
    width = c.n_embd;
    h_pitch = round_up(width, LIN_K_ALIGN);
    side_dim = c.side_dim;
    side_p = round_up(side_dim, LIN_K_ALIGN);
    eps = c.rms_eps;
    final_gain = c.final_gain;
    residual_mult = c.residual_mult;
    plain = c.layers[0].pre_norm1 && !c.layers[0].post_norm1;
    n_group = std::max(1u, c.norm_groups);
    taps = c.conv_taps;
    if (c.final_norm && (rc = upload_now(c.final_norm, width, &final_norm, plain ? final_gain : 1.0f))) return rc;
    L.resize(c.n_layer);
    std::map<std::pair<std::vector<double>, float>, float2 *> tables;
    size_t act = 0, q_n = 0, o_n = 0, o_r = 0, kvp = 0, dq = 0, ex = 0, reach = 0, ff_n = 0, pairs = 0, experts = 0, channels = 0, heads = 0, mixed = 0;
    bool sequential = false;
    for (uint32_t i = 0; i < c.n_layer; ++i) {
        LayerPlan &P = L[i];
        if ((rc = build_layer(c.layers[i], P))) return rc;
        cat_pitch = std::max(cat_pitch, P.out.kp);
        sequential |= P.sequential;
        if (P.sequential && P.n_ff) ff_n = std::max<size_t>(ff_n, T * P.pairs() * P.down.kp);
        if (P.n_expert) {
            pairs = std::max<size_t>(pairs, T * P.pairs());
            experts = std::max<size_t>(experts, P.n_expert + P.n_shared + 1);
        }
    }
    each_mixer([&](MixerPlan &P) {
        const uint32_t H = P.mx.n_head;
        if (!rc) rc = rotation(P, tables);
        act = std::max<size_t>(act, P.act_rows);
        y_pitch = std::max(y_pitch, round_up(P.f32_rows, 4));
        if (P.mx.kind == OB_MIXER_ATTENTION) {
            q_n = std::max<size_t>(q_n, (size_t)H * P.mx.n_map * P.dim_p);
        } else if (P.pool) {
            q_n = std::max<size_t>(q_n, (size_t)H * P.dq);
            o_n = std::max<size_t>(o_n, (size_t)H * P.kv_w);
            kvp = std::max<size_t>(kvp, P.kv_p);
            if (P.expand.rows) {
                dq = std::max<size_t>(dq, P.dq);
                ex = std::max<size_t>(ex, P.paged ? H * P.row : P.expand.rows);
                reach = std::max<size_t>(reach, std::min(P.mx.window ? P.mx.window - 1 : m->cfg.max_seq_len, m->cfg.max_seq_len));
            }
        } else {
            o_r = std::max<size_t>(o_r, (size_t)H * P.mx.vdim);
            if (P.mx.kind == OB_MIXER_STATE_SPACE) {
                channels = std::max<size_t>(channels, P.channels());
                heads = std::max<size_t>(heads, H);
            } else if (P.mx.kind == OB_MIXER_TIME_MIXING) {
                mixed = std::max<size_t>(mixed, (size_t)H * P.mx.dim);
                low_p = std::max(low_p, P.decay2.kp);
            }
        }
    });
    if (rc) return rc;
    {
        if ((rc = dev_alloc(m, &embd, (size_t)c.n_vocab * width))) return rc;
        OB_CUDA(m->ctx, cudaMemcpy(embd, c.token_embd.data, (size_t)c.n_vocab * width * 2, cudaMemcpyHostToDevice));
        if (side_dim) {
            const size_t n = (size_t)c.n_vocab * c.n_layer * side_dim;
            if ((rc = dev_alloc(m, &side_embd, n))) return rc;
            OB_CUDA(m->ctx, cudaMemcpy(side_embd, c.side_embd.data, n * 2, cudaMemcpyHostToDevice));
        }
        HostDense o(round_up(c.n_vocab, LIN_ROW_ALIGN), h_pitch);
        for (uint32_t i = 0; i < c.n_vocab; ++i) o.copy(i, 0, c.output, i);
        if ((rc = upload(o, &output))) return rc;
    }
    if ((rc = scratch(&h, T * h_pitch, es())) || (rc = scratch(&xb, T * h_pitch, es())) || (rc = scratch(&cat, T * cat_pitch, es()))) return rc;
    if ((rc = scratch(&qn, T * act, es())) || (rc = scratch(&q, T * q_n, es())) || (rc = scratch(&o_lat, T * o_n, es()))) return rc;
    if ((rc = scratch_f32(&y, T * y_pitch)) || (rc = scratch_f32(&o_ret, T * o_r))) return rc;
    if (sequential && ((rc = scratch(&ffa, ff_n, es())) || (rc = scratch_f32(&yo, std::max(T, pairs) * width)))) return rc;
    if (pairs) {
        float *row_score;
        if ((rc = dev_alloc(m, &moe.expert, pairs)) || (rc = dev_alloc(m, &moe.rank, pairs)) || (rc = dev_alloc(m, &moe.row, pairs))) return rc;
        if ((rc = scratch_f32(&moe.score, pairs)) || (rc = scratch_f32(&row_score, pairs)) || (rc = scratch_f32(&router_logits, T * experts))) return rc;
        if ((rc = dev_alloc(m, &moe.tiles, pairs / 16 + experts + 1)) || (rc = dev_alloc(m, &moe.n_tiles, 1)) || (rc = dev_alloc(m, &moe.count, experts))) return rc;
        if ((rc = scratch(&moe.gathered, pairs * h_pitch, es()))) return rc;
        OB_CUDA(m->ctx, cudaMemset(moe.count, 0, experts * 4));
        moe.row_score = row_score;
    }
    if (ex) {
        key_cap = round_up((uint32_t)(T + reach), KV_PAGE) + (PREFILL_GROUP + 1) * KV_PAGE;  // (spans in pages begin and end at sixteens)
        std::vector<int32_t> order(key_cap / KV_PAGE);
        for (size_t i = 0; i < order.size(); ++i) order[i] = (int32_t)i;
        if ((rc = dev_alloc(m, &numbers, order.size())) || (rc = dev_alloc(m, &page_tables, T))) return rc;
        OB_CUDA(m->ctx, cudaMemcpy(numbers, order.data(), order.size() * 4, cudaMemcpyHostToDevice));
        if ((rc = scratch(&lat, (size_t)key_cap * dq, 2)) || (rc = scratch(&expanded, (size_t)key_cap * ex, 2))) return rc;
    }
    if (plain) {
        if ((rc = scratch_f32(&inverse, T * n_group))) return rc;
        if (L[0].depth && (rc = scratch_f32(&history, (size_t)c.n_layer * T * width))) return rc;
        if (in_state()) has_state = true;
    }
    if (channels && ((rc = scratch_f32(&conv, T * channels)) || (rc = dev_alloc(m, &steps, T * heads)))) return rc;
    if (mixed && ((rc = scratch(&mix, T * SHIFT_MIXES * h_pitch, es())) || (rc = scratch(&low, T * low_p, es())) || (rc = scratch_f32(&decays, T * mixed)))) return rc;
    if (side_dim && ((rc = scratch(&sg, T * side_p, es())) || (rc = scratch_f32(&sy, T * width)))) return rc;
    if (!f32 && (rc = scratch_f32(&split_part, linear_split_bytes() / 4))) return rc;
    if (kvp && !f32) {  // at most one CTA per SM, of 64 rows, writes partial results at a time (launch_latent_attention)
        part_cap = ((uint64_t)m->ctx->sm_count * 64 + 64) * (kvp + 4);
        if ((rc = scratch_f32(&part, part_cap))) return rc;
    }
    return OB_OK;
}

int check_dense(ob_ctx *ctx, const ob_matrix_desc &d, uint32_t in_dim, uint32_t out_dim, const std::string &name) {
    if (!d.data) return fail(ctx, OB_ERR_INVALID, "layered model: " + name + " has no data");
    if (d.ggml_type != OB_TYPE_BF16) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + name + " is not bfloat16");
    if (d.in_dim != in_dim || d.out_dim != out_dim)
        return fail(ctx, OB_ERR_INVALID, "layered model: " + name + " is [" + std::to_string(d.in_dim) + " -> " + std::to_string(d.out_dim) + "], expected [" +
                                             std::to_string(in_dim) + " -> " + std::to_string(out_dim) + "]");
    return OB_OK;
}

int check_mixer(ob_ctx *ctx, const ob_layered_desc &c, uint32_t i, const ob_mixer_desc &x) {
    const std::string at = "layer " + std::to_string(i) + " ";
    int rc;
    if (!x.n_head || !x.dim || !x.vdim) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "mixer sizes missing");
    const uint32_t H = x.n_head, G = x.n_kv_head, E = c.n_embd, rotating = x.kind == OB_MIXER_LATENT_ATTENTION ? x.rot_dim : x.dim;
    if ((x.rot_dims & 1) || x.rot_dims > rotating) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "rot_dims must be even and fit the rotated vector");
    if (x.rot_dims && !x.rot_freqs && !(x.rot_base > 0)) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "rot_base must be positive");
    if (x.kind == OB_MIXER_LATENT_ATTENTION) {
        if (!x.kv_rank || !x.kv_norm) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "latent size or norm missing");
        if ((uint64_t)(2 * x.kv_rank + x.rot_dim + 256) * 4 > 128 * 1024) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "kv_rank too large");
        if ((rc = check_dense(ctx, x.wq, E, H * (x.dim + x.rot_dim), at + "wq"))) return rc;
        if ((rc = check_dense(ctx, x.w_dkv, E, x.kv_rank + x.rot_dim, at + "w_dkv"))) return rc;
        if ((rc = check_dense(ctx, x.w_uk, x.kv_rank, H * x.dim, at + "w_uk"))) return rc;
        if ((rc = check_dense(ctx, x.w_uv, x.kv_rank, H * x.vdim, at + "w_uv"))) return rc;
        if (x.w_gate.data && (rc = check_dense(ctx, x.w_gate, E, x.w_gate.out_dim == H ? H : H * x.vdim, at + "mixer gate"))) return rc;
    } else if (x.kind == OB_MIXER_RETENTION) {
        if (!x.decay) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "decay missing");
        if (!retention_supported(x.dim)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "retention heads have at most 256 key dimensions");
        if ((rc = check_dense(ctx, x.wq, E, H * x.dim, at + "wq"))) return rc;
        if ((rc = check_dense(ctx, x.wk, E, H * x.dim, at + "wk"))) return rc;
        if ((rc = check_dense(ctx, x.wv, E, H * x.vdim, at + "wv"))) return rc;
        if ((rc = check_dense(ctx, x.w_gate, E, H * x.vdim, at + "mixer gate"))) return rc;
    } else if (x.kind == OB_MIXER_ATTENTION) {
        if (!G || H % G) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "n_kv_head does not divide n_head");
        if (!(x.scale > 0)) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "scale must be positive");
        if (x.n_map != 1 && x.n_map != 2) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "one or two maps per head");
        const bool own = !x.kv_layer;
        if ((x.q_norm != nullptr) != (x.k_norm != nullptr) && own) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "query or key norm missing");
        if (x.n_map != 1 && (x.qk_norm_whole || x.keep_first || x.kv_layer || x.softcap > 0 || x.sink))
            return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "norms of whole projections, kept tokens, shared keys, soft caps and sinks go with one map");
        if (!own) {
            if (x.kv_layer > i) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "keys and values come from an earlier layer");
            const ob_mixer_desc &o = c.layers[x.kv_layer - 1].mixer;
            if (o.kind != OB_MIXER_ATTENTION || o.kv_layer || o.n_kv_head != G || o.dim != x.dim || o.vdim != x.vdim || o.n_map != x.n_map)
                return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "the layer of its keys and values has other ones");
            if (x.wk.data || x.wv.data || x.k_norm || x.k_bias || x.v_bias) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "has keys and values of another layer and of its own");
        }
        if (!attention_supported(x.dim, x.vdim)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "attention head too large");
        if ((rc = check_dense(ctx, x.wq, E, H * x.n_map * x.dim, at + "wq"))) return rc;
        if (own && (rc = check_dense(ctx, x.wk, E, G * x.n_map * x.dim, at + "wk"))) return rc;
        if (!own) {
        } else if (x.wv.data) {
            if ((rc = check_dense(ctx, x.wv, E, G * x.vdim, at + "wv"))) return rc;
        } else if (x.n_map != 1 || x.vdim != x.dim || x.v_bias) {
            return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "keys can be the values of one map of their own size");
        }
        if (x.w_gate.data && x.w_gate.out_dim == H && x.n_map != 1) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "gates of whole heads go with one map");
        if (x.w_gate.data && (rc = check_dense(ctx, x.w_gate, E, x.w_gate.out_dim == H ? H : H * x.vdim, at + "mixer gate"))) return rc;
    } else if (x.kind == OB_MIXER_STATE_SPACE) {
        const uint32_t inner = H * x.vdim, n = inner + 2 * x.n_group * x.dim;
        if (!x.n_group || H % x.n_group) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "n_group does not divide n_head");
        if (!x.n_norm_group || inner % x.n_norm_group) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "n_norm_group does not divide the inner width");
        if (!x.conv_taps || x.conv_taps > CONV_MAX_TAPS) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "the convolution has 1 to 16 taps");
        if (!recurrence_supported(x.dim)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "a state has at most 256 entries per value");
        if (!state_space_out_supported(inner / x.n_norm_group)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "norm group too large");
        if (!x.conv_w || !x.conv_b || !x.dt_bias || !x.a_log || !x.d_skip || !x.out_norm) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "state-space vectors missing");
        if ((rc = check_dense(ctx, x.w_in, E, inner + n + H, at + "w_in"))) return rc;
    } else if (x.kind == OB_MIXER_TIME_MIXING) {
        const uint32_t n = H * x.dim;
        if (x.vdim != x.dim) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "time mixing has values of its keys' size");
        if (!c.layers[i].post_norm1) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "time mixing belongs in sequential blocks");
        if (!recurrence_supported(x.dim)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "a state has at most 256 entries per value");
        if (!x.mu_r || !x.mu_k || !x.mu_v || !x.mu_g || !x.mu_w || !x.decay0 || !x.bonus || !x.out_norm)
            return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "time-mixing vectors missing");
        if ((rc = check_dense(ctx, x.wq, E, n, at + "wq")) || (rc = check_dense(ctx, x.wk, E, n, at + "wk")) || (rc = check_dense(ctx, x.wv, E, n, at + "wv"))) return rc;
        if ((rc = check_dense(ctx, x.w_gate, E, n, at + "mixer gate"))) return rc;
        if (!x.w_decay1.out_dim) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "w_decay1 missing");
        if ((rc = check_dense(ctx, x.w_decay1, E, x.w_decay1.out_dim, at + "w_decay1"))) return rc;
        if ((rc = check_dense(ctx, x.w_decay2, x.w_decay1.out_dim, n, at + "w_decay2"))) return rc;
    } else {
        return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "unknown mixer");
    }
    if (x.kind != OB_MIXER_ATTENTION && (x.q_bias || x.k_bias || x.v_bias)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "the mixer has no biases");
    if (x.kind != OB_MIXER_ATTENTION && x.o_bias) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "the mixer has no biases");
    return check_dense(ctx, x.wo, H * x.vdim, E, at + "wo");
}

int check_block(ob_ctx *ctx, const ob_layered_desc &c, uint32_t i) {
    const ob_block_desc &b = c.layers[i];
    const std::string at = "layer " + std::to_string(i) + " ";
    const uint32_t E = c.n_embd;
    int rc;
    if ((rc = check_mixer(ctx, c, i, b.mixer))) return rc;
    if (b.mixer2.kind) {
        auto scales = [](uint32_t kind) { return kind == OB_MIXER_ATTENTION || kind == OB_MIXER_STATE_SPACE || kind == OB_MIXER_TIME_MIXING; };
        if (!b.post_norm1 || !scales(b.mixer.kind) || !scales(b.mixer2.kind) || b.mixer.o_bias || b.mixer2.o_bias || b.mixer.n_map > 1 || b.mixer2.n_map > 1 ||
            b.mixer2.kv_layer || (b.mixer.kind != OB_MIXER_ATTENTION) == (b.mixer2.kind != OB_MIXER_ATTENTION))
            return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "two mixers: attention with one map beside a recurrent layer, in a sequential block");
        if ((rc = check_mixer(ctx, c, i, b.mixer2))) return rc;
    }
    if ((b.post_norm1 != nullptr) != (c.layers[0].post_norm1 != nullptr)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "blocks of two kinds");
    if ((b.pre_norm1 != nullptr) != (c.layers[0].pre_norm1 != nullptr)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "blocks with and without normed inputs");
    const bool plain = b.pre_norm1 && !b.post_norm1;  // outputs are added as they are
    if (plain && !c.final_norm) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "plain sums go with factors of the last norm");
    if (plain && b.mixer2.kind) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "two mixers go with normed outputs");
    if (!plain && (c.norm_groups > 1 || c.conv_taps || b.depth)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "norms in groups, convolved inputs and averages over depth go with plain sums");
    if (c.conv_taps > CONV_MAX_TAPS) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "the convolution has 1 to 16 taps");
    if (c.norm_groups && E % c.norm_groups) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "norm_groups does not divide the width");
    if (c.conv_taps && (!b.conv1 || (b.n_ff && !b.conv2))) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "convolution of an input missing");
    if ((b.depth != nullptr) != (c.layers[0].depth != nullptr)) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "layers with and without an average over depth");
    if (plain || b.post_norm1) {
        if (c.side_dim) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "sequential blocks have no per-layer token input");
        if (!b.n_ff) return OB_OK;
        if (!plain && !b.post_norm2) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "norm of the feed-forward missing");
        if ((b.pre_norm2 != nullptr) != (b.pre_norm1 != nullptr)) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "norm of the feed-forward's input");
        if (b.ff_kind == OB_FF_GELU_GLU && (rc = check_dense(ctx, b.w_gate, E, b.n_ff, at + "ff gate"))) return rc;
        if (b.ff_kind == OB_FF_RELU2 || b.ff_kind == OB_FF_GELU_GLU) {
            if ((rc = check_dense(ctx, b.w_up, E, b.n_ff, at + "ff up"))) return rc;
            return check_dense(ctx, b.w_down, b.n_ff, E, at + "ff down");
        }
        if (b.ff_kind != OB_FF_EXPERTS) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "unknown feed-forward");
        if (!b.n_expert || !b.n_expert_used || b.n_expert_used > b.n_expert || !b.expert_gate || !b.expert_up || !b.expert_down)
            return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "experts missing");
        if (b.router_softmax > OB_ROUTER_SOFTMAX_ALL) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "unknown scores of the router");
        if (b.n_expert_group && (b.n_expert % b.n_expert_group || !b.n_group_used || b.n_group_used > b.n_expert_group))
            return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "groups do not divide the experts");
        if (b.n_expert_group && b.n_expert_used > b.n_expert / b.n_expert_group * b.n_group_used)
            return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "more experts of a token than its groups hold");
        if (b.shared_ff && !b.router_softmax) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "a shared expert goes with weighted outputs");
        if (b.shared_ff) {
            if ((rc = check_dense(ctx, b.shared_gate, E, b.shared_ff, at + "shared gate")) || (rc = check_dense(ctx, b.shared_up, E, b.shared_ff, at + "shared up")) ||
                (rc = check_dense(ctx, b.shared_down, b.shared_ff, E, at + "shared down")) || (rc = check_dense(ctx, b.w_shared_scale, E, 1, at + "scale of the shared expert")))
                return rc;
        }
        if ((uint64_t)b.n_expert + (b.shared_ff + b.n_ff - 1) / b.n_ff > MOE_MAX_EXPERTS) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "too many experts");
        if ((rc = check_dense(ctx, b.w_router, E, b.n_expert, at + "router"))) return rc;
        for (uint32_t e = 0; e < b.n_expert; ++e) {
            if ((rc = check_dense(ctx, b.expert_gate[e], E, b.n_ff, at + "expert gate"))) return rc;
            if ((rc = check_dense(ctx, b.expert_up[e], E, b.n_ff, at + "expert up"))) return rc;
            if ((rc = check_dense(ctx, b.expert_down[e], b.n_ff, E, at + "expert down"))) return rc;
        }
        return OB_OK;
    }
    if (b.ff_kind != OB_FF_CLAMPED_GLU) return fail(ctx, OB_ERR_UNSUPPORTED, "layered model: " + at + "parallel blocks have the clamped feed-forward");
    if (b.n_ff) {
        if ((rc = check_dense(ctx, b.w_gate, E, b.n_ff, at + "ff gate"))) return rc;
        if ((rc = check_dense(ctx, b.w_up, E, b.n_ff, at + "ff up"))) return rc;
        if ((rc = check_dense(ctx, b.w_down, b.n_ff, E, at + "ff down"))) return rc;
    }
    if (c.side_dim) {
        if (!b.side_norm) return fail(ctx, OB_ERR_INVALID, "layered model: " + at + "side norm missing");
        if ((rc = check_dense(ctx, b.side_gate, E, c.side_dim, at + "side gate"))) return rc;
        if ((rc = check_dense(ctx, b.side_proj, c.side_dim, E, at + "side proj"))) return rc;
    }
    return OB_OK;
}

}  // namespace

extern "C" int ob_layered_model_create(ob_ctx *ctx, const ob_layered_desc *desc, ob_model **out) {
    if (!ctx || !desc || !out) return fail(ctx, OB_ERR_INVALID, "layered_model_create: null argument");
    *out = nullptr;
    const ob_layered_desc &c = *desc;
    if (!c.n_layer || !c.n_embd || !c.n_vocab || !c.layers) return fail(ctx, OB_ERR_INVALID, "layered_model_create: incomplete description");
    if (c.n_embd > 32768) return fail(ctx, OB_ERR_UNSUPPORTED, "layered_model_create: n_embd above 32768");
    int rc;
    if ((rc = check_dense(ctx, c.token_embd, c.n_embd, c.n_vocab, "token_embd"))) return rc;
    if ((rc = check_dense(ctx, c.output, c.n_embd, c.n_vocab, "output"))) return rc;
    if (c.side_dim && (rc = check_dense(ctx, c.side_embd, c.n_layer * c.side_dim, c.n_vocab, "side_embd"))) return rc;
    bool state = c.conv_taps > 1;
    for (uint32_t i = 0; i < c.n_layer; ++i) {
        if ((rc = check_block(ctx, c, i))) return rc;
        state |= recurrent_kind(c.layers[i].mixer.kind) || recurrent_kind(c.layers[i].mixer2.kind);
    }

    std::unique_lock<std::mutex> g(ctx->mu);
    Bind b(ctx);
    OB_CUDA(ctx, linear_configure());
    OB_CUDA(ctx, mixers_configure());
    OB_CUDA(ctx, attention_configure());
    OB_CUDA(ctx, recurrence_configure());
    ob_model *m = new ob_model;
    m->ctx = ctx;
    m->cfg.n_vocab = c.n_vocab;
    m->cfg.n_embd = c.n_embd;
    m->cfg.n_layer = c.n_layer;
    m->cfg.rms_eps = c.rms_eps;
    m->cfg.max_seq_len = c.max_seq_len ? c.max_seq_len : 4096;
    m->cfg.max_batch_tokens = std::max(1u, c.max_batch_tokens);
    m->T = m->cfg.max_batch_tokens;
    auto bail = [&](int code) {
        g.unlock();
        ob_model_destroy(m);
        return code;
    };
    const uint64_t tokens = c.kv_pool_tokens ? c.kv_pool_tokens : m->cfg.max_seq_len;
    m->pool_pages = (uint32_t)((tokens + KV_PAGE - 1) / KV_PAGE);
    for (int32_t p = (int32_t)m->pool_pages - 1; p >= 0; --p) m->free_pages.push_back(p);
    if (state) {
        m->n_state_slots = c.n_state_slots ? c.n_state_slots : 64;
        for (int32_t s = (int32_t)m->n_state_slots - 1; s >= 0; --s) m->free_slots.push_back(s);
    }
    const uint32_t T = m->T;
    // logits of as many rows at a time as fit 1 GiB (a step's rows come in slices of this many)
    m->logit_cap = std::min<uint64_t>(T, std::max<uint64_t>(64, (1ull << 30) / (4ull * c.n_vocab)));
    LayeredGraph *gr = new LayeredGraph;
    gr->m = m;
    m->graph = gr;
    if ((rc = gr->build(c))) return bail(rc);
    if ((rc = dev_alloc(m, &m->x, (size_t)T * c.n_embd))) return bail(rc);
    if ((rc = dev_alloc(m, &m->logits, (size_t)m->logit_cap * c.n_vocab))) return bail(rc);
    const MetaLayout ml(T);
    if ((rc = dev_alloc(m, &m->d_meta, ml.bytes))) return bail(rc);
    if ((rc = dev_alloc(m, &m->d_out_tokens, T))) return bail(rc);
    if ((rc = dev_alloc(m, &m->argmax_scratch, T))) return bail(rc);
    if ((rc = dev_alloc(m, &m->d_step_counter, 4))) return bail(rc);
    if (cudaMallocHost(reinterpret_cast<void **>(&m->h_meta), ml.bytes) != cudaSuccess ||
        cudaMallocHost(reinterpret_cast<void **>(&m->h_out_tokens), (size_t)T * 4) != cudaSuccess)
        return bail(fail(ctx, OB_ERR_OOM, "layered_model_create: pinned host allocation failed"));
    memset(m->h_meta, 0, ml.bytes);
    cudaError_t e = cudaDeviceSynchronize();
    if (e == cudaSuccess) e = cudaGetLastError();
    if (e != cudaSuccess) return bail(fail(ctx, OB_ERR_CUDA, std::string("layered_model_create: ") + cudaGetErrorString(e)));
    *out = m;
    return OB_OK;
}
