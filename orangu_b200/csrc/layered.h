// Launchers of the kernels for models given as a list of layers (layered.cu): bf16-weight products with fused epilogues, norms,
// latent attention over a paged latent cache, retention with a per-sequence state, softmax attention over paged keys and values,
// mixtures of experts, residuals averaged over depth with convolved inputs (internal to the library).
//
// Two precisions share every launcher.  bf16: activations that enter a product are bfloat16, accumulation is fp32.  f32:
// activations are fp32 and every product is plain fp32 multiply-add.  Weights are bfloat16 in both.  The residual stream, norms,
// rotation, attention scores and weights, gates and recurrent states are fp32 in both.
#pragma once

#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "common.cuh"

namespace ob {

// ---- linear.cu -------------------------------------------------------------------------------------------------------
enum LinEpilogue {
    LE_F32 = 0,       // out f32
    LE_ACT = 1,       // out activation
    LE_GLU = 2,       // rows (2j, 2j+1) are (gate j, up j): out activation j = g sigmoid(alpha g) (u + 1) of the limited pair
    LE_RESIDUAL = 3,  // x f32 [t][pitch] += v; out2 (optional) gets the sum as activation
    LE_GELU_EMB = 4,  // out activation = gelu_tanh(v) * emb[token t][emb_col0 + row]
    LE_GATED = 5,     // out activation = v * sigmoid(gate[t * gate_pitch + batch])
    LE_RELU2 = 6,     // out activation = max(v, 0)^2
    LE_SWIGLU = 7,    // rows (2j, 2j+1) are (gate j, up j), both times row_scale[t]: out activation j = silu(g) u, times out_scale[t]
    LE_GELU_GLU = 8,  // rows (2j, 2j+1) are (gate j, up j): out activation j = gelu_tanh(g) u
    LE_TANH = 9,      // out activation = tanh(v)
    LE_DECAY = 10,    // out f32 = exp(-exp(v))
    LE_GATED_EACH = 11  // out activation = v * sigmoid(gate_act[t * gate_pitch + column of the output])
};
struct LinTile {          // rows of a grouped product that share a batch entry
    uint32_t batch, row0, n;
};
struct LinSegment {       // consecutive rows of the weight with one epilogue; row0 is a multiple of 32
    uint32_t row0, n;     // rows [row0, row0 + n)
    int epi;
    void *out;            // element (t, r) goes to out[t * pitch + col0 + batch * batch_cols + (r - row0)] (pairs: (r - row0) / 2)
    uint32_t pitch, col0, batch_cols;
    uint32_t page_pitch = 0;  // > 0: sixteen t's are pitch apart, the sixteens page_pitch
};
struct LinArgs {
    const __nv_bfloat16 *w;   // [n_batch][n_rows][kp], zero padded
    uint32_t n_rows, kp;      // kp: columns, a multiple of 64
    const void *x;            // activations [T][x_pitch]; batch b reads columns [b * x_step, + kp)
    uint32_t x_pitch, x_step; // elements; multiples of 8
    uint32_t T, n_batch;
    LinSegment seg[3];
    int n_seg;
    // epilogue parameters
    void *out2 = nullptr;
    uint32_t out2_pitch = 0;
    float glu_limit = 0.0f, glu_alpha = 0.0f;
    const uint32_t *tokens = nullptr;
    const __nv_bfloat16 *emb = nullptr;
    uint32_t emb_pitch = 0, emb_col0 = 0;
    const float *gate = nullptr;
    const void *gate_act = nullptr;  // activations
    uint32_t gate_pitch = 0;
    float *split_part = nullptr;  // scratch of products that split K, linear_split_bytes
    const float *bias = nullptr;  // [n_batch][n_rows] added to the products before the epilogue
    const float *row_scale = nullptr, *out_scale = nullptr;  // [T]
    // Grouped products: every row of x has a batch entry of its own.  Either row by row, or in tiles of rows with one entry each
    // (rows of one entry next to one another), made on the device: *n_tiles of at most max_tiles, of tile_rows rows or fewer.
    const uint32_t *row_batch = nullptr;  // [T], row t reads row t / x_div of x
    uint32_t x_div = 1;
    const LinTile *tiles = nullptr;
    const uint32_t *n_tiles = nullptr;
    uint32_t max_tiles = 0, tile_rows = 0;
};
// Rows of a tile that a grouped product of `rows` rows over `batches` entries takes best.
uint32_t linear_tile_rows(uint32_t rows, uint32_t batches, bool f32);
constexpr uint32_t LIN_K_ALIGN = 64, LIN_ROW_ALIGN = 32;
cudaError_t linear_configure();  // kernel attributes of the current device (outside stream capture)
uint32_t launch_linear(const LinArgs &a, bool f32, int sm_count, cudaStream_t st);  // kernels launched; 0: a tensor map could not be made
size_t linear_split_bytes();
int linear_take_status();        // 1 when a bounded wait inside a product ran out since the last call
void linear_mark_launched();     // a replayed graph may have run one of the tensor-core products

// ---- mixers.cu -------------------------------------------------------------------------------------------------------
// x = embedding rows; h = x / rms(x) * gain (* w) as activation, or (normed false) x itself; w [width], may be null.
void launch_embed(const __nv_bfloat16 *table, uint32_t width, const uint32_t *tokens, uint32_t T, float *x, bool normed, float eps, float gain, const float *w,
                  void *h, uint32_t h_pitch, bool f32, cudaStream_t st);
// h[i] = x[row i] / rms(x[row i]) * gain (* w), as activation; rows == nullptr: row i; w [width], may be null.
void launch_norm(const float *x, uint32_t width, const uint32_t *rows, uint32_t n, float eps, float gain, const float *w, void *h, uint32_t h_pitch, bool f32,
                 cudaStream_t st);
struct PostNormArgs {        // x += mult * y / rms(y) * w, then h = x, or x / rms(x) * next_w, as activation
    float *x;                // [T][width]
    const float *y;          // [T * top][width]: the `top` rows of a token are added up first
    const uint32_t *rows;    // where they are, [T * top]; null: in order
    uint32_t top;
    const float *w;          // [width]
    uint32_t width, T;
    float eps, mult;
    void *h;                 // null: not needed
    uint32_t h_pitch;
    const float *next_w;     // [width]; null: h is x itself
    uint32_t *zero;          // set to zero for whoever counts next, n_zero words; may be null
    uint32_t n_zero;
};
void launch_post_norm(const PostNormArgs &a, bool f32, cudaStream_t st);
// x += y / rms(y) * w, then (h != nullptr) h = x / rms(x) * gain as activation.
void launch_side_finish(float *x, const float *y, const float *w, uint32_t width, uint32_t T, float eps, float gain, void *h, uint32_t h_pitch, bool f32,
                        cudaStream_t st);

struct Rot {                 // rotation of the first `dims` entries of a vector by position
    const float2 *table;     // [position][dims / 2] (cos, sin)
    uint32_t dims;
    bool interleaved;        // pairs (2i, 2i+1), else (i, i + dims/2)
};

struct LatentArgs {          // latent attention of one layer over T rows
    const float *y;          // projections [T][y_pitch]: rotated query parts [H][rot_dim], latent [kv_rank], shared rotated key part [rot_dim]
    uint32_t y_pitch;
    uint32_t n_head, kv_rank, rot_dim, window;  // window 0: no limit
    uint32_t kv_p, dq;       // padded latent width and padded row width (latent | rotated part) of queries and cache rows
    float eps, scale;
    const float *sink;       // [n_head]: exp of it is added to the softmax's denominator; null: none
    const float *kv_norm;    // [kv_rank]
    Rot rot;
    void *q;                 // activations [T][H][dq]; the latent part is written by the absorbed-query product
    void *cache;             // activations [page][16][dq]
    void *o;                 // activations [T][H * o_pitch_h]: attention output in the latent space
    uint32_t o_head;         // elements between heads in o
    float *part;             // [splits][T * H][kv_p + 4] partial results (unnormalised output, max, sum)
    uint64_t part_cap;       // floats `part` holds
    // rows
    uint32_t T, n_seq;
    const RowSpan *spans;    // device [n_seq]
    const RowSpan *h_spans;  // the same on the host
    bool single;             // every span is one row
    const uint32_t *positions;
    const int32_t *const *tables;
    uint32_t max_pos;        // positions are below this
};
cudaError_t mixers_configure();
void launch_latent_prep(const LatentArgs &a, bool f32, cudaStream_t st);   // norms and appends the latent, rotates and stores the query parts
uint32_t launch_latent_attention(const LatentArgs &a, bool f32, int sm_count, cudaStream_t st);  // returns the kernels launched

// Prompts: the window's latents are gathered from the pages, multiplied out to keys and values (a product), and attended per head:
// on tcgen05 as attention over pages of one key/value head per head (gqa_tc5.cu), or, where that does not take the sizes, by
// latent_prefill_kernel.
constexpr uint32_t PREFILL_SPAN = 64;     // spans of at least this many rows go this way (bf16); in a step they follow the shorter ones
constexpr uint32_t PREFILL_GROUP = 8;     // spans of one launch
struct PrefillSpan {
    uint32_t row0, n, pos0, hist;         // rows, first position, positions before it that are seen
    uint32_t key0, tile0;                 // first gathered key, first tile of the launch
};
struct LatentPrefillArgs {
    PrefillSpan span[PREFILL_GROUP];
    uint32_t n_span, n_keys, n_tiles;
    uint32_t n_head, vdim, window;
    uint32_t dim_k, vdim_k;               // per head in `expanded`, multiples of 16
    uint32_t kv_p, dq, dim_p;
    float scale;
    const int32_t *const *tables;
    const void *cache;                    // [page][16][dq]
    void *lat;                            // [n_keys][dq] gathered rows
    // gathered into pages: spans begin at sixteens, what is past a span's end is zero
    void *pages;                          // [page][n_head][16][page_row]: gets the rotated key part from page_rot0 on; null: no pages
    uint32_t page_row, page_rot0;
    const int32_t *numbers;               // 0, 1, 2 ..
    const int32_t **page_tables;          // [T]: the first row of a span gets its table
    const void *expanded;                 // [n_keys][ex_pitch]: keys [H][dim_k], at ex_v0 values [H][vdim_k]
    uint32_t ex_pitch, ex_v0;
    const void *qn, *q;                   // unrotated query parts [T][qn_pitch] (head h at h * dim_p), rotated ones in [T][H][dq] at kv_p
    uint32_t qn_pitch;
    const float *gate;                    // [T][gate_pitch]: sigmoid of entry h scales head h; null: none
    const void *gate_act;                 // activations [T][gate_pitch]: sigmoid of entry h * vdim + i scales entry i of head h; null: none
    uint32_t gate_pitch;
    const float *sink;                    // as in LatentArgs
    void *out;                            // activations [T][out_pitch], head h at h * vdim
    uint32_t out_pitch;
};
bool latent_prefill_supported(uint32_t dim_k, uint32_t rot_p, uint32_t vdim_k);
uint32_t latent_prefill_tiles(uint32_t n);
void launch_latent_gather(const LatentPrefillArgs &a, cudaStream_t st);
void launch_latent_prefill(const LatentPrefillArgs &a, cudaStream_t st);

struct RetentionArgs {       // retention of one layer over T rows
    float *y;                // projections [T][y_pitch]: q [H][dim], k [H][dim], v [H][vdim], gate [H][vdim]; q and k are rotated in place
    uint32_t y_pitch;
    uint32_t n_head, dim, vdim;
    float eps, k_scale;
    const float *decay;      // [H]
    Rot rot;
    float *state;            // [slot][H][dim][vdim]
    float *o;                // [T][H * vdim] before the norm
    void *out;               // activations [T][out_pitch]: normed, gated
    uint32_t out_pitch;
    uint32_t T, n_seq;
    const RowSpan *spans;
    const uint32_t *positions;
    const int32_t *slots;    // [T]
    uint32_t first_long;     // spans from here on are long (PREFILL_SPAN rows or more)
    float decay_min;         // of decay
};
bool retention_supported(uint32_t dim);
uint32_t launch_retention(const RetentionArgs &a, bool f32, int sm_count, cudaStream_t st);
// ---- gqa.cu ----------------------------------------------------------------------------------------------------------
struct AttentionArgs {       // softmax attention of one layer over T rows
    const float *y;          // f32 projections [T][y_pitch]: queries [n_head][n_map][dim], keys [n_kv][n_map][dim] (own_kv)
    uint32_t y_pitch;
    const void *va;          // activations [T][va_pitch]: values [n_kv][vdim] (has_v; else the values are the keys as projected), gates [n_head][vdim] from gate0
    uint32_t va_pitch, gate0;
    bool has_v, has_gate;
    uint32_t n_head, n_kv, n_map, dim, vdim, window;  // window 0: no limit
    uint32_t dim_p, vdim_p, row;  // padded sizes; elements of a cache row: keys [n_map][dim_p], value [vdim_p], padding
    float eps, scale, map_weight, head_gain;  // head_gain: of every head's output
    const float *q_norm, *k_norm;  // [dim], with norm_whole [n_head * dim] and [n_kv * dim]; null: no norm
    bool norm_whole;         // a token's queries (keys) are normed all together
    bool own_kv;             // keys and values are appended to the cache; else another layer has done so
    uint32_t keep;           // first positions that stay visible beyond the window
    float softcap;           // > 0: score = softcap tanh(score / softcap)
    const float *sink;       // [n_head]: exp of it is added to the softmax's denominator; null: none
    const float *head_gate;  // f32 [T][y_pitch]: sigmoid of entry h scales head h; null: none.  These four: one map
    Rot rot;
    void *q;                 // activations [T][n_head][n_map][dim_p]
    const void *q2 = nullptr;  // prompts on tcgen05, one map: columns from q_split on come from here
    uint32_t q_split = 0, q_pitch = 0, q_head = 0, q2_pitch = 0, q2_head = 0;  // with q2: pitches of a token and of a head, of both
    void *cache;             // activations [page][n_kv][16][row]
    uint32_t n_pages;        // of the pool
    void *out;               // activations [T][out_pitch], head h at h * vdim
    uint32_t out_pitch;
    uint32_t T, n_seq, n_short;   // spans [0, n_short) are short, the others long (PREFILL_SPAN rows or more)
    const RowSpan *spans;    // device [n_seq]
    const RowSpan *h_spans;  // the same on the host
    bool single;             // every span is one row
    const uint32_t *positions;
    const int32_t *const *tables;
    uint32_t max_pos;        // positions are below this
};
cudaError_t attention_configure();
bool attention_supported(uint32_t dim, uint32_t vdim);
uint32_t attention_cache_row(uint32_t n_map, uint32_t dim_p, uint32_t vdim_p);  // elements of a cache row
void launch_attention_prep(const AttentionArgs &a, bool f32, cudaStream_t st);  // norms, rotates and stores queries; appends keys and values
uint32_t launch_attention(const AttentionArgs &a, bool f32, int sm_count, cudaStream_t st);  // returns the kernels launched; 0: a tensor map could not be made
// gqa_tc5.cu: the long spans on tcgen05 (bf16)
cudaError_t attention_prompt_configure();
bool attention_prompt_supported(uint32_t n_map, uint32_t dim_p, uint32_t vdim_p);
bool launch_attention_prompt(const AttentionArgs &a, int sm_count, cudaStream_t st);  // false: a tensor map could not be made
int attention_take_status();  // as linear_take_status

// ---- moe.cu ----------------------------------------------------------------------------------------------------------
struct MoeArgs {             // routing of T tokens to `top` of n_expert experts; a (token, choice) is a pair, t * (top + n_shared) + choice
    const void *x;           // activations [T][x_pitch], x_pitch a multiple of 64
    uint32_t x_pitch;
    const __nv_bfloat16 *w;  // router [n_expert (+ 1 with n_shared) or more][x_pitch]
    const float *logits;     // [T][logit_pitch]: logits made by a product; null: the routing kernel makes them
    uint32_t logit_pitch;
    uint32_t n_expert, top, T;
    uint32_t n_shared;       // experts n_expert .. that every token uses after its chosen ones; their score is the sigmoid of logit n_expert
    uint32_t score_of;       // OB_ROUTER_*: what a chosen expert's logit becomes
    float scale;             // OB_ROUTER_SOFTMAX_ALL: factor of the scores
    uint32_t n_group, keep;  // n_group equal groups of neighbours: only the experts of the `keep` groups with the largest logits can be chosen
    uint32_t *expert;        // [pairs]
    float *score;            // [pairs]
    // grouping (null: pairs stay in order): pairs of one expert next to one another
    uint32_t *count;         // [n_expert + n_shared], zero before and left for the caller to zero
    uint32_t *rank, *row;    // [pairs]: place among the expert's pairs; row of the pair
    void *gathered;          // activations [pairs][x_pitch]
    float *row_score;        // [pairs], by row
    LinTile *tiles;          // tiles of tile_rows rows or fewer, *n_tiles of them
    uint32_t *n_tiles, tile_rows;
};
constexpr uint32_t MOE_MAX_EXPERTS = 1024;
constexpr uint32_t MOE_DOT_TOKENS = 64;  // up to this many tokens the routing kernel makes the logits itself
uint32_t launch_moe_route(const MoeArgs &a, bool f32, cudaStream_t st);  // returns the kernels launched

// ---- recurrence.cu ---------------------------------------------------------------------------------------------------
// Per head a state S [dim][vdim] in fp32.  With a decay per token: S = a S + k (s v)^T, o = S^T q.  With a decay per key entry:
// o = S^T q, then S = diag(w) S + k v^T.
struct RecurrenceArgs {
    const float *q, *k, *v;  // rows of [n_head / share][dim], the same, [n_head][vdim]
    uint32_t pitch;          // of all three
    uint32_t share;          // consecutive heads that share q and k
    const float2 *step;      // [T][n_head] (a, s); null: decay per key entry
    const float *w;          // rows of [n_head][dim]
    uint32_t w_pitch;
    uint32_t n_head, dim, vdim;
    float *state;            // [slot][n_head][dim][vdim]
    float *o;                // [T][n_head * vdim]
    uint32_t n_seq, first_long;  // spans from first_long on are long (PREFILL_SPAN rows or more)
    const RowSpan *spans;
    const uint32_t *positions;
    const int32_t *slots;    // [T]
};
cudaError_t recurrence_configure();
bool recurrence_supported(uint32_t dim);
uint32_t launch_recurrence(const RecurrenceArgs &a, int sm_count, cudaStream_t st);  // returns the kernels launched

struct ConvArgs {            // causal convolution per channel, silu; and the steps of a state-space layer
    const float *y;          // projections [T][y_pitch]: inputs of the channels, then [n_head] raw step sizes
    uint32_t y_pitch, n_channel, taps, n_head;
    const float *w, *b;      // [n_channel][taps] (the last tap meets the current token), [n_channel]
    float *state;            // [slot][taps - 1][n_channel]: the last inputs, the oldest first
    float *u;                // [T][n_channel]
    const float *dt_bias, *a_log;  // [n_head]
    float2 *step;            // [T][n_head]: (exp(-exp(a_log) dt), dt) with dt = softplus(raw + dt_bias)
    uint32_t T, n_seq;
    const RowSpan *spans, *h_spans;
    bool single;
    const uint32_t *positions;
    const int32_t *slots;
};
constexpr uint32_t CONV_MAX_TAPS = 16;
void launch_conv(const ConvArgs &a, cudaStream_t st);

struct StateSpaceOutArgs {   // (o + skip x) silu(z), normed in n_part equal parts, times norm
    const float *o, *x;      // [T][inner]; rows of [inner]
    uint32_t x_pitch;
    const void *z;           // activations [T][z_pitch]
    uint32_t z_pitch, inner, vdim, n_part, T;
    const float *skip, *norm;  // [inner / vdim], [inner]
    float eps;
    void *out;               // activations [T][out_pitch]
    uint32_t out_pitch;
};
bool state_space_out_supported(uint32_t part);
void launch_state_space_out(const StateSpaceOutArgs &a, bool f32, cudaStream_t st);

constexpr uint32_t SHIFT_MIXES = 5;
struct ShiftMixArgs {        // h = x / rms(x) * norm; mix i = h + (h' - h) mu[i], h' the previous token's h
    const float *x;          // [T][width]
    const float *norm;       // null: h is x
    const float *mu[SHIFT_MIXES];
    float *state;            // [slot][width]: the last token's h
    void *mix;               // activations [T][SHIFT_MIXES * pitch]
    uint32_t width, pitch, T, n_seq;
    float eps;
    const RowSpan *spans;
    bool single;
    const uint32_t *positions;
    const int32_t *slots;
};
void launch_shift_mix(const ShiftMixArgs &a, bool f32, cudaStream_t st);

struct TimeMixOutArgs {      // per head: (o + (sum r bonus k) v) over its root mean square, times norm, times silu(gate)
    const float *o;          // [T][n_head * dim]
    const float *r, *k, *v, *gate;  // rows of [n_head * dim]
    uint32_t pitch, n_head, dim, T;
    const float *bonus, *norm;  // [n_head * dim]
    float eps;
    void *out;
    uint32_t out_pitch;
};
void launch_time_mix_out(const TimeMixOutArgs &a, bool f32, cudaStream_t st);

// ---- residual.cu -----------------------------------------------------------------------------------------------------
struct ResidualArgs {        // s = x + mult y; v = depth average of s, or s; n = grouped norm of v; h = n + causal convolution of n (or n)
    const float *x;          // [..][width]; null: the tokens' embeddings
    const uint32_t *x_rows;  // row of x of each token; null: in order
    const __nv_bfloat16 *table;
    const uint32_t *tokens;
    const float *y;          // null: nothing is added; else the sum of a token's `top` rows, as in PostNormArgs
    const uint32_t *rows;
    uint32_t top;
    float mult;
    float *sum;              // [T][width] gets s; may be null, may be x.  With a convolution one of this and average is given
    const float *depth;      // [n_history + 1]: factors of the rows of `history`, then of s; null: no average
    const float *history;    // n_history arrays [T][width], history_step apart
    uint64_t history_step;
    uint32_t n_history;
    float *average;          // [T][width] gets v; may be null
    const float *norm;       // [width]; null: h is not made
    uint32_t n_group;        // equal parts of the width that are normed each by itself; at least 1
    float eps;
    const float *conv;       // [taps][width], the last tap meets the current token
    uint32_t taps;           // 0: no convolution
    float *state;            // [slot][taps - 1][width]: the last n, the oldest first
    float *inverse;          // scratch [T][n_group]
    void *h;                 // activations [T][h_pitch]
    uint32_t h_pitch;
    uint32_t *zero;          // as in PostNormArgs
    uint32_t n_zero;
    uint32_t width, T, n_seq;
    const RowSpan *spans, *h_spans;
    bool single;             // every span is one row
    const uint32_t *positions;
    const int32_t *slots;
};
uint32_t launch_residual(const ResidualArgs &a, bool f32, cudaStream_t st);  // returns the kernels launched

// Pages [0, n_pages) of one sequence's table to another's within a pool of pages of page_bytes (a multiple of 16).
void launch_copy_pages(void *pool, uint64_t page_bytes, const int32_t *src_table, const int32_t *dst_table, uint32_t n_pages, cudaStream_t st);

}  // namespace ob
