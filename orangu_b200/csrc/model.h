// The device-resident model and its per-sequence cache, shared by the translation units that build models (model.cu for the
// Llama graph, layered.cu for models given as a list of layers) and the one that steps them.
#pragma once

#include <algorithm>
#include <map>
#include <string>
#include <vector>

#include "layered.h"
#include "runtime.h"
#include "tp.h"

namespace obrt {

struct LayerDev {
    float *attn_norm = nullptr, *ffn_norm = nullptr;
    float *q_bias = nullptr, *k_bias = nullptr, *v_bias = nullptr, *q_norm = nullptr, *k_norm = nullptr;  // this rank's part; null: absent
    bool variant = false;  // any of the above, or the NEOX pairing: the layer takes the operator-by-operator path
    ob_weight *wq = nullptr, *wk = nullptr, *wv = nullptr, *wo = nullptr, *gate = nullptr, *up = nullptr, *down = nullptr;
};

struct ActPair {  // both granularities for one product input
    ActBuf k, flat;
};

// Per-step metadata, one pinned host block mirrored by one device block.
struct MetaLayout {
    uint32_t T;
    size_t off_tokens, off_positions, off_npos, off_tables, off_slots, off_spans, off_logit_rows, bytes;
    explicit MetaLayout(uint32_t t) : T(t) {
        off_tokens = 0;
        off_positions = off_tokens + (size_t)t * 4;
        off_npos = off_positions + (size_t)t * 4;
        off_tables = (off_npos + (size_t)t * 4 + 15) & ~(size_t)15;
        off_slots = off_tables + (size_t)t * 8;       // state slot of each row's sequence
        off_spans = off_slots + (size_t)t * 4;        // rows of each sequence of the step
        off_spans = (off_spans + 7) & ~(size_t)7;
        off_logit_rows = off_spans + (size_t)t * sizeof(RowSpan);
        bytes = off_logit_rows + (size_t)t * 4;
    }
};

// What a model family other than the Llama graph of model.cu supplies.  Everything around it -- the page pool and the page
// tables, the state slots, the metadata block, sampling, captured graphs, the slot pool -- is the model's.
struct StepGraph {
    virtual ~StepGraph() {}
    // All layers for the T rows that d_meta describes: n_seq spans of rows (MetaLayout::off_spans), one batch.
    // single: every span is one row.  max_pos bounds the positions of the rows (exclusive).
    virtual void layers(uint32_t T, uint32_t n_seq, const RowSpan *spans, uint32_t max_pos, cudaStream_t st) = 0;
    // Logits of n rows, the numbers of which are at d_rows (null: rows 0 .. n-1), into m->logits [n][n_vocab].
    virtual void head(const uint32_t *d_rows, uint32_t n, cudaStream_t st) = 0;
    virtual bool take_failure() = 0;  // a launch was refused since the last call
    // Something other than pages carries the sequence: it can be emptied and copied whole, not cut.
    virtual bool recurrent() const = 0;
    // The first n positions' pages (and the state, when n is all of them) of one sequence to another.
    virtual int copy_prefix(ob_kv *dst, const ob_kv *src, uint32_t n) = 0;
    virtual int read_pages(const ob_kv *kv, uint32_t layer, uint32_t pos0, uint32_t n, float *k_out, float *v_out) = 0;
    virtual int read_state(const ob_kv *kv, uint32_t layer, float *out) = 0;
};

}  // namespace obrt

using namespace obrt;

struct ob_model {
    ob_ctx *ctx = nullptr;
    ob_model_desc cfg{};
    uint32_t tp_rank = 0, tp_size = 1;
    uint32_t n_head_l = 0, n_head_kv_l = 0, n_ff_l = 0, vocab_l = 0, vocab0 = 0;
    std::vector<LayerDev> layers;
    ob_weight *token_embd = nullptr, *output = nullptr;
    float *output_norm = nullptr;
    float *rope_table = nullptr;
    std::vector<void *> owned;  // plain cudaMalloc blocks

    // KV pool: [layer][page][n_head_kv_l][16][head_dim] fp16, K and V
    uint32_t pool_pages = 0;
    __half *k_pool = nullptr, *v_pool = nullptr;
    size_t layer_stride = 0;  // elements
    std::vector<int32_t> free_pages;

    // A model whose layers are not the Llama graph below: its step, and the slots of its per-sequence state.
    StepGraph *graph = nullptr;
    uint32_t n_state_slots = 0;
    std::vector<int32_t> free_slots;
    uint32_t logit_cap = 0;  // rows m->logits holds

    uint32_t T = 0;  // max rows per step
    float *x = nullptr, *q = nullptr, *k = nullptr, *v = nullptr, *attn = nullptr, *gate = nullptr, *up = nullptr, *proj = nullptr,
          *logits = nullptr;
    ActPair act_embd, act_attn, act_ff;
    float *part_o = nullptr, *part_ml = nullptr;
    uint32_t *ff_counters = nullptr;    // [n_ff / 256] arrival counters of the SwiGLU outputs, zero between launches
    uint32_t *attn_counters = nullptr;  // [rows][kv heads] arrival counters of the fused attention kernel, zero between launches
    float *norm_scale = nullptr;      // [2] RMSNorm scales for the fused decode kernels (attention norm, FFN / output norm)
    uint8_t *ready_embd = nullptr, *ready_attn = nullptr, *ready_ff = nullptr;  // quantized activations of the single decode token
    float *scores = nullptr;          // exact-order attention scratch [T][n_head_l][score_stride]
    uint32_t score_stride = 0, exact_attn_max_pos = 0;
    uint32_t max_splits = 1;
    size_t row_splits_cap = 0;  // (row, split) pairs part_o / part_ml hold
    uint8_t *d_meta = nullptr, *h_meta = nullptr;
    uint32_t *d_out_tokens = nullptr, *h_out_tokens = nullptr;
    unsigned long long *argmax_scratch = nullptr;
    uint32_t *d_history = nullptr, *d_step_counter = nullptr;
    uint32_t history_cap = 0;
    uint32_t last_T = 0;
    std::map<uint64_t, cudaGraphExec_t> graphs;
    std::map<uint64_t, uint64_t> graph_launches;  // kernels one replay stands for
    obtp::Comm *comm = nullptr;
    obtp::PeerXchg px{};         // size > 1: the single-token step exchanges partials through peer memory instead of NCCL
    obtp::PeerBulk bulk{};       // cap > 0: so do steps of a few rows (decode batches, short prefill chunks)
    bool use_stream = true;  // OB_STREAM_GEMV=0 keeps batch-1 decode on the unfused kernels
    bool stream_ok = false;      // every fused decode kernel of this model's shapes fits (shared memory)
    bool use_fused_attn = true;  // OB_FUSED_ATTN=0 keeps the two-kernel flash-decode
    bool use_prefill_attn = true;  // OB_PREFILL_ATTN=0: prefill chunks take the decode kernel row by row
    bool comm_failed = false;    // a collective could not be enqueued during the last step (reported by check_peer)
    obtp::Rendezvous *rdv = nullptr;  // host-side meeting of the ranks before a step is enqueued (tensor parallel only)
    uint32_t rdv_timeout_ms = 30000;  // OB_TP_RENDEZVOUS_MS; 0 = off
    bool out_of_step = false;         // a rendezvous failed: the ranks no longer run the same sequence of steps
    // Persistent layer kernel (layer_stream.cu): the single-token products between two attention kernels as one launch.
    // Phase list: [q/k/v of layer 0] then per layer [attention-output, gate/up, down, q/k/v of the next layer | output projection].
    bool use_persist = false;    // OB_PERSIST=1; measured slower than one launch per product (barrier waits and the synchronous norm outweigh the launches saved)
    bool persist_ok = false;
    bool launch_failed = false;  // a launch of the persistent kernel was refused (reported after the step)
    std::vector<LsPhase> h_phases;
    LsPhase *d_phases = nullptr;
    LsLayout ls_layout{};
    uint32_t *ls_barriers = nullptr;  // one word per launch of a step, zeroed when the step starts
    uint32_t *ls_status = nullptr;    // set by the kernel when a barrier wait ran out of time
    uint32_t *h_ls_status = nullptr;  // pinned host copy, fetched with every step's results
    uint32_t ls_timeout_ms = 2000;
    bool ls_split = false;            // OB_LS_SPLIT=1: every phase is its own launch
};

struct ob_kv {
    ob_model *m = nullptr;
    uint32_t capacity = 0, len = 0;
    std::vector<int32_t> pages;   // pages held, in position order
    int32_t *d_table = nullptr;   // device copy, room for ceil(capacity / 16) entries
    int32_t slot = -1;            // state slot (models with recurrent layers): held while the sequence holds tokens
    bool on_demand = false;       // pages are taken from the pool as the sequence grows (ob_kv_create_paged) and go back on truncate
};

namespace obrt {

template <typename Tp>
inline int dev_alloc(ob_model *m, Tp **out, size_t count) {
    void *p = nullptr;
    OB_CUDA(m->ctx, cudaMalloc(&p, std::max<size_t>(count * sizeof(Tp), 16)));
    m->owned.push_back(p);
    *out = static_cast<Tp *>(p);
    return OB_OK;
}

inline int upload_f32(ob_model *m, const float *src, size_t n, float **out) {
    int rc = dev_alloc(m, out, n);
    if (rc) return rc;
    OB_CUDA(m->ctx, cudaMemcpyAsync(*out, src, n * 4, cudaMemcpyHostToDevice, m->ctx->stream));
    return OB_OK;
}

}  // namespace obrt
