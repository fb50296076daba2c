// Host-side objects of libswlm_cuda.so shared by its executors: the context (weight store), the compiled plan and the
// runtime state behind the handles of include/swlm.h.
#pragma once

#include <algorithm>
#include <map>
#include <string>
#include <vector>

#include "swlm_internal.h"

namespace swlm {

template <typename T>
inline int dev_alloc(T** p, size_t count, int64_t* total = nullptr) {
    *p = nullptr;
    if (count == 0) return SWLM_OK;
    SWLM_CUDA(cudaMalloc((void**)p, count * sizeof(T)));
    if (total) *total += (int64_t)(count * sizeof(T));
    return SWLM_OK;
}


enum LaunchKind { L_EMBED, L_RMSNORM, L_QGEMV, L_QK_NORM, L_ATTN, L_SWIGLU, L_CONV, L_ARGMAX, L_SSM,
                  L_PRODUCT, L_LATENT, L_DELTA, L_ROUTED, L_SOFTCAP, L_GROUPED, L_RETENTION, L_JOIN, L_TOKEN_GATE };   // from L_PRODUCT on: fp32-stream plans only

// What a launch over the residual stream does, in this order; parts that are not set are left out (see JoinLaunch).
struct JoinParts {
    const DenseTensor* table = nullptr; float table_scale = 1.f;               // starts the stream
    int keep = -1;                                                             // convolution whose last inputs go to its state
    bool adds = false; int in_buf = -1, gate_buf = -1; const DenseTensor* w = nullptr; float eps = 0.f, weight_bias = 0.f;
    int store = -1; const DenseTensor* avg_w = nullptr; int avg = 0;           // results of the layers
    int copy_buf = -1;
    int conv = -1, conv_buf = -1; const DenseTensor* conv_w = nullptr;
    bool changes() const { return table || adds || avg; }
};

struct Launch {
    int kind = 0;
    swlm_step st{};            // the (first) step this launch came from
    const Q4Tiled* w = nullptr;
    std::vector<std::string> w_names;
    int w_mode = 0;
    int epilogue = QGEMV_EPI_STORE;
    int gated_act = GATED_ACT_SILU;
    int n_seg = 1;
    int seg_buf[kMaxProductSegs] = {-1, -1, -1, -1, -1, -1, -1, -1};
    int seg_off[kMaxProductSegs] = {};     // first column in the buffer (fp32-stream plans)
    int seg_end[kMaxProductSegs] = {};
    const DenseTensor* d1 = nullptr;
    const DenseTensor* d2 = nullptr;
    const Q4Raw* q_embed = nullptr;  // embedding step over a quantized table
    const DenseF32* f1 = nullptr;    // recurrent step: norm weight, A_log (d1 = conv taps, d2 = dt_bias)
    const DenseF32* f2 = nullptr;
    int rope_table = -1;       // index into plan->rope_tables
    std::string label;
    int steps_covered = 1;
    // residual add / copy / RMSNorm folded into this product's prologue (norm.kind == 0: none)
    swlm_step norm{};
    const DenseTensor* norm_w = nullptr;
    int x_buf = -1;            // buffer the product reads (the norm's input when fused)
    int push = 0, in_tp = 0;   // tensor parallel: partial rows pushed to all ranks / pushed partials consumed
    int res_in = 0, res_out = 0;  // physical residual buffers (0 or 1) this launch reads / writes
    int prefetch_launch = -1;     // index of the later product whose weights this launch pulls into L2
    // products of fp32-stream plans: one matrix (possibly the rows of several tensors), or gate and up
    const Matrix* m1 = nullptr;
    const Matrix* m2 = nullptr;
    const Matrix* m3 = nullptr;               // routed feed-forward: the experts' down rows (m1, m2: gate, up)
    const Matrix *m4 = nullptr, *m5 = nullptr;   // and the shared feed-forward's up and down
    GatedAct act;
    float softcap = 0.f;                      // of the output head's logits
    const DenseTensor* seg_bias[kMaxProductSegs] = {};
    Matrix part[2];                           // products of two inputs: the rows that meet the first and the second one
    int x2_buf = -1, first_segs = 0;          // the second input, and how many results belong to the first
    JoinParts join;
    int fused = 0;                            // single tokens: this many launches behind this one are part of it (a token input)
    const DenseTensor* dv[6] = {};            // gated delta rule: taps of q, k, v, norm weight, A_log, dt_bias; latent attention: [0] sink; norms: [0] table that joins
    int window_set = 0;                       // latent attention: index into plan->windows
    const DenseTensor* norm_post = nullptr;   // norm steps: weight of the norm applied to the input before it is added
    int kv_prefetch_attn = -1;    // index of the attention launch whose K/V rows this product pulls into L2
};

// Angle per position of every rotated pair, with the scaling the table was built for (factor 0: none); cos and sin are
// multiplied by `magnitude`.
struct RopeTable {
    int rope_dim; float base; float* inv_freq;
    float factor = 0.f, original = 0.f, fast = 0.f, slow = 0.f, magnitude = 1.f, divisor = 1.f;
};

// One latent-attention layer's share of the page pool.
struct LatentLayer { int rank = 0, rot = 0; LatentRow row{}; };

// One grouped-attention layer's share of the page pool.
struct GroupedLayer { GroupedRow row{}; };

// One convolution over the stream: its last taps - 1 inputs per sequence, in fp32.
struct StreamConv { int taps = 0; };

// One gated-delta or retention layer: per sequence an fp32 state and the last inputs of the convolutions (retention: no taps).
struct DeltaLayer {
    DeltaShape shape;
    size_t state_elems() const { return (size_t)shape.heads * shape.dim * shape.vdim; }
    size_t ring_elems() const { return (size_t)shape.taps * shape.channels(); }
};

// Activation buffers and scratch of the row executor of fp32-stream plans. A state holds two sets: one sized for a decode
// step (its pointers are captured in CUDA graphs and never change), one that grows with the largest batch of rows seen.
struct StreamBufs {
    int rows = 0, wants = 0;              // capacity: activation rows, rows of the output head
    void* buf[SWLM_BUF_COUNT] = {};       // HIDDEN, RESIDUAL, SCRATCH3, SCRATCH4, LOGITS fp32; the others in the plan's activation type
    float* res2 = nullptr;                // ping-pong partner of RESIDUAL
    int32_t* meta = nullptr; size_t meta_cap = 0;        // row descriptors: token, sequence, position per row, row lists, spans, tiles
    int32_t* argmax_out = nullptr;
    float* qcat = nullptr; size_t qcat_cap = 0;          // latent attention: absorbed queries
    float* partial = nullptr; size_t partial_cap = 0;    // latent attention: partial results per split
    float* part = nullptr; size_t part_cap = 0;          // products: sums of K ranges
    unsigned char* expand = nullptr; size_t expand_cap = 0;
    float* delta = nullptr; size_t delta_cap = 0;        // gated delta rule: records and read-outs of portions
    unsigned char* routed = nullptr; size_t routed_cap = 0;
    float* argmax_val = nullptr; int32_t* argmax_idx = nullptr;
    float* results = nullptr;             // depth-wise average: [result][rows][width of RESIDUAL]
};

// One batch of rows for the row executor (device pointers).
struct RowBatch {
    int rows = 0;
    const int32_t *tok = nullptr, *seq = nullptr, *pos = nullptr;
    int wants = 0; const int32_t* wants_idx = nullptr;              // rows that get logits; null: rows 0 .. wants - 1
    int n_short = 0; const int32_t* short_rows = nullptr; int splits_pages = 1;   // latent attention one by one; longest context in pages
    int n_long = 0; const int32_t* long_rows = nullptr;             // and in spans
    int n_spans = 0; int n_tiles = 0; const int2* tiles = nullptr;
    std::vector<const LatentSpan*> spans; std::vector<int> total_ctx;   // per window of the plan: what is gathered depends on it
    int n_single = 0; const int32_t* single_rows = nullptr;         // gated delta rule: single tokens (null: rows 0 .. n_single - 1)
    int n_runs = 0; const RowRun* runs = nullptr; int n_blocks = 0; const int32_t* block_run = nullptr;   // and longer portions
    bool advance = false;                                           // decode step over all sequences: feed tokens back, advance positions
};

}  // namespace swlm

using namespace swlm;

struct swlm_ctx {
    int device = 0, tp_rank = 0, tp_size = 1;
    cudaStream_t stream = nullptr;
    std::map<std::string, Q4Raw> raw;
    std::map<std::string, Q4Tiled> tiled;  // plain and fused tensors, keyed by name ("a|b|c" for fused)
    std::map<std::string, Q4Raw> raw_cat;  // source-layout tensors with the rows of several raw tensors one after the other ("a|b|c")
    std::map<std::string, DenseTensor> dense;
    std::map<std::string, Matrix> matrices;      // bf16 matrices of the dense products
    std::map<std::string, Matrix> matrix_cat;    // the rows of several of them one after the other ("a|b|c"); the parts become views of it
    std::map<std::string, DenseF32> densef;   // fp32 tensors (recurrent layers' norm weight and A_log)
    int64_t bytes = 0;
    float* op_partial = nullptr; size_t op_partial_floats = 0;
    unsigned char* op_xh = nullptr; size_t op_xh_bytes = 0;   // scratch of the op-level tensor-core product
    unsigned* op_attn_counters = nullptr; size_t op_attn_counter_count = 0;
    unsigned* op_counters = nullptr; size_t op_counter_count = 0;
    int* tc_status = nullptr;  // device word the tcgen05 GEMM sets when one of its bounded waits expired
    // Lifetime: plans keep their context alive, states their plan. A destroy call on an object that still has
    // users only marks it; the memory goes when the last user is destroyed (hosts with garbage-collected
    // wrappers release objects in no particular order).
    int users = 0;
    bool destroy_requested = false;
};

struct swlm_plan {
    swlm_ctx* ctx = nullptr;
    swlm_buffers_desc desc{};
    std::vector<swlm_step> steps;
    std::vector<Launch> launches;
    std::vector<RopeTable> rope_tables;
    int attn_splits = 1;
    size_t attn_scratch = 0, qgemv_partial = 0, qgemv_counters = 0;
    int final_res = 0;  // physical residual buffer that holds the residual stream after a step
    // Row-wise execution (prompt chunks, more than 16 sequences): consecutive products of one input run as one product
    // over their concatenated rows. Per step: how many steps the product starting there covers (0: covered by an
    // earlier one) and the tensor it multiplies.
    struct RowsGroup { int count = 1; const Q4Raw* raw = nullptr; };
    std::vector<RowsGroup> rows_groups;
    bool rows_groups_ready = false;
    // fp32-stream plans (desc.stream_dtype != 0)
    std::vector<LatentLayer> latent;      // by step.layer
    std::vector<GroupedLayer> grouped;    // by step.layer
    std::vector<DeltaLayer> delta;        // by step.layer
    std::vector<StreamConv> convs;        // by step.layer
    bool biased = false;                  // do products have biases?
    std::vector<int> windows;             // distinct sliding windows of the attention layers
    int stream_width[SWLM_BUF_COUNT] = {};
    int latent_heads_max = 0, latent_q_floats = 0, latent_part_floats = 0;   // largest over the layers, per row / per row and split
    bool stream() const { return desc.stream_dtype != 0; }
    bool all_f32() const { return desc.stream_dtype == SWLM_STREAM_ALL_F32; }
    int users = 0;
    bool destroy_requested = false;
};

struct swlm_state {
    swlm_plan* plan = nullptr;
    cudaStream_t own_stream = nullptr, stream = nullptr;
    __nv_bfloat16* buf[SWLM_BUF_COUNT] = {};
    int width[SWLM_BUF_COUNT] = {};
    __nv_bfloat16* kcache = nullptr; __nv_bfloat16* vcache = nullptr; size_t kv_layer_elems = 0;
    // rotated KV schemes: rotors [kv_layers][kv_heads][groups][4], projection matrix [head_dim][qjl_dim], projected K
    // residuals [kv_layers][seq][kv_heads][max_seq][qjl_dim], all fp16
    __half* rotors = nullptr; size_t rotor_layer_elems = 0;
    __half* qjl_matrix = nullptr;
    __half* qjl_res = nullptr; size_t qjl_layer_elems = 0;
    std::vector<uint16_t> rotors_host, qjl_matrix_host;   // host copies for the cache probes
    __nv_bfloat16* conv = nullptr; size_t conv_layer_elems = 0;
    __nv_bfloat16* ssm_conv = nullptr; size_t ssm_conv_layer_elems = 0;   // [layer][seq][kernel][conv_dim]
    float* ssm_state = nullptr; size_t ssm_state_layer_elems = 0;         // [layer][seq][heads][key_dim][value_dim]
    int32_t* position = nullptr; int32_t* step_counter = nullptr;
    int32_t* token_in = nullptr; int32_t* token_out = nullptr; int32_t* ring = nullptr;
    int32_t* prompt = nullptr; size_t prompt_cap = 0;
    int ring_cap = 4096;
    float* attn_scratch = nullptr; float* qgemv_partial = nullptr; unsigned* qgemv_counters = nullptr;
    size_t attn_scratch_cap = 0, qgemv_partial_cap = 0, qgemv_counters_cap = 0;
    unsigned* attn_counters = nullptr;
    float* argmax_val = nullptr; int32_t* argmax_idx = nullptr;
    __nv_bfloat16* res2 = nullptr;  // second physical residual buffer (ping-pong partner of buf[RESIDUAL])
    // tensor-parallel exchange (tp_size > 1): this rank's buffer, the peers' mappings, local counters
    TpParams tp{};
    bool tp_attached = false;
    int32_t* tp_words = nullptr;  // [0] all-reduce epoch, [1] rows-done counter, [2] status, [3] argmax epoch, [4] CTAs done pushing a prompt chunk
    int tp_rows_epoch = 0;        // prompt-chunk exchanges issued so far (the same count on every rank)
    int32_t* h_tok = nullptr;  // pinned host staging, 2 * max_batch
    std::vector<int> pos_host;   // host mirror of the per-sequence positions
    long long steps_host = 0;
    cudaGraphExec_t graph_full = nullptr, graph_body = nullptr;
    int graph_full_launches = 0, graph_body_launches = 0;
    int64_t launches = 0;
    // prompt ingestion in chunks: activation rows for `pf_rows` tokens per logical buffer, attention scratch
    __nv_bfloat16* pf_buf[SWLM_BUF_COUNT] = {};
    int pf_rows = 0;
    unsigned* pf_attn_counters = nullptr;
    unsigned char* wide_xh = nullptr;  // the same for a decode step of more than kQGemvMaxRows sequences
    unsigned char* pf_xh = nullptr;  // scratch of the tensor-core product: fp16 copy of a chunk's widest activations
    int* pf_status = nullptr;      // device word: a bounded wait of the tensor-core product expired
    int prefill_chunk = 2048;      // tokens per chunk; 0 = one token at a time through the decode graph
    int* tc_status = nullptr;      // pinned host word (mapped): a bounded wait of a kernel expired
    // fp32-stream plans: paged pools, those of the latent layers first, then the grouped ones (one page list per sequence, the same page numbers in every layer's
    // pool), the page table on host and device, and the two activation sets
    std::vector<void*> pool; std::vector<size_t> pool_bytes;
    std::vector<float*> delta_state; std::vector<void*> delta_ring;   // per gated-delta layer: [max_batch][state_elems], [max_batch][ring_elems]
    std::vector<float*> conv_state;                                   // per convolution over the stream: [max_batch][taps - 1][hidden]
    unsigned* routed_counts = nullptr;                                // rows per expert, zero between launches
    int pool_pages = 0, pages_per_seq = 0;
    std::vector<int> free_pages;
    std::vector<std::vector<int>> seq_pages;
    std::vector<int32_t> page_table_host; int32_t* page_table = nullptr; bool page_table_dirty = false;
    StreamBufs dec, big;
    StreamBufs* last_bufs = nullptr; int last_res = 0;     // what the buffer probes read
    int32_t* seq_identity = nullptr;
    std::map<int, cudaGraphExec_t> row_graphs;   // decode steps of n rows, any sequences
    std::map<int, int> row_graph_launches;
    int32_t* h_rows = nullptr; size_t h_rows_cap = 0;      // pinned staging of row descriptors
};

struct swlm_snap {
    std::vector<void*> dev;
    std::vector<size_t> bytes;
    std::vector<int> pos_host;
    std::vector<std::vector<int>> seq_pages;   // fp32-stream plans: page lists and the free list
    std::vector<int> free_pages;
};


// ---- fp32-stream plans (stream_exec.cu) -----------------------------------------------------------------------------
namespace swlm {
int stream_compile(swlm_plan* plan);
void stream_plan_free(swlm_plan* plan);
int stream_state_create(swlm_state* s);
void stream_state_free(swlm_state* s);
// pages for `tokens` tokens of a sequence (more are taken, surplus ones given back when `shrink`)
int stream_reserve(swlm_state* s, int seq, int tokens, bool shrink = false);
void stream_release_all(swlm_state* s);
int stream_upload_pages(swlm_state* s);
int stream_enqueue_step(swlm_state* s, bool body_only, cudaStream_t stream, int only_kind);
int stream_launches_per_step(const swlm_plan* plan);
void stream_drop_graphs(swlm_state* s);
// the entries of swlm_run_batch, at most row_cap rows at a time
int stream_run(swlm_state* s, int n_entries, const int32_t* seqs, const int32_t* counts, const int32_t* tokens, const int32_t* want_counts,
               const int32_t* wants, float* logits_out, int32_t* tokens_out, int row_cap);
int stream_profile(swlm_state* s, int seq, const int32_t* tokens, int n, int only_kind, int repeats);
int stream_run_step(swlm_state* s, const swlm_step* step, const int32_t* token_in, int32_t* token_out);
int stream_check_status(swlm_state* s);
}  // namespace swlm
