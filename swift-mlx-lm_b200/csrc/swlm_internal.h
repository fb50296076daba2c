// Internal declarations shared by the translation units of libswlm_cuda.so.
#pragma once

#include <cuda_bf16.h>
#include <cuda_fp16.h>
#include <cuda_runtime.h>

#include <cstdint>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "../../include/swlm.h"
#include "tp_device.cuh"

namespace swlm {

// ---- errors ------------------------------------------------------------------
void set_error(const char* fmt, ...);
int cuda_fail(cudaError_t e, const char* what);  // records the message, returns SWLM_ERR_CUDA
#define SWLM_CUDA(call)                                          \
    do {                                                         \
        cudaError_t e__ = (call);                                \
        if (e__ != cudaSuccess) return ::swlm::cuda_fail(e__, #call); \
    } while (0)

// ---- launches ------------------------------------------------------------------
// Every kernel of the decode step is launched with programmatic stream serialization (programmatic
// dependent launch): a kernel may start while its predecessor drains, does what does not depend on it
// (the GEMV kernels start streaming weights), and executes `griddepcontrol.wait` before it touches
// anything the predecessor wrote. SWLM_NO_PDL=1 in the environment turns the attribute off.
bool pdl_enabled();
template <typename... P, typename... A>
inline cudaError_t launch_k(void (*kernel)(P...), dim3 grid, dim3 block, size_t smem, cudaStream_t s, A... args) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = grid; cfg.blockDim = block; cfg.dynamicSmemBytes = smem; cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[0].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl_enabled() ? 1 : 0;
    return cudaLaunchKernelEx(&cfg, kernel, static_cast<P>(args)...);
}
#ifdef __CUDACC__
// Wait until the preceding kernel in the stream has completed and its writes are visible.
__device__ __forceinline__ void pdl_wait() { asm volatile("griddepcontrol.wait;" ::: "memory"); }
// Allow the next kernel in the stream to begin launching.
__device__ __forceinline__ void pdl_launch_dependents() { asm volatile("griddepcontrol.launch_dependents;" ::: "memory"); }
#endif

// ---- device tensors -----------------------------------------------------------
//
// Q4 group-64 tensor in the streaming layout of the GEMV/GEMM kernels.
//   tiles : uint4[row_tiles][kt_pad][32]   one 512-byte tile = 16 rows x 64 columns,
//           lane (g = lane>>2, t = lane&3) owns 16 bytes = 4 words; word j, nibble e holds
//           W[16*rt + g + 8*(e&1)][64*kt + 16*t + 4*j + (e>>2) + 2*((e>>1)&1)]:
//           the A-fragment order of mma.m16n8k16 for k-step j, with the group's columns assigned to
//           k-steps so that lane t's B fragments are the 16 consecutive activations 16t..16t+15.
//   sb    : uint4[row_tiles][kt_pad/4][16]  per row, four consecutive groups' (scale, zero)
//           pairs, each pair two 16-bit floats (bf16, or fp16 when the source was STAF).
// kt_pad = K/64 rounded up to a multiple of 4; padding tiles hold q = 0, scale = zero = 0.
struct Q4Tiled {
    int n = 0, k = 0;           // logical (per-rank) shape
    int row_tiles = 0;          // ceil(n / 16)
    int kt_pad = 0;             // k-tiles including padding
    bool sb_f16 = false;        // scale/zero stored as fp16 instead of bf16
    bool interleaved = false;   // rows 0-7 of each tile from source A, rows 8-15 from source B
    uint4* tiles = nullptr;
    uint4* sb = nullptr;
    size_t bytes() const { return (size_t)row_tiles * kt_pad * 512 + (size_t)row_tiles * (kt_pad / 4) * 256; }
};

// Raw source copy kept on the device so that fused tensors can be assembled at plan time.
struct Q4Raw {
    int n = 0, k = 0;
    bool sb_f16 = false;
    int shard_kind = 0;
    uint32_t* w = nullptr;      // [n][k/8]
    uint16_t* scales = nullptr; // [n][k/64]
    uint16_t* biases = nullptr;
};

struct DenseTensor {
    int64_t rows = 0, cols = 0;
    int shard_kind = 0;
    __nv_bfloat16* data = nullptr;
};

struct DenseF32 {
    int64_t count = 0;
    float* data = nullptr;
};

// ---- kernels: launch wrappers (each returns a status; no synchronisation) -------

struct RepackSrc {
    const uint32_t* w;
    const uint16_t* scales;
    const uint16_t* biases;
    int n;
};
// Build a tiled tensor from up to three raw sources that share K.
// mode 0: rows concatenated; mode 1: two sources interleaved 8 rows each per tile.
int launch_repack(const RepackSrc* src, int n_src, int mode, int k, const Q4Tiled& dst, cudaStream_t s);
int launch_untile_bf16(const Q4Tiled& t, __nv_bfloat16* out, cudaStream_t s);

enum { QGEMV_EPI_STORE = 0, QGEMV_EPI_SWIGLU = 1 };   // SWIGLU: the gated-activation epilogue (SiLU or GELU, see gated_act)
enum { GATED_ACT_SILU = 0, GATED_ACT_GELU_TANH = 1, GATED_ACT_CLAMPED = 2 };
// Activation of a gated feed-forward. CLAMPED: g = min(gate, limit), u = clamp(up, -limit, limit), g sigmoid(alpha g) (u + 1).
struct GatedAct { int kind = GATED_ACT_SILU; float alpha = 0.f, limit = 0.f; };
#ifdef __CUDACC__
// the exact GELU
__device__ __forceinline__ float gelu_erf(float v) { return 0.5f * v * (1.0f + erff(v * 0.70710678f)); }
// activation(gate) * up of the gated MLP (Generator/MetalSourceGenerator+NormAndElementwise.swift:176-208):
// SiLU for SwiGLU, the tanh approximation of GELU for GEGLU.
__device__ __forceinline__ float gated_activation(float g, float up, int act) {
    const float a = act == GATED_ACT_GELU_TANH ? 0.5f * g * (1.0f + tanhf(0.7978845608f * (g + 0.044715f * g * g * g)))
                                               : g * (1.0f / (1.0f + expf(-g)));
    return a * up;
}
__device__ __forceinline__ float gated_activation(float g, float up, const GatedAct& act) {
    if (act.kind != GATED_ACT_CLAMPED) return gated_activation(g, up, act.kind);
    g = fminf(g, act.limit);
    up = fminf(fmaxf(up, -act.limit), act.limit);
    return g * (1.0f / (1.0f + expf(-act.alpha * g))) * (up + 1.0f);
}
#endif

// Weights of a later launch that this launch asks the memory system to bring from HBM into L2 while it runs
// (its own data comes from L2 or is small, so HBM would otherwise idle). Two arrays, sizes multiples of 256.
struct PrefetchTarget {
    const void* p[2] = {nullptr, nullptr};
    unsigned long long bytes[2] = {0, 0};
    // heads > 0: the two arrays are the K and V caches of one layer and sequence; what is requested is the first
    // position[0] rows (row_bytes each) of every head, heads being head_stride bytes apart. The position is only a
    // hint here: a stale value requests a row too few.
    int heads = 0, row_bytes = 0;
    unsigned long long head_stride = 0;
    const int* position = nullptr;
};
#ifdef __CUDACC__
// CTA `part` of `nparts` requests its share, 16 KB per instruction, one instruction per thread and round.
__device__ __forceinline__ void prefetch_target_slice(const PrefetchTarget& t, int part, int nparts, int tid, int nthreads) {
    if (t.heads > 0) {
        // KV rows: 256-byte granules, numbered head-major over both caches
        const unsigned long long per_head = ((unsigned long long)t.position[0] * (unsigned)t.row_bytes) >> 8;
        if (per_head == 0) return;
        const unsigned long long gran = per_head * (unsigned)t.heads * 2ull;
        const unsigned long long g0 = gran * (unsigned long long)part / (unsigned long long)nparts;
        const unsigned long long g1 = gran * (unsigned long long)(part + 1) / (unsigned long long)nparts;
        for (unsigned long long g = g0 + 16ull * tid; g < g1; g += 16ull * nthreads) {  // 4 KB per instruction
            const unsigned long long hd = g / per_head, off = g - hd * per_head;        // head index over both caches
            const unsigned long long run = per_head - off < 16ull ? per_head - off : 16ull;
            const unsigned n = (unsigned)((g1 - g < run ? g1 - g : run) << 8);
            const unsigned char* base = static_cast<const unsigned char*>(t.p[hd >= (unsigned)t.heads ? 1 : 0]) +
                                        (hd % (unsigned)t.heads) * t.head_stride + (off << 8);
            asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(base), "r"(n) : "memory");
        }
        return;
    }
#pragma unroll
    for (int a = 0; a < 2; ++a) {
        if (!t.p[a]) continue;
        const unsigned long long gran = t.bytes[a] >> 8;
        const unsigned long long g0 = gran * (unsigned long long)part / (unsigned long long)nparts;
        const unsigned long long g1 = gran * (unsigned long long)(part + 1) / (unsigned long long)nparts;
        for (unsigned long long g = g0 + 64ull * tid; g < g1; g += 64ull * nthreads) {
            const unsigned n = (unsigned)((g1 - g < 64ull ? g1 - g : 64ull) << 8);
            asm volatile("cp.async.bulk.prefetch.L2.global [%0], %1;" ::"l"(static_cast<const unsigned char*>(t.p[a]) + (g << 8)), "r"(n) : "memory");
        }
    }
}
#endif

// Residual add / copy / RMSNorm fused in front of a product (mode = the step kind it replaces, 0 = none).
// x of the launch is then the un-normalised input; res_in and res_out must be different buffers.
struct XNorm {
    int mode = 0;
    const __nv_bfloat16* res_in = nullptr;
    __nv_bfloat16* res_out = nullptr;
    int res_stride = 0;
    const __nv_bfloat16* weight = nullptr;
    float eps = 0.f, weight_bias = 0.f;
};

struct QGemvLaunch {
    const Q4Tiled* w = nullptr;
    XNorm norm;
    int push = 0, in_tp = 0;   // tensor parallel: push partial rows to every rank / consume pushed partials
    TpParams tp{};
    const __nv_bfloat16* x = nullptr;  // [m][x_stride]
    int x_stride = 0;
    // result rows [0, seg_end[0]) go to y[0], [seg_end[0], seg_end[1]) to y[1], ... each [m][y_stride[i]]
    __nv_bfloat16* y[3] = {nullptr, nullptr, nullptr};
    int y_stride[3] = {0, 0, 0};
    int seg_end[3] = {0, 0, 0};
    int m = 1;
    int epilogue = QGEMV_EPI_STORE;
    int gated_act = GATED_ACT_SILU;   // activation of the gated epilogue
    float* partial = nullptr;     // split-K scratch, see qgemv_scratch_floats()
    unsigned* counters = nullptr; // one per CTA row group, zero between launches
    PrefetchTarget prefetch;      // batch-1 kernel only
};
size_t qgemv_scratch_floats(const Q4Tiled& w, int m);
int qgemv_counter_count(const Q4Tiled& w);
int launch_qgemv(const QGemvLaunch& a, cudaStream_t s);
// SWLM_TRACE=1: slot for the phase timestamps of one launch (nullptr when tracing is off or the slots are used up)
unsigned long long* qgemv_trace_slot(int ctas, int row_tiles, int kt4, int epi, int norm);
int qgemv_init();  // sets shared-memory attributes once per process
void qgemv_trace_report();  // SWLM_TRACE=1: phase timeline of the batch-1 launches, to stderr

// rmsnorm family: mode = SWLM_STEP_COPY_RMSNORM / RESADD_COPY_RMSNORM / RESADD_RMSNORM
int launch_rmsnorm(int mode, int m, int dim, const __nv_bfloat16* in, int in_stride, __nv_bfloat16* residual,
                   int res_stride, const __nv_bfloat16* weight, float eps, float weight_bias,
                   __nv_bfloat16* out, int out_stride, cudaStream_t s);
int launch_qk_norm(int m, int heads, int kv_heads, int head_dim, __nv_bfloat16* q, int q_stride,
                   __nv_bfloat16* k, int k_stride, const __nv_bfloat16* wq, const __nv_bfloat16* wk,
                   float eps, float weight_bias, cudaStream_t s);
int launch_embed(int m, int dim, const int32_t* tokens, int vocab, const __nv_bfloat16* table,
                 __nv_bfloat16* out, int out_stride, cudaStream_t s);
// the same gather from a Q4 group-64 table (packed source copy): out = bf16(q * scale + zero)
int launch_embed_q4(int m, int dim, const int32_t* tokens, const Q4Raw& table, __nv_bfloat16* out, int out_stride, cudaStream_t s);
int launch_swiglu(int m, int n, const __nv_bfloat16* gate, int g_stride, const __nv_bfloat16* up, int u_stride,
                  __nv_bfloat16* out, int o_stride, int act, cudaStream_t s);
int launch_conv_step(int m, int dim, int kernel, __nv_bfloat16* state, size_t state_seq_stride,
                     const __nv_bfloat16* in, int in_stride, const __nv_bfloat16* weight,
                     __nv_bfloat16* out, int out_stride, cudaStream_t s);
// conv_state_update over `tokens` consecutive tokens of one sequence (state of that sequence), bit-identical to
// `tokens` single steps.
// One step of the gated delta rule for m sequences (see SWLM_STEP_SSM_RECURRENCE): conv shift + SiLU over the q|k|v
// channels, per-head state update and read-out, RMS norm and z gate. conv_state [m][kernel][conv_dim] bf16 (row pitch
// conv_seq_stride elements per sequence), state [m][heads][key_dim][value_dim] fp32.
struct SsmLaunch {
    int m = 1, heads = 0, groups = 1, key_dim = 0, value_dim = 0, kernel = 0;
    // > 1 (with m == 1): the rows are consecutive prompt tokens of one sequence, walked in order inside the kernel
    // (ssm_recurrence_seq, Generator/MetalSourceGenerator+ConvAndState.swift:502-): the same code as the single step,
    // so a chunk leaves the state repeated decode steps would
    int tokens = 1;
    const __nv_bfloat16* qkv = nullptr; int qkv_stride = 0;
    const __nv_bfloat16* z = nullptr; int z_stride = 0;
    const __nv_bfloat16* beta = nullptr; int beta_stride = 0;
    const __nv_bfloat16* alpha = nullptr; int alpha_stride = 0;
    const __nv_bfloat16* conv_weight = nullptr;   // [conv_dim][kernel]
    const float* norm_weight = nullptr;           // [value_dim]
    const __nv_bfloat16* dt_bias = nullptr;       // [heads]
    const float* a_log = nullptr;                 // [heads]
    __nv_bfloat16* conv_state = nullptr; size_t conv_seq_stride = 0;
    float* state = nullptr; size_t state_seq_stride = 0;
    __nv_bfloat16* out = nullptr; int out_stride = 0;
};
int launch_ssm_recurrence(const SsmLaunch& a, cudaStream_t s);
int launch_conv_prefill(int tokens, int dim, int kernel, __nv_bfloat16* state, const __nv_bfloat16* in, int in_stride,
                        const __nv_bfloat16* weight, __nv_bfloat16* out, int out_stride, cudaStream_t s);
// argmax over [m][n] bf16, lowest index wins. Writes token_out[m], token_in_next[m] (may be null) and
// ring[(step_counter % ring_cap) * m + b] (ring may be null); when advance != 0 the last thread also
// increments the device-side position and step counter. Two launches.
int launch_argmax(int m, int n, const __nv_bfloat16* logits, int stride, int32_t* token_out,
                  int32_t* token_in_next, int32_t* ring, int32_t* step_counter, int ring_cap,
                  int32_t* position, int advance, float* scratch_val, int32_t* scratch_idx, const TpParams& tp,
                  int32_t* am_epoch, int shard_offset, cudaStream_t s);
size_t argmax_scratch_elems(int m);

// Sequences decoded together: 1..16 ride in the GEMV kernels (one weight pass for all of them), 17..kMaxSequences
// take the tensor-core product, one row per sequence.
constexpr int kMaxSequences = 64;
constexpr int kQGemvMaxRows = 16;

struct AttnLaunch {
    int m = 1;            // sequences
    int heads = 0, kv_heads = 0, head_dim = 0;
    int rope_dim = 0;
    const float* inv_freq = nullptr;  // [rope_dim/2] device
    float scale = 1.f;
    const __nv_bfloat16* q = nullptr; int q_stride = 0;   // [m][heads*hd]
    const __nv_bfloat16* k = nullptr; int k_stride = 0;   // new token's k [m][kv_heads*hd]
    const __nv_bfloat16* v = nullptr; int v_stride = 0;
    __nv_bfloat16* kcache = nullptr;  // [m][kv_heads][max_seq][hd]
    __nv_bfloat16* vcache = nullptr;
    int max_seq = 0;
    const int32_t* position = nullptr;  // device array [m]: index of each sequence's new token
    __nv_bfloat16* out = nullptr; int out_stride = 0;
    float* scratch = nullptr;   // attn_scratch_floats()
    unsigned* counters = nullptr;  // m * kv_heads arrival counters, zero between launches
    int splits = 1;             // KV splits per (sequence, kv head)
    // >= 0: prompt ingestion. The m rows are consecutive tokens of sequence 0 starting at this position; their
    // k/v rows are appended first, then token b attends cache rows 0..pos_base+b. `position` is not read.
    int pos_base = -1;
    int window = 0;       // sliding window: the current token and the window - 1 before it; 0 = everything
    int kv_scheme = 0;    // one of the quantized SWLM_KV_* schemes: the cache rows are blocks of 8- or 4-bit values (decode steps only)
    // rotated schemes: this layer's rotors [kv_heads][ceil(head_dim / 3)][4], the projection matrix [head_dim][qjl_dim]
    // and this layer's projected K residuals [m][kv_heads][max_seq][qjl_dim] (qjl_dim 0: no correction)
    const __half* rotors = nullptr;
    const __half* qjl_matrix = nullptr;
    __half* qjl_res = nullptr;
    int qjl_dim = 0;
    PrefetchTarget prefetch;
};
int attn_pick_splits(int m, int kv_heads, int max_ctx);
size_t attn_scratch_floats(int m, int heads, int head_dim, int splits);
// decode: q rows are unrotated; RoPE, KV append and the current token's unrounded term are handled inside.
int launch_attn_decode(const AttnLaunch& a, cudaStream_t s);
// generic flash-decode over an existing cache (q already rotated), ctx_len fixed on the host.
int launch_flash_decode_plain(int m, int heads, int kv_heads, int hd, int ctx_len, int ctx_stride, float scale,
                              const __nv_bfloat16* q, const __nv_bfloat16* k, const __nv_bfloat16* v,
                              __nv_bfloat16* out, float* scratch, unsigned* counters, int splits, cudaStream_t s);
int attn_init();
size_t flash_decode_static_capacity();
int launch_flash_decode_static(int device, int m, int heads, int kv_heads, int hd, int ctx_len, int ctx_stride, float scale,
                               const __nv_bfloat16* q, const __nv_bfloat16* k, const __nv_bfloat16* v, __nv_bfloat16* out,
                               cudaStream_t s);

// Tensor-core (tcgen05) form of the quantised product for m >= kQGemmTcMinRows, fed from the packed source copy.
constexpr int kQGemmTcMinRows = 17;   // 17..63 token rows ride in a 64-token tile whose other rows are zero
int qgemm_tc_init();
size_t qgemm_tc_scratch_bytes(int m, int k);   // fp16 copy of the activations + one float per token row
// kernels one call of launch_qgemm_tc issues: the fp16 copy of the rows (unless reused), the product, and the sum over
// K ranges when a short launch is split
int qgemm_tc_launch_count(const Q4Raw& w, int m, bool reuse_x);
// Where the rows of a product over concatenated weights go: rows [end[q-1], end[q]) to y[q] (up to three outputs,
// e.g. q | k | v); null = all rows to `y`.
struct TcSegments {
    int count = 1;
    int end[3] = {0, 0, 0};
    __nv_bfloat16* y[3] = {nullptr, nullptr, nullptr};
    int stride[3] = {0, 0, 0};
};
int launch_qgemm_tc(const Q4Raw& w, int m, const __nv_bfloat16* x, int x_stride, __nv_bfloat16* y, int y_stride,
                    void* scratch, int* status, cudaStream_t s, bool reuse_x = false, const TcSegments* segments = nullptr);

// Tensor-parallel sum of `rows` bf16 partial rows (prompt chunks): every rank copies its partials into every rank's
// exchange buffer and raises a flag carrying `epoch` (the host counts exchanges); then each rank waits (bounded) for
// all flags and adds the partials in rank order into `x` (in place). Two launches.
int launch_tp_rows_allreduce(const TpParams& tp, __nv_bfloat16* x, int x_stride, int rows, int hidden, int epoch,
                             unsigned* done_counter, cudaStream_t s);
int launch_fill_u32(uint32_t* p, size_t n, uint32_t v, cudaStream_t s);
int launch_advance(int m, int32_t* position, int32_t* step_counter, cudaStream_t s);

// =====================================================================================================================
// fp32-stream plans: dense bf16 products, sandwich norms, latent attention over a paged cache
// =====================================================================================================================

// Dense bf16 matrix [n][k], row pitch ld (k rounded up to 8, the padding is zero).
struct Matrix {
    int n = 0, k = 0, ld = 0;
    __nv_bfloat16* data = nullptr;
    bool view = false;   // rows of a concatenated matrix that owns the memory
};
constexpr int kMaxProductSegs = 8;

// Where a product's rows go: rows [end[q-1], end[q]) to y[q], an fp32 or bf16 buffer [m][stride[q]].
struct ProductOut {
    int count = 1;
    int end[kMaxProductSegs] = {};
    void* y[kMaxProductSegs] = {};
    int stride[kMaxProductSegs] = {};
    int f32[kMaxProductSegs] = {};
    const __nv_bfloat16* bias[kMaxProductSegs] = {};   // added to the rows of a segment; null: none
    int biased = 0;        // are there any?
    float softcap = 0.f;   // > 0: every value v becomes softcap * tanh(v / softcap)
    int gelu = 0;          // every value v becomes v * (1 + erf(v / sqrt(2))) / 2
};

// A norm step over the fp32 stream. mode = its step kind (0: none).
//   COPY_RMSNORM             h = in
//   RESADD_*                 h = res_in + in
//   POSTNORM_*               h = res_in + norm(in; w_post), and with a table + table[tokens[row]] * table_scale
// res_out (unless null) = h; the result is norm(h; w).
struct StreamNorm {
    int mode = 0;
    const float* in = nullptr; int in_stride = 0;
    const float* res_in = nullptr; float* res_out = nullptr; int res_stride = 0;
    const __nv_bfloat16* w_post = nullptr;
    const __nv_bfloat16* w = nullptr;
    float eps = 0.f, weight_bias = 0.f;
    const __nv_bfloat16* table = nullptr; const int32_t* tokens = nullptr; int vocab = 0; float table_scale = 0.f;
    // row r's entry of the table
    __device__ const __nv_bfloat16* table_row(int r, int dim) const { return table + (size_t)min(max(tokens[r], 0), vocab - 1) * dim; }
};
// rows_idx (may be null): output row r is computed from input row rows_idx[r].
int launch_stream_norm(const StreamNorm& a, int m, int dim, const int32_t* rows_idx, void* out, int out_stride, bool out_f32, cudaStream_t s);
// out[r] = table[tok[r]] * scale, fp32
int launch_stream_embed(int m, int dim, const int32_t* tokens, int vocab, const __nv_bfloat16* table, float scale, float* out, int out_stride, cudaStream_t s);
int launch_stream_gated(int m, int n, const void* gate, int g_stride, const void* up, int u_stride, void* out, int o_stride, bool f32, GatedAct act, cudaStream_t s);
// logits = cap * tanh(logits / cap), in place
int launch_stream_softcap(int m, int n, float* logits, int stride, float cap, cudaStream_t s);
// argmax over fp32 rows, any m (blocks of kMaxSequences rows); the advancing form of launch_argmax for m <= kMaxSequences
int launch_argmax_f32(int m, int n, const float* logits, int stride, int32_t* token_out, int32_t* token_in_next, int32_t* ring,
                      int32_t* step_counter, int ring_cap, int32_t* position, int advance, float* scratch_val, int32_t* scratch_idx, cudaStream_t s);

struct ProductLaunch {
    const Matrix* w = nullptr;
    const Matrix* w2 = nullptr;     // gated form: out = act(w x) * (w2 x), rows of both side by side
    GatedAct act;
    int m = 0;
    const void* x = nullptr; int x_stride = 0; bool x_f32 = false;   // x_f32: activations fp32, true fp32 products
    const void* x2 = nullptr; int x2_stride = 0, split = 0;   // weight rows from `split` on meet these activations (only when product_takes_two)
    StreamNorm norm;                // x = this norm's result (only when product_takes_norm)
    ProductOut out;
    float* part = nullptr; size_t part_floats = 0;   // split-K sums
    int* status = nullptr;          // device word set when a bounded wait expired
    // Grouped form (bf16, tensor cores): w holds the rows of `experts` matrices one after the other, activation rows are sorted
    // by expert, and tiles[i] = (expert, first row, rows, 0) names the rows of tile i (at most group_bn; 0 rows: nothing to do).
    int experts = 0;
    const int4* tiles = nullptr; int max_tiles = 0, group_bn = 0;
};
int bgemm_init();
int launch_product(const ProductLaunch& a, cudaStream_t s);
// rows per tile of a grouped product over `rows` activation rows, and the most tiles they can make
int grouped_bn(int rows, int experts);
int grouped_max_tiles(int rows, int experts);
bool product_takes_norm(int m, int k);
bool product_takes_gate(int m, int k, bool x_f32);
bool product_takes_two(int m, int k, int split, bool x_f32);
int product_launch_count(const ProductLaunch& a);
size_t product_part_floats(int n, int k, int m, bool gated);

// Geometry of one cached latent row: rank latent entries padded to rp, then rot rotated entries padded to rotp; `pitch`
// entries from row to row (in bf16 pools an odd multiple of 16 bytes, so that eight consecutive rows of a page copied
// to shared memory as they are lie in different bank groups). Padding entries are zero.
struct LatentRow { int rank = 0, rot = 0, rp = 0, rotp = 0, pitch = 0; };
LatentRow latent_row(int rank, int rot, bool f32);
// Consecutive rows of one sequence inside a batch: rows row0 .. row0 + count - 1 at positions pos0 ..; ctx0 = first of the
// pos0 + count gathered rows of this span.
// With a sliding window the rows in front of `lo` (a multiple of the page size) are not gathered.
struct LatentSpan { int row0, count, pos0, seq, ctx0, lo; };

struct LatentLaunch {
    LatentRow row;
    int heads = 0, dim = 0, vdim = 0, rot_dims = 0, rot_neighbours = 0;
    float scale = 1.f, eps = 0.f, weight_bias = 0.f, magnitude = 1.f;
    int window = 0;                                        // > 0: a row sees its own and the window - 1 positions before it
    const __nv_bfloat16* sink = nullptr;                   // [heads]: exp(sink) joins the denominator; null: none
    const float* inv_freq = nullptr;
    bool f32 = false;
    void* q = nullptr; int q_stride = 0;                   // [rows][heads * (dim + rot)]; rotated in place for span rows
    const float* kv = nullptr; int kv_stride = 0;          // [rows][rank + rot]
    const float* gate = nullptr; int gate_stride = 0;      // [rows][heads] or null
    const __nv_bfloat16* norm_w = nullptr;
    const Matrix* uk = nullptr; const Matrix* uv = nullptr;
    const Matrix* ukv = nullptr;                           // uk's rows, then uv's
    void* pool = nullptr;
    const int32_t* page_table = nullptr; int pages_per_seq = 0;
    const int32_t* row_seq = nullptr; const int32_t* row_pos = nullptr;
    void* out = nullptr; int out_stride = 0;
    // rows that are attended one by one in the latent space (row numbers; null: rows 0 .. n_short - 1)
    int n_short = 0; const int32_t* short_rows = nullptr; int splits = 1;
    float* qcat = nullptr; float* partial = nullptr;
    // rows attended in spans over expanded keys and values: row numbers, the spans, (span, query tile) pairs
    int n_long = 0; const int32_t* long_rows = nullptr;
    int n_spans = 0; const LatentSpan* spans = nullptr; int n_tiles = 0; const int2* tiles = nullptr; int total_ctx = 0;
    unsigned char* expand = nullptr;
    float* part = nullptr; size_t part_floats = 0;
    int* status = nullptr;
    bool only_attention = false;   // timing hook: the attention kernel alone
};
int latent_init();
int latent_pick_splits(int rows, int heads, int max_pages, int window);
size_t latent_qcat_floats(const LatentRow& r, int heads);              // per row
size_t latent_partial_floats(const LatentRow& r, int heads);           // per row and split
size_t latent_expand_bytes(const LatentRow& r, int heads, int dim, int vdim, int total_ctx);
// can rows of this layer be attended in spans over expanded keys and values?
bool latent_expands(const LatentRow& r, int dim, int vdim, bool f32);
constexpr int kLatentQueryTile = 128;
// launches (for the counters): short part 3, span part 4 or 5
int launch_latent(const LatentLaunch& a, cudaStream_t s, int* launches);

// ---- the residual stream between sublayers (stream_join.cu) ------------------------------------------------------------
// Parts that are not set are left out:
//   x = table[token] * table_scale, or res_in
//   keep_ring: x of a portion's last rows goes to the state of the convolution that read it
//   x += norm(in * sigmoid(gate); w)
//   results[store] = x;  x = sum over j < avg of avg_w[j] * results[j] (x itself is the last of them)
//   res_out = x, copy_out = x, conv_out = x + conv(x)
struct JoinLaunch {
    int rows = 0, width = 0; bool f32 = false;             // f32: copy_out and conv_out are fp32
    bool singles = false;                                  // every row is the only one of its sequence
    const int32_t *row_seq = nullptr, *row_pos = nullptr, *tokens = nullptr;
    const __nv_bfloat16* table = nullptr; int vocab = 0; float table_scale = 1.f;
    const float* res_in = nullptr; float* res_out = nullptr; int res_stride = 0;
    const float* in = nullptr; int in_stride = 0;
    const float* gate = nullptr; int gate_stride = 0;
    const __nv_bfloat16* w = nullptr; float eps = 0.f, weight_bias = 0.f;
    float* keep_ring = nullptr; int keep_taps = 0;         // [sequence][taps - 1][width], slot = position % (taps - 1)
    float* results = nullptr; size_t result_step = 0; int store = -1;   // [result][row][res_stride]
    const __nv_bfloat16* avg_w = nullptr; int avg = 0;
    const __nv_bfloat16* conv_w = nullptr; const float* conv_ring = nullptr; int taps = 0; void* conv_out = nullptr; int conv_stride = 0;   // conv_w [width][taps]
    void* copy_out = nullptr; int copy_stride = 0;
};
bool join_supported(int width, int taps);
int launch_join(const JoinLaunch& a, cudaStream_t s, int* launches);
// A token's own input to a layer, for single tokens: y = proj (gelu_tanh(gate x) * table[token][col ..]) between two joins that do
// nothing else with what lies between them: `first` ends with x, `last` starts with it and adds norm(y).
struct TokenInput {
    int n = 0;
    const __nv_bfloat16 *gate = nullptr, *proj = nullptr; int gate_ld = 0, proj_ld = 0;   // [n][width], [width][n]
    const __nv_bfloat16* table = nullptr; int cols = 0, col = 0;
    int* status = nullptr;
    int gate_here = 0, proj_here = 0;                      // (decided at the launch) which weights are held in shared memory
};
bool token_input_fits(const TokenInput& t, int rows, int width);
int launch_token_input(const JoinLaunch& first, const TokenInput& t, const JoinLaunch& last, cudaStream_t s);
// out = gelu_tanh(in) * table[token][col ..]
int launch_token_gate(int m, int n, const void* in, int in_stride, const int32_t* tokens, int vocab, const __nv_bfloat16* table, int cols, int col, void* out,
                      int out_stride, bool f32, cudaStream_t s);

// ---- rotary positions --------------------------------------------------------------------------------------------------
// Entry i of a vector whose first `dims` entries turn: the pair it belongs to, its partner, and whether it is the pair's first.
struct RotaryEntry { int pair, partner; bool first; };
#ifdef __CUDACC__
__device__ __forceinline__ RotaryEntry rotary_entry(int i, int dims, int neighbours) {
    if (neighbours) return RotaryEntry{i >> 1, i ^ 1, (i & 1) == 0};
    const int half = dims >> 1;
    return i < half ? RotaryEntry{i, i + half, true} : RotaryEntry{i - half, i - half, false};
}
// first entry of pair i, and the distance to the second
__device__ __forceinline__ int rotary_first(int i, int neighbours) { return neighbours ? 2 * i : i; }
__device__ __forceinline__ int rotary_step(int dims, int neighbours) { return neighbours ? 1 : dims >> 1; }
#endif

// ---- gated delta rule (delta_rule.cu) ----------------------------------------------------------------------------------
// Consecutive rows of one sequence: rows row0 .. row0 + count - 1 of the batch at positions pos0 ..; walked in blocks of
// kDeltaBlock tokens, blk0 = number of blocks of the runs before it.
struct RowRun { int row0, count, pos0, seq, blk0; };
constexpr int kDeltaBlock = 4;
struct DeltaShape { int heads = 0, groups = 0, dim = 0, vdim = 0, taps = 0; __host__ __device__ int channels() const { return 2 * groups * dim + heads * vdim; } };
struct DeltaLaunch {
    DeltaShape shape;
    int decay_dim = 1;                                     // decay inputs per head: 1 or dim
    int gate_act = 0;                                      // SWLM_GATE_*
    float eps = 0.f, unit_eps = 0.f, q_scale = 1.f;
    bool f32 = false;
    const void* qkv = nullptr; int qkv_stride = 0;
    const float* beta = nullptr; int beta_stride = 0;
    const float* decay = nullptr; int decay_stride = 0;
    const void* gate = nullptr; int gate_stride = 0;
    const __nv_bfloat16 *conv_q = nullptr, *conv_k = nullptr, *conv_v = nullptr, *norm_w = nullptr, *a_log = nullptr, *dt_bias = nullptr;
    void* ring = nullptr;                                  // [sequence][taps][channels]: inputs of the convolutions, slot = position % taps
    float* state = nullptr;                                // [sequence][heads][dim][vdim]
    const int32_t* row_seq = nullptr; const int32_t* row_pos = nullptr;
    void* out = nullptr; int out_stride = 0;
    int n_single = 0; const int32_t* single_rows = nullptr;   // rows that are one token of their sequence (null: rows 0 ..)
    int n_runs = 0; const RowRun* runs = nullptr;             // longer portions
    int n_blocks = 0; const int32_t* block_run = nullptr;     // the run of every block
    float* scratch = nullptr;
    int* status = nullptr;
};
int delta_init();
bool delta_supported(const DeltaShape& s);
bool delta_step_fits(const DeltaShape& s);                    // single tokens in one fused launch
size_t delta_scratch_floats(const DeltaShape& s, int blocks, int rows);
int launch_delta(const DeltaLaunch& a, cudaStream_t s, int* launches);

// ---- retention (retention.cu) -------------------------------------------------------------------------------------------
struct RetentionLaunch {
    int heads = 0, dim = 0, vdim = 0;
    float eps = 0.f, scale = 1.f, out_scale = 1.f;
    bool f32 = false;
    const float* decay = nullptr;                          // [heads]
    const void* qkv = nullptr; int qkv_stride = 0;
    const void* gate = nullptr; int gate_stride = 0;
    float* state = nullptr;                                // [sequence][heads][dim][vdim]
    const int32_t* row_seq = nullptr; const int32_t* row_pos = nullptr;
    void* out = nullptr; int out_stride = 0;
    int n_single = 0; const int32_t* single_rows = nullptr;   // as DeltaLaunch
    int n_runs = 0; const RowRun* runs = nullptr;
    int n_blocks = 0; const int32_t* block_run = nullptr;
    float* scratch = nullptr;                              // [row][heads][vdim]
};
int retention_init();
bool retention_supported(int heads, int dim, int vdim);
bool retention_step_fits(int dim, int vdim);
int launch_retention(const RetentionLaunch& a, cudaStream_t s, int* launches);

// ---- grouped-query attention over pages (grouped_attention.cu) -----------------------------------------------------------
// A page holds, head after head, 64 key rows of `pk` entries and 64 value rows of `pv` (in bf16 pools odd multiples of 16 bytes,
// see LatentRow); dp and vp are the sizes padded to 16, padding entries are zero. block: entries of a (page, head) pair.
// shared: the values are the keys before their norm. One row per token is kept, and behind the 64 rows 64 fp32 numbers that turn
// a row into its key.
struct GroupedRow { int groups = 0, dim = 0, vdim = 0, dp = 0, vp = 0, pk = 0, pv = 0, block = 0, shared = 0; };
GroupedRow grouped_row(int groups, int dim, int vdim, bool f32, bool shared);
struct GroupedLaunch {
    GroupedRow row;
    int heads = 0, rot_dims = 0, rot_neighbours = 0, window = 0, chunk = 0, sink_one = 0;
    float scale = 1.f, eps = 0.f, weight_bias = 0.f, magnitude = 1.f, out_scale = 1.f;
    int head_norm = 0, temp_every = 0; float temp_coef = 0.f;   // norm of q and k without weights; query temperature
    const float* inv_freq = nullptr;
    bool f32 = false;
    const __nv_bfloat16 *q_norm = nullptr, *k_norm = nullptr;
    void* qkv = nullptr; int qkv_stride = 0;               // q | k | v per row; q is normed and rotated in place
    const float* gate = nullptr; int gate_stride = 0;
    const void* entry_gate = nullptr; int entry_gate_stride = 0;   // [rows][heads * vdim], in the activation type
    void* pool = nullptr;
    const int32_t* page_table = nullptr; int pages_per_seq = 0;
    const int32_t* row_seq = nullptr; const int32_t* row_pos = nullptr;
    void* out = nullptr; int out_stride = 0;
    int n_rows = 0;                                        // all rows of the batch
    int n_short = 0; const int32_t* short_rows = nullptr; int max_pages = 1;   // attended one by one; longest context of theirs
    const LatentSpan* spans = nullptr; int n_tiles = 0; const int2* tiles = nullptr;   // and in spans: tiles of kLatentQueryTile rows
    int* status = nullptr;
    bool singles = false;          // every row is the only one of its sequence
    bool only_attention = false;   // timing hook
};
int grouped_init();
bool grouped_supported(const GroupedRow& r);
// do batches of single tokens take one launch (norm and append in the attention kernel)?
bool grouped_appends(const GroupedRow& r, bool f32, int rot_dims);
// can rows of this layer be attended in spans?
bool grouped_spans(const GroupedRow& r, bool f32);
int launch_grouped(const GroupedLaunch& a, cudaStream_t s, int* launches);

// ---- routed feed-forward (routed_mlp.cu) -------------------------------------------------------------------------------
// shared_ff > 0: inner size of the feed-forward that every row takes. The last `identity` of the experts + identity that are scored
// hand their input through.
struct RoutedShape { int experts = 0, top = 0, groups = 1, keep = 1, width = 0, ff = 0, shared_ff = 0, identity = 0; __host__ __device__ int scored() const { return experts + identity; } };
struct RoutedLaunch {
    RoutedShape shape;
    float scale = 1.f;
    GatedAct act;
    int softmax = 0, group_best = 2, raw_weights = 0;      // scores, what a group counts as, whether weights are renormalised
    int m = 0; bool f32 = false;
    const void* x = nullptr; int x_stride = 0;
    const float* z = nullptr; int z_stride = 0;            // router logits; with a shared feed-forward its gate behind them
    // the experts' rows one after the other; gate == null: an expert is down(gelu(up x))
    const Matrix *gate = nullptr, *up = nullptr, *down = nullptr;
    const Matrix *shared_up = nullptr, *shared_down = nullptr;
    const __nv_bfloat16* correction = nullptr;             // [scored]: joins the scores for the choice only
    float* out = nullptr; int out_stride = 0;
    unsigned char* scratch = nullptr;
    unsigned* counts = nullptr;                            // [kMaxExperts], zero between launches
    float* part = nullptr; size_t part_floats = 0;         // split-K sums of the shared products
    int* status = nullptr;
};
constexpr int kMaxExperts = 1024, kMaxTop = 64;
int routed_init();
bool routed_supported(const RoutedShape& s);
size_t routed_scratch_bytes(const RoutedShape& s, int m, bool f32);
int launch_routed(const RoutedLaunch& a, cudaStream_t s, int* launches);

}  // namespace swlm
