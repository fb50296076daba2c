/*
 * swlm_plan.h — the execution record shared by the host and the CUDA backend.
 *
 * A plan is a flat array of `swlm_step` records, one per reference dispatch.
 * It replaces the reference's `MetalDispatchStep` / `MetalDispatchPlan`
 * (Sources/MetalCompiler/Execution/MetalDecodePlan.swift:6-193): where the
 * reference stores {pipeline, grid, buffer bindings, constants}, a step here
 * stores {operation kind, logical buffer slots, tensor names, dimensions}.
 * The backend is free to fuse adjacent steps into one launch as long as every
 * value that the reference stores to a decode buffer is rounded to bf16 at the
 * same point.
 *
 * Logical buffers follow the reference's decode buffer set
 * (Sources/MetalCompiler/Buffer/MetalBufferAllocator.swift:4-132): `hidden`,
 * `residual`, five scratch slots of `slot_dim` elements, `logits`, all bf16,
 * one row per sequence of the batch.
 */
#ifndef SWLM_PLAN_H
#define SWLM_PLAN_H

#include <stdint.h>

#ifdef __cplusplus
extern "C" {
#endif

#define SWLM_NAME_MAX 96

/* Logical buffer ids used by swlm_step.in_buf / in2_buf / out_buf. */
enum {
    SWLM_BUF_NONE = -1,
    SWLM_BUF_HIDDEN = 0,
    SWLM_BUF_RESIDUAL = 1,
    SWLM_BUF_SCRATCH0 = 2, /* block output: attention / conv / swiglu result, norm output */
    SWLM_BUF_SCRATCH1 = 3, /* q, gate, packed B|C|x */
    SWLM_BUF_SCRATCH2 = 4, /* k, up */
    SWLM_BUF_SCRATCH3 = 5, /* v */
    SWLM_BUF_SCRATCH4 = 6,
    SWLM_BUF_LOGITS = 7,
    SWLM_BUF_COUNT = 8
};

/* Step kinds. The comment names the reference kernel each one stands for. */
enum {
    /* embedding_lookup_bf16 — Generator/MetalSourceGenerator+Embedding.swift:3-48.
       hidden[b] = table[token_in[b]]; weight = table [vocab, n] bf16. */
    SWLM_STEP_EMBED = 1,
    /* fused_copy_rms_norm — Primitives/Reduction.swift:74-115 + CopyFragment.
       residual = in; out = bf16(in * rsqrt(mean(in^2)+eps) * (w + weight_bias)). */
    SWLM_STEP_COPY_RMSNORM = 2,
    /* fused_residual_add_copy_rms_norm — Compiler/MetalEntryCollector.swift:143-218.
       h = float(in) + float(residual); residual = bf16(h);
       out = bf16(h * rsqrt(mean(h^2)+eps) * (w + weight_bias)). */
    SWLM_STEP_RESADD_COPY_RMSNORM = 3,
    /* fused_residual_add_rms_norm (final norm): as above without the residual store. */
    SWLM_STEP_RESADD_RMSNORM = 4,
    /* gemv_q4_g64 — Generator/MetalSourceGenerator+Quantized.swift:496-575.
       out[n] = bf16(sum_k (scale*q + zero) * in[k]), fp32 accumulation. */
    SWLM_STEP_QGEMV = 5,
    /* batched_qk_rms_norm_2 — Generator/MetalSourceGenerator+Batched.swift:681-760.
       per-head RMSNorm of q (in_buf, `heads`) with `weight` and of k (in2_buf,
       `kv_heads`) with `weight2`, in place. */
    SWLM_STEP_QK_NORM = 6,
    /* rope_flash_attn_decode — Generator/MetalSourceGenerator+Attention.swift:551-930.
       q = in_buf, k = in2_buf, v = in3_buf, result = out_buf. Inline rotate-half
       RoPE on q and the new k, append k,v at `position`, attend over [0, position]. */
    SWLM_STEP_ATTN_DECODE = 7,
    /* swiglu — Primitives/ElementwiseFragment.swift:49-54.
       out = bf16(g/(1+exp(-g)) * up), g = in_buf, up = in2_buf. */
    SWLM_STEP_SWIGLU = 8,
    /* conv_state_update_bf16 — Generator/MetalSourceGenerator+ConvAndState.swift:27-70.
       in_buf holds B|C|x (3*n); state [conv_kernel][n] bf16; weight [n][conv_kernel] bf16. */
    SWLM_STEP_CONV_STATE_UPDATE = 9,
    /* argmax — Generator/MetalSourceGenerator+Sampling.swift:62-107; lowest index
       wins among equal maxima. token_out[b] = argmax(in_buf[b][0..n)). */
    SWLM_STEP_ARGMAX = 10,
    /* geglu — the gated activation with GELU (tanh approximation) instead of SiLU
       (Generator/MetalSourceGenerator+NormAndElementwise.swift:176-208, GatedActivation.geluTanh):
       out = bf16(0.5 g (1 + tanh(0.7978845608 (g + 0.044715 g^3))) * up), g = in_buf, up = in2_buf. */
    SWLM_STEP_GEGLU = 11,
    /* ssm_recurrence (gated delta rule of the DeltaNet / Qwen3.5 linear-attention layers) —
       Generator/MetalSourceGenerator+ConvAndState.swift:282-500, Primitives/SSMRecurrenceFragment.swift.
       in_buf = projected q|k|v (2*groups*key_dim + heads*value_dim values), in2_buf = z (heads*value_dim),
       in3_buf = beta (heads), in4_buf = alpha (heads), out_buf = heads*value_dim values.
       Per channel: causal conv over conv_kernel taps (state [conv_kernel][conv_dim], weight dtype) + SiLU; per head:
       decay = exp(-exp(A_log) * softplus(alpha + dt_bias)), beta = sigmoid(beta), q and k L2-normalised (q also scaled
       by key_dim^-1/2), S = decay * S + k (x) beta (v - S^T k), out = S^T q (state S [key_dim][value_dim] fp32); then
       RMS norm over value_dim with `weight2` and the gate z * sigmoid(z).
       weight = conv taps [conv_dim][conv_kernel] bf16, weight2 = norm weight [value_dim] fp32, weight3 = dt_bias
       [heads] bf16, weight4 = A_log [heads] fp32 (the two fp32 tensors: swlm_weights_add_dense_f32). */
    SWLM_STEP_SSM_RECURRENCE = 12,
    /* ---- steps of fp32-stream plans (swlm_buffers_desc.stream_dtype != 0); no counterpart in the reference ----
       Such plans also use EMBED (times `scale` when it is not 0), the three norm steps, SWIGLU / GEGLU and ARGMAX. */
    /* out[n] = sum_k W[n][k] in[k], W a dense bf16 matrix (swlm_weights_add_matrix_bf16), fp32 accumulation.
       weight3 not empty: a bias [n] is added.
       weight2 not empty: a second matrix [n][k2] times the k2 columns that start at the next multiple of 8 behind the first
       k ones is added (the two are kept side by side and run as one product). */
    SWLM_STEP_PRODUCT = 13,
    /* Sandwich norm: t = in * rsqrt(mean(in^2)+eps) * (weight + weight_bias); residual += t;
       out = residual * rsqrt(mean(residual^2)+eps) * (weight2 + weight_bias).
       weight3 not empty: an embedding table; the row of the token times `scale` is added to the residual with t. */
    SWLM_STEP_POSTNORM_RESADD_COPY_RMSNORM = 14,
    /* the same in front of the output head: the sum is not stored */
    SWLM_STEP_POSTNORM_RESADD_RMSNORM = 15,
    /* Latent attention. in_buf = q (heads * (head_dim + key_dim): per head head_dim plain, then key_dim rotated entries),
       in2_buf = n latent entries followed by key_dim entries of the key part that all heads share, in3_buf = gate (heads,
       before the sigmoid; SWLM_BUF_NONE: no gate), out_buf = heads * value_dim.
       The latent c is RMS-normed (`weight`, eps, weight_bias); rotate-half rotary positions act on the first rope_dim of
       the key_dim entries of q and of the shared key part (rope_pairs 1: entries 2i and 2i + 1 form a pair instead). Cached per token: c and the rotated key part. Per head the
       plain key is weight2 [heads * head_dim][n] c, the value weight3 [heads * value_dim][n] c; score = (q . k over both
       parts) * scale, softmax over all positions up to the token's own; out = sigmoid(gate) * value sum.
       window_left > 0: only the last window_left positions, the token's own among them. weight4 not empty: a sink, one
       number per head whose exponential is added to the softmax's denominator as it is. */
    SWLM_STEP_LATENT_ATTN = 16,
    /* Gated activation with limits: g = min(in, limit), u = clamp(in2, -limit, limit),
       out = g * sigmoid(scale * g) * (u + 1). */
    SWLM_STEP_CLAMPED_GLU = 17,
    /* Gated delta rule with a state per sequence. in_buf = q | k | v before their convolutions (groups * key_dim, the same
       again, heads * value_dim), in2_buf = step sizes before the sigmoid (heads), in3_buf = decay inputs (heads * k, k = 1 or
       key_dim: one decay per head or per key channel), in4_buf = output gate before its activation (heads * value_dim),
       out_buf = heads * value_dim (may be in4_buf). Head h reads q and k of group h / (heads / groups).
       Every channel of q, k, v: causal convolution over conv_kernel tokens (weight, weight2, weight3: [channels][conv_kernel],
       the last column meets the current token; zeros before the start), then SiLU. q and k per group: x / sqrt(sum(x^2) +
       eps2), q also times scale. decay = exp(-exp(A_log) * softplus(in3 + dt_bias)), beta = sigmoid(in2);
       S = decay * S; u = beta * (v - S^T k); S = S + k u^T; o = S^T q with S [key_dim][value_dim] fp32, zero at position 0.
       out = o * rsqrt(mean(o^2) + eps) * weight4 * activation(in4); gate_act: one of SWLM_GATE_*.
       weight5 = A_log [heads], weight6 = dt_bias [heads * k]. in2, in3 and in4 are read from columns in2_off, in3_off, in4_off on. */
    SWLM_STEP_GATED_DELTA = 18,
    /* Routed feed-forward: in_buf = input (n values), in2_buf = router logits (experts), out_buf = n values in hidden.
       s = sigmoid(logits); the experts form `groups` equal groups of neighbours, a group counts as the sum of its two largest
       s, and only experts of the groups_keep best groups can be chosen; the `top` largest s among them are. Expert i is the
       clamped gated feed-forward (CLAMPED_GLU with glu_alpha, limit) of the matrices <weight>i<weight2>, <weight>i<weight3>
       [k][n] and <weight>i<weight4> [n][k]; its output is weighted with s / (sum of the chosen s + 1e-20) * scale.
       score_act SWLM_SCORE_SOFTMAX: s = softmax(logits) over all experts. group_best 1: a group counts as its largest s.
       raw_weights 1: an expert's output is weighted with s * scale. weight2 empty: expert i is <weight4>(gelu(<weight3> in))
       with the exact (erf) GELU. weight5 not empty (only then): a feed-forward weight6 [n][k2] (gelu(weight5 [k2][n] in)) that every
       token takes, its output times sigmoid(in2[experts]) is added.
       expert_act SWLM_EXPERT_SILU: gate and up are combined as silu(gate) * up. identity > 0: in2_buf holds experts + identity
       logits; the last ones stand for experts without tensors whose output is the input (no groups then). weight7 not empty: a
       vector [experts + identity] that is added to the scores for the choice only. */
    SWLM_STEP_ROUTED_MLP = 19,
    /* logits = scale * tanh(logits / scale), in place */
    SWLM_STEP_SOFTCAP = 20,
    /* Grouped-query attention over a paged cache. in_buf from column in_off on = q | k | v (heads * head_dim, kv_heads *
       head_dim, kv_heads * value_dim), in3_buf = gate (heads, before the sigmoid; SWLM_BUF_NONE: none), out_buf from column
       out_off on = heads * value_dim. Query head h reads key / value head h / (heads / kv_heads).
       q and k per head: RMS norm with weight / weight2 [head_dim] (eps, weight_bias; empty: none), then rotary positions on
       the first rope_dim entries (rope_pairs as in LATENT_ATTN). Cached per token: k after that, and v. score = (q . k) *
       scale, softmax over the positions up to the token's own: window_left > 0: the last window_left of them; chunk > 0:
       those of the token's own chunk of `chunk` positions, counted from position 0. sink_one 1: one is added to the softmax's
       denominator. out = sigmoid(gate) * value sum * out_scale.
       head_norm 1: q and k per head are divided by their root mean square (eps) without a weight. value_is_key 1: in_buf holds
       q | k only and the values are the keys before their norm (value_dim = head_dim, no rotation); one row per token is cached.
       temp_every > 0: q at position p is multiplied by 1 + temp_coef * ln((p + 1) div temp_every + 1). in4_buf from column
       in4_off on (SWLM_BUF_NONE: none) = a gate per entry of the result, before its sigmoid, in the activation type. */
    SWLM_STEP_GROUPED_ATTN = 21,
    /* Retention with a state per sequence. in_buf from column in_off on = q | k | v (heads * key_dim, the same again, heads *
       value_dim), in4_buf from column in4_off on = output gate before its SiLU (heads * value_dim), out_buf from column
       out_off on = heads * value_dim (may not be in_buf or in4_buf).
       S = decay_h * S + (scale * k) v^T; o = S^T q with S [key_dim][value_dim] fp32, zero at position 0;
       out = o * rsqrt(mean(o^2) + eps) * silu(gate) * out_scale. weight = decay [heads], an fp32 tensor.
       `layer` indexes the same states as GATED_DELTA. */
    SWLM_STEP_RETENTION = 22,
    /* ---- steps that act on the residual stream itself (sublayers that read the stream without a norm in front) ----
       EMBED with out_buf = RESIDUAL starts such a stream; COPY_RMSNORM with in_buf = RESIDUAL norms it as it is.
       Neighbours among the following steps run as one launch. */
    /* t = in_buf (fp32), times sigmoid(in3_buf) (fp32; SWLM_BUF_NONE: no gate); residual += t * rsqrt(mean(t^2)+eps) * (weight + weight_bias) */
    SWLM_STEP_GATED_POSTNORM_ADD = 23,
    /* Depth-wise average: the stream is kept as result k - 1 of the pass (the embedding output is result 0), and becomes
       sum over j < k of weight[j] * result j. */
    SWLM_STEP_DEPTH_AVG = 24,
    /* out_buf = h + conv(h), h the residual stream and conv a causal convolution over conv_kernel tokens per channel (weight
       [n][conv_kernel], the last column meets the current token; zeros before the start). `layer` indexes the stream_convs
       states that keep the last inputs of a sequence. */
    SWLM_STEP_STREAM_CONV = 25,
    /* out_buf = the residual stream, in the activation type */
    SWLM_STEP_STREAM_COPY = 26,
    /* out = gelu_tanh(in) * weight[token][in2_off ..], weight a table with a row per token of the vocabulary */
    SWLM_STEP_TOKEN_GATE = 27
};
enum { SWLM_EXPERT_CLAMPED = 0, SWLM_EXPERT_SILU = 1 };
enum { SWLM_GATE_SILU = 0, SWLM_GATE_SIGMOID = 1 };
enum { SWLM_SCORE_SIGMOID = 0, SWLM_SCORE_SOFTMAX = 1 };
enum { SWLM_ROPE_HALVES = 0, SWLM_ROPE_NEIGHBOURS = 1 };

typedef struct swlm_step {
    int32_t kind;
    int32_t layer;       /* index of the KV-cache / conv-state slab this step owns, else -1 */
    int32_t in_buf;
    int32_t in2_buf;
    int32_t in3_buf;
    int32_t out_buf;
    int32_t n;           /* output width (rows of the weight) / vector dimension */
    int32_t k;           /* input width (columns of the weight) */
    int32_t heads;
    int32_t kv_heads;
    int32_t head_dim;
    int32_t rope_dim;    /* 0 = no RoPE */
    int32_t conv_kernel;
    float   eps;
    float   weight_bias;
    float   scale;       /* attention scale */
    float   rope_base;
    char    weight[SWLM_NAME_MAX];
    char    weight2[SWLM_NAME_MAX];
    /* attention: sliding window. 0 = attend everything; W > 0 = the current token and the W - 1 before it
       (windowLeft, Generator/MetalSourceGenerator+Attention.swift:851-853; decode and prompt chunks alike). */
    int32_t window_left;
    /* SWLM_STEP_SSM_RECURRENCE only */
    int32_t in4_buf;
    int32_t groups;      /* key groups; heads / groups value heads share one q and k */
    int32_t key_dim;
    int32_t value_dim;
    char    weight3[SWLM_NAME_MAX];
    char    weight4[SWLM_NAME_MAX];
    /* SWLM_STEP_LATENT_ATTN: rotary frequencies interpolated by parts (YaRN). rope_factor 0 = plain frequencies; else pairs
       that turn fewer than rope_slow times over rope_original positions are divided by rope_factor, pairs that turn more
       than rope_fast times stay, a linear ramp in between, and cos and sin are multiplied by 0.1 ln(rope_factor) + 1. */
    float   rope_factor;
    float   rope_original;
    float   rope_fast;
    float   rope_slow;
    /* fp32-stream plans */
    int32_t in_off;      /* first column of the input in in_buf (a multiple of 8) */
    int32_t out_off;     /* and of the result in out_buf, so that several results share a buffer */
    int32_t experts;
    int32_t top;
    int32_t groups_keep;
    int32_t gate_act;
    float   limit;
    float   glu_alpha;
    float   eps2;
    char    weight5[SWLM_NAME_MAX];
    char    weight6[SWLM_NAME_MAX];
    int32_t rope_pairs;    /* SWLM_ROPE_* */
    float   rope_divisor;  /* every rotary frequency is divided by it; 0 = 1 */
    int32_t chunk;
    int32_t sink_one;
    int32_t k2;
    int32_t in4_off;
    float   out_scale;     /* GROUPED_ATTN, RETENTION */
    int32_t score_act;     /* SWLM_SCORE_* */
    int32_t group_best;    /* 0 = 2 */
    int32_t raw_weights;
    int32_t in2_off;
    int32_t in3_off;
    int32_t value_is_key;  /* GROUPED_ATTN */
    int32_t head_norm;
    float   temp_coef;
    int32_t temp_every;
    int32_t identity;      /* ROUTED_MLP */
    int32_t expert_act;    /* SWLM_EXPERT_* */
    char    weight7[SWLM_NAME_MAX];
} swlm_step;

/* Sizes of the runtime buffer set; mirrors the inputs of
   MetalBufferAllocator.makeDecodeBufferAllocation (Buffer/MetalBufferAllocator.swift:4-132)
   and KVCacheSpecification (Buffer/MetalGraphAllocator.swift:15-223). */
typedef struct swlm_buffers_desc {
    int32_t hidden;       /* hidden size */
    int32_t slot_dim;     /* elements per scratch slot */
    int32_t vocab;
    int32_t max_seq;      /* KV slots per sequence (maximumSequenceLength) */
    int32_t max_batch;    /* sequences decoded together; the reference is 1 */
    int32_t kv_layers;    /* number of attention layers (KV slabs) */
    int32_t kv_heads;
    int32_t head_dim;
    int32_t conv_layers;  /* number of short-conv layers (state slabs) */
    int32_t conv_dim;
    int32_t conv_kernel;
    /* recurrent layers (SWLM_STEP_SSM_RECURRENCE): per layer and sequence a conv state [ssm_conv_kernel][conv_dim]
       (conv_dim = 2*ssm_groups*ssm_key_dim + ssm_heads*ssm_value_dim) and an fp32 state [ssm_heads][ssm_key_dim][ssm_value_dim].
       All zero when the plan has no such layer. */
    int32_t ssm_layers;
    int32_t ssm_heads;
    int32_t ssm_groups;
    int32_t ssm_key_dim;
    int32_t ssm_value_dim;
    int32_t ssm_conv_kernel;
    /* KV cache element scheme (KVCacheSpecification, Buffer/MetalGraphAllocator.swift): 0 or SWLM_KV_BF16 = dense bf16;
       the quantized schemes keep groups of 32 / 64 / 128 values along the head dimension as blocks fp16 scale | fp16 zero
       | payload (8-bit: one byte per value; 4-bit: two values per byte, the even one in the low nibble), value = scale *
       q + zero (kv_quant_bits / _group_size / _bytes_per_block, read_kv_element, write_kv_quantized_q8 / _q4:
       Generator/MetalSourceGenerator+Attention.swift:1894-1956, 2057-2155). K and V use the same scheme; a group may not
       be wider than head_dim. */
    int32_t kv_scheme;
    /* The two rotated schemes (is_rotor_scheme / rotor_base_scheme, :1791-1800) store rows in the block layout of their
       base scheme after every group of three consecutive values of a K or V row was turned by a unit rotor of Cl(3,0)
       (rotor_sandwich, :1807-1813; one rotor per attention layer, KV head and group, ceil(head_dim / 3) groups, the
       last one padded with zeros); q is turned the same way and the attention output turned back
       (rotor_sandwich_inverse, :1815-1821). kv_qjl_dim > 0 (at most 64; rotated schemes only) adds the correction of
       the K quantisation error: per cached row kv_qjl_dim fp16 values Phi . (k_rotated - dequantised row) with the fixed
       +-1/sqrt(kv_qjl_dim) matrix Phi [head_dim][kv_qjl_dim], and every score over a cached row gains
       (Phi . q_rotated) . (that row's values) (qjl_compute_residual, qjl_project_query, qjl_score_correction,
       :1983-2048). */
    int32_t kv_qjl_dim;
    /* fp32-stream plans: hidden, residual and logits are kept in fp32 (as are scratch slots 3 and 4), the other scratch
       slots and the cache in bf16 (SWLM_STREAM_F32) or everything in fp32 with true fp32 products (SWLM_STREAM_ALL_F32).
       0 = the bf16 buffers of the reference. Buffer widths follow from the steps (slot_dim is not used). */
    int32_t stream_dtype;
    int32_t latent_layers;   /* number of latent-attention layers (page pools) */
    /* tokens the page pools of the cached rows hold over all sequences, rounded up to pages of 64;
       0 = max_batch * max_seq. Sequences take pages as they grow and give them back when they are reset. */
    int32_t kv_pool_tokens;
    int32_t delta_layers;    /* number of SWLM_STEP_GATED_DELTA and SWLM_STEP_RETENTION layers: fp32 state (and convolution
                                inputs) per sequence */
    int32_t grouped_layers;  /* number of SWLM_STEP_GROUPED_ATTN layers (page pools of keys and values) */
    int32_t stream_convs;    /* number of SWLM_STEP_STREAM_CONV states */
    int32_t depth_results;   /* results SWLM_STEP_DEPTH_AVG keeps (the embedding output among them); 0: none */
} swlm_buffers_desc;

enum { SWLM_STREAM_BF16 = 0, SWLM_STREAM_F32 = 1, SWLM_STREAM_ALL_F32 = 2 };
#define SWLM_PAGE_TOKENS 64

enum {
    SWLM_KV_BF16 = 0x01,
    SWLM_KV_Q8G32 = 0x10, SWLM_KV_Q8G64 = 0x11, SWLM_KV_Q8G128 = 0x12,   /* 36 / 68 / 132 bytes per block */
    SWLM_KV_Q4G64 = 0x40, SWLM_KV_Q4G128 = 0x41, SWLM_KV_Q4G128Z = 0x42, /* 36 / 68 / 68 bytes per block (0x42, the
                                                                            reference's q4Group128ScaleF16Zero, reads and
                                                                            writes cache rows exactly as 0x41 does) */
    SWLM_KV_ROTOR_Q8G32 = 0x70, SWLM_KV_ROTOR_Q4G64 = 0x71               /* rotated rows in the layout of 0x10 / 0x40 */
};
static inline int swlm_kv_is_rotor(int scheme) { return scheme == 0x70 || scheme == 0x71; }
static inline int swlm_kv_base_scheme(int scheme) { return scheme == 0x70 ? 0x10 : scheme == 0x71 ? 0x40 : scheme; }
/* rotors per KV head: groups of three values along the head dimension (KVCacheSpecification.numRotorGroups) */
static inline int swlm_kv_rotor_groups(int head_dim) { return (head_dim + 2) / 3; }
/* bits per value (0: dense), values per group, bytes per block and bytes per row of head_dim values */
static inline int swlm_kv_bits(int scheme) {
    scheme = swlm_kv_base_scheme(scheme);
    return scheme >= 0x10 && scheme <= 0x12 ? 8 : (scheme >= 0x40 && scheme <= 0x42) ? 4 : 0;
}
static inline int swlm_kv_group(int scheme) {
    scheme = swlm_kv_base_scheme(scheme);
    return scheme == 0x10 ? 32 : (scheme == 0x11 || scheme == 0x40) ? 64 : (scheme == 0x12 || scheme == 0x41 || scheme == 0x42) ? 128 : 0;
}
static inline int swlm_kv_block_bytes(int scheme) { return swlm_kv_bits(scheme) ? 4 + swlm_kv_group(scheme) * swlm_kv_bits(scheme) / 8 : 0; }
static inline int swlm_kv_row_bytes(int scheme, int head_dim) {
    return swlm_kv_bits(scheme) ? head_dim / swlm_kv_group(scheme) * swlm_kv_block_bytes(scheme) : head_dim * 2;
}

#ifdef __cplusplus
}
#endif
#endif /* SWLM_PLAN_H */
