// Grouped-query attention of fp32-stream plans over a paged cache: norm of q and k per head, rotary positions, a softmax over the
// positions a window or a chunk lets through with an optional constant in the denominator, and a gate per head.
//
// A page holds 64 tokens of every key / value head: per head 64 key rows, then 64 value rows, so that the keys and values of a
// (page, head) pair are one contiguous piece of memory. grouped_append_kernel norms and rotates q in place and k and v into the
// cache; then a batch's rows go one of two ways:
//   * one by one (decode steps, short portions): grouped_decode_kernel, a cluster of CTAs per (row, key / value head) that deal the
//     context out to their warps; every warp copies its keys and values by itself and keeps its own running softmax, the
//     results are merged through shared memory and then through distributed shared memory. Where every row is a token of its own
//     and nothing is rotated, the kernel norms and appends by itself: the cached rows in front of the token are requested before
//     the preceding kernel has finished, the token's own key does not go through the cache.
//   * in spans (prompt portions): grouped_prefill_kernel, a tiled attention of 128 queries by 64 keys.
// Both multiply on tensor cores with fp32 sums; softmax weights enter as bf16 hi + lo pairs. grouped_simple_kernel (fp32 FMAs)
// serves fp32 caches and head sizes beyond the others. The newest rows are read back from the cache like all others, so a row's
// result does not depend on how a sequence was cut into batches.
//
// Where the values are the keys before their norm, one row per token is kept and read as key and as value; the norm is a number
// per row that scales the row's score.
#include <cooperative_groups.h>

#include <algorithm>
#include <utility>

#include "swlm_internal.h"
#include "tc_device.cuh"

namespace cg = cooperative_groups;

namespace swlm {
namespace {

constexpr int kPage = SWLM_PAGE_TOKENS;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ga_get(const float* p) { return *p; }
__device__ __forceinline__ float ga_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void ga_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void ga_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ unsigned ga_pack(float a, float b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const unsigned*>(&v);
}
__device__ __forceinline__ float ga_round(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }
__device__ __forceinline__ void ga_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ga_ldsm(unsigned (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
// lane (g, t) gives entries 2t and 2t + 1 of row g of an 8 x 8 matrix and gets those of row g of its transpose
__device__ __forceinline__ unsigned ga_transpose(unsigned v) {
    unsigned r;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(r) : "r"(v));
    return r;
}
__device__ __forceinline__ void ga_ldsm_trans(unsigned (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}

struct GroupedParams {
    GroupedRow row;
    int heads, share, rot_dims, rot_neighbours, window, chunk, sink_one;
    float scale_log2, eps, weight_bias, magnitude, out_scale;
    const float* inv_freq;
    const __nv_bfloat16 *q_norm, *k_norm;
    void* qkv; int qkv_stride;
    const float* gate; int gate_stride;
    const void* entry_gate; int entry_gate_stride;
    int head_norm, temp_every; float temp_coef;
    void* pool;
    const int32_t* page_table; int pages_per_seq;
    const int32_t* row_seq; const int32_t* row_pos;
    void* out; int out_stride;
    int n_rows; const int32_t* rows;     // the rows of this launch; null: 0 .. n_rows - 1
    const LatentSpan* spans; const int2* tiles;
    int* status;
};

// first position a row at `pos` sees; never falls as pos grows
__device__ __forceinline__ int ga_first_seen(const GroupedParams& p, int pos) {
    const int w = p.window > 0 ? max(0, pos - p.window + 1) : 0, c = p.chunk > 0 ? pos / p.chunk * p.chunk : 0;
    return max(w, c);
}
__device__ __forceinline__ int ga_row(const GroupedParams& p, int i) { return p.rows ? p.rows[i] : i; }
// keys of head g in the page of a position; ga_values: where its values lie, ga_factors: what turns shared rows into keys
template <typename T>
__device__ __forceinline__ T* ga_block(const GroupedParams& p, int seq, int page_index, int g) {
    const int page = p.page_table[(size_t)seq * p.pages_per_seq + page_index];
    return static_cast<T*>(p.pool) + ((size_t)page * p.row.groups + g) * p.row.block;
}
__device__ __forceinline__ int ga_values(const GroupedRow& r) { return r.shared ? 0 : kPage * r.pk; }
template <typename T>
__device__ __forceinline__ float* ga_factors(const GroupedParams& p, const T* block) { return reinterpret_cast<float*>(const_cast<T*>(block) + (size_t)kPage * p.row.pk); }
// the gate of entry c of head h
template <typename T>
__device__ __forceinline__ float ga_entry_gate(const GroupedParams& p, int r, int h, int c) {
    return 1.0f / (1.0f + expf(-ga_get(static_cast<const T*>(p.entry_gate) + (size_t)r * p.entry_gate_stride + (size_t)h * p.row.vdim + c)));
}
// a sigmoid by the hardware's approximations (an fp32 number, a few units in the last place off)
__device__ __forceinline__ float ga_sigmoid(float x) { return __fdividef(1.0f, 1.0f + __expf(-x)); }
// two neighbours, bf16
__device__ __forceinline__ float2 ga_entry_gates(const GroupedParams& p, int r, int h, int c) {
    const unsigned v = __ldcg(reinterpret_cast<const unsigned*>(static_cast<const __nv_bfloat16*>(p.entry_gate) + (size_t)r * p.entry_gate_stride + (size_t)h * p.row.vdim + c));
    return make_float2(ga_sigmoid(__uint_as_float(v << 16)), ga_sigmoid(__uint_as_float(v & 0xFFFF0000u)));
}
__device__ __forceinline__ float ga_gate(const GroupedParams& p, int r, int h) {
    return (p.gate ? 1.0f / (1.0f + expf(-p.gate[(size_t)r * p.gate_stride + h])) : 1.0f) * p.out_scale;
}

// ---- norm, rotation, append -------------------------------------------------------------------------------------------
// CTA (row, eight vectors of the row): a warp per query, key or value vector.
constexpr int kAppWarps = 8;
template <typename T>
__global__ void __launch_bounds__(kAppWarps * 32) grouped_append_kernel(const GroupedParams p) {
    extern __shared__ __align__(16) float app_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, r = blockIdx.x, i = blockIdx.y * kAppWarps + warp;
    const int G = p.row.groups, dim = p.row.dim, vdim = p.row.vdim;
    if (i >= p.heads + (p.row.shared ? G : 2 * G)) return;
    const int pos = p.row_pos[r], seq = p.row_seq[r];
    T* base = static_cast<T*>(p.qkv) + (size_t)r * p.qkv_stride;
    if (i >= p.heads + G) {
        const int g = i - p.heads - G;
        const T* src = base + (size_t)(p.heads + G) * dim + (size_t)g * vdim;
        T* dst = ga_block<T>(p, seq, pos / kPage, g) + (size_t)kPage * p.row.pk + (size_t)(pos % kPage) * p.row.pv;
        for (int c = lane; c < vdim; c += 32) dst[c] = src[c];
        return;
    }
    float* x = app_smem + (size_t)warp * dim;
    T* src = base + (size_t)i * dim;
    float ss = 0.f;
    for (int c = lane; c < dim; c += 32) { const float v = ga_get(src + c); x[c] = v; ss = fmaf(v, v, ss); }
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const __nv_bfloat16* w = i < p.heads ? p.q_norm : p.k_norm;
    if (w) {
        const float sc = 1.0f / sqrtf(ss / (float)dim + p.eps);
        for (int c = lane; c < dim; c += 32) x[c] = x[c] * sc * (__bfloat162float(w[c]) + p.weight_bias);
    }
    float f = p.head_norm ? 1.0f / sqrtf(ss / (float)dim + p.eps) : 1.0f;
    if (p.row.shared && i >= p.heads) {   // the row as it is; its norm becomes a factor of the scores
        if (lane == 0) ga_factors(p, ga_block<T>(p, seq, pos / kPage, i - p.heads))[pos % kPage] = f;
        f = 1.0f;
    }
    if (i < p.heads && p.temp_every > 0) f *= 1.0f + p.temp_coef * logf((float)((pos + 1) / p.temp_every) + 1.0f);
    __syncwarp();
    T* dst = i < p.heads ? src : ga_block<T>(p, seq, pos / kPage, i - p.heads) + (size_t)(pos % kPage) * p.row.pk;
    for (int c = lane; c < dim; c += 32) {
        float v = x[c];
        if (c < p.rot_dims) {
            const RotaryEntry e = rotary_entry(c, p.rot_dims, p.rot_neighbours);
            float cs, sn;
            sincosf((float)pos * p.inv_freq[e.pair], &sn, &cs);
            const float o = x[e.partner];
            v = p.magnitude * (e.first ? v * cs - o * sn : v * cs + o * sn);
        }
        ga_put(dst + c, v * f);
    }
}

// ---- rows one by one, fp32 FMAs ---------------------------------------------------------------------------------------
// CTA (row, head), four warps that take the keys in turn.
constexpr int kSimpleWarps = 4;
template <typename T>
__global__ void __launch_bounds__(kSimpleWarps * 32) grouped_simple_kernel(const GroupedParams p) {
    extern __shared__ __align__(16) float simple_smem[];
    __shared__ float ms[kSimpleWarps], ls[kSimpleWarps];
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, dim = p.row.dim, vdim = p.row.vdim, h = blockIdx.y, g = h / p.share;
    const int r = ga_row(p, blockIdx.x), pos = p.row_pos[r], seq = p.row_seq[r];
    float* q = simple_smem;                                     // [dim]
    float* acc = simple_smem + dim + (size_t)warp * vdim;       // [warps][vdim]
    const T* src = static_cast<const T*>(p.qkv) + (size_t)r * p.qkv_stride + (size_t)h * dim;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) q[i] = ga_get(src + i);
    for (int i = lane; i < vdim; i += 32) acc[i] = 0.f;
    __syncthreads();
    float m = -INFINITY, l = 0.f;
    for (int key = ga_first_seen(p, pos) + warp; key <= pos; key += kSimpleWarps) {
        const T* block = ga_block<T>(p, seq, key / kPage, g);
        const T* k = block + (size_t)(key % kPage) * p.row.pk;
        const T* v = block + ga_values(p.row) + (size_t)(key % kPage) * p.row.pv;
        float s = 0.f;
        for (int i = lane; i < dim; i += 32) s = fmaf(q[i], ga_get(k + i), s);
        for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        s *= p.scale_log2;
        if (p.row.shared) s *= ga_factors(p, block)[key % kPage];
        const float m_new = fmaxf(m, s), corr = exp2f(m - m_new), w = exp2f(s - m_new);
        l = l * corr + w;
        m = m_new;
        for (int i = lane; i < vdim; i += 32) acc[i] = acc[i] * corr + w * ga_get(v + i);
    }
    if (lane == 0) { ms[warp] = m; ls[warp] = l; }
    __syncthreads();
    float top = p.sink_one ? 0.f : -INFINITY;
    for (int w = 0; w < kSimpleWarps; ++w) top = fmaxf(top, ms[w]);
    float total = p.sink_one ? exp2f(-top) : 0.f;
    for (int w = 0; w < kSimpleWarps; ++w) total += ls[w] * exp2f(ms[w] - top);
    const float f = ga_gate(p, r, h) / total;
    T* out = static_cast<T*>(p.out) + (size_t)r * p.out_stride + (size_t)h * vdim;
    for (int i = threadIdx.x; i < vdim; i += blockDim.x) {
        float v = 0.f;
        for (int w = 0; w < kSimpleWarps; ++w) v += simple_smem[dim + (size_t)w * vdim + i] * exp2f(ms[w] - top);
        ga_put(out + i, v * f * (p.entry_gate ? ga_entry_gate<T>(p, r, h, i) : 1.0f));
    }
}

// ---- rows one by one, tensor cores ------------------------------------------------------------------------------------
// Cluster of CTAs per (row, key / value head, eight query heads of it): the context in units of UK keys, dealt out to all warps of the
// cluster. A unit is two bulk copies (keys, values) into a stage of the warp's own. Keys (and entries of the values) are the rows of the
// multiplications, the few heads their columns.
constexpr int kDecStages = 2;   // units under way per warp, as far as shared memory goes
constexpr int kDecWarps = 8, kDecThreads = kDecWarps * 32, kDecHeads = 8, kDecCluster = 16;
template <int KQ, int NV, int UK, bool APPENDS>   // 16-column steps of query / key and value rows, keys of a unit; norm and append in here
__global__ void __launch_bounds__(kDecThreads, 1) grouped_decode_kernel(const GroupedParams p, int stages, int recv_at) {
    extern __shared__ __align__(128) unsigned char dec_smem[];
    __shared__ __align__(8) unsigned long long bar[kDecWarps][kDecStages];
    constexpr int QP = 16 * KQ + 8;
    __shared__ __align__(16) __nv_bfloat16 q_s[APPENDS ? kDecHeads * QP : 1], k_s[APPENDS ? 16 * KQ : 1], v_s[APPENDS ? 16 * NV : 1];
    __shared__ float own_factor;
    __shared__ float warp_m[kDecWarps][kDecHeads], warp_l[kDecWarps][kDecHeads], all_m[kDecCluster][kDecHeads], all_l[kDecCluster][kDecHeads];
    const cg::cluster_group cluster = cg::this_cluster();
    auto started = cluster.barrier_arrive();   // waited for before anything is written to another CTA's shared memory
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int nz = gridDim.x, rank = blockIdx.x, kv = blockIdx.y / ((p.share + kDecHeads - 1) / kDecHeads), tile = blockIdx.y % ((p.share + kDecHeads - 1) / kDecHeads);
    const int h0 = kv * p.share + tile * kDecHeads, nh = min(kDecHeads, p.share - tile * kDecHeads);   // query heads of this CTA
    pdl_launch_dependents();
    if (tid < kDecWarps * kDecStages) mbar_init(&bar[0][0] + tid, 1);
    if (tid == 0) asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    __syncthreads();
    if (!APPENDS) pdl_wait();   // (otherwise what is read first was there before this step)
    const int r = ga_row(p, blockIdx.z), pos = p.row_pos[r], seq = p.row_seq[r];
    const int past_end = APPENDS ? pos : pos + 1;   // first position whose row is not read from the cache
    const int seen0 = ga_first_seen(p, pos), unit0 = seen0 / UK, units = past_end > seen0 ? (past_end - 1) / UK + 1 - unit0 : 0;
    const int pk = p.row.pk, pv = p.row.pv, k_bytes = UK * pk * 2, v_bytes = p.row.shared ? UK * 4 : UK * pv * 2;   // (shared rows: their factors instead of values)
    unsigned char* stage0 = dec_smem + (size_t)warp * stages * (k_bytes + v_bytes);
    auto request = [&](int u, int st) {   // lane 0
        const unsigned bar_at = smem_u32(&bar[warp][st]);
        unsigned char* stage = stage0 + (size_t)st * (k_bytes + v_bytes);
        const int key0 = (unit0 + u) * UK;
        const __nv_bfloat16* block = ga_block<__nv_bfloat16>(p, seq, key0 / kPage, kv);
        mbar_expect(bar_at, (unsigned)(k_bytes + v_bytes));
        bulk_load(smem_u32(stage), block + (size_t)(key0 % kPage) * pk, (unsigned)k_bytes, bar_at);
        bulk_load(smem_u32(stage) + (unsigned)k_bytes, block + (size_t)kPage * pk + (size_t)(key0 % kPage) * (p.row.shared ? 2 : pv), (unsigned)v_bytes, bar_at);
    };
    const int first = rank * kDecWarps + warp, step = nz * kDecWarps;
    if (lane == 0) for (int st = 0; st < stages && first + st * step < units; ++st) request(first + st * step, st);
    const bool keeps = APPENDS && rank == 0 && tile == 0;   // puts the token's row into the cache
    __nv_bfloat16* own_block = keeps ? ga_block<__nv_bfloat16>(p, seq, pos / kPage, kv) : nullptr;
    const float temperature = APPENDS && p.temp_every > 0 ? 1.0f + p.temp_coef * logf((float)((pos + 1) / p.temp_every) + 1.0f) : 1.0f;
    if (APPENDS) pdl_wait();
    const float gate = tid >> 4 < nh ? ga_gate(p, r, h0 + (tid >> 4)) : 0.f;   // of the head whose results this thread merges
    const int ksteps = p.row.dp >> 4, n_vt = p.row.vp >> 4;
    const __nv_bfloat16* qkv = static_cast<const __nv_bfloat16*>(p.qkv) + (size_t)r * p.qkv_stride;
    const __nv_bfloat16* q = qkv + (size_t)h0 * p.row.dim;
    if (APPENDS) {
        // a warp per vector: the queries of this CTA, then the key; the value is copied
        const int dim = p.row.dim, vdim = p.row.vdim;
        for (int i = warp; i <= nh; i += kDecWarps) {
            const bool is_key = i == nh;
            const __nv_bfloat16* src = is_key ? qkv + (size_t)(p.heads + kv) * dim : q + (size_t)i * dim;
            __nv_bfloat16* dst = is_key ? k_s : q_s + (size_t)i * QP;
            float x[KQ / 2];
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < KQ / 2; ++j) { const int c = lane + 32 * j; x[j] = c < dim ? ga_get(src + c) : 0.f; ss = fmaf(x[j], x[j], ss); }
            for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            const __nv_bfloat16* w = is_key ? p.k_norm : p.q_norm;
            float f = p.head_norm || w ? 1.0f / sqrtf(ss / (float)dim + p.eps) : 1.0f;
            if (is_key && p.row.shared) {
                if (lane == 0) own_factor = f;
                f = 1.0f;
            }
            if (!is_key) f *= temperature;
#pragma unroll
            for (int j = 0; j < KQ / 2; ++j) {
                const int c = lane + 32 * j;
                if (c < 16 * KQ) ga_put(dst + c, c < dim ? x[j] * f * (w ? __bfloat162float(w[c]) + p.weight_bias : 1.0f) : 0.f);
            }
        }
        const __nv_bfloat16* v = qkv + (size_t)(p.heads + p.row.groups) * dim + (size_t)kv * vdim;
        if (!p.row.shared) for (int c = tid; c < 16 * NV; c += kDecThreads) v_s[c] = c < vdim ? v[c] : __float2bfloat16_rn(0.f);
        __syncthreads();
        if (keeps) {   // for the tokens to come
            for (int c = tid; c < dim; c += kDecThreads) own_block[(size_t)(pos % kPage) * pk + c] = k_s[c];
            if (p.row.shared) { if (tid == 0) ga_factors(p, own_block)[pos % kPage] = own_factor; }
            else for (int c = tid; c < vdim; c += kDecThreads) own_block[(size_t)kPage * pk + (size_t)(pos % kPage) * pv + c] = v_s[c];
        }
    }
    const __nv_bfloat16* own_v = APPENDS && p.row.shared ? k_s : v_s;
    // A column is a head. Up to four heads fill the columns twice: the first four carry the high parts of the softmax weights, the
    // others the low parts.
    const bool twice = nh <= kDecHeads / 2;
    const int hq = twice ? g & 3 : g;          // the head of column g
    unsigned qb[KQ][2];
#pragma unroll
    for (int k = 0; k < KQ; ++k)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int c = 16 * k + 8 * e + 2 * t;
            if (APPENDS) qb[k][e] = hq < nh ? *reinterpret_cast<const unsigned*>(q_s + (size_t)hq * QP + c) : 0u;
            else qb[k][e] = hq < nh && c < p.row.dim ? __ldcg(reinterpret_cast<const unsigned*>(q + (size_t)hq * p.row.dim + c)) : 0u;
        }
    // lane (g, t): rows g and g + 8 of every tile (keys, or entries of the values), columns 2t and 2t + 1
    float oacc[NV][4];
#pragma unroll
    for (int j = 0; j < NV; ++j) oacc[j][0] = oacc[j][1] = oacc[j][2] = oacc[j][3] = 0.f;
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
    if (APPENDS && rank == 0 && warp == 0) {   // the token's own key: the first row of a tile whose others are zero
        float own[4] = {0.f, 0.f, 0.f, 0.f}, odd[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int k = 0; k < KQ; ++k) {
            const unsigned ka[4] = {g == 0 ? *reinterpret_cast<const unsigned*>(k_s + 16 * k + 2 * t) : 0u, 0u, g == 0 ? *reinterpret_cast<const unsigned*>(k_s + 16 * k + 8 + 2 * t) : 0u, 0u};
            ga_mma(k & 1 ? odd : own, ka, qb[k][0], qb[k][1]);
        }
        const float f = p.row.shared ? p.scale_log2 * own_factor : p.scale_log2;
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            m[e] = f * __shfl_sync(0xffffffffu, own[e] + odd[e], t);
            l[e] = g == 0 ? 1.f : 0.f;
        }
        if (!twice || t < 2) {
#pragma unroll
            for (int j = 0; j < NV; ++j) {
                oacc[j][0] = oacc[j][1] = __bfloat162float(own_v[16 * j + g]);
                oacc[j][2] = oacc[j][3] = __bfloat162float(own_v[16 * j + 8 + g]);
            }
        }
    }
    constexpr int MT = UK / 16;
    int at = 0;
    unsigned phase = 0;
    for (int u = first; u < units; u += step) {
        const unsigned ks = smem_u32(stage0) + (unsigned)(at * (k_bytes + v_bytes)), vs = p.row.shared ? ks : ks + (unsigned)k_bytes;
        const float* factors = reinterpret_cast<const float*>(stage0 + (size_t)at * (k_bytes + v_bytes) + k_bytes);
        if (!mbar_wait(&bar[warp][at], phase)) {
            if (lane == 0) atomicExch(p.status, 61);
            // leave the loop only when the copies under way have landed (bounded)
            for (int st = 0; st < stages && u + st * step < units; ++st) mbar_wait(&bar[warp][(at + st) % stages], phase ^ (unsigned)(at + st >= stages));
            break;
        }
        float sacc[MT][4];
#pragma unroll
        for (int i = 0; i < MT; ++i) sacc[i][0] = sacc[i][1] = sacc[i][2] = sacc[i][3] = 0.f;
        unsigned kf[2][MT][4];   // the next fragments are on their way while these multiply
        auto keys = [&](int k) {
#pragma unroll
            for (int i = 0; i < MT; ++i) ga_ldsm(kf[k & 1][i], ks + (unsigned)((16 * i + (lane & 15)) * pk + 16 * k + 8 * (lane >> 4)) * 2u);
        };
        keys(0);
#pragma unroll
        for (int k = 0; k < KQ; ++k)
            if (k < ksteps) {
                if (k + 1 < KQ && k + 1 < ksteps) keys(k + 1);
#pragma unroll
                for (int i = 0; i < MT; ++i) ga_mma(sacc[i], kf[k & 1][i], qb[k][0], qb[k][1]);
            }
        const int key0 = (unit0 + u) * UK;
        float mx[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int i = 0; i < MT; ++i)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int at_key = 16 * i + 8 * half + g, key = key0 + at_key;
                const bool seen = key < past_end && key >= seen0;
                const float f = p.row.shared ? p.scale_log2 * factors[at_key] : p.scale_log2;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float& v = sacc[i][2 * half + e];
                    v = seen ? v * f : -INFINITY;
                    mx[e] = fmaxf(mx[e], v);
                }
            }
#pragma unroll
        for (int o = 4; o < 32; o <<= 1) { mx[0] = fmaxf(mx[0], __shfl_xor_sync(0xffffffffu, mx[0], o)); mx[1] = fmaxf(mx[1], __shfl_xor_sync(0xffffffffu, mx[1], o)); }
        // (every unit holds at least one key that is seen, by all heads alike)
        float corr[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const float next = fmaxf(m[e], mx[e]);
            corr[e] = exp2f(m[e] - next);
            m[e] = next;
            l[e] *= corr[e];
        }
#pragma unroll
        for (int j = 0; j < NV; ++j) { oacc[j][0] *= corr[0]; oacc[j][1] *= corr[1]; oacc[j][2] *= corr[0]; oacc[j][3] *= corr[1]; }
#pragma unroll
        for (int i = 0; i < MT; ++i) {
            unsigned hi[2], lo[2];   // weights of keys 2t, 2t + 1 (and + 8) for head g, after the transposition
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const float x = exp2f(sacc[i][2 * half] - m[0]), y = exp2f(sacc[i][2 * half + 1] - m[1]);
                l[0] += x; l[1] += y;
                const float xh = ga_round(x), yh = ga_round(y);
                const unsigned high = ga_pack(xh, yh), low = ga_pack(x - xh, y - yh);
                hi[half] = ga_transpose(twice && t >= 2 ? low : high);
                lo[half] = ga_transpose(low);
            }
            unsigned vf[2][4];
            auto values = [&](int j) { ga_ldsm_trans(vf[j & 1], vs + (unsigned)((16 * i + (lane & 7) + 8 * (lane >> 4)) * pv + 16 * j + 8 * ((lane >> 3) & 1)) * 2u); };
            values(0);
#pragma unroll
            for (int j = 0; j < NV; ++j)
                if (j < n_vt) {
                    if (j + 1 < NV && j + 1 < n_vt) values(j + 1);
                    ga_mma(oacc[j], vf[j & 1], hi[0], hi[1]);
                    if (!twice) ga_mma(oacc[j], vf[j & 1], lo[0], lo[1]);
                }
        }
        __syncwarp();   // the stage is free
        if (lane == 0 && u + stages * step < units) request(u + stages * step, at);
        if (++at == stages) { at = 0; phase ^= 1; }
    }
#pragma unroll
    for (int o = 4; o < 32; o <<= 1) { l[0] += __shfl_xor_sync(0xffffffffu, l[0], o); l[1] += __shfl_xor_sync(0xffffffffu, l[1], o); }
    if (twice) {   // high and low parts
#pragma unroll
        for (int j = 0; j < NV; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) oacc[j][e] += __shfl_xor_sync(0xffffffffu, oacc[j][e], 2);
    }
    if (g == 0) {
#pragma unroll
        for (int e = 0; e < 2; ++e) { warp_m[warp][2 * t + e] = m[e]; warp_l[warp][2 * t + e] = l[e]; }
    }
    __syncthreads();
    // the stages now hold the warps' sums: [warps][heads of this CTA][pitch]
    const int vp = p.row.vp, pitch = vp + 4, share = (nh * vp + nz - 1) / nz;   // share: entries of the result that a CTA of the cluster finishes
    float* sums = reinterpret_cast<float*>(dec_smem);
    float* recv = reinterpret_cast<float*>(dec_smem + recv_at);   // [nz][share], written by the other CTAs
#pragma unroll
    for (int e = 0; e < 2; ++e)
        if (2 * t + e < nh) {
            float* row = sums + ((size_t)warp * nh + 2 * t + e) * pitch + g;
#pragma unroll
            for (int j = 0; j < NV; ++j)
                if (j < n_vt) { row[16 * j] = oacc[j][e]; row[16 * j + 8] = oacc[j][2 + e]; }
        }
    // the gate of the first entry this thread finishes is on its way during the merge
    const __nv_bfloat16* egate = static_cast<const __nv_bfloat16*>(p.entry_gate) + (size_t)r * p.entry_gate_stride + (size_t)h0 * p.row.vdim;
    float entry = 1.f;
    if (p.entry_gate && tid < share && rank * share + tid < nh * vp && (rank * share + tid) % vp < p.row.vdim)
        entry = ga_sigmoid(__bfloat162float(egate[(size_t)((rank * share + tid) / vp) * p.row.vdim + (rank * share + tid) % vp]));
    cluster.barrier_wait(std::move(started));
    static_assert(kDecWarps <= 16 && kDecCluster == 16 && kDecHeads * 16 <= kDecThreads, "sixteen lanes per head");
    auto merge = [](float& top, float& total, float mine, float sum) {   // maximum and rescaled sum over sixteen lanes; this lane's factor
        top = mine;
#pragma unroll
        for (int o = 1; o < 16; o <<= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
        const float f = mine == -INFINITY ? 0.f : exp2f(mine - top);
        total = f * sum;
#pragma unroll
        for (int o = 1; o < 16; o <<= 1) total += __shfl_xor_sync(0xffffffffu, total, o);
        return f;
    };
    const int part = tid & 15, of_head = tid >> 4;   // (the first warps, two heads each)
    if (warp < kDecHeads / 2) {
        const bool there = part < kDecWarps;
        float top, total;
        const float f = merge(top, total, there ? warp_m[part][of_head] : -INFINITY, there ? warp_l[part][of_head] : 0.f);
        if (there) warp_l[part][of_head] = f;
        if (part < nz) {
            cluster.map_shared_rank(all_m[rank], part)[of_head] = top;
            cluster.map_shared_rank(all_l[rank], part)[of_head] = total;
        }
    }
    __syncthreads();
    for (int i = tid; i < nh * vp; i += kDecThreads) {
        const int hh = i / vp, z = i / share;
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kDecWarps; ++w) v = fmaf(warp_l[w][hh], sums[((size_t)w * nh + hh) * pitch + i - hh * vp], v);
        cluster.map_shared_rank(recv, z)[rank * share + i - z * share] = v;
    }
    cluster.sync();   // (nobody reaches into another CTA's shared memory behind this)
    if (warp < kDecHeads / 2) {
        const bool there = part < nz;
        float top, total;
        float f = merge(top, total, there ? all_m[part][of_head] : -INFINITY, there ? all_l[part][of_head] : 0.f);
        if (p.sink_one) {   // one joins the sum
            const float scale = top > 0.f ? 1.f : exp2f(top);
            f *= scale;
            total = total * scale + exp2f(-fmaxf(top, 0.f));
        }
        all_m[part][of_head] = f * gate / total;
    }
    __syncthreads();
    for (int q = tid; q < share && rank * share + q < nh * vp; q += kDecThreads) {
        const int i = rank * share + q, hh = i / vp, c = i - hh * vp;
        if (c >= p.row.vdim) continue;
        float v = 0.f;
        for (int z = 0; z < nz; ++z) v = fmaf(all_m[z][hh], recv[z * share + q], v);
        if (p.entry_gate) v *= q == tid ? entry : ga_sigmoid(__bfloat162float(egate[(size_t)hh * p.row.vdim + c]));
        static_cast<__nv_bfloat16*>(p.out)[(size_t)r * p.out_stride + (size_t)(h0 + hh) * p.row.vdim + c] = __float2bfloat16_rn(v);
    }
}

// ---- spans ------------------------------------------------------------------------------------------------------------
// CTA (tile of 128 query rows of a span, head), 8 warps of 16 query rows; a key tile is a page, one bulk copy of keys and values.
constexpr int kPfThreads = 256, kPfStages = 3;
template <int KQ, int NV, bool SHARED>
__global__ void __launch_bounds__(kPfThreads, 1) grouped_prefill_kernel(const GroupedParams p) {
    extern __shared__ __align__(128) unsigned char pf_smem[];
    __shared__ __align__(8) unsigned long long full_bar[kPfStages];
    __shared__ int bad;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3, h = blockIdx.y, kv = h / p.share;
    const int pk = p.row.pk, pv = p.row.pv, stage_bytes = p.row.block * 2;
    pdl_launch_dependents();
    if (tid == 0) {
        for (int s = 0; s < kPfStages; ++s) mbar_init(&full_bar[s], 1);
        bad = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    const int2 tile = p.tiles[blockIdx.x];
    const LatentSpan span = p.spans[tile.x];
    const int q0 = tile.y * kLatentQueryTile, nq = min(kLatentQueryTile, span.count - q0);
    const int first_pos = span.pos0 + q0, last_pos = first_pos + nq - 1;
    const int kt0 = ga_first_seen(p, first_pos) / kPage, n_tiles = last_pos / kPage + 1 - kt0;
    auto request = [&](int i) {   // thread 0: key tile kt0 + i
        const unsigned at = smem_u32(&full_bar[i % kPfStages]);
        mbar_expect(at, (unsigned)stage_bytes);
        bulk_load(smem_u32(pf_smem) + (unsigned)(i % kPfStages * stage_bytes), ga_block<__nv_bfloat16>(p, span.seq, kt0 + i, kv), (unsigned)stage_bytes, at);
    };
    if (tid == 0) for (int i = 0; i < min(kPfStages, n_tiles); ++i) request(i);
    unsigned qa[KQ][4];
    const __nv_bfloat16* q = static_cast<const __nv_bfloat16*>(p.qkv) + (size_t)(span.row0 + q0) * p.qkv_stride + (size_t)h * p.row.dim;
#pragma unroll
    for (int k = 0; k < KQ; ++k)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int rr = warp * 16 + g + 8 * (e & 1), c = 16 * k + 8 * (e >> 1) + 2 * t;
            qa[k][e] = rr < nq && c < p.row.dim ? __ldcg(reinterpret_cast<const unsigned*>(q + (size_t)rr * p.qkv_stride + c)) : 0u;
        }
    const int pos_a = first_pos + warp * 16 + g, pos_b = pos_a + 8;
    const int warp_first = first_pos + warp * 16, warp_last = min(warp_first + 15, last_pos);
    const int seen_a = ga_first_seen(p, pos_a), seen_b = ga_first_seen(p, pos_b), warp_seen = ga_first_seen(p, warp_first), full_from = ga_first_seen(p, warp_last);
    float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;
    float oacc[2 * NV][4];
#pragma unroll
    for (int j = 0; j < 2 * NV; ++j) oacc[j][0] = oacc[j][1] = oacc[j][2] = oacc[j][3] = 0.f;
    const int ksteps = p.row.dp >> 4, n_vt = p.row.vp >> 4;
    int i = 0;
    for (; i < n_tiles; ++i) {
        if (!mbar_wait(&full_bar[i % kPfStages], (unsigned)((i / kPfStages) & 1))) { atomicExch(p.status, 62); bad = 1; }
        const int key0 = (kt0 + i) * kPage;
        const unsigned kb = smem_u32(pf_smem) + (unsigned)(i % kPfStages * stage_bytes), vb = SHARED ? kb : kb + (unsigned)(kPage * pk) * 2u;
        const float* factors = reinterpret_cast<const float*>(pf_smem + (size_t)(i % kPfStages) * stage_bytes + (size_t)kPage * pk * 2);
        if (warp_first <= last_pos && key0 <= warp_last && key0 + kPage > warp_seen) {
            float sacc[8][4];
#pragma unroll
            for (int j = 0; j < 8; ++j) sacc[j][0] = sacc[j][1] = sacc[j][2] = sacc[j][3] = 0.f;
#pragma unroll
            for (int k = 0; k < KQ; ++k)
                if (k < ksteps) {
#pragma unroll
                    for (int jp = 0; jp < 4; ++jp) {
                        unsigned b[4];
                        ga_ldsm(b, kb + (unsigned)((jp * 16 + (lane & 7) + 8 * (lane >> 4)) * pk + 16 * k + 8 * ((lane >> 3) & 1)) * 2u);
                        ga_mma(sacc[2 * jp], qa[k], b[0], b[1]);
                        ga_mma(sacc[2 * jp + 1], qa[k], b[2], b[3]);
                    }
                }
            const bool edge = key0 + kPage - 1 > warp_first || key0 < full_from;   // some row does not see the whole tile
            float mx_a = -INFINITY, mx_b = -INFINITY;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                float2 ff = make_float2(p.scale_log2, p.scale_log2);
                if (SHARED) { const float2 v = *reinterpret_cast<const float2*>(factors + 8 * j + 2 * t); ff.x *= v.x; ff.y *= v.y; }
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int key = key0 + 8 * j + 2 * t + e;
                    const float f = e ? ff.y : ff.x;
                    const float a = !edge || (key <= pos_a && key >= seen_a) ? sacc[j][e] * f : -INFINITY;
                    const float b = !edge || (key <= pos_b && key >= seen_b) ? sacc[j][2 + e] * f : -INFINITY;
                    sacc[j][e] = a; sacc[j][2 + e] = b;
                    mx_a = fmaxf(mx_a, a); mx_b = fmaxf(mx_b, b);
                }
            }
#pragma unroll
            for (int o = 1; o < 4; o <<= 1) { mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, o)); mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, o)); }
            const float mn_a = fmaxf(m_a, mx_a), mn_b = fmaxf(m_b, mx_b);
            // a row that sees nothing yet keeps a maximum of -inf, weights of zero and sums of zero
            const float ra = mn_a == -INFINITY ? 0.f : mn_a, rb = mn_b == -INFINITY ? 0.f : mn_b;
            const float ca = m_a == -INFINITY ? 1.f : exp2f(m_a - mn_a), cb = m_b == -INFINITY ? 1.f : exp2f(m_b - mn_b);
            m_a = mn_a; m_b = mn_b;
            float sa = 0.f, sb = 0.f;
#pragma unroll
            for (int j = 0; j < 8; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    sacc[j][e] = exp2f(sacc[j][e] - ra); sa += sacc[j][e];
                    sacc[j][2 + e] = exp2f(sacc[j][2 + e] - rb); sb += sacc[j][2 + e];
                }
            l_a = l_a * ca + sa; l_b = l_b * cb + sb;
            if (__any_sync(0xffffffffu, ca != 1.0f || cb != 1.0f)) {
#pragma unroll
                for (int j = 0; j < 2 * NV; ++j) { oacc[j][0] *= ca; oacc[j][1] *= ca; oacc[j][2] *= cb; oacc[j][3] *= cb; }
            }
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                unsigned ah[4], al[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float x = sacc[2 * kk + (e >> 1)][(e & 1) * 2], y = sacc[2 * kk + (e >> 1)][(e & 1) * 2 + 1];
                    const float xh = ga_round(x), yh = ga_round(y);
                    ah[e] = ga_pack(xh, yh);
                    al[e] = ga_pack(x - xh, y - yh);
                }
#pragma unroll
                for (int j = 0; j < NV; ++j)
                    if (j < n_vt) {
                        unsigned b[4];
                        ga_ldsm_trans(b, vb + (unsigned)((16 * kk + (lane & 7) + 8 * ((lane >> 3) & 1)) * pv + 16 * j + 8 * (lane >> 4)) * 2u);
                        ga_mma(oacc[2 * j], ah, b[0], b[1]);
                        ga_mma(oacc[2 * j], al, b[0], b[1]);
                        ga_mma(oacc[2 * j + 1], ah, b[2], b[3]);
                        ga_mma(oacc[2 * j + 1], al, b[2], b[3]);
                    }
            }
        }
        __syncthreads();   // the stage is free
        if (bad) break;    // uniform: written before the barrier by whoever gave up
        if (tid == 0 && i + kPfStages < n_tiles) request(i + kPfStages);
    }
    if (bad) {
        // leave only when the copies that may still be under way have landed (bounded)
        if (tid == 0) for (int k = i; k < i + kPfStages && k < n_tiles; ++k) mbar_wait(&full_bar[k % kPfStages], (unsigned)((k / kPfStages) & 1));
        return;
    }
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) { l_a += __shfl_xor_sync(0xffffffffu, l_a, o); l_b += __shfl_xor_sync(0xffffffffu, l_b, o); }
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int rr = warp * 16 + g + 8 * half;
        if (rr >= nq) continue;
        const int row = span.row0 + q0 + rr;
        // (every row sees its own key, so its maximum is finite)
        const float m = half ? m_b : m_a, top = p.sink_one ? fmaxf(m, 0.f) : m, own = exp2f(m - top);
        const float f = ga_gate(p, row, h) * own / ((half ? l_b : l_a) * own + (p.sink_one ? exp2f(-top) : 0.f));
        __nv_bfloat16* o = static_cast<__nv_bfloat16*>(p.out) + (size_t)row * p.out_stride + (size_t)h * p.row.vdim;
#pragma unroll
        for (int j = 0; j < 2 * NV; ++j) {
            const int c = 8 * j + 2 * t;
            if (c < p.row.vdim) {
                float x = oacc[j][2 * half] * f, y = oacc[j][2 * half + 1] * f;
                if (p.entry_gate) { const float2 s = ga_entry_gates(p, row, h, c); x *= s.x; y *= s.y; }
                *reinterpret_cast<unsigned*>(o + c) = ga_pack(x, y);
            }
        }
    }
}

// ---- launches ---------------------------------------------------------------------------------------------------------
enum { FORM_MEDIUM, FORM_LARGE, FORM_SIMPLE };
// up to 128 entries per head: decode and prefill kernels; up to 256: the decode kernel for all rows; else fp32 FMAs
int form_of(const GroupedRow& r, bool f32) {
    if (f32 || ((r.dim | r.vdim) & 7)) return FORM_SIMPLE;
    return r.dp <= 128 && r.vp <= 128 ? FORM_MEDIUM : r.dp <= 256 && r.vp <= 256 ? FORM_LARGE : FORM_SIMPLE;
}
constexpr size_t kGaMaxSmem = 200 * 1024, kDecSmem = 160 * 1024;
// stages, then sums in their place
size_t decode_recv_at(const GroupedRow& r, int share, int unit, int stage_count) {
    const size_t stages = (size_t)stage_count * kDecWarps * unit * (r.shared ? 2 * r.pk + 4 : 2 * (r.pk + r.pv)), sums = (size_t)kDecWarps * std::min(share, kDecHeads) * (r.vp + 4) * 4;
    return (std::max(stages, sums) + 15) / 16 * 16;
}
// and what the other CTAs of the cluster send
size_t decode_smem(const GroupedRow& r, int share, int unit, int stage_count) {
    return decode_recv_at(r, share, unit, stage_count) + ((size_t)std::min(share, kDecHeads) * r.vp + kDecCluster) * 4;
}
size_t simple_bytes(const GroupedRow& r) { return ((size_t)r.dim + (size_t)kSimpleWarps * r.vdim) * 4; }
constexpr int kUnitMedium = 32, kUnitLarge = 16;
// CTAs per cluster: enough warps for the longest context, about one CTA per SM over all rows; the largest clusters only when all of them
// run at once with room to spare (`clusters`: how many fit an empty GPU)
int decode_cluster(const GroupedLaunch& a, int unit, int clusters) {
    int keys = a.max_pages * kPage;
    if (a.window > 0) keys = std::min(keys, a.window);
    if (a.chunk > 0) keys = std::min(keys, a.chunk);
    const int units = (keys + unit - 2) / unit + 1, tiles = a.n_short * a.row.groups * ((a.heads / a.row.groups + kDecHeads - 1) / kDecHeads);
    int nz = 2 * tiles <= clusters + 1 ? kDecCluster : kDecCluster / 2;
    while (nz > 1 && ((nz >> 1) * kDecWarps >= units || (long long)tiles * nz > 148)) nz >>= 1;
    return nz;
}
// how many of the largest clusters of a kernel the GPU runs at once
template <typename K>
int largest_clusters(K kernel) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(kDecCluster); cfg.blockDim = dim3(kDecThreads); cfg.dynamicSmemBytes = kDecSmem;
    cudaLaunchAttribute cluster[1];
    cluster[0].id = cudaLaunchAttributeClusterDimension;
    cluster[0].val.clusterDim.x = kDecCluster; cluster[0].val.clusterDim.y = 1; cluster[0].val.clusterDim.z = 1;
    cfg.attrs = cluster;
    cfg.numAttrs = 1;
    int n = 0;
    return cudaOccupancyMaxActiveClusters(&n, kernel, &cfg) == cudaSuccess ? n : 0;
}
template <int KQ, int NV, int UK, bool APPENDS>
cudaError_t decode_launch(const GroupedParams& p, const GroupedLaunch& a, cudaStream_t s) {
    static const int clusters = largest_clusters(grouped_decode_kernel<KQ, NV, UK, APPENDS>);
    const int nz = decode_cluster(a, UK, clusters);
    int stages = kDecStages;
    while (stages > 1 && decode_smem(p.row, p.share, UK, stages) > kDecSmem) --stages;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(nz, p.row.groups * ((p.share + kDecHeads - 1) / kDecHeads), p.n_rows); cfg.blockDim = dim3(kDecThreads); cfg.stream = s;
    cfg.dynamicSmemBytes = decode_smem(p.row, p.share, UK, stages);
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = nz; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl_enabled() ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, grouped_decode_kernel<KQ, NV, UK, APPENDS>, p, stages, (int)decode_recv_at(p.row, p.share, UK, stages));
}
template <typename K>
int decode_attr(K kernel) {
    SWLM_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGaMaxSmem));
    SWLM_CUDA(cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1));
    return SWLM_OK;
}

}  // namespace

GroupedRow grouped_row(int groups, int dim, int vdim, bool f32, bool shared) {
    GroupedRow r;
    r.groups = groups; r.dim = dim; r.vdim = vdim; r.shared = shared;
    r.dp = (dim + 15) / 16 * 16; r.vp = (vdim + 15) / 16 * 16;
    r.pk = r.dp + (f32 ? 0 : 8); r.pv = r.vp + (f32 ? 0 : 8);
    r.block = shared ? kPage * (r.pk + (f32 ? 1 : 2)) : kPage * (r.pk + r.pv);
    return r;
}
bool grouped_supported(const GroupedRow& r) { return r.dim <= 4096 && simple_bytes(r) <= kGaMaxSmem; }
bool grouped_appends(const GroupedRow& r, bool f32, int rot_dims) { return form_of(r, f32) != FORM_SIMPLE && rot_dims == 0; }
bool grouped_spans(const GroupedRow& r, bool f32) { return form_of(r, f32) == FORM_MEDIUM; }

int grouped_init() {
    SWLM_CUDA(cudaFuncSetAttribute(grouped_append_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGaMaxSmem));
    SWLM_CUDA(cudaFuncSetAttribute(grouped_append_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGaMaxSmem));
    SWLM_CUDA(cudaFuncSetAttribute(grouped_simple_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGaMaxSmem));
    SWLM_CUDA(cudaFuncSetAttribute(grouped_simple_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGaMaxSmem));
    int rc;
    if ((rc = decode_attr(grouped_decode_kernel<8, 8, kUnitMedium, false>)) || (rc = decode_attr(grouped_decode_kernel<8, 8, kUnitMedium, true>)) ||
        (rc = decode_attr(grouped_decode_kernel<16, 16, kUnitLarge, false>)) || (rc = decode_attr(grouped_decode_kernel<16, 16, kUnitLarge, true>))) return rc;
    SWLM_CUDA(cudaFuncSetAttribute(grouped_prefill_kernel<8, 8, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGaMaxSmem));
    SWLM_CUDA(cudaFuncSetAttribute(grouped_prefill_kernel<8, 8, true>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGaMaxSmem));
    return SWLM_OK;
}

int launch_grouped(const GroupedLaunch& a, cudaStream_t s, int* launches) {
    GroupedParams p{};
    p.row = a.row; p.heads = a.heads; p.share = a.heads / a.row.groups; p.rot_dims = a.rot_dims; p.rot_neighbours = a.rot_neighbours;
    p.window = a.window; p.chunk = a.chunk; p.sink_one = a.sink_one;
    p.scale_log2 = a.scale * kLog2e; p.eps = a.eps; p.weight_bias = a.weight_bias; p.magnitude = a.magnitude; p.out_scale = a.out_scale; p.inv_freq = a.inv_freq;
    p.head_norm = a.head_norm; p.temp_every = a.temp_every; p.temp_coef = a.temp_coef; p.entry_gate = a.entry_gate; p.entry_gate_stride = a.entry_gate_stride;
    p.q_norm = a.q_norm; p.k_norm = a.k_norm; p.qkv = a.qkv; p.qkv_stride = a.qkv_stride; p.gate = a.gate; p.gate_stride = a.gate_stride;
    p.pool = a.pool; p.page_table = a.page_table; p.pages_per_seq = a.pages_per_seq; p.row_seq = a.row_seq; p.row_pos = a.row_pos;
    p.out = a.out; p.out_stride = a.out_stride; p.spans = a.spans; p.tiles = a.tiles; p.status = a.status;
    cudaError_t e;
    const bool appends = grouped_appends(a.row, a.f32, a.rot_dims) && a.singles && a.n_short == a.n_rows && !a.only_attention;
    if (!a.only_attention && !appends) {
        const dim3 grid(a.n_rows, (a.heads + (a.row.shared ? 1 : 2) * a.row.groups + kAppWarps - 1) / kAppWarps);
        const size_t smem = (size_t)kAppWarps * a.row.dim * 4;
        e = a.f32 ? launch_k(grouped_append_kernel<float>, grid, dim3(kAppWarps * 32), smem, s, p) : launch_k(grouped_append_kernel<__nv_bfloat16>, grid, dim3(kAppWarps * 32), smem, s, p);
        if (e != cudaSuccess) return cuda_fail(e, "grouped append launch");
        *launches += 1;
    }
    if (a.n_short > 0) {
        p.n_rows = a.n_short; p.rows = a.short_rows;
        switch (form_of(a.row, a.f32)) {
        case FORM_MEDIUM: e = appends ? decode_launch<8, 8, kUnitMedium, true>(p, a, s) : decode_launch<8, 8, kUnitMedium, false>(p, a, s); break;
        case FORM_LARGE: e = appends ? decode_launch<16, 16, kUnitLarge, true>(p, a, s) : decode_launch<16, 16, kUnitLarge, false>(p, a, s); break;
        default:
            e = a.f32 ? launch_k(grouped_simple_kernel<float>, dim3(a.n_short, a.heads), dim3(kSimpleWarps * 32), simple_bytes(a.row), s, p)
                      : launch_k(grouped_simple_kernel<__nv_bfloat16>, dim3(a.n_short, a.heads), dim3(kSimpleWarps * 32), simple_bytes(a.row), s, p);
        }
        if (e != cudaSuccess) return cuda_fail(e, "grouped attention launch");
        *launches += 1;
    }
    if (a.n_tiles > 0) {
        const dim3 grid(a.n_tiles, a.heads);
        const size_t smem = (size_t)kPfStages * a.row.block * 2;
        e = a.row.shared ? launch_k(grouped_prefill_kernel<8, 8, true>, grid, dim3(kPfThreads), smem, s, p) : launch_k(grouped_prefill_kernel<8, 8, false>, grid, dim3(kPfThreads), smem, s, p);
        if (e != cudaSuccess) return cuda_fail(e, "grouped prompt attention launch");
        *launches += 1;
    }
    return SWLM_OK;
}

}  // namespace swlm
