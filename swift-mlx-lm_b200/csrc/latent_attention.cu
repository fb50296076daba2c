// Latent attention: keys and values of all heads come out of one cached row per token (a normed latent and a rotated key
// part shared by the heads), kept in pages of 64 rows that sequences take from a pool.
//
// Two ways through it, chosen per row of a batch:
//   * one by one, in the latent space (decode steps, short portions): latent_query_kernel folds the key projection into the
//     query (q_plain . W_uk c = (W_uk^T q_plain) . c), rotates, and appends the row's own latent; an attention kernel works
//     on the cached rows as one key / value head shared by all query heads, split over the context; latent_out_kernel merges
//     the splits, applies the value projection and the output gate.
//   * in spans (prompt portions): latent_append_kernel appends and rotates, latent_gather_kernel lines the cached rows of the
//     spans up, one tensor-core product expands them to keys and values per head, latent_prefill_kernel is a tiled causal
//     attention over them with the gate in its epilogue.
//
// Scores, softmax and sums are fp32. Where tensor cores take fp32 quantities (absorbed queries, softmax weights) these enter
// as bf16 hi + lo pairs. With a sliding window only the pages it reaches into are touched; a sink joins the denominator when
// the splits are merged, or at the end of a query tile. The newest rows are read back from the cache like all others, so a row's result does not depend on
// how a sequence was cut into batches.
#include <cooperative_groups.h>

#include <algorithm>
#include <cstdlib>
#include <utility>

#include "swlm_internal.h"
#include "tc_device.cuh"

namespace cg = cooperative_groups;

namespace swlm {
namespace {

constexpr int kPage = SWLM_PAGE_TOKENS;
constexpr int kPartialTail = 4;   // behind a partial's rp sums: running maximum, sum of weights, padding to 16 bytes
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float lat_get(const float* p) { return *p; }
__device__ __forceinline__ float lat_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void lat_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void lat_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ unsigned lat_pack(float a, float b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const unsigned*>(&v);
}
__device__ __forceinline__ float lat_round(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }
__device__ __forceinline__ float lat_lo(unsigned w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float lat_hi(unsigned w) { return __uint_as_float(w & 0xFFFF0000u); }
__device__ __forceinline__ void lat_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void lat_ldsm(unsigned (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void lat_ldsm_trans(unsigned (&r)[4], unsigned addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}

struct LatentParams {
    LatentRow row;
    int heads, dim, vdim, rot_dims, rot_neighbours;
    float scale_log2, eps, weight_bias, magnitude;
    int window; const __nv_bfloat16* sink;
    const float* inv_freq;
    void* q; int q_stride;
    const float* kv; int kv_stride;
    const float* gate; int gate_stride;
    const __nv_bfloat16* norm_w;
    const __nv_bfloat16* uk; int uk_ld;
    const __nv_bfloat16* uv; int uv_ld;
    void* pool;
    const int32_t* page_table; int pages_per_seq;
    const int32_t* row_seq; const int32_t* row_pos;
    void* out; int out_stride;
    int n_rows; const int32_t* rows;     // the rows of this launch; null: 0 .. n_rows - 1
    int splits;
    float* qcat; float* partial;
    int frag;                            // qcat holds bf16 hi + lo fragments of the tensor-core kernel instead of fp32 rows
    int* status;
    // spans
    const LatentSpan* spans; const int2* tiles; int n_spans, total_ctx;
    __nv_bfloat16* ctx_latent; __nv_bfloat16* ctx_rot; int ctx_ld, rot_ld;
    const __nv_bfloat16* ctx_k; const __nv_bfloat16* ctx_v;
};

// Entry (row of the launch, head, column) of the queries. As fragments: per 16 heads and 16 columns, lane (g, t) holds 8 words:
// the four words of an m16n8k16 A fragment from the high bf16 halves, then the four from the low ones.
__device__ __forceinline__ void store_query(const LatentParams& p, int rl, int h, int col, float v) {
    const int qw = p.row.rp + p.row.rotp;
    if (!p.frag) { p.qcat[((size_t)rl * p.heads + h) * qw + col] = v; return; }
    const int tiles = (p.heads + 15) >> 4, hr = h & 15, k = col & 15;
    const int lane = (hr & 7) * 4 + ((k & 7) >> 1), word = (hr >> 3) + 2 * (k >> 3);
    __nv_bfloat16* d = reinterpret_cast<__nv_bfloat16*>(p.qcat) + ((((size_t)rl * tiles + (h >> 4)) * (qw >> 4) + (col >> 4)) * 32 + lane) * 16 + word * 2 + (k & 1);
    const __nv_bfloat16 hi = __float2bfloat16_rn(v);
    d[0] = hi;
    d[8] = __float2bfloat16_rn(v - __bfloat162float(hi));
}

// first position a row at `pos` sees
__device__ __forceinline__ int first_seen(const LatentParams& p, int pos) { return p.window > 0 ? max(0, pos - p.window + 1) : 0; }
// a head's sink as a score in base 2, -inf when there is none
__device__ __forceinline__ float sink_log2(const LatentParams& p, int h) { return p.sink ? __bfloat162float(p.sink[h]) * kLog2e : -INFINITY; }

__device__ __forceinline__ int batch_row(const LatentParams& p, int i) { return p.rows ? p.rows[i] : i; }
template <typename T>
__device__ __forceinline__ T* cached_row(const LatentParams& p, int seq, int pos) {
    const int page = p.page_table[(size_t)seq * p.pages_per_seq + pos / kPage];
    return static_cast<T*>(p.pool) + ((size_t)page * kPage + pos % kPage) * p.row.pitch;
}
// cos and sin of pair i at a position, times the scaling's magnitude
__device__ __forceinline__ void angle(const LatentParams& p, int pos, int i, float& c, float& s) {
    sincosf((float)pos * p.inv_freq[i], &s, &c);
    c *= p.magnitude;
    s *= p.magnitude;
}
// entry i of a rotated part x[0 .. rot) at position pos
template <typename V>
__device__ __forceinline__ float rotated(const LatentParams& p, const V& x, int pos, int i) {
    if (i >= p.rot_dims) return x(i);
    const RotaryEntry e = rotary_entry(i, p.rot_dims, p.rot_neighbours);
    float c, s;
    angle(p, pos, e.pair, c, s);
    return e.first ? x(i) * c - x(e.partner) * s : x(i) * c + x(e.partner) * s;
}

// The row a warp appends: norm of the latent, rotation of the shared key part, zeros in the padding.
constexpr int kAppendRegs = 16;   // latent entries per lane that are read once
template <typename T>
__device__ __forceinline__ void append_row(const LatentParams& p, int r, int lane) {
    const float* src = p.kv + (size_t)r * p.kv_stride;
    const int pos = p.row_pos[r], seq = p.row_seq[r];
    float v[kAppendRegs];
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < kAppendRegs; ++j) { const int i = lane + 32 * j; v[j] = i < p.row.rank ? src[i] : 0.f; }
    T* dst = cached_row<T>(p, seq, pos);
#pragma unroll
    for (int j = 0; j < kAppendRegs; ++j) ss = fmaf(v[j], v[j], ss);
    for (int i = lane + 32 * kAppendRegs; i < p.row.rank; i += 32) { const float x = src[i]; ss = fmaf(x, x, ss); }
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    const float sc = 1.0f / sqrtf(ss / (float)p.row.rank + p.eps);
#pragma unroll
    for (int j = 0; j < kAppendRegs; ++j) {
        const int i = lane + 32 * j;
        if (i < p.row.rp) lat_put(dst + i, i < p.row.rank ? v[j] * sc * (__bfloat162float(p.norm_w[i]) + p.weight_bias) : 0.f);
    }
    for (int i = lane + 32 * kAppendRegs; i < p.row.rp; i += 32)
        lat_put(dst + i, i < p.row.rank ? src[i] * sc * (__bfloat162float(p.norm_w[i]) + p.weight_bias) : 0.f);
    const float* rot = src + p.row.rank;
    auto at = [&](int i) { return rot[i]; };
    for (int i = lane; i < p.row.pitch - p.row.rp; i += 32) lat_put(dst + p.row.rp + i, i < p.row.rot ? rotated(p, at, pos, i) : 0.f);
}

// The same by a CTA of 256 threads: everything that does not depend on something else is requested at once.
constexpr int kAppendThreads = 256;
template <typename T>
__device__ __forceinline__ void append_row_cta(const LatentParams& p, int r, float* red) {
    const int tid = threadIdx.x, half = p.row.rp;
    const float* src = p.kv + (size_t)r * p.kv_stride;
    const int pos = p.row_pos[r], seq = p.row_seq[r];
    float v[2], w[2];
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int i = tid + kAppendThreads * j;
        v[j] = i < p.row.rank ? src[i] : 0.f;
        w[j] = i < p.row.rank ? __bfloat162float(p.norm_w[i]) + p.weight_bias : 0.f;
    }
    const float* rot = src + p.row.rank;
    auto at = [&](int i) { return rot[i]; };
    const int tail = p.row.pitch - p.row.rp;
    const float turned = tid < p.row.rot ? rotated(p, at, pos, tid) : 0.f;
    T* dst = cached_row<T>(p, seq, pos);
    float ss = fmaf(v[0], v[0], v[1] * v[1]);
    for (int i = tid + 2 * kAppendThreads; i < p.row.rank; i += kAppendThreads) { const float x = src[i]; ss = fmaf(x, x, ss); }
    for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
    if ((tid & 31) == 0) red[tid >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < kAppendThreads / 32; ++i) ss += red[i];
    __syncthreads();
    const float sc = 1.0f / sqrtf(ss / (float)p.row.rank + p.eps);
#pragma unroll
    for (int j = 0; j < 2; ++j) {
        const int i = tid + kAppendThreads * j;
        if (i < half) lat_put(dst + i, v[j] * sc * w[j]);
    }
    for (int i = tid + 2 * kAppendThreads; i < half; i += kAppendThreads)
        lat_put(dst + i, i < p.row.rank ? src[i] * sc * (__bfloat162float(p.norm_w[i]) + p.weight_bias) : 0.f);
    if (tid < tail) lat_put(dst + half + tid, turned);
    for (int i = tid + kAppendThreads; i < tail; i += kAppendThreads) lat_put(dst + half + i, i < p.row.rot ? rotated(p, at, pos, i) : 0.f);
}

// ---- rows one by one: queries -----------------------------------------------------------------------------------------
// CTA (h < heads, group of MR rows, 128 latent columns): absorbed query of one head, qcat[row][h] =
// [W_uk^T q_plain | rotated part], fp32, padding zero (the CTA of the first columns adds rotated part and padding). Thread
// (group g of 16, chunk of 8 columns): rows d = g, g + 16, ... of the head's key projection; the first batch of them is read
// before the preceding kernel has finished. CTA h == heads: the rows' own latents go to the cache.
constexpr int kQueryThreads = 256, kQueryChunks = 16, kQueryGroups = kQueryThreads / kQueryChunks, kQueryBatch = 8;
template <typename T, int MR>
__global__ void __launch_bounds__(kQueryThreads) latent_query_kernel(const LatentParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float query_smem[];
    const int tid = threadIdx.x, h = blockIdx.x, r0 = blockIdx.y * MR;
    const int nr = min(MR, p.n_rows - r0);
    if (h == p.heads) {
        static_assert(kQueryThreads == kAppendThreads, "a CTA appends a row");
        pdl_wait();
        for (int i = blockIdx.z; i < nr; i += gridDim.z) append_row_cta<T>(p, batch_row(p, r0 + i), query_smem);
        return;
    }
    const int cc = tid % kQueryChunks, g = tid / kQueryChunks, chunk = blockIdx.z * kQueryChunks + cc;
    const bool live = chunk < (p.uk_ld >> 3);
    const __nv_bfloat16* w = p.uk + (size_t)h * p.dim * p.uk_ld + 8 * (live ? chunk : 0);
    uint4 wv[kQueryBatch];
    auto load = [&](int d0) {
#pragma unroll
        for (int u = 0; u < kQueryBatch; ++u) {
            const int d = d0 + u * kQueryGroups;
            wv[u] = live && d < p.dim ? __ldg(reinterpret_cast<const uint4*>(w + (size_t)d * p.uk_ld)) : make_uint4(0, 0, 0, 0);
        }
    };
    load(g);
    pdl_wait();
    const int per_head = p.dim + p.row.rot, qw = p.row.rp + p.row.rotp;
    float* qs = query_smem;                                          // [MR][per_head]
    float* acc_s = query_smem + (MR * per_head + 3) / 4 * 4; // [groups][MR][chunks * 8]
    for (int i = tid; i < nr * per_head; i += kQueryThreads) {
        const int rr = i / per_head, c = i - rr * per_head;
        qs[rr * per_head + c] = lat_get(static_cast<const T*>(p.q) + (size_t)batch_row(p, r0 + rr) * p.q_stride + (size_t)h * per_head + c);
    }
    __syncthreads();
    if (blockIdx.z == 0) {
        for (int i = tid; i < nr * (qw - p.row.rank); i += kQueryThreads) {
            const int rr = i / (qw - p.row.rank), c = p.row.rank + i - rr * (qw - p.row.rank);
            const int rc = c - p.row.rp;
            const float* x = qs + rr * per_head + p.dim;
            auto at = [&](int e) { return x[e]; };
            const float v = rc >= 0 && rc < p.row.rot ? rotated(p, at, p.row_pos[batch_row(p, r0 + rr)], rc) : 0.f;
            store_query(p, r0 + rr, h, c, v);
        }
    }
    float acc[MR][8];
#pragma unroll
    for (int rr = 0; rr < MR; ++rr)
#pragma unroll
        for (int e = 0; e < 8; ++e) acc[rr][e] = 0.f;
    for (int d0 = g; d0 < p.dim; d0 += kQueryBatch * kQueryGroups) {
        if (d0 != g) load(d0);
#pragma unroll
        for (int u = 0; u < kQueryBatch; ++u) {
            const int d = d0 + u * kQueryGroups;
            if (d < p.dim) {
                const uint4 v = wv[u];
                const float wf[8] = {lat_lo(v.x), lat_hi(v.x), lat_lo(v.y), lat_hi(v.y), lat_lo(v.z), lat_hi(v.z), lat_lo(v.w), lat_hi(v.w)};
#pragma unroll
                for (int rr = 0; rr < MR; ++rr) {
                    if (rr < nr) {
                        const float x = qs[rr * per_head + d];
#pragma unroll
                        for (int e = 0; e < 8; ++e) acc[rr][e] = fmaf(x, wf[e], acc[rr][e]);
                    }
                }
            }
        }
    }
    constexpr int COLS = kQueryChunks * 8;
#pragma unroll
    for (int rr = 0; rr < MR; ++rr) {
        float4* d = reinterpret_cast<float4*>(acc_s + (size_t)(g * MR + rr) * COLS + cc * 8);
        d[0] = make_float4(acc[rr][0], acc[rr][1], acc[rr][2], acc[rr][3]);
        d[1] = make_float4(acc[rr][4], acc[rr][5], acc[rr][6], acc[rr][7]);
    }
    __syncthreads();
    for (int i = tid; i < nr * COLS; i += kQueryThreads) {
        const int rr = i / COLS, col = i - rr * COLS, c = blockIdx.z * COLS + col;
        float v = 0.f;
#pragma unroll
        for (int q = 0; q < kQueryGroups; ++q) v += acc_s[(size_t)(q * MR + rr) * COLS + col];
        if (c < p.row.rank) store_query(p, r0 + rr, h, c, v);
    }
}
template <typename T, int MR>
cudaError_t launch_query(const LatentLaunch& a, const LatentParams& p, cudaStream_t s) {
    const size_t smem = ((size_t)(MR * (a.dim + a.row.rot) + 3) / 4 * 4 + (size_t)kQueryGroups * MR * kQueryChunks * 8) * 4;
    const dim3 grid(a.heads + 1, (a.n_short + MR - 1) / MR, (a.uk->ld / 8 + kQueryChunks - 1) / kQueryChunks);
    return launch_k(latent_query_kernel<T, MR>, grid, dim3(kQueryThreads), smem, s, p);
}

// ---- rows one by one: attention on tensor cores (bf16 pool) -----------------------------------------------------------
// CTA (split, 16 heads, row): of the pages the row sees, number split, split + splits, ... A page is one bulk copy (rows pitched to
// be free of bank conflicts), two pages in flight. Scores: warp (kq, tq) multiplies its quarter of the query columns, held in
// registers as hi + lo fragments, with 32 of the page's 64 rows; the quarters are added in shared memory. Values: the same
// page again, 16 latent columns per warp and step, softmax weights as hi + lo.
constexpr int kSplWarps = 8, kSplThreads = kSplWarps * 32, kSplHeads = 16;
constexpr int kSPitch = 68, kPPitch = 72;
template <int KPW, int NPW>
__global__ void __launch_bounds__(kSplThreads, 1) latent_split_kernel(const LatentParams p) {
    extern __shared__ __align__(128) unsigned char split_smem[];
    __shared__ __align__(8) unsigned long long full_bar[2];
    __shared__ float corr_s[kSplHeads];
    __shared__ int bad;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3;
    const int split = blockIdx.x, h0 = blockIdx.y * kSplHeads, rl = blockIdx.z;
    const int page_bytes = kPage * p.row.pitch * 2;
    unsigned char* pages = split_smem;
    float* s_sm = reinterpret_cast<float*>(split_smem + 2 * (size_t)page_bytes);            // [4][16][kSPitch]
    __nv_bfloat16* p_hi = reinterpret_cast<__nv_bfloat16*>(s_sm + 4 * kSplHeads * kSPitch); // [16][kPPitch]
    __nv_bfloat16* p_lo = p_hi + kSplHeads * kPPitch;
    pdl_launch_dependents();
    if (tid == 0) {
        mbar_init(&full_bar[0], 1);
        mbar_init(&full_bar[1], 1);
        bad = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    const int r = batch_row(p, rl), pos = p.row_pos[r], seq = p.row_seq[r];
    const int32_t* table = p.page_table + (size_t)seq * p.pages_per_seq;
    const int seen0 = first_seen(p, pos), page0 = seen0 / kPage;
    const int n_pages = pos / kPage + 1 - page0;
    if (split >= n_pages) return;
    const int first_page = table[page0 + split];
    const int mine = (n_pages - split + p.splits - 1) / p.splits;
    auto request = [&](int i) {   // thread 0: the i-th page of this CTA
        const unsigned bar = smem_u32(&full_bar[i & 1]);
        mbar_expect(bar, (unsigned)page_bytes);
        bulk_load(smem_u32(pages + (size_t)(i & 1) * page_bytes),
                  static_cast<const unsigned char*>(p.pool) + (size_t)(i == 0 ? first_page : table[page0 + split + i * p.splits]) * page_bytes, (unsigned)page_bytes, bar);
    };
    if (tid == 0) { request(0); if (mine > 1) request(1); }

    // query fragments of this warp's quarter of the columns
    const int kq = warp & 3, tq = warp >> 2;
    const int qw = p.row.rp + p.row.rotp, ksteps = qw >> 4;
    unsigned qh[KPW][4], ql[KPW][4];
    {
        // (heads past the last one hold whatever was there: their results are dropped)
        const uint4* f = reinterpret_cast<const uint4*>(p.qcat) + (((size_t)rl * gridDim.y + blockIdx.y) * ksteps * 32 + lane) * 2;
#pragma unroll
        for (int k = 0; k < KPW; ++k) {
            const int ks = kq * KPW + k;
            const uint4 zero = make_uint4(0, 0, 0, 0);
            const uint4 hi = ks < ksteps ? __ldcg(f + (size_t)ks * 64) : zero, lo = ks < ksteps ? __ldcg(f + (size_t)ks * 64 + 1) : zero;
            qh[k][0] = hi.x; qh[k][1] = hi.y; qh[k][2] = hi.z; qh[k][3] = hi.w;
            ql[k][0] = lo.x; ql[k][1] = lo.y; ql[k][2] = lo.z; ql[k][3] = lo.w;
        }
    }
    float oacc[NPW][2][4];
#pragma unroll
    for (int j = 0; j < NPW; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) oacc[j][0][e] = oacc[j][1][e] = 0.f;
    const int srow = tid >> 4, scol = (tid & 15) * 4;   // softmax: head and first of four rows of the page
    float m_run = -INFINITY, l_run = 0.f;
    const int n_ct = p.row.rp >> 4;

    int i = 0;
    for (; i < mine; ++i) {
        if (!mbar_wait(&full_bar[i & 1], (unsigned)((i >> 1) & 1))) { atomicExch(p.status, 41); bad = 1; }
        const unsigned page = smem_u32(pages + (size_t)(i & 1) * page_bytes);
        float sacc[4][4];
#pragma unroll
        for (int n = 0; n < 4; ++n) sacc[n][0] = sacc[n][1] = sacc[n][2] = sacc[n][3] = 0.f;
        const unsigned brow = page + (unsigned)((tq * 32 + (lane & 7) + 8 * (lane >> 4)) * p.row.pitch + 8 * ((lane >> 3) & 1)) * 2u;
#pragma unroll
        for (int k = 0; k < KPW; ++k) {
            const int ks = kq * KPW + k;
            if (ks < ksteps) {
#pragma unroll
                for (int tp = 0; tp < 2; ++tp) {
                    unsigned b[4];
                    lat_ldsm(b, brow + (unsigned)(tp * 16 * p.row.pitch + 16 * ks) * 2u);
                    lat_mma(sacc[2 * tp], qh[k], b[0], b[1]);
                    lat_mma(sacc[2 * tp], ql[k], b[0], b[1]);
                    lat_mma(sacc[2 * tp + 1], qh[k], b[2], b[3]);
                    lat_mma(sacc[2 * tp + 1], ql[k], b[2], b[3]);
                }
            }
        }
#pragma unroll
        for (int n = 0; n < 4; ++n) {
            float* d = s_sm + (kq * kSplHeads + g) * kSPitch + tq * 32 + n * 8 + 2 * t;
            *reinterpret_cast<float2*>(d) = make_float2(sacc[n][0], sacc[n][1]);
            *reinterpret_cast<float2*>(d + 8 * kSPitch) = make_float2(sacc[n][2], sacc[n][3]);
        }
        __syncthreads();
        if (bad) break;   // uniform: written before the barrier by whoever gave up
        {
            float4 s4 = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
            for (int q = 0; q < 4; ++q) {
                const float4 v = *reinterpret_cast<const float4*>(s_sm + (q * kSplHeads + srow) * kSPitch + scol);
                s4.x += v.x; s4.y += v.y; s4.z += v.z; s4.w += v.w;
            }
            const int key0 = (page0 + split + i * p.splits) * kPage + scol;
            float s[4] = {s4.x, s4.y, s4.z, s4.w};
            float mx = -INFINITY;
#pragma unroll
            for (int e = 0; e < 4; ++e) { s[e] = key0 + e <= pos && key0 + e >= seen0 ? s[e] * p.scale_log2 : -INFINITY; mx = fmaxf(mx, s[e]); }
#pragma unroll
            for (int o = 1; o < 16; o <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float m_new = fmaxf(m_run, mx);       // every page holds at least one row that is seen
            const float corr = exp2f(m_run - m_new);
            float sum = 0.f;
            unsigned hi[2], lo[2];
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const float a = exp2f(s[2 * e] - m_new), b = exp2f(s[2 * e + 1] - m_new);
                sum += a + b;
                const float ah = lat_round(a), bh = lat_round(b);
                hi[e] = lat_pack(ah, bh);
                lo[e] = lat_pack(a - ah, b - bh);
            }
#pragma unroll
            for (int o = 1; o < 16; o <<= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            l_run = l_run * corr + sum;
            m_run = m_new;
            *reinterpret_cast<uint2*>(p_hi + srow * kPPitch + scol) = make_uint2(hi[0], hi[1]);
            *reinterpret_cast<uint2*>(p_lo + srow * kPPitch + scol) = make_uint2(lo[0], lo[1]);
            if ((tid & 15) == 0) corr_s[srow] = corr;
        }
        __syncthreads();
        const float c0 = corr_s[g], c1 = corr_s[g + 8];
#pragma unroll
        for (int j = 0; j < NPW; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) { oacc[j][e][0] *= c0; oacc[j][e][1] *= c0; oacc[j][e][2] *= c1; oacc[j][e][3] *= c1; }
#pragma unroll
        for (int kk = 0; kk < kPage / 16; ++kk) {
            unsigned ah[4], al[4];
            const unsigned pa = (unsigned)((lane & 15) * kPPitch + 16 * kk + 8 * (lane >> 4)) * 2u;
            lat_ldsm(ah, smem_u32(p_hi) + pa);
            lat_ldsm(al, smem_u32(p_lo) + pa);
            const unsigned vrow = page + (unsigned)((16 * kk + (lane & 7) + 8 * ((lane >> 3) & 1)) * p.row.pitch + 8 * (lane >> 4)) * 2u;
#pragma unroll
            for (int j = 0; j < NPW; ++j) {
                const int ct = warp + kSplWarps * j;
                if (ct < n_ct) {
                    unsigned b[4];
                    lat_ldsm_trans(b, vrow + (unsigned)ct * 32u);
                    lat_mma(oacc[j][0], ah, b[0], b[1]);
                    lat_mma(oacc[j][0], al, b[0], b[1]);
                    lat_mma(oacc[j][1], ah, b[2], b[3]);
                    lat_mma(oacc[j][1], al, b[2], b[3]);
                }
            }
        }
        __syncthreads();   // the page's stage is free
        if (tid == 0 && i + 2 < mine) request(i + 2);
    }
    if (bad) {
        // leave only when the copies that may still be under way have landed (bounded)
        if (tid == 0) for (int k = i; k < i + 2 && k < mine; ++k) mbar_wait(&full_bar[k & 1], (unsigned)((k >> 1) & 1));
        return;
    }
    const size_t pw = (size_t)p.row.rp + kPartialTail;
    float* po = p.partial + ((size_t)rl * p.heads * p.splits + split) * pw;
#pragma unroll
    for (int j = 0; j < NPW; ++j) {
        const int ct = warp + kSplWarps * j;
        if (ct < n_ct)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int col = ct * 16 + e * 8 + 2 * t;
                if (h0 + g < p.heads) *reinterpret_cast<float2*>(po + (size_t)(h0 + g) * p.splits * pw + col) = make_float2(oacc[j][e][0], oacc[j][e][1]);
                if (h0 + g + 8 < p.heads) *reinterpret_cast<float2*>(po + (size_t)(h0 + g + 8) * p.splits * pw + col) = make_float2(oacc[j][e][2], oacc[j][e][3]);
            }
    }
    if ((tid & 15) == 0 && h0 + srow < p.heads) {
        float* d = po + (size_t)(h0 + srow) * p.splits * pw + p.row.rp;
        d[0] = m_run;
        d[1] = l_run;
    }
}

// ---- rows one by one: attention with fp32 FMAs (fp32 pool, or a geometry the kernel above does not hold) ---------------
// CTA (row, head), four warps that take the keys in turn; writes one partial (splits == 1).
constexpr int kSimpleWarps = 4;
template <typename T>
__global__ void __launch_bounds__(kSimpleWarps * 32) latent_simple_kernel(const LatentParams p) {
    extern __shared__ __align__(16) float simple_smem[];
    const int qw = p.row.rp + p.row.rotp, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    float* q = simple_smem;                                       // [qw]
    float* acc = simple_smem + qw + (size_t)warp * p.row.rp;      // [warps][rp]
    __shared__ float ms[kSimpleWarps], ls[kSimpleWarps];
    pdl_launch_dependents();
    pdl_wait();
    const int rl = blockIdx.x, h = blockIdx.y, r = batch_row(p, rl), pos = p.row_pos[r], seq = p.row_seq[r];
    for (int i = threadIdx.x; i < qw; i += blockDim.x) q[i] = p.qcat[((size_t)rl * p.heads + h) * qw + i];
    for (int i = lane; i < p.row.rp; i += 32) acc[i] = 0.f;
    __syncthreads();
    float m = -INFINITY, l = 0.f;
    for (int key = first_seen(p, pos) + warp; key <= pos; key += kSimpleWarps) {
        const T* c = cached_row<T>(p, seq, key);
        float s = 0.f;
        for (int i = lane; i < qw; i += 32) s = fmaf(q[i], lat_get(c + i), s);
        for (int o = 16; o > 0; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
        s *= p.scale_log2;
        const float m_new = fmaxf(m, s), corr = exp2f(m - m_new), w = exp2f(s - m_new);
        l = l * corr + w;
        m = m_new;
        for (int i = lane; i < p.row.rp; i += 32) acc[i] = acc[i] * corr + w * lat_get(c + i);
    }
    if (lane == 0) { ms[warp] = m; ls[warp] = l; }
    __syncthreads();
    float top = ms[0];
    for (int w = 1; w < kSimpleWarps; ++w) top = fmaxf(top, ms[w]);
    float total = 0.f;
    for (int w = 0; w < kSimpleWarps; ++w) total += ls[w] * exp2f(ms[w] - top);
    float* po = p.partial + ((size_t)rl * p.heads + h) * ((size_t)p.row.rp + kPartialTail);
    for (int i = threadIdx.x; i < p.row.rp; i += blockDim.x) {
        float v = 0.f;
        for (int w = 0; w < kSimpleWarps; ++w) v += simple_smem[qw + (size_t)w * p.row.rp + i] * exp2f(ms[w] - top);
        po[i] = v;
    }
    if (threadIdx.x == 0) { po[p.row.rp] = top; po[p.row.rp + 1] = total; }
}

// ---- rows one by one: merge, value projection, gate --------------------------------------------------------------------
// A cluster of CTAs per (head, row): each merges its share of the latent columns over the splits and hands it to the others
// through distributed shared memory, then multiplies its share of the head's value rows.
constexpr int kOutThreads = 256, kOutWarps = kOutThreads / 32, kLatMaxSplits = 296, kOutBatch = 4, kOutRows = 2, kOutCluster = 8;
template <typename T>
__global__ void __launch_bounds__(kOutThreads) latent_out_kernel(const LatentParams p) {
    extern __shared__ __align__(16) float out_smem[];   // [rp] merged, then [groups][share] the thread groups' sums
    __shared__ float w_s[kLatMaxSplits];
    const cg::cluster_group cluster = cg::this_cluster();
    auto started = cluster.barrier_arrive();   // waited for before anything is written to another CTA's shared memory
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.x, rl = blockIdx.y, z = blockIdx.z, nz = gridDim.z;
    const int per = (p.vdim + nz - 1) / nz, v0 = z * per, v1 = min(p.vdim, v0 + per);
    // value rows v0 + warp, + 8, ... of this warp, their first 512 columns: not the preceding kernel's business
    const int chunks = p.uv_ld >> 3;
    const __nv_bfloat16* rows = p.uv + (size_t)h * p.vdim * p.uv_ld;
    uint4 wv[kOutRows][2];
#pragma unroll
    for (int j = 0; j < kOutRows; ++j)
#pragma unroll
        for (int q = 0; q < 2; ++q) {
            const int v = v0 + warp + j * kOutWarps, cq = lane + 32 * q;
            wv[j][q] = v < v1 && cq < chunks ? __ldg(reinterpret_cast<const uint4*>(rows + (size_t)v * p.uv_ld) + cq) : make_uint4(0, 0, 0, 0);
        }
    pdl_wait();
    const int r = batch_row(p, rl);
    const int pos = p.row_pos[r], used = min(p.splits, pos / kPage + 1 - first_seen(p, pos) / kPage);
    const float sink = sink_log2(p, h);
    const size_t pw = (size_t)p.row.rp + kPartialTail;
    const float* base = p.partial + ((size_t)rl * p.heads + h) * p.splits * pw;
    if (warp == 0) {
        float top = sink;
        for (int s = lane; s < used; s += 32) top = fmaxf(top, __ldcg(base + s * pw + p.row.rp));
        for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
        float total = 0.f;
        for (int s = lane; s < used; s += 32) {
            const float2 ml = __ldcg(reinterpret_cast<const float2*>(base + s * pw + p.row.rp));
            const float w = exp2f(ml.x - top);
            w_s[s] = w;
            total = fmaf(w, ml.y, total);
        }
        for (int o = 16; o > 0; o >>= 1) total += __shfl_xor_sync(0xffffffffu, total, o);
        const float inv = 1.0f / (total + exp2f(sink - top));
        __syncwarp();
        for (int s = lane; s < used; s += 32) w_s[s] *= inv;
    }
    __syncthreads();
    // this CTA's latent columns, four per thread, the splits dealt to groups of threads
    const int quads = p.row.rp >> 2, share = (quads + nz - 1) / nz, q0 = z * share, nq = max(0, min(share, quads - q0));
    const int cols = min(share, kOutThreads), groups = kOutThreads / cols, g = tid / cols, c = tid - g * cols;
    float4* sums = reinterpret_cast<float4*>(out_smem + p.row.rp);
    for (int c0 = 0; c0 < nq; c0 += cols) {
        if (g < groups && c0 + c < nq) {
            const float* src = base + 4 * (q0 + c0 + c);
            float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll kOutBatch
            for (int s = g; s < used; s += groups) {
                const float4 x = __ldcg(reinterpret_cast<const float4*>(src + s * pw));
                const float w = w_s[s];
                v.x = fmaf(w, x.x, v.x); v.y = fmaf(w, x.y, v.y); v.z = fmaf(w, x.z, v.z); v.w = fmaf(w, x.w, v.w);
            }
            sums[g * share + c0 + c] = v;
        }
    }
    __syncthreads();
    cluster.barrier_wait(std::move(started));
    for (int i = tid; i < nq * 4; i += kOutThreads) {
        float v = 0.f;
        for (int q = 0; q < groups; ++q) v += reinterpret_cast<const float*>(sums)[(size_t)q * share * 4 + i];
        out_smem[q0 * 4 + i] = v;
        for (int o = 1; o < nz; ++o) cluster.map_shared_rank(out_smem, (z + o) % nz)[q0 * 4 + i] = v;
    }
    cluster.sync();
    const float gate = p.gate ? 1.0f / (1.0f + expf(-p.gate[(size_t)r * p.gate_stride + h])) : 1.0f;
    auto dot = [&](const uint4& x, int cq) {
        const float4 a = *reinterpret_cast<const float4*>(out_smem + 8 * cq), b = *reinterpret_cast<const float4*>(out_smem + 8 * cq + 4);
        float acc = lat_lo(x.x) * a.x;
        acc = fmaf(lat_hi(x.x), a.y, acc); acc = fmaf(lat_lo(x.y), a.z, acc); acc = fmaf(lat_hi(x.y), a.w, acc);
        acc = fmaf(lat_lo(x.z), b.x, acc); acc = fmaf(lat_hi(x.z), b.y, acc); acc = fmaf(lat_lo(x.w), b.z, acc);
        return fmaf(lat_hi(x.w), b.w, acc);
    };
    auto finish = [&](int v, float acc) {
        for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (lane == 0) lat_put(static_cast<T*>(p.out) + (size_t)r * p.out_stride + (size_t)h * p.vdim + v, acc * gate);
    };
#pragma unroll
    for (int j = 0; j < kOutRows; ++j) {
        const int v = v0 + warp + j * kOutWarps;
        if (v < v1) {   // uniform across the warp
            float acc = 0.f;
#pragma unroll
            for (int q = 0; q < 2; ++q) if (lane + 32 * q < chunks) acc += dot(wv[j][q], lane + 32 * q);
            for (int cq = lane + 64; cq < chunks; cq += 32) acc += dot(__ldg(reinterpret_cast<const uint4*>(rows + (size_t)v * p.uv_ld) + cq), cq);
            finish(v, acc);
        }
    }
#pragma unroll 1
    for (int v = v0 + warp + kOutRows * kOutWarps; v < v1; v += kOutWarps) {
        float acc = 0.f;
        for (int cq = lane; cq < chunks; cq += 32) acc += dot(__ldg(reinterpret_cast<const uint4*>(rows + (size_t)v * p.uv_ld) + cq), cq);
        finish(v, acc);
    }
}
// CTAs per (head, row): as many as the portable cluster size while the launch stays below four CTAs per SM
int out_cluster(int heads, int rows, int vdim) {
    int nz = kOutCluster;
    while (nz > 1 && ((long long)heads * rows * nz > 4 * 148 || nz > vdim)) nz >>= 1;
    return nz;
}
template <typename T>
cudaError_t launch_out(const LatentLaunch& a, const LatentParams& p, cudaStream_t s) {
    const int nz = out_cluster(a.heads, a.n_short, a.vdim);
    const int share = (a.row.rp / 4 + nz - 1) / nz, cols = std::min(share, kOutThreads), groups = kOutThreads / cols;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(a.heads, a.n_short, nz); cfg.blockDim = dim3(kOutThreads); cfg.stream = s;
    cfg.dynamicSmemBytes = ((size_t)a.row.rp + (size_t)groups * share * 4) * 4;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = nz;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl_enabled() ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, latent_out_kernel<T>, p);
}

// ---- spans: append and rotate ------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(128) latent_append_kernel(const LatentParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int r = batch_row(p, blockIdx.x), lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    if (warp == 0) { append_row<__nv_bfloat16>(p, r, lane); return; }
    const int half = p.rot_dims >> 1, per_head = p.dim + p.row.rot, pos = p.row_pos[r];
    __nv_bfloat16* q = static_cast<__nv_bfloat16*>(p.q) + (size_t)r * p.q_stride + p.dim;
    const int step = rotary_step(p.rot_dims, p.rot_neighbours);
    for (int i = lane; i < half; i += 32) {
        float c, s;
        angle(p, pos, i, c, s);
        for (int h = warp - 1; h < p.heads; h += 3) {
            __nv_bfloat16* x = q + (size_t)h * per_head + rotary_first(i, p.rot_neighbours);
            const float u = __bfloat162float(x[0]), v = __bfloat162float(x[step]);
            x[0] = __float2bfloat16_rn(u * c - v * s);
            x[step] = __float2bfloat16_rn(v * c + u * s);
        }
    }
}

// Cached rows of the spans (from position `lo` on), one after the other: latents [total_ctx][ctx_ld], rotated parts [total_ctx][rot_ld].
__global__ void __launch_bounds__(128) latent_gather_kernel(const LatentParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.x * 4 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    if (row >= p.total_ctx) return;
    int sp = 0;
    while (sp + 1 < p.n_spans && p.spans[sp + 1].ctx0 <= row) ++sp;
    const LatentSpan span = p.spans[sp];
    const __nv_bfloat16* src = cached_row<__nv_bfloat16>(p, span.seq, span.lo + row - span.ctx0);
    for (int i = lane; i < p.ctx_ld / 8; i += 32) reinterpret_cast<uint4*>(p.ctx_latent + (size_t)row * p.ctx_ld)[i] = reinterpret_cast<const uint4*>(src)[i];
    for (int i = lane; i < p.rot_ld / 8; i += 32) reinterpret_cast<uint4*>(p.ctx_rot + (size_t)row * p.rot_ld)[i] = reinterpret_cast<const uint4*>(src + p.row.rp)[i];
}

// ---- spans: tiled causal attention over expanded keys and values --------------------------------------------------------
// CTA (tile of 128 query rows of a span, head), 8 warps of 16 query rows; key tiles of 64 through two shared-memory stages.
constexpr int kPfThreads = 256, kPfKeys = 64;
template <int KQ, int NV>
constexpr size_t latent_prefill_smem() {
    return (size_t)2 * kPfKeys * ((KQ * 16 + 8) + (NV * 16 + 8)) * 2 + (size_t)kLatentQueryTile * (KQ * 16 + 8) * 2;
}
template <int KQ, int NV>   // 16-column steps of query / key rows, 16-column steps of value rows
__global__ void __launch_bounds__(kPfThreads, 1) latent_prefill_kernel(const LatentParams p) {
    constexpr int PK = KQ * 16 + 8, PV = NV * 16 + 8;          // row pitches in entries: odd multiples of 16 bytes
    constexpr int STAGE = kPfKeys * (PK + PV);
    extern __shared__ __align__(16) unsigned char pf_raw[];
    __nv_bfloat16* kv_sm = reinterpret_cast<__nv_bfloat16*>(pf_raw);
    __nv_bfloat16* q_sm = kv_sm + 2 * STAGE;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t = lane & 3, h = blockIdx.y;
    const int dim_p = (p.dim + 15) & ~15;
    // zeros in the padding columns of both stages and of the query tile, written once
    for (int i = tid; i < 2 * STAGE / 8; i += kPfThreads) reinterpret_cast<uint4*>(kv_sm)[i] = make_uint4(0, 0, 0, 0);
    for (int i = tid; i < kLatentQueryTile * PK / 8; i += kPfThreads) reinterpret_cast<uint4*>(q_sm)[i] = make_uint4(0, 0, 0, 0);
    pdl_launch_dependents();
    __syncthreads();
    pdl_wait();
    const int2 tile = p.tiles[blockIdx.x];
    const LatentSpan span = p.spans[tile.x];
    const int q0 = tile.y * kLatentQueryTile, nq = min(kLatentQueryTile, span.count - q0);
    const int first_pos = span.pos0 + q0, last_pos = first_pos + nq - 1;
    const int kt0 = first_seen(p, first_pos) / kPfKeys, n_tiles = last_pos / kPfKeys + 1;   // key tiles the first row sees from, and all
    const int cd = p.dim >> 3, cr = p.row.rot >> 3, cv = p.vdim >> 3;
    // 16-byte chunk tid, tid + 256, ... of a tile as (row, chunk of the row), without divisions in the loop
    const int per_row = cd + cr + cv, r_first = tid / per_row, c_first = tid - r_first * per_row, r_step = kPfThreads / per_row, c_step = kPfThreads - r_step * per_row;
    auto load_tile = [&](int kt, int stage) {
        __nv_bfloat16* ks = kv_sm + stage * STAGE;
        __nv_bfloat16* vs = ks + kPfKeys * PK;
        for (int r = r_first, c = c_first; r < kPfKeys; r += r_step + (c + c_step >= per_row), c += c_step - (c + c_step >= per_row ? per_row : 0)) {
            const size_t row = span.ctx0 + min(kt * kPfKeys + r, last_pos) - span.lo;
            const __nv_bfloat16* src;
            __nv_bfloat16* dst;
            if (c < cd) { src = p.ctx_k + row * ((size_t)p.heads * p.dim) + (size_t)h * p.dim + 8 * c; dst = ks + r * PK + 8 * c; }
            else if (c < cd + cr) { src = p.ctx_rot + row * p.rot_ld + 8 * (c - cd); dst = ks + r * PK + dim_p + 8 * (c - cd); }
            else { src = p.ctx_v + row * ((size_t)p.heads * p.vdim) + (size_t)h * p.vdim + 8 * (c - cd - cr); dst = vs + r * PV + 8 * (c - cd - cr); }
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    {
        const int per_head = p.dim + p.row.rot, per_row = cd + cr;
        for (int i = tid; i < nq * per_row; i += kPfThreads) {
            const int r = i / per_row, c = i - r * per_row;
            const __nv_bfloat16* src = static_cast<const __nv_bfloat16*>(p.q) + (size_t)(span.row0 + q0 + r) * p.q_stride + (size_t)h * per_head + 8 * c;
            __nv_bfloat16* dst = q_sm + r * PK + (c < cd ? 8 * c : dim_p + 8 * (c - cd));
            asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
        }
    }
    load_tile(kt0, kt0 & 1);   // one group with the query rows
    unsigned qa[KQ][4];
    const int pos_a = first_pos + warp * 16 + g, pos_b = pos_a + 8;   // positions of this lane's two rows
    const int warp_first = first_pos + warp * 16, warp_last = min(warp_first + 15, last_pos);
    float m_a = -INFINITY, m_b = -INFINITY, l_a = 0.f, l_b = 0.f;
    float oacc[2 * NV][4];
#pragma unroll
    for (int j = 0; j < 2 * NV; ++j) oacc[j][0] = oacc[j][1] = oacc[j][2] = oacc[j][3] = 0.f;

    const int seen_a = first_seen(p, pos_a), seen_b = first_seen(p, pos_b), warp_seen = first_seen(p, warp_first);
    const int full_from = p.window > 0 ? max(0, warp_last - p.window + 1) : 0;   // first position that no row of the warp has left behind

    for (int kt = kt0; kt < n_tiles; ++kt) {
        if (kt + 1 < n_tiles) load_tile(kt + 1, (kt + 1) & 1);
        else asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        if (kt == kt0) {
#pragma unroll
            for (int k = 0; k < KQ; ++k) lat_ldsm(qa[k], smem_u32(q_sm) + (unsigned)((warp * 16 + (lane & 15)) * PK + 16 * k + 8 * (lane >> 4)) * 2u);
        }
        if (warp_first <= last_pos && kt * kPfKeys <= warp_last && (kt + 1) * kPfKeys > warp_seen) {
            const unsigned kb = smem_u32(kv_sm + (kt & 1) * STAGE), vb = kb + (unsigned)(kPfKeys * PK) * 2u;
            float sacc[8][4];
#pragma unroll
            for (int j = 0; j < 8; ++j) sacc[j][0] = sacc[j][1] = sacc[j][2] = sacc[j][3] = 0.f;
#pragma unroll
            for (int k = 0; k < KQ; ++k)
#pragma unroll
                for (int jp = 0; jp < 4; ++jp) {
                    unsigned b[4];
                    lat_ldsm(b, kb + (unsigned)((jp * 16 + (lane & 7) + 8 * (lane >> 4)) * PK + 16 * k + 8 * ((lane >> 3) & 1)) * 2u);
                    lat_mma(sacc[2 * jp], qa[k], b[0], b[1]);
                    lat_mma(sacc[2 * jp + 1], qa[k], b[2], b[3]);
                }
            const bool edge = (kt + 1) * kPfKeys - 1 > warp_first || kt * kPfKeys < full_from;   // some row does not see the whole tile
            float mx_a = -INFINITY, mx_b = -INFINITY;
#pragma unroll
            for (int j = 0; j < 8; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int key = kt * kPfKeys + 8 * j + 2 * t + e;
                    const float a = !edge || (key <= pos_a && key >= seen_a) ? sacc[j][e] * p.scale_log2 : -INFINITY;
                    const float b = !edge || (key <= pos_b && key >= seen_b) ? sacc[j][2 + e] * p.scale_log2 : -INFINITY;
                    sacc[j][e] = a; sacc[j][2 + e] = b;
                    mx_a = fmaxf(mx_a, a); mx_b = fmaxf(mx_b, b);
                }
#pragma unroll
            for (int o = 1; o < 4; o <<= 1) { mx_a = fmaxf(mx_a, __shfl_xor_sync(0xffffffffu, mx_a, o)); mx_b = fmaxf(mx_b, __shfl_xor_sync(0xffffffffu, mx_b, o)); }
            const float mn_a = fmaxf(m_a, mx_a), mn_b = fmaxf(m_b, mx_b);
            m_a = m_a == -INFINITY ? mn_a : m_a; m_b = m_b == -INFINITY ? mn_b : m_b;   // (nothing seen so far: sums are zero)
            // a row whose window starts in a later tile sees nothing of this one: its weights must come out zero
            const float ra = mn_a == -INFINITY ? 0.f : mn_a, rb = mn_b == -INFINITY ? 0.f : mn_b;
            const float ca = mn_a == -INFINITY ? 1.f : exp2f(m_a - mn_a), cb = mn_b == -INFINITY ? 1.f : exp2f(m_b - mn_b);
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
                for (int e = 0; e < 4; ++e) {   // (row g, keys 0-7), (row g + 8, keys 0-7), (row g, keys 8-15), (row g + 8, keys 8-15)
                    const float x = sacc[2 * kk + (e >> 1)][(e & 1) * 2], y = sacc[2 * kk + (e >> 1)][(e & 1) * 2 + 1];
                    const float xh = lat_round(x), yh = lat_round(y);
                    ah[e] = lat_pack(xh, yh);
                    al[e] = lat_pack(x - xh, y - yh);
                }
#pragma unroll
                for (int j = 0; j < NV; ++j) {
                    unsigned b[4];
                    lat_ldsm_trans(b, vb + (unsigned)((16 * kk + (lane & 7) + 8 * ((lane >> 3) & 1)) * PV + 16 * j + 8 * (lane >> 4)) * 2u);
                    lat_mma(oacc[2 * j], ah, b[0], b[1]);
                    lat_mma(oacc[2 * j], al, b[0], b[1]);
                    lat_mma(oacc[2 * j + 1], ah, b[2], b[3]);
                    lat_mma(oacc[2 * j + 1], al, b[2], b[3]);
                }
            }
        }
        __syncthreads();
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int o = 1; o < 4; o <<= 1) { l_a += __shfl_xor_sync(0xffffffffu, l_a, o); l_b += __shfl_xor_sync(0xffffffffu, l_b, o); }
    const float sink = sink_log2(p, h);
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int rr = warp * 16 + g + 8 * half;
        if (rr >= nq) continue;
        const int row = span.row0 + q0 + rr;
        const float gate = p.gate ? 1.0f / (1.0f + expf(-p.gate[(size_t)row * p.gate_stride + h])) : 1.0f;
        // (every row sees its own key, so its maximum is finite)
        const float m = half ? m_b : m_a, top = fmaxf(m, sink), own = exp2f(m - top);
        const float f = gate * own / ((half ? l_b : l_a) * own + exp2f(sink - top));
        __nv_bfloat16* o = static_cast<__nv_bfloat16*>(p.out) + (size_t)row * p.out_stride + (size_t)h * p.vdim;
#pragma unroll
        for (int j = 0; j < 2 * NV; ++j) {
            const int c = 8 * j + 2 * t;
            if (c < p.vdim) *reinterpret_cast<unsigned*>(o + c) = lat_pack(oacc[j][2 * half] * f, oacc[j][2 * half + 1] * f);
        }
    }
}

LatentParams latent_params(const LatentLaunch& a) {
    LatentParams p{};
    p.row = a.row; p.heads = a.heads; p.dim = a.dim; p.vdim = a.vdim; p.rot_dims = a.rot_dims; p.rot_neighbours = a.rot_neighbours;
    p.window = a.window; p.sink = a.sink;
    p.scale_log2 = a.scale * kLog2e; p.eps = a.eps; p.weight_bias = a.weight_bias; p.magnitude = a.magnitude; p.inv_freq = a.inv_freq;
    p.q = a.q; p.q_stride = a.q_stride; p.kv = a.kv; p.kv_stride = a.kv_stride; p.gate = a.gate; p.gate_stride = a.gate_stride;
    p.norm_w = a.norm_w; p.uk = a.uk->data; p.uk_ld = a.uk->ld; p.uv = a.uv->data; p.uv_ld = a.uv->ld;
    p.pool = a.pool; p.page_table = a.page_table; p.pages_per_seq = a.pages_per_seq; p.row_seq = a.row_seq; p.row_pos = a.row_pos;
    p.out = a.out; p.out_stride = a.out_stride; p.qcat = a.qcat; p.partial = a.partial; p.status = a.status; p.splits = 1;
    return p;
}

constexpr int kSplKpwSmall = 3, kSplNpwSmall = 2, kSplKpw = 9, kSplNpw = 4;
bool split_small(const LatentRow& r) { return (r.rp + r.rotp) / 16 <= 4 * kSplKpwSmall && r.rp / 16 <= kSplWarps * kSplNpwSmall; }
bool split_fits(const LatentRow& r) { return (r.rp + r.rotp) / 16 <= 4 * kSplKpw && r.rp / 16 <= kSplWarps * kSplNpw; }
size_t split_smem_bytes(const LatentRow& r) { return (size_t)2 * kPage * r.pitch * 2 + (size_t)4 * kSplHeads * kSPitch * 4 + (size_t)2 * kSplHeads * kPPitch * 2; }
constexpr size_t kSimpleMaxSmem = 200 * 1024;
size_t simple_smem_bytes(const LatentRow& r) { return ((size_t)r.rp + r.rotp + (size_t)kSimpleWarps * r.rp) * 4; }

template <typename T>
int launch_short(const LatentLaunch& a, cudaStream_t s, int* launches) {
    LatentParams p = latent_params(a);
    p.n_rows = a.n_short; p.rows = a.short_rows; p.splits = a.splits;
    cudaError_t e;
    const bool mma = !a.f32 && split_fits(a.row);
    p.frag = mma ? 1 : 0;
    if (!mma) p.splits = 1;
    if (!a.only_attention) {
        e = a.n_short == 1 ? launch_query<T, 1>(a, p, s) : launch_query<T, 4>(a, p, s);
        if (e != cudaSuccess) return cuda_fail(e, "latent query launch");
        *launches += 1;
    }
    if (mma) {
        const dim3 grid(p.splits, (a.heads + kSplHeads - 1) / kSplHeads, a.n_short);
        e = split_small(a.row) ? launch_k(latent_split_kernel<kSplKpwSmall, kSplNpwSmall>, grid, dim3(kSplThreads), split_smem_bytes(a.row), s, p)
                               : launch_k(latent_split_kernel<kSplKpw, kSplNpw>, grid, dim3(kSplThreads), split_smem_bytes(a.row), s, p);
    } else {
        e = launch_k(latent_simple_kernel<T>, dim3(a.n_short, a.heads), dim3(kSimpleWarps * 32), simple_smem_bytes(a.row), s, p);
    }
    if (e != cudaSuccess) return cuda_fail(e, "latent attention launch");
    *launches += 1;
    if (!a.only_attention) {
        e = launch_out<T>(a, p, s);
        if (e != cudaSuccess) return cuda_fail(e, "latent output launch");
        *launches += 1;
    }
    return SWLM_OK;
}

// expanded scratch: latents, rotated parts, keys, values of total_ctx rows
struct ExpandLayout { size_t latent, rot, k, v, total; int ctx_ld, rot_ld; };
ExpandLayout expand_layout(const LatentRow& r, int heads, int dim, int vdim, int ctx) {
    ExpandLayout l;
    auto up = [](size_t x) { return (x + 255) / 256 * 256; };
    l.ctx_ld = (r.rank + 7) / 8 * 8; l.rot_ld = r.rot;
    l.latent = 0;
    l.rot = l.latent + up((size_t)ctx * l.ctx_ld * 2);
    l.k = l.rot + up((size_t)ctx * l.rot_ld * 2);
    l.v = l.k + up((size_t)ctx * heads * dim * 2);
    l.total = l.v + up((size_t)ctx * heads * vdim * 2);
    return l;
}
enum { PF_SMALL, PF_MEDIUM, PF_LARGE, PF_NONE };
int prefill_form(int dim, int rot, int vdim) {
    const int kq = (dim + 15) / 16 + (rot + 15) / 16, nv = (vdim + 15) / 16;
    return kq <= 4 && nv <= 5 ? PF_SMALL : kq <= 8 && nv <= 8 ? PF_MEDIUM : kq <= 12 && nv <= 8 ? PF_LARGE : PF_NONE;
}

int launch_long(const LatentLaunch& a, cudaStream_t s, int* launches) {
    LatentParams p = latent_params(a);
    const ExpandLayout l = expand_layout(a.row, a.heads, a.dim, a.vdim, a.total_ctx);
    p.n_rows = a.n_long; p.rows = a.long_rows; p.spans = a.spans; p.tiles = a.tiles; p.n_spans = a.n_spans; p.total_ctx = a.total_ctx;
    p.ctx_latent = reinterpret_cast<__nv_bfloat16*>(a.expand + l.latent); p.ctx_ld = l.ctx_ld;
    p.ctx_rot = reinterpret_cast<__nv_bfloat16*>(a.expand + l.rot); p.rot_ld = l.rot_ld;
    p.ctx_k = reinterpret_cast<__nv_bfloat16*>(a.expand + l.k);
    p.ctx_v = reinterpret_cast<__nv_bfloat16*>(a.expand + l.v);
    cudaError_t e;
    if (!a.only_attention) {
        e = launch_k(latent_append_kernel, dim3(a.n_long), dim3(128), 0, s, p);
        if (e != cudaSuccess) return cuda_fail(e, "latent append launch");
        e = launch_k(latent_gather_kernel, dim3((a.total_ctx + 3) / 4), dim3(128), 0, s, p);
        if (e != cudaSuccess) return cuda_fail(e, "latent gather launch");
        ProductLaunch x;
        x.w = a.ukv; x.m = a.total_ctx; x.x = p.ctx_latent; x.x_stride = l.ctx_ld;
        x.out.count = 2;
        x.out.end[0] = a.heads * a.dim; x.out.end[1] = x.out.end[2] = x.out.end[3] = a.ukv->n;
        x.out.y[0] = a.expand + l.k; x.out.stride[0] = a.heads * a.dim;
        x.out.y[1] = a.expand + l.v; x.out.stride[1] = a.heads * a.vdim;
        x.part = a.part; x.part_floats = a.part_floats; x.status = a.status;
        const int rc = launch_product(x, s);
        if (rc) return rc;
        *launches += 2 + product_launch_count(x);
    }
    const dim3 grid(a.n_tiles, a.heads);
    switch (prefill_form(a.dim, a.row.rot, a.vdim)) {
    case PF_SMALL: e = launch_k(latent_prefill_kernel<4, 5>, grid, dim3(kPfThreads), latent_prefill_smem<4, 5>(), s, p); break;
    case PF_MEDIUM: e = launch_k(latent_prefill_kernel<8, 8>, grid, dim3(kPfThreads), latent_prefill_smem<8, 8>(), s, p); break;
    default: e = launch_k(latent_prefill_kernel<12, 8>, grid, dim3(kPfThreads), latent_prefill_smem<12, 8>(), s, p); break;
    }
    if (e != cudaSuccess) return cuda_fail(e, "latent prompt attention launch");
    *launches += 1;
    return SWLM_OK;
}

}  // namespace

LatentRow latent_row(int rank, int rot, bool f32) {
    LatentRow r;
    r.rank = rank; r.rot = rot;
    r.rp = (rank + 15) / 16 * 16; r.rotp = (rot + 15) / 16 * 16;
    r.pitch = r.rp + r.rotp + (f32 ? 0 : 8);
    return r;
}

int latent_init() {
    SWLM_CUDA(cudaFuncSetAttribute(latent_split_kernel<kSplKpwSmall, kSplNpwSmall>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    SWLM_CUDA(cudaFuncSetAttribute(latent_split_kernel<kSplKpw, kSplNpw>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    SWLM_CUDA(cudaFuncSetAttribute(latent_simple_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSimpleMaxSmem));
    SWLM_CUDA(cudaFuncSetAttribute(latent_simple_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSimpleMaxSmem));
    SWLM_CUDA(cudaFuncSetAttribute(latent_query_kernel<float, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    SWLM_CUDA(cudaFuncSetAttribute(latent_query_kernel<float, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    SWLM_CUDA(cudaFuncSetAttribute(latent_query_kernel<__nv_bfloat16, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    SWLM_CUDA(cudaFuncSetAttribute(latent_query_kernel<__nv_bfloat16, 4>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    SWLM_CUDA(cudaFuncSetAttribute(latent_out_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024));
    SWLM_CUDA(cudaFuncSetAttribute(latent_out_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 100 * 1024));
    SWLM_CUDA(cudaFuncSetAttribute(latent_prefill_kernel<4, 5>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)latent_prefill_smem<4, 5>()));
    SWLM_CUDA(cudaFuncSetAttribute(latent_prefill_kernel<8, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)latent_prefill_smem<8, 8>()));
    SWLM_CUDA(cudaFuncSetAttribute(latent_prefill_kernel<12, 8>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)latent_prefill_smem<12, 8>()));
    return SWLM_OK;
}

// CTAs of the attention kernel fill the GPU once; no more splits than a row can see pages.
int latent_pick_splits(int rows, int heads, int max_pages, int window) {
    if (window > 0) max_pages = std::min(max_pages, (window + kPage - 2) / kPage + 1);
    const int per_split = rows * ((heads + kSplHeads - 1) / kSplHeads);
    return std::max(1, std::min(std::min(148 / std::max(1, per_split), max_pages), kLatMaxSplits));
}
size_t latent_qcat_floats(const LatentRow& r, int heads) { return (size_t)(heads + 15) / 16 * 16 * (r.rp + r.rotp); }
size_t latent_partial_floats(const LatentRow& r, int heads) { return (size_t)heads * (r.rp + kPartialTail); }
size_t latent_expand_bytes(const LatentRow& r, int heads, int dim, int vdim, int total_ctx) { return expand_layout(r, heads, dim, vdim, total_ctx).total; }
bool latent_expands(const LatentRow& r, int dim, int vdim, bool f32) {
    return !f32 && !((dim | vdim | r.rot | r.rank) & 7) && prefill_form(dim, r.rot, vdim) != PF_NONE;
}

int launch_latent(const LatentLaunch& a, cudaStream_t s, int* launches) {
    int rc = SWLM_OK;
    if (a.n_short > 0) rc = a.f32 ? launch_short<float>(a, s, launches) : launch_short<__nv_bfloat16>(a, s, launches);
    if (!rc && a.n_long > 0) rc = launch_long(a, s, launches);
    return rc;
}

}  // namespace swlm
