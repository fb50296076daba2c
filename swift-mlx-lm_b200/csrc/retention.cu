// Retention: linear attention with a fixed decay per head over an fp32 state per sequence and head, a norm of every head's read-out
// and a SiLU gate.
//
//   S_t = decay S_(t-1) + (scale k_t) v_t^T,  o_t = S_t^T q_t
//
// Three ways through it:
//   * a single token of a sequence (decode steps): retention_step_kernel does all of it in one launch, a cluster of CTAs per head
//     that each own 32 columns of the state; the state is requested before the preceding kernel has finished.
//   * portions, bf16: retention_chunk_kernel takes 64 tokens at a time on tensor cores, a CTA per 32 columns of a head's state.
//     With S the state in front of a chunk of n tokens,
//       o_t = decay^(t+1) S^T q_t + sum_{s <= t} decay^(t-s) scale (q_t . k_s) v_s
//       S'  = decay^n S + sum_s k_s (decay^(n-1-s) scale v_s)^T
//     q, k and v enter as they are; every fp32 factor (the state, the weighted scores, the decayed values) enters as a bf16
//     hi + lo pair, the sums are fp32 and the state itself stays fp32.
//   * anything else (fp32 plans, sizes beyond those): retention_walk_kernel, token by token.
// The read-outs of portions are normed and gated by retention_gate_kernel.
#include <cooperative_groups.h>

#include <algorithm>
#include <utility>

#include "swlm_internal.h"
#include "tc_device.cuh"

namespace cg = cooperative_groups;

namespace swlm {
namespace {

constexpr int kRetCols = 32, kRetWarps = 8, kRetThreads = kRetWarps * 32, kRetCluster = 8;
constexpr int kRetChunk = 64;

struct RetentionParams {
    int heads, dim, vdim;
    float eps, scale, out_scale;
    const float* decay;
    const void* qkv; int qkv_stride;
    const void* gate; int gate_stride;
    float* state;
    const int32_t* row_seq; const int32_t* row_pos;
    void* out; int out_stride;
    const int32_t* single_rows;
    const RowRun* runs; const int32_t* block_run;   // runs == null: every single row is a run of one token
    float* o;                                       // [row][heads][vdim]
};

__device__ __forceinline__ float rn_get(const float* p) { return *p; }
__device__ __forceinline__ float rn_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void rn_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void rn_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ float rn_silu(float x) { return x / (1.0f + expf(-x)); }
__device__ __forceinline__ float rn_sum(float v) {
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
__device__ __forceinline__ unsigned rn_pack(float a, float b) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
    return *reinterpret_cast<const unsigned*>(&v);
}
__device__ __forceinline__ float rn_round(float v) { return __bfloat162float(__float2bfloat16_rn(v)); }
__device__ __forceinline__ void rn_mma(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void rn_ldsm(unsigned (&r)[4], const __nv_bfloat16* at) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(at)) : "memory");
}
__device__ __forceinline__ void rn_ldsm_trans(unsigned (&r)[4], const __nv_bfloat16* at) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(smem_u32(at)) : "memory");
}
// decay^n; log2_decay may be -inf
__device__ __forceinline__ float rn_power(float log2_decay, int n) { return n == 0 ? 1.0f : exp2f(log2_decay * (float)n); }

__device__ __forceinline__ RowRun rn_run(const RetentionParams& p, int i) {
    if (p.runs) return p.runs[i];
    const int row = p.single_rows ? p.single_rows[i] : i;
    return RowRun{row, 1, p.row_pos[row], p.row_seq[row], i};
}

// ---- single tokens ----------------------------------------------------------------------------------------------------
// Cluster of CTAs per (head, row), 32 state columns each: warp w holds key channels w, w + 8, ... of the CTA's columns, lane =
// column. Nothing of this layer's state is touched by the kernels in front of this one, so it is read ahead of them.
template <typename T, int R>
__global__ void __launch_bounds__(kRetThreads, R <= 16 ? 3 : 2) retention_step_kernel(const RetentionParams p) {
    extern __shared__ __align__(16) float step_smem[];   // q [dim], scale * k [dim]
    __shared__ float part[kRetWarps][kRetCols], ssq[kRetCluster];
    const cg::cluster_group cluster = cg::this_cluster();
    auto started = cluster.barrier_arrive();   // waited for before anything is written to another CTA's shared memory
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, vb = blockIdx.x, h = blockIdx.y, dim = p.dim, vdim = p.vdim;
    const int row = p.single_rows ? p.single_rows[blockIdx.z] : blockIdx.z, pos = p.row_pos[row], seq = p.row_seq[row];
    const int col = vb * kRetCols + lane;
    const bool live = col < vdim;
    float* st = p.state + ((size_t)seq * p.heads + h) * dim * vdim + col;
    float S[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = warp + kRetWarps * i;
        S[i] = live && pos > 0 && d < dim ? st[(size_t)d * vdim] : 0.f;
    }
    const float decay = p.decay[h];
    pdl_wait();
    const T* base = static_cast<const T*>(p.qkv) + (size_t)row * p.qkv_stride;
    const float v = live ? rn_get(base + (size_t)2 * p.heads * dim + (size_t)h * vdim + col) : 0.f;
    const float gate = live && warp == 0 ? rn_silu(rn_get(static_cast<const T*>(p.gate) + (size_t)row * p.gate_stride + (size_t)h * vdim + col)) : 0.f;
    for (int i = tid; i < 2 * dim; i += kRetThreads) {
        const bool is_k = i >= dim;
        const int d = is_k ? i - dim : i;
        step_smem[i] = rn_get(base + (size_t)(is_k ? p.heads : 0) * dim + (size_t)h * dim + d) * (is_k ? p.scale : 1.0f);
    }
    __syncthreads();
    float a = 0.f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = warp + kRetWarps * i;
        if (d < dim) {
            S[i] = fmaf(decay, S[i], step_smem[dim + d] * v);
            a = fmaf(S[i], step_smem[d], a);
            if (live) st[(size_t)d * vdim] = S[i];
        }
    }
    part[warp][lane] = a;
    __syncthreads();
    float o = 0.f;
#pragma unroll
    for (int w = 0; w < kRetWarps; ++w) o += part[w][lane];
    const int nz = gridDim.x;
    cluster.barrier_wait(std::move(started));
    if (warp == 0) {
        const float ss = rn_sum(o * o);
        if (lane < nz) cluster.map_shared_rank(ssq, lane)[vb] = ss;
    }
    cluster.sync();
    if (warp == 0 && live) {
        float ss = 0.f;
        for (int i = 0; i < nz; ++i) ss += ssq[i];
        rn_put(static_cast<T*>(p.out) + (size_t)row * p.out_stride + (size_t)h * vdim + col, o / sqrtf(ss / (float)vdim + p.eps) * gate * p.out_scale);
    }
}

// ---- token by token ---------------------------------------------------------------------------------------------------
// CTA (32 columns, head, run), the state in registers (R channels per warp and lane) or, with R = 0, in memory.
template <typename T, int R>
__global__ void __launch_bounds__(kRetThreads) retention_walk_kernel(const RetentionParams p) {
    extern __shared__ __align__(16) float walk_smem[];   // two stages of q [dim], scale * k [dim]
    __shared__ float part[2][kRetWarps][kRetCols];
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, h = blockIdx.y, dim = p.dim, vdim = p.vdim, col = blockIdx.x * kRetCols + lane;
    const RowRun run = rn_run(p, blockIdx.z);
    const bool live = col < vdim;
    const float decay = p.decay[h];
    float* st = p.state + ((size_t)run.seq * p.heads + h) * dim * vdim + col;
    float S[R > 0 ? R : 1];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = warp + kRetWarps * i;
        S[i] = live && run.pos0 > 0 && d < dim ? st[(size_t)d * vdim] : 0.f;
    }
    for (int t = 0; t < run.count; ++t) {
        const T* base = static_cast<const T*>(p.qkv) + (size_t)(run.row0 + t) * p.qkv_stride;
        float* q = walk_smem + (size_t)(t & 1) * 2 * dim;
        float* k = q + dim;
        for (int i = tid; i < 2 * dim; i += kRetThreads) {
            const bool is_k = i >= dim;
            const int d = is_k ? i - dim : i;
            q[i] = rn_get(base + (size_t)(is_k ? p.heads : 0) * dim + (size_t)h * dim + d) * (is_k ? p.scale : 1.0f);
        }
        const float v = live ? rn_get(base + (size_t)2 * p.heads * dim + (size_t)h * vdim + col) : 0.f;
        __syncthreads();
        float a = 0.f;
        if constexpr (R > 0) {
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int d = warp + kRetWarps * i;
                if (d < dim) { S[i] = fmaf(decay, S[i], k[d] * v); a = fmaf(S[i], q[d], a); }
            }
        } else if (live) {
            for (int d = warp; d < dim; d += kRetWarps) {
                const float s = fmaf(decay, run.pos0 + t > 0 ? st[(size_t)d * vdim] : 0.f, k[d] * v);
                st[(size_t)d * vdim] = s;
                a = fmaf(s, q[d], a);
            }
        }
        part[t & 1][warp][lane] = a;
        __syncthreads();
        if (warp == 0 && live) {
            float o = 0.f;
#pragma unroll
            for (int w = 0; w < kRetWarps; ++w) o += part[t & 1][w][lane];
            p.o[((size_t)(run.row0 + t) * p.heads + h) * vdim + col] = o;
        }
    }
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = warp + kRetWarps * i;
        if (live && d < dim) st[(size_t)d * vdim] = S[i];
    }
}

// ---- portions on tensor cores -----------------------------------------------------------------------------------------
// CTA (32 columns, head, run), eight warps, chunks of 64 tokens through two stages. Warps 0 .. 3: scores and their products with
// the values for 16 tokens each; warps 4 .. 7: the same tokens' products with the state; then all warps update the state, 16 MT
// key channels each, kept in the accumulators.
constexpr int kRetVPitch = kRetCols + 8, kRetOPitch = kRetCols + 4;
template <int MT> __host__ __device__ constexpr int ret_pitch() { return MT * 128 + 8; }   // entries of a staged q or k row
template <int MT> constexpr size_t ret_smem() {
    return (size_t)2 * 2 * kRetChunk * ret_pitch<MT>() * 2 + (size_t)2 * kRetChunk * kRetVPitch * 2 + (size_t)2 * kRetChunk * kRetVPitch * 2 +
           (size_t)2 * MT * 128 * kRetVPitch * 2 + (size_t)kRetChunk * kRetOPitch * 4;
}
template <int MT>
__global__ void __launch_bounds__(kRetThreads, 1) retention_chunk_kernel(const RetentionParams p) {
    constexpr int PITCH = ret_pitch<MT>(), QK = kRetChunk * PITCH, VS = kRetChunk * kRetVPitch, SS = MT * 128 * kRetVPitch, KS = MT * 8;
    extern __shared__ __align__(128) unsigned char ret_raw[];
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(ret_raw);   // [2][64][PITCH]
    __nv_bfloat16* ks = qs + 2 * QK;
    __nv_bfloat16* vs = ks + 2 * QK;                                 // [2][64][kRetVPitch]
    __nv_bfloat16* dv = vs + 2 * VS;                                 // decayed values, hi then lo
    __nv_bfloat16* sb = dv + 2 * VS;                                 // state, hi then lo: [MT * 128][kRetVPitch]
    float* os = reinterpret_cast<float*>(sb + 2 * SS);               // [64][kRetOPitch] products with the state
    __shared__ float pw[kRetChunk + 1];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g = lane >> 2, t4 = lane & 3;
    const int h = blockIdx.y, c0 = blockIdx.x * kRetCols, dim = p.dim, vdim = p.vdim, nv = min(kRetCols, vdim - c0);
    for (int i = tid; i < (4 * QK + 2 * VS) / 8; i += kRetThreads) reinterpret_cast<uint4*>(qs)[i] = make_uint4(0, 0, 0, 0);   // columns that no copy writes
    const float decay = p.decay[h], log2_decay = log2f(decay);
    if (tid <= kRetChunk) pw[tid] = tid == 1 ? decay : rn_power(log2_decay, tid);
    pdl_launch_dependents();
    __syncthreads();
    pdl_wait();
    const RowRun run = rn_run(p, blockIdx.z);
    const int chunks = (run.count + kRetChunk - 1) / kRetChunk;
    const int cd = dim >> 3, cv = nv >> 3, per_row = 2 * cd + cv;
    const __nv_bfloat16* base = static_cast<const __nv_bfloat16*>(p.qkv) + (size_t)run.row0 * p.qkv_stride;
    const size_t k_at = (size_t)p.heads * dim + (size_t)h * dim, v_at = (size_t)2 * p.heads * dim + (size_t)h * vdim + c0;
    // 16-byte piece tid, tid + 256, ... of a chunk as (row, piece of the row), without divisions in the loop
    const int r_first = tid / per_row, c_first = tid - r_first * per_row, r_step = kRetThreads / per_row, c_step = kRetThreads - r_step * per_row;
    auto load = [&](int b) {
        const int st = b & 1, n = min(kRetChunk, run.count - b * kRetChunk);
        for (int r = r_first, c = c_first; r < kRetChunk; r += r_step + (c + c_step >= per_row), c += c_step - (c + c_step >= per_row ? per_row : 0)) {
            __nv_bfloat16* dst = c < cd ? qs + st * QK + r * PITCH + 8 * c : c < 2 * cd ? ks + st * QK + r * PITCH + 8 * (c - cd) : vs + st * VS + r * kRetVPitch + 8 * (c - 2 * cd);
            if (r < n) {
                const __nv_bfloat16* src = base + (size_t)(b * kRetChunk + r) * p.qkv_stride + (c < cd ? (size_t)h * dim + 8 * c : c < 2 * cd ? k_at + 8 * (c - cd) : v_at + 8 * (c - 2 * cd));
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(dst)), "l"(src) : "memory");
            } else *reinterpret_cast<uint4*>(dst) = make_uint4(0, 0, 0, 0);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    load(0);
    // state rows 16 (warp + 8 m) + g and + 8, columns 8 j + 2 t4 (+ 1)
    float* st = p.state + ((size_t)run.seq * p.heads + h) * dim * vdim + c0;
    float S[MT][4][4];
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int d = 16 * (warp + 8 * m) + g + 8 * e, c = 8 * j + 2 * t4;
                const float2 x = run.pos0 > 0 && d < dim && c < nv ? *reinterpret_cast<const float2*>(st + (size_t)d * vdim + c) : make_float2(0.f, 0.f);
                S[m][j][2 * e] = x.x; S[m][j][2 * e + 1] = x.y;
            }
    auto publish = [&] {   // the state as hi + lo
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const float x = S[m][j][2 * e], y = S[m][j][2 * e + 1], xh = rn_round(x), yh = rn_round(y);
                    const int at = (16 * (warp + 8 * m) + g + 8 * e) * kRetVPitch + 8 * j + 2 * t4;
                    *reinterpret_cast<unsigned*>(sb + at) = rn_pack(xh, yh);
                    *reinterpret_cast<unsigned*>(sb + SS + at) = rn_pack(x - xh, y - yh);
                }
    };
    publish();
    const int ksteps = (dim + 15) >> 4;
    for (int b = 0; b < chunks; ++b) {
        const int n = min(kRetChunk, run.count - b * kRetChunk);
        const __nv_bfloat16 *q = qs + (b & 1) * QK, *k = ks + (b & 1) * QK, *v = vs + (b & 1) * VS;
        if (b + 1 < chunks) load(b + 1);
        else asm volatile("cp.async.commit_group;" ::: "memory");
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();   // the chunk is here, the state is published
        // decayed values
        for (int i = tid; i < kRetChunk * (kRetCols / 2); i += kRetThreads) {
            const int s = i / (kRetCols / 2), c = 2 * (i % (kRetCols / 2));
            const float f = s < n ? pw[n - 1 - s] * p.scale : 0.f;
            const float x = f * __bfloat162float(v[s * kRetVPitch + c]), y = f * __bfloat162float(v[s * kRetVPitch + c + 1]);
            const float xh = rn_round(x), yh = rn_round(y);
            *reinterpret_cast<unsigned*>(dv + s * kRetVPitch + c) = rn_pack(xh, yh);
            *reinterpret_cast<unsigned*>(dv + VS + s * kRetVPitch + c) = rn_pack(x - xh, y - yh);
        }
        const int mt = warp & 3;   // tokens 16 mt .. 16 mt + 15 of the chunk
        float oacc[4][4];
#pragma unroll
        for (int j = 0; j < 4; ++j) oacc[j][0] = oacc[j][1] = oacc[j][2] = oacc[j][3] = 0.f;
        if (warp < 4) {
            float sacc[8][4];
#pragma unroll
            for (int j = 0; j < 8; ++j) sacc[j][0] = sacc[j][1] = sacc[j][2] = sacc[j][3] = 0.f;
#pragma unroll
            for (int kk = 0; kk < KS; ++kk)
                if (kk < ksteps) {
                    unsigned a[4];
                    rn_ldsm(a, q + (16 * mt + (lane & 15)) * PITCH + 16 * kk + 8 * (lane >> 4));
#pragma unroll
                    for (int jp = 0; jp < 4; ++jp)
                        if (jp <= mt) {
                            unsigned bf[4];
                            rn_ldsm(bf, k + (jp * 16 + (lane & 7) + 8 * (lane >> 4)) * PITCH + 16 * kk + 8 * ((lane >> 3) & 1));
                            rn_mma(sacc[2 * jp], a, bf[0], bf[1]);
                            rn_mma(sacc[2 * jp + 1], a, bf[2], bf[3]);
                        }
                }
#pragma unroll
            for (int jp = 0; jp < 4; ++jp)
                if (jp <= mt) {
                    unsigned ah[4], al[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {   // (row g, keys 0-7), (row g + 8, keys 0-7), (row g, keys 8-15), (row g + 8, keys 8-15)
                        const int tok = 16 * mt + g + 8 * (e & 1), s = 16 * jp + 8 * (e >> 1) + 2 * t4;
                        const float x = s <= tok ? sacc[2 * jp + (e >> 1)][(e & 1) * 2] * pw[tok - s] * p.scale : 0.f;
                        const float y = s + 1 <= tok ? sacc[2 * jp + (e >> 1)][(e & 1) * 2 + 1] * pw[tok - s - 1] * p.scale : 0.f;
                        const float xh = rn_round(x), yh = rn_round(y);
                        ah[e] = rn_pack(xh, yh);
                        al[e] = rn_pack(x - xh, y - yh);
                    }
#pragma unroll
                    for (int j = 0; j < 2; ++j) {
                        unsigned bf[4];
                        rn_ldsm_trans(bf, v + (16 * jp + (lane & 7) + 8 * ((lane >> 3) & 1)) * kRetVPitch + 16 * j + 8 * (lane >> 4));
                        rn_mma(oacc[2 * j], ah, bf[0], bf[1]);
                        rn_mma(oacc[2 * j], al, bf[0], bf[1]);
                        rn_mma(oacc[2 * j + 1], ah, bf[2], bf[3]);
                        rn_mma(oacc[2 * j + 1], al, bf[2], bf[3]);
                    }
                }
        } else {
#pragma unroll
            for (int kk = 0; kk < KS; ++kk)
                if (kk < ksteps) {
                    unsigned a[4];
                    rn_ldsm(a, q + (16 * mt + (lane & 15)) * PITCH + 16 * kk + 8 * (lane >> 4));
#pragma unroll
                    for (int j = 0; j < 2; ++j)
#pragma unroll
                        for (int half = 0; half < 2; ++half) {
                            unsigned bf[4];
                            rn_ldsm_trans(bf, sb + half * SS + (16 * kk + (lane & 7) + 8 * ((lane >> 3) & 1)) * kRetVPitch + 16 * j + 8 * (lane >> 4));
                            rn_mma(oacc[2 * j], a, bf[0], bf[1]);
                            rn_mma(oacc[2 * j + 1], a, bf[2], bf[3]);
                        }
                }
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int tok = 16 * mt + g + 8 * e;
                    const float f = pw[tok + 1];
                    *reinterpret_cast<float2*>(os + tok * kRetOPitch + 8 * j + 2 * t4) = make_float2(oacc[j][2 * e] * f, oacc[j][2 * e + 1] * f);
                }
        }
        __syncthreads();   // decayed values and the products with the state are there; nobody reads the published state any more
        if (warp < 4) {
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int tok = 16 * mt + g + 8 * e, c = 8 * j + 2 * t4;
                    const float2 x = *reinterpret_cast<const float2*>(os + tok * kRetOPitch + c);
                    if (tok < n && c < nv)
                        *reinterpret_cast<float2*>(p.o + ((size_t)(run.row0 + b * kRetChunk + tok) * p.heads + h) * vdim + c0 + c) = make_float2(oacc[j][2 * e] + x.x, oacc[j][2 * e + 1] + x.y);
                }
        }
        const float all = pw[n];
#pragma unroll
        for (int m = 0; m < MT; ++m) {
            const int d0 = 16 * (warp + 8 * m);
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[m][j][e] *= all;
            if (d0 < dim) {
#pragma unroll
                for (int kk = 0; kk < kRetChunk / 16; ++kk) {
                    unsigned a[4];   // rows: key channels, columns: tokens
                    rn_ldsm_trans(a, k + (16 * kk + (lane & 7) + 8 * (lane >> 4)) * PITCH + d0 + 8 * ((lane >> 3) & 1));
#pragma unroll
                    for (int j = 0; j < 2; ++j)
#pragma unroll
                        for (int half = 0; half < 2; ++half) {
                            unsigned bf[4];
                            rn_ldsm_trans(bf, dv + half * VS + (16 * kk + (lane & 7) + 8 * ((lane >> 3) & 1)) * kRetVPitch + 16 * j + 8 * (lane >> 4));
                            rn_mma(S[m][2 * j], a, bf[0], bf[1]);
                            rn_mma(S[m][2 * j + 1], a, bf[2], bf[3]);
                        }
                }
            }
        }
        publish();
        __syncthreads();   // the chunk's stage and the decayed values are free
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int m = 0; m < MT; ++m)
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int d = 16 * (warp + 8 * m) + g + 8 * e, c = 8 * j + 2 * t4;
                if (d < dim && c < nv) *reinterpret_cast<float2*>(st + (size_t)d * vdim + c) = make_float2(S[m][j][2 * e], S[m][j][2 * e + 1]);
            }
}

// ---- portions: norm and gate ------------------------------------------------------------------------------------------
// CTA (block of kDeltaBlock tokens, head), a warp per token.
template <typename T>
__global__ void __launch_bounds__(kDeltaBlock * 32) retention_gate_kernel(const RetentionParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, blk = blockIdx.x, h = blockIdx.y, vdim = p.vdim;
    const RowRun run = rn_run(p, p.block_run ? p.block_run[blk] : blk);
    const int i = (blk - run.blk0) * kDeltaBlock + (threadIdx.x >> 5);
    if (i >= run.count) return;
    const int row = run.row0 + i;
    const float* o = p.o + ((size_t)row * p.heads + h) * vdim;
    float ss = 0.f;
    for (int c = lane; c < vdim; c += 32) ss = fmaf(o[c], o[c], ss);
    const float sc = p.out_scale / sqrtf(rn_sum(ss) / (float)vdim + p.eps);
    const T* gate = static_cast<const T*>(p.gate) + (size_t)row * p.gate_stride + (size_t)h * vdim;
    T* out = static_cast<T*>(p.out) + (size_t)row * p.out_stride + (size_t)h * vdim;
    for (int c = lane; c < vdim; c += 32) rn_put(out + c, o[c] * sc * rn_silu(rn_get(gate + c)));
}

// ---- launches ---------------------------------------------------------------------------------------------------------
int col_blocks(int vdim) { return (vdim + kRetCols - 1) / kRetCols; }
int regs_of(int dim) { return dim <= 64 ? 8 : dim <= 128 ? 16 : dim <= 256 ? 32 : 0; }
bool step_fits(int dim, int vdim) { return regs_of(dim) > 0 && col_blocks(vdim) <= kRetCluster; }
bool chunk_fits(const RetentionLaunch& a) {
    return !a.f32 && !((a.dim | a.vdim) & 7) && a.dim <= 256 && !(a.qkv_stride & 7) && !(reinterpret_cast<uintptr_t>(a.qkv) & 15);
}

template <typename T, int R>
cudaError_t step_launch(const RetentionParams& p, int rows, cudaStream_t s) {
    const int nz = col_blocks(p.vdim);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(nz, p.heads, rows); cfg.blockDim = dim3(kRetThreads); cfg.stream = s;
    cfg.dynamicSmemBytes = (size_t)2 * p.dim * 4;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = nz; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl_enabled() ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, retention_step_kernel<T, R>, p);
}
template <typename T>
int portions(const RetentionLaunch& a, const RetentionParams& p, int runs, int blocks, bool chunked, cudaStream_t s, int* launches) {
    const dim3 grid(col_blocks(p.vdim), p.heads, runs);
    const size_t smem = (size_t)4 * p.dim * 4;
    cudaError_t e;
    if (chunked && p.dim <= 128) e = launch_k(retention_chunk_kernel<1>, grid, dim3(kRetThreads), ret_smem<1>(), s, p);
    else if (chunked) e = launch_k(retention_chunk_kernel<2>, grid, dim3(kRetThreads), ret_smem<2>(), s, p);
    else switch (regs_of(p.dim)) {
        case 8: e = launch_k(retention_walk_kernel<T, 8>, grid, dim3(kRetThreads), smem, s, p); break;
        case 16: e = launch_k(retention_walk_kernel<T, 16>, grid, dim3(kRetThreads), smem, s, p); break;
        case 32: e = launch_k(retention_walk_kernel<T, 32>, grid, dim3(kRetThreads), smem, s, p); break;
        default: e = launch_k(retention_walk_kernel<T, 0>, grid, dim3(kRetThreads), smem, s, p);
        }
    if (e != cudaSuccess) return cuda_fail(e, "retention launch");
    e = launch_k(retention_gate_kernel<T>, dim3(blocks, p.heads), dim3(kDeltaBlock * 32), 0, s, p);
    if (e != cudaSuccess) return cuda_fail(e, "retention gate launch");
    *launches += 2;
    return SWLM_OK;
}
template <typename T>
int run(const RetentionLaunch& a, RetentionParams p, cudaStream_t s, int* launches) {
    if (a.n_single > 0) {
        if (step_fits(a.dim, a.vdim)) {
            const int regs = regs_of(a.dim);
            const cudaError_t e = regs == 8 ? step_launch<T, 8>(p, a.n_single, s) : regs == 16 ? step_launch<T, 16>(p, a.n_single, s) : step_launch<T, 32>(p, a.n_single, s);
            if (e != cudaSuccess) return cuda_fail(e, "retention step launch");
            *launches += 1;
        } else {
            const int rc = portions<T>(a, p, a.n_single, a.n_single, false, s, launches);
            if (rc) return rc;
        }
    }
    if (a.n_runs > 0) {
        p.runs = a.runs;
        p.block_run = a.block_run;
        return portions<T>(a, p, a.n_runs, a.n_blocks, chunk_fits(a), s, launches);
    }
    return SWLM_OK;
}

}  // namespace

bool retention_supported(int heads, int dim, int vdim) { return heads > 0 && dim > 0 && vdim > 0 && dim <= 2048; }
bool retention_step_fits(int dim, int vdim) { return step_fits(dim, vdim); }

int retention_init() {
    SWLM_CUDA(cudaFuncSetAttribute(retention_chunk_kernel<1>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ret_smem<1>()));
    SWLM_CUDA(cudaFuncSetAttribute(retention_chunk_kernel<2>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)ret_smem<2>()));
    return SWLM_OK;
}

int launch_retention(const RetentionLaunch& a, cudaStream_t s, int* launches) {
    RetentionParams p{};
    p.heads = a.heads; p.dim = a.dim; p.vdim = a.vdim; p.eps = a.eps; p.scale = a.scale; p.out_scale = a.out_scale; p.decay = a.decay;
    p.qkv = a.qkv; p.qkv_stride = a.qkv_stride; p.gate = a.gate; p.gate_stride = a.gate_stride; p.state = a.state;
    p.row_seq = a.row_seq; p.row_pos = a.row_pos; p.out = a.out; p.out_stride = a.out_stride; p.single_rows = a.single_rows; p.o = a.scratch;
    return a.f32 ? run<float>(a, p, s, launches) : run<__nv_bfloat16>(a, p, s, launches);
}

}  // namespace swlm
