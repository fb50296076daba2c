// The residual stream between the sublayers of designs whose sublayers read the stream itself: what a sublayer returns is gated,
// normed and added, results of layers are averaged over the depth, and the next sublayer gets the stream with a short causal
// convolution over it. All of it is fp32.
//
//   single tokens   stream_step_kernel: everything between two products in one launch, a cluster of CTAs per row that share its
//                   columns; the norm's sum crosses the cluster through distributed shared memory. With a token input in between
//                   (two small products with a gated table row between them, then a second norm) that is part of it: a CTA
//                   multiplies its columns of the stream, the sums cross the cluster, and it works out its columns of the result.
//                   Its weights come to shared memory before the preceding kernel has finished, as far as they fit.
//   portions        stream_join_kernel (a CTA per row) and stream_conv_kernel (a thread walks a few rows of four channels).
//
// A convolution finds the tokens in front of a portion in the state of the sequence. The state is written by the launch that
// changes the stream next (it reads the same rows), so nobody writes what others still read.
#include <cooperative_groups.h>

#include <algorithm>
#include <utility>

#include "swlm_internal.h"
#include "tc_device.cuh"

namespace cg = cooperative_groups;

namespace swlm {
namespace {

constexpr int kConvRows = 8, kConvThreads = 128;
constexpr int kStepCluster = 8;
constexpr int kSideThreads = 256, kSideCluster = 16, kSideMaxRows = 16;   // rows beyond which the products of a token input run on their own
constexpr int kStepResults = 128;   // earlier results whose weights are kept at hand
constexpr size_t kSideSmem = 160 * 1024;

__device__ __forceinline__ void jn_put4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void jn_put4(__nv_bfloat16* p, const float (&v)[4]) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v[0], v[1]), hi = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}
// four fp32 values of a buffer row (rows are padded to eight and 16-byte aligned)
__device__ __forceinline__ void jn_get4(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
// four values of a bf16 vector of n entries, zeros past its end; `whole`: rows of it are 8-byte aligned and n a multiple of four
__device__ __forceinline__ void jn_weights4(const __nv_bfloat16* p, int i, int n, bool whole, float (&v)[4]) {
    if (whole && i < n) {
        const uint2 a = __ldg(reinterpret_cast<const uint2*>(p + i));
        v[0] = __uint_as_float(a.x << 16); v[1] = __uint_as_float(a.x & 0xFFFF0000u);
        v[2] = __uint_as_float(a.y << 16); v[3] = __uint_as_float(a.y & 0xFFFF0000u);
        return;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = i + e < n ? __bfloat162float(p[i + e]) : 0.f;
}
__device__ __forceinline__ float jn_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }

// sum over j < avg - 1 of weight(j) * results[j] at four entries of a row
template <typename W>
__device__ __forceinline__ void jn_results(const JoinLaunch& p, W weight, int r, int i, float (&sum)[4]) {
    sum[0] = sum[1] = sum[2] = sum[3] = 0.f;
    const float* at = p.results + (size_t)r * p.res_stride + i;
#pragma unroll 8
    for (int q = 0; q < p.avg - 1; ++q) {
        float v[4];
        jn_get4(at + q * p.result_step, v);
        const float w = weight(q);
#pragma unroll
        for (int e = 0; e < 4; ++e) sum[e] = fmaf(w, v[e], sum[e]);
    }
}
__device__ __forceinline__ void jn_average(const JoinLaunch& p, int r, int i, float (&h)[4]) {
    float sum[4];
    jn_results(p, [&](int q) { return __bfloat162float(p.avg_w[q]); }, r, i, sum);
    const float w = __bfloat162float(p.avg_w[p.avg - 1]);
#pragma unroll
    for (int e = 0; e < 4; ++e) h[e] = fmaf(w, h[e], sum[e]);
}

// ---- portions: gate, norm, sum, average -------------------------------------------------------------------------------
// CTA per row; a thread keeps entries 4 (tid + NT j) .. + 3.
template <typename T, int J, int NT>
__global__ void __launch_bounds__(NT, 1024 / NT) stream_join_kernel(const JoinLaunch p) {
    __shared__ float red[NT / 32];
    const int tid = threadIdx.x, width = p.width, r = blockIdx.x;
    const bool whole = (width & 3) == 0;
    pdl_launch_dependents();
    pdl_wait();
    const int seq = p.row_seq[r];
    float h[J][4], t[J][4];
    const __nv_bfloat16* row = p.table ? p.table + (size_t)min(max(p.tokens[r], 0), p.vocab - 1) * width : nullptr;
    float ss = 0.f;
#pragma unroll
    for (int j = 0; j < J; ++j) {
        const int i = 4 * (tid + NT * j);
        h[j][0] = h[j][1] = h[j][2] = h[j][3] = t[j][0] = t[j][1] = t[j][2] = t[j][3] = 0.f;
        if (i >= width) continue;
        if (row) jn_weights4(row, i, width, whole, h[j]);
        else jn_get4(p.res_in + (size_t)r * p.res_stride + i, h[j]);
        if (p.in) jn_get4(p.in + (size_t)r * p.in_stride + i, t[j]);
        float gate[4];
        if (p.gate) jn_get4(p.gate + (size_t)r * p.gate_stride + i, gate);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            if (row) h[j][e] *= p.table_scale;
            if (p.gate) t[j][e] *= jn_sigmoid(gate[e]);
            if (i + e >= width) h[j][e] = t[j][e] = 0.f;
            ss = fmaf(t[j][e], t[j][e], ss);
        }
    }
    if (p.keep_ring && !(r + p.keep_taps - 1 < p.rows && p.row_seq[r + p.keep_taps - 1] == seq)) {   // among the last of its portion
        float* keep = p.keep_ring + ((size_t)seq * (p.keep_taps - 1) + p.row_pos[r] % (p.keep_taps - 1)) * width;
#pragma unroll
        for (int j = 0; j < J; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) { const int i = 4 * (tid + NT * j) + e; if (i < width) keep[i] = h[j][e]; }
    }
    float scale = 0.f;
    if (p.in) {
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if ((tid & 31) == 0) red[tid >> 5] = ss;
        __syncthreads();
        float total = 0.f;
#pragma unroll
        for (int i = 0; i < NT / 32; ++i) total += red[i];
        scale = 1.0f / sqrtf(total / (float)width + p.eps);
    }
#pragma unroll
    for (int j = 0; j < J; ++j) {
        const int i = 4 * (tid + NT * j);
        if (i >= width) continue;
        if (p.in) {
            float w[4];
            jn_weights4(p.w, i, width, whole, w);
#pragma unroll
            for (int e = 0; e < 4; ++e) h[j][e] = fmaf(t[j][e] * scale, w[e] + p.weight_bias, h[j][e]);
        }
        if (p.store >= 0) jn_put4(p.results + p.store * p.result_step + (size_t)r * p.res_stride + i, h[j]);
        if (p.avg) jn_average(p, r, i, h[j]);
        if (p.res_out) jn_put4(p.res_out + (size_t)r * p.res_stride + i, h[j]);
        if (p.copy_out) jn_put4(static_cast<T*>(p.copy_out) + (size_t)r * p.copy_stride + i, h[j]);
    }
}

// ---- portions: the convolution ----------------------------------------------------------------------------------------
// CTA (128 quads of channels, kConvRows rows). `stream` are the rows the join left behind; TAPS 0: any number, rows read again.
template <typename T, int TAPS>
__global__ void __launch_bounds__(kConvThreads) stream_conv_kernel(const JoinLaunch p, const float* stream) {
    constexpr int PAST = TAPS > 1 ? TAPS - 1 : 1;
    const int width = p.width, i = 4 * (blockIdx.x * kConvThreads + threadIdx.x), r0 = blockIdx.y * kConvRows, r1 = min(r0 + kConvRows, p.rows), past = p.taps - 1;
    const bool live = i < width;
    pdl_launch_dependents();
    float w[TAPS > 0 ? TAPS : 1][4];
    if (TAPS > 0 && live)
#pragma unroll
        for (int k = 0; k < (TAPS > 0 ? TAPS : 1); ++k)
#pragma unroll
            for (int e = 0; e < 4; ++e) w[k][e] = i + e < width ? __bfloat162float(p.conv_w[(size_t)(i + e) * TAPS + k]) : 0.f;
    pdl_wait();
    if (!live) return;
    // the stream d tokens in front of row r
    auto back = [&](int r, int d, float (&v)[4]) {
        if (r - d >= 0 && p.row_seq[r - d] == p.row_seq[r]) { jn_get4(stream + (size_t)(r - d) * p.res_stride + i, v); return; }
        const int at = p.row_pos[r] - d;
        const float* from = p.conv_ring + ((size_t)p.row_seq[r] * past + (at >= 0 ? at % past : 0)) * width;
#pragma unroll
        for (int e = 0; e < 4; ++e) v[e] = at >= 0 && i + e < width ? from[i + e] : 0.f;
    };
    if (TAPS > 0 && r1 - r0 == kConvRows && r0 >= past && p.row_seq[r0 - past] == p.row_seq[r1 - 1]) {   // all rows of one portion: requested at once
        float h[kConvRows + (TAPS > 1 ? TAPS - 1 : 0)][4];
#pragma unroll
        for (int n = 0; n < kConvRows + TAPS - 1; ++n) jn_get4(stream + (size_t)(r0 - past + n) * p.res_stride + i, h[n]);
#pragma unroll
        for (int n = 0; n < kConvRows; ++n) {
            float y[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                y[e] = fmaf(w[TAPS > 0 ? TAPS - 1 : 0][e], h[n + TAPS - 1][e], h[n + TAPS - 1][e]);
#pragma unroll
                for (int d = 1; d < TAPS; ++d) y[e] = fmaf(w[TAPS - 1 - d][e], h[n + TAPS - 1 - d][e], y[e]);
            }
            jn_put4(static_cast<T*>(p.conv_out) + (size_t)(r0 + n) * p.conv_stride + i, y);
        }
        return;
    }
    float hist[PAST][4];   // hist[d - 1]: d tokens back
    for (int r = r0; r < r1; ++r) {
        float h[4], y[4];
        jn_get4(stream + (size_t)r * p.res_stride + i, h);
        if (TAPS > 0) {
            if (TAPS > 1 && (r == r0 || p.row_seq[r - 1] != p.row_seq[r]))
#pragma unroll
                for (int d = 1; d <= PAST; ++d) back(r, d, hist[d - 1]);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                y[e] = fmaf(w[TAPS > 0 ? TAPS - 1 : 0][e], h[e], h[e]);
                if (TAPS > 1)
#pragma unroll
                    for (int d = 1; d <= PAST; ++d) y[e] = fmaf(w[TAPS > 1 ? TAPS - 1 - d : 0][e], hist[d - 1][e], y[e]);
            }
#pragma unroll
            for (int d = PAST; d > 1; --d)
#pragma unroll
                for (int e = 0; e < 4; ++e) hist[d - 1][e] = hist[d - 2][e];
#pragma unroll
            for (int e = 0; e < 4; ++e) hist[0][e] = h[e];
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e) y[e] = h[e];
            for (int d = 0; d <= past; ++d) {
                float v[4] = {h[0], h[1], h[2], h[3]};
                if (d > 0) back(r, d, v);
#pragma unroll
                for (int e = 0; e < 4; ++e)
                    if (i + e < width) y[e] = fmaf(__bfloat162float(p.conv_w[(size_t)(i + e) * p.taps + past - d]), v[e], y[e]);
            }
        }
        jn_put4(static_cast<T*>(p.conv_out) + (size_t)r * p.conv_stride + i, y);
    }
}

// ---- single tokens ----------------------------------------------------------------------------------------------------
// Sums over LANES neighbouring lanes of V values each; the sum of value (lane % LANES) * V / LANES is left in this lane.
template <int LANES, int V>
__device__ __forceinline__ float jn_sums(float (&v)[V], int lane) {
    int o = LANES / 2;
#pragma unroll
    for (int n = V / 2; n > 0; n >>= 1, o >>= 1) {
        const bool upper = lane & o;
#pragma unroll
        for (int j = 0; j < n; ++j) {
            const float give = upper ? v[j] : v[j + n], keep = upper ? v[j + n] : v[j];
            v[j] = keep + __shfl_xor_sync(0xffffffffu, give, o);
        }
    }
    float r = v[0];
    for (; o > 0; o >>= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
    return r;
}
// out[n] = W[n][0 .. 8 chunks) . x for n < rows, by the whole CTA, LANES lanes to a row; x and out in shared memory, W anywhere
template <int LANES, int V>
__device__ __forceinline__ void jn_rows_by(const __nv_bfloat16* w, int ld, int rows, int chunks, const float* x, float* out) {
    constexpr int PER = 32 / LANES;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, part = lane / LANES, l = lane % LANES;
    for (int n0 = warp * V * PER; n0 < rows; n0 += kSideThreads / 32 * V * PER) {
        float acc[V];
#pragma unroll
        for (int q = 0; q < V; ++q) acc[q] = 0.f;
        for (int c = l; c < chunks; c += LANES) {
            uint4 v[V];
#pragma unroll
            for (int q = 0; q < V; ++q) v[q] = n0 + q * PER + part < rows ? *(reinterpret_cast<const uint4*>(w + (size_t)(n0 + q * PER + part) * ld) + c) : make_uint4(0, 0, 0, 0);
            float f[8];
            *reinterpret_cast<float4*>(f) = *reinterpret_cast<const float4*>(x + 8 * c);
            *reinterpret_cast<float4*>(f + 4) = *reinterpret_cast<const float4*>(x + 8 * c + 4);
#pragma unroll
            for (int q = 0; q < V; ++q) {
                const unsigned b[4] = {v[q].x, v[q].y, v[q].z, v[q].w};
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    acc[q] = fmaf(__uint_as_float(b[e] << 16), f[2 * e], acc[q]);
                    acc[q] = fmaf(__uint_as_float(b[e] & 0xFFFF0000u), f[2 * e + 1], acc[q]);
                }
            }
        }
        const float sum = jn_sums<LANES, V>(acc, lane);
        const int n = n0 + l * V / LANES * PER + part;
        if (l % (LANES / V) == 0 && n < rows) out[n] = sum;
    }
}
__device__ __forceinline__ void jn_rows(const __nv_bfloat16* w, int ld, int rows, int chunks, const float* x, float* out) {
    if (chunks > 16) jn_rows_by<32, 16>(w, ld, rows, chunks, x, out);
    else if (chunks > 8) jn_rows_by<16, 16>(w, ld, rows, chunks, x, out);
    else jn_rows_by<8, 8>(w, ld, rows, chunks, x, out);
}
__device__ __forceinline__ float jn_rounded(float v, float) { return v; }
__device__ __forceinline__ float jn_rounded(float v, __nv_bfloat16) { return __bfloat162float(__float2bfloat16_rn(v)); }

// Cluster of CTAs per row, a thread per four columns. p: start, keep and first norm; f: what follows (SIDE: behind the token input,
// whose result f's norm is for; else the same as p).
template <typename T, bool SIDE, int NT>
__global__ void __launch_bounds__(NT) stream_step_kernel(const JoinLaunch p, const TokenInput side, const JoinLaunch f) {
    extern __shared__ __align__(128) float step_smem[];
    __shared__ float red[NT / 32], ssq[2][SIDE ? kSideCluster : kStepCluster], avg_s[kStepResults];
    __shared__ __align__(8) unsigned long long landed[2];
    const cg::cluster_group cluster = cg::this_cluster();
    auto started = cluster.barrier_arrive();   // waited for before anything is written to another CTA's shared memory
    pdl_launch_dependents();
    const int tid = threadIdx.x, nz = gridDim.x, rank = blockIdx.x, row = blockIdx.y, width = p.width;
    const int chunks = (width + 7) / 8, share = (chunks + nz - 1) / nz, chunk0 = share * rank, own = max(0, min(share, chunks - chunk0));   // chunks of eight columns
    // shared memory of a token input: this CTA's columns of the stream, later of the result; its sums; everybody's; its columns of the
    // first matrix; its rows of the second
    const int np = (side.n + 7) / 8 * 8, own_rows = max(0, min(8 * own, width - 8 * chunk0));
    float* xs = step_smem;
    float* part = xs + 8 * share;
    float* all = part + np;
    __nv_bfloat16* gate_s = reinterpret_cast<__nv_bfloat16*>(all + (size_t)nz * np);
    __nv_bfloat16* proj_s = gate_s + (side.gate_here ? (size_t)side.n * 8 * share : 0);
    if (SIDE && (side.gate_here || side.proj_here)) {
        if (tid == 0) {
            mbar_init(&landed[0], 1);
            mbar_init(&landed[1], 1);
            asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
            mbar_expect(smem_u32(&landed[0]), side.gate_here ? (unsigned)(side.n * own * 16) : 0u);
            mbar_expect(smem_u32(&landed[1]), side.proj_here ? (unsigned)(own_rows * np * 2) : 0u);
        }
        __syncthreads();
        if (side.gate_here && own > 0)
            for (int n = tid; n < side.n; n += NT) bulk_load(smem_u32(gate_s + (size_t)n * 8 * share), side.gate + (size_t)n * side.gate_ld + 8 * chunk0, own * 16, smem_u32(&landed[0]));
        if (side.proj_here)
            for (int n = 16 * tid; n < own_rows; n += 16 * NT)
                bulk_load(smem_u32(proj_s + (size_t)n * np), side.proj + (size_t)(8 * chunk0 + n) * side.proj_ld, (unsigned)(min(16, own_rows - n) * np * 2), smem_u32(&landed[1]));
    }
    const int i = 8 * chunk0 + 4 * tid;
    const bool mine = 4 * tid < 8 * own, whole = (width & 3) == 0;
    const int seq = p.row_seq[row], pos = p.row_pos[row], past = max(0, f.taps - 1);
    // what does not depend on the kernels in front of this one: weights, and the convolution's past
    for (int q = tid; q < min(f.avg, kStepResults); q += NT) avg_s[q] = __bfloat162float(f.avg_w[q]);
    float nw[4] = {}, fw[4] = {}, before[4] = {}, last[4] = {};
    if (mine) {
        if (p.in) jn_weights4(p.w, i, width, whole, nw);
        if (SIDE) jn_weights4(f.w, i, width, whole, fw);
        if (f.conv_out) {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (i + e < width) {
                    const __nv_bfloat16* w = f.conv_w + (size_t)(i + e) * f.taps;
                    last[e] = __bfloat162float(w[past]);
                    for (int d = 1; d <= past && d <= pos; ++d) before[e] = fmaf(__bfloat162float(w[past - d]), f.conv_ring[((size_t)seq * past + (pos - d) % past) * width + i + e], before[e]);
                }
        }
    }
    if (SIDE && !side.gate_here) {   // the other weights come closer
        const int lines = (own + 7) / 8;   // of 128 bytes per row of this CTA's columns
        for (int n = tid; n < side.n * lines; n += NT)
            asm volatile("prefetch.global.L2 [%0];" ::"l"(side.gate + (size_t)(n / lines) * side.gate_ld + 8 * chunk0 + 64 * (n % lines)));
    }
    if (SIDE && !side.proj_here)
        for (int n = tid; n < (own_rows * side.proj_ld + 63) / 64; n += NT) asm volatile("prefetch.global.L2 [%0];" ::"l"(side.proj + (size_t)8 * chunk0 * side.proj_ld + 64 * n));
    __syncthreads();   // (avg_s)
    pdl_wait();
    float h[4] = {}, t[4] = {}, sum[4] = {};
    if (mine) {
        if (p.table) jn_weights4(p.table + (size_t)min(max(p.tokens[row], 0), p.vocab - 1) * width, i, width, whole, h);
        else jn_get4(p.res_in + (size_t)row * p.res_stride + i, h);
        if (p.in) jn_get4(p.in + (size_t)row * p.in_stride + i, t);
        float gate[4];
        if (p.gate) jn_get4(p.gate + (size_t)row * p.gate_stride + i, gate);
        if (f.avg) jn_results(f, [&](int q) { return q < kStepResults ? avg_s[q] : __bfloat162float(f.avg_w[q]); }, row, i, sum);
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            if (p.table) h[e] *= p.table_scale;
            if (p.gate) t[e] *= jn_sigmoid(gate[e]);
            if (i + e >= width) h[e] = t[e] = 0.f;
        }
        if (p.keep_ring) {
            float* keep = p.keep_ring + ((size_t)seq * (p.keep_taps - 1) + pos % (p.keep_taps - 1)) * width;
#pragma unroll
            for (int e = 0; e < 4; ++e) if (i + e < width) keep[i + e] = h[e];
        }
    }
    // 1 / root mean square over the row of what the threads hold; slot: 0 for the first norm, 1 for the second
    auto over_rms = [&](const float (&v)[4], int slot, float eps) {
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) ss = fmaf(v[e], v[e], ss);
        for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        if ((tid & 31) == 0) red[tid >> 5] = ss;
        __syncthreads();
        if (tid < nz) {
            float total = 0.f;
#pragma unroll
            for (int q = 0; q < NT / 32; ++q) total += red[q];
            cluster.map_shared_rank(ssq[slot], tid)[rank] = total;
        }
        cluster.sync();
        float total = 0.f;
        for (int q = 0; q < nz; ++q) total += ssq[slot][q];
        return 1.0f / sqrtf(total / (float)width + eps);
    };
    auto wait = [&](int which) {   // for the weights in shared memory; never leave with a copy under way (bounded)
        if (mbar_wait(&landed[which], 0u)) return;
        if (tid == 0) atomicExch(side.status, 71);
        mbar_wait(&landed[which], 0u);
    };
    cluster.barrier_wait(std::move(started));
    if (p.in) {
        const float scale = over_rms(t, 0, p.eps);
#pragma unroll
        for (int e = 0; e < 4; ++e) h[e] = fmaf(t[e] * scale, nw[e] + p.weight_bias, h[e]);
    }
    if (SIDE) {
        if (4 * tid < 8 * share)
#pragma unroll
            for (int e = 0; e < 4; ++e) xs[4 * tid + e] = mine && i + e < width ? jn_rounded(h[e], T(0.f)) : 0.f;
        __syncthreads();
        if (side.gate_here) {
            wait(0);
            jn_rows(gate_s, 8 * share, side.n, own, xs, part);
        } else jn_rows(side.gate + 8 * chunk0, side.gate_ld, side.n, own, xs, part);
        __syncthreads();
        for (int n = tid; n < side.n * nz; n += NT) cluster.map_shared_rank(all, n / side.n)[rank * np + n % side.n] = part[n % side.n];
        cluster.sync();
        const __nv_bfloat16* token = side.table + (size_t)min(max(p.tokens[row], 0), p.vocab - 1) * side.cols + side.col;
        for (int n = tid; n < np; n += NT) {
            float v = 0.f;
            if (n < side.n) {
                for (int q = 0; q < nz; ++q) v += all[q * np + n];
                v = jn_rounded(gated_activation(jn_rounded(v, T(0.f)), __bfloat162float(token[n]), GATED_ACT_GELU_TANH), T(0.f));
            }
            part[n] = v;
        }
        __syncthreads();
        if (side.proj_here) {
            wait(1);
            jn_rows(proj_s, np, own_rows, np / 8, part, xs);
        } else jn_rows(side.proj + (size_t)8 * chunk0 * side.proj_ld, side.proj_ld, own_rows, np / 8, part, xs);
        __syncthreads();
#pragma unroll
        for (int e = 0; e < 4; ++e) t[e] = mine && i + e < width ? xs[4 * tid + e] : 0.f;
        const float scale = over_rms(t, 1, f.eps);
#pragma unroll
        for (int e = 0; e < 4; ++e) h[e] = fmaf(t[e] * scale, fw[e] + f.weight_bias, h[e]);
    }
    if (!mine) return;   // (nobody reaches into this CTA's shared memory any more)
    if (f.store >= 0) jn_put4(f.results + f.store * f.result_step + (size_t)row * f.res_stride + i, h);
    if (f.avg) {
        const float w = __bfloat162float(f.avg_w[f.avg - 1]);
#pragma unroll
        for (int e = 0; e < 4; ++e) h[e] = fmaf(w, h[e], sum[e]);
    }
    if (f.res_out) jn_put4(f.res_out + (size_t)row * f.res_stride + i, h);
    if (f.copy_out) jn_put4(static_cast<T*>(f.copy_out) + (size_t)row * f.copy_stride + i, h);
    if (f.conv_out) {
        float y[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) y[e] = h[e] + fmaf(last[e], h[e], before[e]);
        jn_put4(static_cast<T*>(f.conv_out) + (size_t)row * f.conv_stride + i, y);
    }
}

// ---- a gate out of a table --------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) token_gate_kernel(int n, const T* in, int in_stride, const int32_t* tokens, int vocab, const __nv_bfloat16* table, int cols, int col,
                                                         T* out, int out_stride, int m) {
    pdl_launch_dependents();
    pdl_wait();
    const int at = blockIdx.x * blockDim.x + threadIdx.x, r = at / n, i = at - r * n;
    if (r >= m) return;
    const int tok = min(max(tokens[r], 0), vocab - 1);
    const float v = gated_activation((float)in[(size_t)r * in_stride + i], __bfloat162float(table[(size_t)tok * cols + col + i]), GATED_ACT_GELU_TANH);
    out[(size_t)r * out_stride + i] = (T)v;
}

// ---- launches ---------------------------------------------------------------------------------------------------------
template <typename T, int J, int NT>
cudaError_t join_launch(const JoinLaunch& a, cudaStream_t s) { return launch_k(stream_join_kernel<T, J, NT>, dim3(a.rows), dim3(NT), 0, s, a); }
template <typename T, int TAPS>
cudaError_t conv_launch(const JoinLaunch& a, cudaStream_t s) {
    return launch_k(stream_conv_kernel<T, TAPS>, dim3((a.width + 4 * kConvThreads - 1) / (4 * kConvThreads), (a.rows + kConvRows - 1) / kConvRows), dim3(kConvThreads), 0, s, a,
                    a.res_out ? (const float*)a.res_out : a.res_in);
}
template <typename T>
int portions(const JoinLaunch& a, cudaStream_t s, int* launches) {
    cudaError_t e = cudaSuccess;
    if (a.res_out || a.copy_out || a.keep_ring) {
        e = a.width <= 4 * 128 ? join_launch<T, 1, 128>(a, s) : a.width <= 4 * 256 ? join_launch<T, 1, 256>(a, s) : a.width <= 4 * 512 ? join_launch<T, 2, 256>(a, s)
            : a.width <= 4 * 1024 ? join_launch<T, 2, 512>(a, s) : join_launch<T, 8, 512>(a, s);
        *launches += 1;
    }
    if (e == cudaSuccess && a.conv_out) {
        e = a.taps == 1 ? conv_launch<T, 1>(a, s) : a.taps == 2 ? conv_launch<T, 2>(a, s) : a.taps == 3 ? conv_launch<T, 3>(a, s) : a.taps == 4 ? conv_launch<T, 4>(a, s) : conv_launch<T, 0>(a, s);
        *launches += 1;
    }
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "stream join launch");
}

size_t side_smem(const TokenInput& t, int width, int nz) {
    const size_t np = (t.n + 7) / 8 * 8, share = ((width + 7) / 8 + nz - 1) / nz;
    return (8 * share + np * (nz + 1)) * 4 + (t.gate_here ? (size_t)t.n * share * 16 : 0) + (t.proj_here ? 8 * share * np * 2 : 0);
}
template <typename T, bool SIDE, int NT>
int step_launch(const JoinLaunch& p, const TokenInput& side, const JoinLaunch& f, int nz, cudaStream_t s) {
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(nz, p.rows); cfg.blockDim = dim3(NT); cfg.stream = s;
    cfg.dynamicSmemBytes = SIDE ? side_smem(side, p.width, nz) : 0;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = nz; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl_enabled() ? 2 : 1;
    const cudaError_t e = cudaLaunchKernelEx(&cfg, stream_step_kernel<T, SIDE, NT>, p, side, f);
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "stream step launch");
}
constexpr int kStepThreads = 128;
bool step_fits(int width) { return width <= 4 * kSideThreads * kStepCluster; }

// What of the weights fits shared memory, and the size of the cluster: as many CTAs as the GPU runs together, so that most does.
TokenInput side_shape(TokenInput t, int width, int nz) {
    t.gate_here = 1;
    if (side_smem(t, width, nz) > kSideSmem) t.gate_here = 0;
    t.proj_here = t.proj_ld == (t.n + 7) / 8 * 8;
    if (side_smem(t, width, nz) > kSideSmem) t.proj_here = 0;
    return t;
}
template <typename T>
int side_launch(const JoinLaunch& first, const TokenInput& t, const JoinLaunch& last, cudaStream_t s) {
    const auto kernel = stream_step_kernel<T, true, kSideThreads>;
    static const cudaError_t attr = [&] {
        const cudaError_t e = cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kSideSmem);
        return e != cudaSuccess ? e : cudaFuncSetAttribute(kernel, cudaFuncAttributeNonPortableClusterSizeAllowed, 1);
    }();
    if (attr != cudaSuccess) return cuda_fail(attr, "stream step attributes");
    static const int largest = [&] {   // are clusters of 16 CTAs with all of the shared memory possible here?
        cudaLaunchConfig_t cfg = {};
        cfg.gridDim = dim3(kSideCluster); cfg.blockDim = dim3(kSideThreads); cfg.dynamicSmemBytes = kSideSmem;
        cudaLaunchAttribute cluster[1];
        cluster[0].id = cudaLaunchAttributeClusterDimension;
        cluster[0].val.clusterDim.x = kSideCluster; cluster[0].val.clusterDim.y = 1; cluster[0].val.clusterDim.z = 1;
        cfg.attrs = cluster;
        cfg.numAttrs = 1;
        int n = 0;
        return cudaOccupancyMaxActiveClusters(&n, kernel, &cfg) == cudaSuccess && n > 0 ? kSideCluster : kStepCluster;
    }();
    // (many rows: smaller clusters that read the weights where they are, so that all run at once)
    if (first.rows * largest > 148) return step_launch<T, true, kSideThreads>(first, t, last, kStepCluster, s);
    return step_launch<T, true, kSideThreads>(first, side_shape(t, first.width, largest), last, largest, s);
}

}  // namespace

bool join_supported(int width, int taps) { return width > 0 && width <= 4 * 512 * 8 && taps >= 0; }

int launch_join(const JoinLaunch& a, cudaStream_t s, int* launches) {
    if (a.rows <= 0) return SWLM_OK;
    if (!join_supported(a.width, a.taps)) { set_error("stream of %d entries with convolutions of %d taps", a.width, a.taps); return SWLM_ERR_UNSUPPORTED; }
    if (a.singles && step_fits(a.width)) {
        *launches += 1;
        int nz = 1;
        while (nz < kStepCluster && nz * 4 * kStepThreads < a.width) nz <<= 1;
        const TokenInput none;
        if (nz * 4 * kStepThreads >= a.width) return a.f32 ? step_launch<float, false, kStepThreads>(a, none, a, nz, s) : step_launch<__nv_bfloat16, false, kStepThreads>(a, none, a, nz, s);
        return a.f32 ? step_launch<float, false, kSideThreads>(a, none, a, nz, s) : step_launch<__nv_bfloat16, false, kSideThreads>(a, none, a, nz, s);
    }
    return a.f32 ? portions<float>(a, s, launches) : portions<__nv_bfloat16>(a, s, launches);
}

bool token_input_fits(const TokenInput& t, int rows, int width) {
    TokenInput none = t;
    none.gate_here = none.proj_here = 0;
    return rows <= kSideMaxRows && step_fits(width) && side_smem(none, width, kSideCluster) <= kSideSmem && side_smem(none, width, kStepCluster) <= kSideSmem;
}
int launch_token_input(const JoinLaunch& first, const TokenInput& t, const JoinLaunch& last, cudaStream_t s) {
    if (first.rows <= 0) return SWLM_OK;
    if (!token_input_fits(t, first.rows, first.width)) { set_error("token input of %d entries into %d x %d", t.n, first.rows, first.width); return SWLM_ERR_UNSUPPORTED; }
    return first.f32 ? side_launch<float>(first, t, last, s) : side_launch<__nv_bfloat16>(first, t, last, s);
}

int launch_token_gate(int m, int n, const void* in, int in_stride, const int32_t* tokens, int vocab, const __nv_bfloat16* table, int cols, int col, void* out,
                      int out_stride, bool f32, cudaStream_t s) {
    if (m <= 0) return SWLM_OK;
    const dim3 grid((unsigned)(((size_t)m * n + 255) / 256));
    const cudaError_t e = f32 ? launch_k(token_gate_kernel<float>, grid, dim3(256), 0, s, n, static_cast<const float*>(in), in_stride, tokens, vocab, table, cols, col,
                                         static_cast<float*>(out), out_stride, m)
                              : launch_k(token_gate_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, n, static_cast<const __nv_bfloat16*>(in), in_stride, tokens, vocab, table, cols,
                                         col, static_cast<__nv_bfloat16*>(out), out_stride, m);
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "token gate launch");
}

}  // namespace swlm
