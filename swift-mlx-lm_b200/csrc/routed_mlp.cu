// Routed feed-forward: a router picks `top` of the experts for every row, the row's result is the weighted sum of theirs; a
// shared feed-forward that every row takes, weighted by a sigmoid, may join the sum.
//
//   few rows (and fp32 plans)  routed_gate_kernel: every CTA works out its row's choice from the router's logits, then its warps
//                              stream gate and up rows of the chosen experts (and of the shared feed-forward);
//                              routed_down_kernel: a warp per output runs through the chosen experts' down rows one after the
//                              other, so the sum over experts needs no pass of its own.
//   more rows (bf16)           routed_choose_kernel, routed_sort_kernel (rows sorted by expert, table of tiles), two grouped
//                              tensor-core products, two plain ones for the shared feed-forward, routed_sum_kernel.
//
// An expert's place among the candidates is the number of candidates before it (larger score, or equal score and lower index),
// so the choice takes one pass without a sequence of maxima.
#include <algorithm>

#include "swlm_internal.h"

namespace swlm {
namespace {

constexpr int kRtThreads = 256, kRtWarps = kRtThreads / 32;
constexpr int kRtFewRows = 4;       // bf16 rows that go one by one

struct RoutedParams {
    RoutedShape sh;
    float scale;
    GatedAct act;
    int softmax, group_best, raw_weights;
    const __nv_bfloat16* correction;
    int m;
    const void* x; int x_stride;
    const float* z; int z_stride;
    const __nv_bfloat16 *gate, *up, *down; int in_ld, mid_ld;   // row pitches of gate / up and of down; gate == null: GELU of up
    const __nv_bfloat16 *shared_up, *shared_down; int shared_ld;
    void* shared_mid; int shared_stride;     // [rows][shared_stride]
    const float* shared_y; int shared_y_stride;
    float* out; int out_stride;
    int* sel; float* weight; int* rank;      // [rows][top]
    unsigned* counts;                        // [experts]
    void* mid; int mid_stride;               // [rows * top][mid_stride]
    __nv_bfloat16* sorted; int sorted_stride;
    float* y; int y_stride;
    int4* tiles; int max_tiles, bn;
};

__device__ __forceinline__ float rt_get(const float* p) { return *p; }
__device__ __forceinline__ float rt_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void rt_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void rt_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
// eight consecutive values, 16-byte aligned
__device__ __forceinline__ void rt_get8(const float* p, float (&f)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void rt_get8(const __nv_bfloat16* p, float (&f)[8]) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    const unsigned w[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) { f[2 * i] = __uint_as_float(w[i] << 16); f[2 * i + 1] = __uint_as_float(w[i] & 0xFFFF0000u); }
}
__device__ __forceinline__ float rt_lo(unsigned w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float rt_hi(unsigned w) { return __uint_as_float(w & 0xFFFF0000u); }
__device__ __forceinline__ uint4 rt_stream(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
__device__ __forceinline__ float rt_dot8(const uint4& w, const float* x, float acc) {
    const float4 a = *reinterpret_cast<const float4*>(x), b = *reinterpret_cast<const float4*>(x + 4);
    acc = fmaf(rt_lo(w.x), a.x, acc); acc = fmaf(rt_hi(w.x), a.y, acc); acc = fmaf(rt_lo(w.y), a.z, acc); acc = fmaf(rt_hi(w.y), a.w, acc);
    acc = fmaf(rt_lo(w.z), b.x, acc); acc = fmaf(rt_hi(w.z), b.y, acc); acc = fmaf(rt_lo(w.w), b.z, acc); return fmaf(rt_hi(w.w), b.w, acc);
}

__device__ __forceinline__ float shared_weight(const RoutedParams& p, int row) { return 1.0f / (1.0f + expf(-p.z[(size_t)row * p.z_stride + p.sh.experts])); }

// from the chosen scores to the weights
template <int THREADS>
__device__ __forceinline__ void weigh(const RoutedParams& p, float* w, int tid) {
    float total = 0.f;
    for (int i = 0; i < p.sh.top; ++i) total += w[i];
    if (THREADS == 32) __syncwarp(); else __syncthreads();
    for (int i = tid; i < p.sh.top; i += THREADS) w[i] = p.raw_weights ? w[i] * p.scale : w[i] / (total + 1e-20f) * p.scale;
}

// Experts with tensors first, those that hand the input through behind them (one warp; top <= 64); returns the number of the first.
__device__ __forceinline__ int real_first(const RoutedShape& sh, int* sel, float* w, int lane) {
    const int a = lane < sh.top ? sel[lane] : 0, b = lane + 32 < sh.top ? sel[lane + 32] : 0;
    const float wa = lane < sh.top ? w[lane] : 0.f, wb = lane + 32 < sh.top ? w[lane + 32] : 0.f;
    const unsigned lower = (1u << lane) - 1u;
    const unsigned la = __ballot_sync(0xffffffffu, lane < sh.top), lb = __ballot_sync(0xffffffffu, lane + 32 < sh.top);
    const unsigned ra = __ballot_sync(0xffffffffu, lane < sh.top && a < sh.experts), rb = __ballot_sync(0xffffffffu, lane + 32 < sh.top && b < sh.experts);
    const int real = __popc(ra) + __popc(rb);
    __syncwarp();
    if (lane < sh.top) { const int at = a < sh.experts ? __popc(ra & lower) : real + __popc(la & ~ra & lower); sel[at] = a; w[at] = wa; }
    if (lane + 32 < sh.top) { const int at = b < sh.experts ? __popc(ra) + __popc(rb & lower) : real + __popc(la & ~ra) + __popc(lb & ~rb & lower); sel[at] = b; w[at] = wb; }
    return real;
}

// The choice of one row by THREADS threads (a warp or the CTA). s: [experts] scores, gs: [groups] group scores, both shared;
// sel / w: [top] in order of falling score. With a correction the choice looks at s + correction, kept in cs: [scored]; the weights
// are the plain scores. MORE: corrections and identity experts are possible (others do without that code).
template <int THREADS, bool MORE>
__device__ __forceinline__ void choose(const RoutedParams& p, const float* z, float* s, float* gs, float* cs, int* sel, float* w, int tid) {
    auto sync = [] { if (THREADS == 32) __syncwarp(); else __syncthreads(); };
    const int E = MORE ? p.sh.scored() : p.sh.experts, G = p.sh.groups, per = E / G;
    for (int i = tid; i < p.sh.top; i += THREADS) { sel[i] = i; w[i] = 0.f; }   // indices stay valid whatever the logits are
    if (p.softmax) {   // every warp works out maximum and sum for itself
        float top = -INFINITY, sum = 0.f;
        for (int e = tid & 31; e < E; e += 32) top = fmaxf(top, z[e]);
        for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
        for (int e = tid & 31; e < E; e += 32) sum += expf(z[e] - top);
        for (int o = 16; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        for (int e = tid; e < E; e += THREADS) s[e] = expf(z[e] - top) / sum;
    } else {
        for (int e = tid; e < E; e += THREADS) s[e] = 1.0f / (1.0f + expf(-z[e]));
    }
    sync();
    if (MORE && p.correction) {
        for (int e = tid; e < E; e += THREADS) cs[e] = s[e] + __bfloat162float(p.correction[e]);
        sync();
        for (int e = tid; e < E; e += THREADS) {
            const float v = cs[e];
            int before = 0;
            for (int o = 0; o < E; ++o) before += cs[o] > v || (cs[o] == v && o < e);
            if (before < p.sh.top) { sel[before] = e; w[before] = s[e]; }
        }
        sync();
        weigh<THREADS>(p, w, tid);
        sync();
        return;
    }
    for (int g = tid; g < G; g += THREADS) {
        float first = 0.f, second = 0.f;   // scores are not negative
        for (int e = g * per; e < (g + 1) * per; ++e) {
            const float v = s[e];
            second = fmaxf(second, fminf(first, v));
            first = fmaxf(first, v);
        }
        gs[g] = p.group_best == 1 ? first : first + second;
    }
    sync();
    auto kept = [&](int g) {
        int before = 0;
        for (int o = 0; o < G; ++o) before += gs[o] > gs[g] || (gs[o] == gs[g] && o < g);
        return before < p.sh.keep;
    };
    if (p.sh.keep < G) {
        // experts of the other groups leave the race (a score is never below zero)
        for (int e = tid; e < E; e += THREADS) { const bool in = kept(e / per); if (!in) s[e] = -1.0f; }
        sync();
    }
    for (int e = tid; e < E; e += THREADS) {
        const float v = s[e];
        int before = 0;
        for (int o = 0; o < E; ++o) before += s[o] > v || (s[o] == v && o < e);
        if (v >= 0.f && before < p.sh.top) { sel[before] = e; w[before] = v; }
    }
    sync();
    weigh<THREADS>(p, w, tid);
    sync();
}

// ---- few rows ---------------------------------------------------------------------------------------------------------
// CTA (share of the work, row). A unit of work is one row of an expert's gate with the same row of its up, or without a gate two
// rows of up; those of the shared feed-forward come first, because they are known before the choice.
__host__ __device__ __forceinline__ int routed_units(int ff, bool gated) { return gated ? ff : (ff + 1) / 2; }
template <typename T, bool GATED, bool MORE>
__global__ void __launch_bounds__(kRtThreads) routed_gate_kernel(const RoutedParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) float rt_smem[];
    __shared__ int sel[kMaxTop];
    __shared__ float weight[kMaxTop];
    __shared__ int real_s;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = blockIdx.y;
    const int per = routed_units(p.sh.ff, GATED), shared = routed_units(p.sh.shared_ff, GATED);
    const int chunks = p.in_ld >> 3;
    constexpr int U = 4;
    uint4 av[U], bv[U];
    const __nv_bfloat16 *ar = nullptr, *br = nullptr;
    int slot = 0, f = 0;
    auto place = [&](int u) {   // rows of unit u
        const bool mine = u >= shared;
        slot = mine ? (u - shared) / per : p.sh.top;
        f = mine ? u - shared - slot * per : u;
        const __nv_bfloat16* up = mine ? p.up + (size_t)sel[slot] * p.sh.ff * p.in_ld : p.shared_up;
        if (GATED) {
            ar = up + (size_t)f * p.in_ld;
            br = p.gate + ((size_t)sel[slot] * p.sh.ff + f) * p.in_ld;
        } else {
            f *= 2;
            ar = up + (size_t)f * p.in_ld;
            br = ar + (f + 1 < (mine ? p.sh.ff : p.sh.shared_ff) ? p.in_ld : 0);
        }
    };
    auto load = [&](int c0) {
#pragma unroll
        for (int j = 0; j < U; ++j) {
            const int c = c0 + 32 * j;
            av[j] = c < chunks ? rt_stream(ar + 8 * c) : make_uint4(0, 0, 0, 0);
            bv[j] = c < chunks ? rt_stream(br + 8 * c) : make_uint4(0, 0, 0, 0);
        }
    };
    const int first = blockIdx.x * kRtWarps + warp;
    if (first < shared) { place(first); load(lane); }
    pdl_wait();
    float* x = rt_smem;                    // [in_ld]
    float* s = x + p.in_ld;                // [scored], then [groups], then [scored]
    const T* src = static_cast<const T*>(p.x) + (size_t)row * p.x_stride;
    for (int i = tid; i < p.in_ld; i += kRtThreads) x[i] = i < p.sh.width ? rt_get(src + i) : 0.f;
    choose<kRtThreads, MORE>(p, p.z + (size_t)row * p.z_stride, s, s + p.sh.scored(), s + p.sh.scored() + p.sh.groups, sel, weight, tid);
    int real = p.sh.top;
    if (MORE && p.sh.identity) {
        if (warp == 0) { const int n = real_first(p.sh, sel, weight, lane); if (lane == 0) real_s = n; }
        __syncthreads();
        real = real_s;
    }
    const int units = shared + real * per;
    if (blockIdx.x == 0 && tid < p.sh.top) {
        p.sel[row * p.sh.top + tid] = sel[tid];
        p.weight[row * p.sh.top + tid] = weight[tid];
    }
    for (int u = first; u < units; u += gridDim.x * kRtWarps) {
        if (u != first || u >= shared) place(u);
        float a = 0.f, b = 0.f;
        for (int c0 = lane; c0 < chunks; c0 += 32 * U) {
            if (c0 != lane || u != first || u >= shared) load(c0);
#pragma unroll
            for (int j = 0; j < U; ++j) {
                const int c = c0 + 32 * j;
                if (c < chunks) { a = rt_dot8(av[j], x + 8 * c, a); b = rt_dot8(bv[j], x + 8 * c, b); }
            }
        }
        for (int o = 16; o > 0; o >>= 1) { a += __shfl_xor_sync(0xffffffffu, a, o); b += __shfl_xor_sync(0xffffffffu, b, o); }
        if (lane == 0) {
            T* mid = slot == p.sh.top ? static_cast<T*>(p.shared_mid) + (size_t)row * p.shared_stride : static_cast<T*>(p.mid) + (size_t)(row * p.sh.top + slot) * p.mid_stride;
            if (GATED) rt_put(mid + f, gated_activation(b, a, p.act));
            else {
                rt_put(mid + f, gelu_erf(a));
                if (f + 1 < (slot == p.sh.top ? p.sh.shared_ff : p.sh.ff)) rt_put(mid + f + 1, gelu_erf(b));
            }
        }
    }
}

// CTA (share of the outputs, row): mid rows of all chosen experts, weighted, in shared memory; two warps per output, each with
// half of the 16-byte chunks of the chosen experts' rows, those of the shared feed-forward behind them.
constexpr int kDownUnroll = 8, kDownWarps = 2;
template <typename T, bool MORE>
__global__ void __launch_bounds__(kRtThreads) routed_down_kernel(const RoutedParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float rt_smem[];   // [top][mid_ld], [shared_ld]
    __shared__ float part[kRtWarps];
    __shared__ int sel[kMaxTop];
    __shared__ float weight[kMaxTop];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, row = blockIdx.y, all_top = p.sh.top;
    if (tid < all_top) { sel[tid] = p.sel[row * all_top + tid]; weight[tid] = p.weight[row * all_top + tid]; }
    __syncthreads();
    int top = all_top;         // experts with tensors come first
    float through = 0.f;       // weight of the others
    if (MORE && p.sh.identity)
        while (top > 0 && sel[top - 1] >= p.sh.experts) through += weight[--top];
    const T* input = static_cast<const T*>(p.x) + (size_t)row * p.x_stride;
    const int chunks = p.mid_ld >> 3, routed = chunks * top, all = routed + (p.shared_ld >> 3), half = warp % kDownWarps;
    uint4 v[kDownUnroll];
    auto load = [&](int n, int c0) {
        int t = min(c0 / chunks, top), c = c0 - t * chunks;
#pragma unroll
        for (int j = 0; j < kDownUnroll; ++j) {
            const bool live = n < p.sh.width && (t < top || c < all - routed);
            const __nv_bfloat16* src = t < top ? p.down + ((size_t)sel[t] * p.sh.width + n) * p.mid_ld : p.shared_down + (size_t)n * p.shared_ld;
            v[j] = live ? rt_stream(src + 8 * c) : make_uint4(0, 0, 0, 0);
            c += 32 * kDownWarps;
            while (t < top && c >= chunks) { c -= chunks; ++t; }
        }
    };
    const int first = half * 32 + lane;
    int n = (blockIdx.x * kRtWarps + warp) / kDownWarps;
    load(n, first);   // the first weights are on their way while the activations are gathered
    const float shared_w = p.shared_ld ? shared_weight(p, row) : 0.f;
    for (int i = tid; i < all; i += kRtThreads) {   // eight activations each, times their weight; zeros in the padding
        const int t = min(i / chunks, top), c = 8 * (i - t * chunks), ff = t < top ? p.sh.ff : p.sh.shared_ff;
        const T* mid = t < top ? static_cast<const T*>(p.mid) + (size_t)(row * all_top + t) * p.mid_stride : static_cast<const T*>(p.shared_mid) + (size_t)row * p.shared_stride;
        const float w = t < top ? weight[t] : shared_w;
        float f[8];
        rt_get8(mid + c, f);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] = c + e < ff ? f[e] * w : 0.f;
        *reinterpret_cast<float4*>(rt_smem + 8 * i) = make_float4(f[0], f[1], f[2], f[3]);
        *reinterpret_cast<float4*>(rt_smem + 8 * i + 4) = make_float4(f[4], f[5], f[6], f[7]);
    }
    __syncthreads();
    const int step = gridDim.x * kRtWarps / kDownWarps, rounds = (p.sh.width + step - 1) / step;
    for (int it = 0; it < rounds; ++it, n += step) {
        float acc = 0.f;
        for (int c0 = first; c0 < all; c0 += 32 * kDownWarps * kDownUnroll) {
            if (it > 0 || c0 != first) load(n, c0);
#pragma unroll
            for (int j = 0; j < kDownUnroll; ++j) {
                const int i = c0 + 32 * kDownWarps * j;
                if (i < all) acc = rt_dot8(v[j], rt_smem + 8 * i, acc);
            }
        }
        for (int o = 16; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
        if (lane == 0) part[warp] = acc;
        __syncthreads();
        if (lane == 0 && half == 0 && n < p.sh.width) {
            float total = 0.f;
#pragma unroll
            for (int w = 0; w < kDownWarps; ++w) total += part[warp + w];
            if (MORE && p.sh.identity) total = fmaf(through, rt_get(input + n), total);
            p.out[(size_t)row * p.out_stride + n] = total;
        }
        __syncthreads();
    }
}

// ---- many rows --------------------------------------------------------------------------------------------------------
// A warp per row; an expert's rows are numbered as they come.
constexpr int kChooseWarps = 4;
__global__ void __launch_bounds__(kChooseWarps * 32) routed_choose_kernel(const RoutedParams p) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float rt_smem[];
    __shared__ int sel[kChooseWarps][kMaxTop];
    __shared__ float weight[kChooseWarps][kMaxTop];
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, row = blockIdx.x * kChooseWarps + warp;
    if (row >= p.m) return;
    float* s = rt_smem + (size_t)warp * (2 * p.sh.scored() + p.sh.groups);
    choose<32, true>(p, p.z + (size_t)row * p.z_stride, s, s + p.sh.scored(), s + p.sh.scored() + p.sh.groups, sel[warp], weight[warp], lane);
    for (int t = lane; t < p.sh.top; t += 32) {
        p.sel[row * p.sh.top + t] = sel[warp][t];
        p.weight[row * p.sh.top + t] = weight[warp][t];
        p.rank[row * p.sh.top + t] = sel[warp][t] < p.sh.experts ? (int)atomicAdd(p.counts + sel[warp][t], 1u) : -1;
    }
}

// Every CTA works out where each expert's rows start; then a warp per (row, slot) copies the row to its place, which replaces
// its rank. CTA 0 also writes the table of tiles.
__global__ void __launch_bounds__(kRtThreads) routed_sort_kernel(const RoutedParams p) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ int start[kMaxExperts], tile0[kMaxExperts], warp_rows[kRtWarps], warp_tiles[kRtWarps];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, E = p.sh.experts;
    constexpr int PER = kMaxExperts / kRtThreads;   // experts per thread
    int c[PER], rows = 0, tiles = 0;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int e = tid * PER + j;
        c[j] = e < E ? (int)__ldcg(p.counts + e) : 0;
        rows += c[j];
        tiles += (c[j] + p.bn - 1) / p.bn;
    }
    int r = rows, t = tiles;
    for (int o = 1; o < 32; o <<= 1) {
        const int a = __shfl_up_sync(0xffffffffu, r, o), b = __shfl_up_sync(0xffffffffu, t, o);
        if (lane >= o) { r += a; t += b; }
    }
    if (lane == 31) { warp_rows[warp] = r; warp_tiles[warp] = t; }
    __syncthreads();
    for (int w = 0; w < warp; ++w) { r += warp_rows[w]; t += warp_tiles[w]; }
    r -= rows; t -= tiles;
#pragma unroll
    for (int j = 0; j < PER; ++j) {
        const int e = tid * PER + j;
        start[e] = r; tile0[e] = t;
        r += c[j]; t += (c[j] + p.bn - 1) / p.bn;
    }
    __syncthreads();
    if (blockIdx.x == 0) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int e = tid * PER + j;
            for (int i = 0; i * p.bn < c[j]; ++i) p.tiles[tile0[e] + i] = make_int4(e, start[e] + i * p.bn, min(p.bn, c[j] - i * p.bn), 0);
        }
        int used = 0;
        for (int w = 0; w < kRtWarps; ++w) used += warp_tiles[w];
        for (int i = used + tid; i < p.max_tiles; i += kRtThreads) p.tiles[i] = make_int4(0, 0, 0, 0);
    }
    const int chunks = p.sorted_stride >> 3, all = p.m * p.sh.top;
    for (int a = blockIdx.x * kRtWarps + warp; a < all; a += gridDim.x * kRtWarps) {
        if (p.sel[a] >= p.sh.experts) continue;   // hands its input through
        const int at = start[p.sel[a]] + p.rank[a];
        const uint4* src = reinterpret_cast<const uint4*>(static_cast<const __nv_bfloat16*>(p.x) + (size_t)(a / p.sh.top) * p.x_stride);
        uint4* dst = reinterpret_cast<uint4*>(p.sorted + (size_t)at * p.sorted_stride);
        for (int i = lane; i < chunks; i += 32) dst[i] = src[i];
        __syncwarp();
        if (lane == 0) p.rank[a] = at;
    }
}

__global__ void __launch_bounds__(kRtThreads) routed_sum_kernel(const RoutedParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int row = blockIdx.y, i = (blockIdx.x * kRtThreads + threadIdx.x) * 4;
    if (blockIdx.x == 0 && blockIdx.y == 0)
        for (int e = threadIdx.x; e < p.sh.experts; e += kRtThreads) p.counts[e] = 0;
    if (i >= p.sh.width) return;
    float4 v = make_float4(0.f, 0.f, 0.f, 0.f);
    for (int t = 0; t < p.sh.top; ++t) {
        const float w = p.weight[row * p.sh.top + t];
        const int at = p.rank[row * p.sh.top + t];
        float4 y;   // (rows are padded to 8)
        if (at >= 0) y = *reinterpret_cast<const float4*>(p.y + (size_t)at * p.y_stride + i);
        else {
            const uint2 x = *reinterpret_cast<const uint2*>(static_cast<const __nv_bfloat16*>(p.x) + (size_t)row * p.x_stride + i);
            y = make_float4(rt_lo(x.x), rt_hi(x.x), rt_lo(x.y), rt_hi(x.y));
        }
        v.x = fmaf(w, y.x, v.x); v.y = fmaf(w, y.y, v.y); v.z = fmaf(w, y.z, v.z); v.w = fmaf(w, y.w, v.w);
    }
    if (p.shared_y) {
        const float w = shared_weight(p, row);
        const float4 y = *reinterpret_cast<const float4*>(p.shared_y + (size_t)row * p.shared_y_stride + i);
        v.x = fmaf(w, y.x, v.x); v.y = fmaf(w, y.y, v.y); v.z = fmaf(w, y.z, v.z); v.w = fmaf(w, y.w, v.w);
    }
    float* o = p.out + (size_t)row * p.out_stride + i;
    const float r[4] = {v.x, v.y, v.z, v.w};
    for (int j = 0; j < 4 && i + j < p.sh.width; ++j) o[j] = r[j];
}

// ---- launches ---------------------------------------------------------------------------------------------------------
int up8(int v) { return (v + 7) / 8 * 8; }
size_t up256(size_t v) { return (v + 255) / 256 * 256; }
bool few(int m, bool f32) { return f32 || m <= kRtFewRows; }
struct RoutedScratch { size_t sel, weight, rank, tiles, mid, sorted, y, shared_mid, shared_y, total; };
RoutedScratch layout(const RoutedShape& s, int m, bool f32) {
    RoutedScratch l;
    const size_t a = (size_t)m * s.top;
    l.sel = 0;
    l.weight = l.sel + up256(a * 4);
    l.rank = l.weight + up256(a * 4);
    l.tiles = l.rank + up256(a * 4);
    l.mid = l.tiles + (few(m, f32) ? 0 : up256((size_t)grouped_max_tiles((int)a, s.experts) * 16));
    l.sorted = l.mid + up256(a * up8(s.ff) * (f32 ? 4 : 2));
    l.y = l.sorted + (few(m, f32) ? 0 : up256(a * up8(s.width) * 2));
    l.shared_mid = l.y + (few(m, f32) ? 0 : up256(a * up8(s.width) * 4));
    l.shared_y = l.shared_mid + up256((size_t)m * up8(s.shared_ff) * (f32 ? 4 : 2));
    l.total = l.shared_y + (few(m, f32) || !s.shared_ff ? 0 : up256((size_t)m * up8(s.width) * 4));
    return l;
}
constexpr size_t kRtMaxSmem = 200 * 1024;
size_t gate_smem(const RoutedShape& s) { return ((size_t)up8(s.width) + 2 * s.scored() + s.groups) * 4; }
size_t down_smem(const RoutedShape& s) { return ((size_t)s.top * up8(s.ff) + up8(s.shared_ff)) * 4; }

template <typename T, bool MORE>
int few_rows(const RoutedParams& p, cudaStream_t s, int* launches) {
    // up to four CTAs per SM, all with the same number of rounds
    const bool gated = p.gate != nullptr;
    const int units = p.sh.top * routed_units(p.sh.ff, gated) + routed_units(p.sh.shared_ff, gated);
    const int most = std::max(1, (4 * 148 + p.m - 1) / p.m), rounds = (units + kRtWarps * most - 1) / (kRtWarps * most), gx = (units + kRtWarps * rounds - 1) / (kRtWarps * rounds);
    cudaError_t e = gated ? launch_k(routed_gate_kernel<T, true, MORE>, dim3(gx, p.m), dim3(kRtThreads), gate_smem(p.sh), s, p)
                          : launch_k(routed_gate_kernel<T, false, MORE>, dim3(gx, p.m), dim3(kRtThreads), gate_smem(p.sh), s, p);
    if (e != cudaSuccess) return cuda_fail(e, "routed gate launch");
    const int outs = (p.sh.width * kDownWarps + kRtWarps - 1) / kRtWarps, dx = std::max(1, std::min(outs, (4 * 148 + p.m - 1) / p.m));
    e = launch_k(routed_down_kernel<T, MORE>, dim3(dx, p.m), dim3(kRtThreads), down_smem(p.sh), s, p);
    if (e != cudaSuccess) return cuda_fail(e, "routed down launch");
    *launches += 2;
    return SWLM_OK;
}

}  // namespace

template <typename T, bool MORE>
static int few_attr() {
    SWLM_CUDA(cudaFuncSetAttribute(routed_gate_kernel<T, true, MORE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kRtMaxSmem));
    SWLM_CUDA(cudaFuncSetAttribute(routed_gate_kernel<T, false, MORE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kRtMaxSmem));
    SWLM_CUDA(cudaFuncSetAttribute(routed_down_kernel<T, MORE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kRtMaxSmem));
    return SWLM_OK;
}
int routed_init() {
    int rc;
    if ((rc = few_attr<float, false>()) || (rc = few_attr<float, true>()) || (rc = few_attr<__nv_bfloat16, false>()) || (rc = few_attr<__nv_bfloat16, true>())) return rc;
    return SWLM_OK;
}
bool routed_supported(const RoutedShape& s) {
    return s.experts > 0 && s.identity >= 0 && s.scored() <= kMaxExperts && s.top > 0 && s.top <= kMaxTop && s.groups > 0 && s.scored() % s.groups == 0 && s.keep > 0 &&
           s.keep <= s.groups && (!s.identity || s.groups == 1) && s.top <= s.keep * (s.scored() / s.groups) && s.width > 0 && s.ff > 0 && s.shared_ff >= 0 && gate_smem(s) <= kRtMaxSmem && down_smem(s) <= kRtMaxSmem;
}
size_t routed_scratch_bytes(const RoutedShape& s, int m, bool f32) { return layout(s, m, f32).total; }

int launch_routed(const RoutedLaunch& a, cudaStream_t s, int* launches) {
    if (a.m <= 0) return SWLM_OK;
    const RoutedScratch l = layout(a.shape, a.m, a.f32);
    RoutedParams p{};
    p.sh = a.shape; p.scale = a.scale; p.act = a.act; p.m = a.m; p.x = a.x; p.x_stride = a.x_stride; p.z = a.z; p.z_stride = a.z_stride;
    p.correction = a.correction;
    p.softmax = a.softmax; p.group_best = a.group_best; p.raw_weights = a.raw_weights;
    p.gate = a.gate ? a.gate->data : nullptr; p.up = a.up->data; p.down = a.down->data; p.in_ld = a.up->ld; p.mid_ld = a.down->ld; p.out = a.out; p.out_stride = a.out_stride;
    p.sel = reinterpret_cast<int*>(a.scratch + l.sel); p.weight = reinterpret_cast<float*>(a.scratch + l.weight); p.rank = reinterpret_cast<int*>(a.scratch + l.rank);
    p.counts = a.counts; p.mid = a.scratch + l.mid; p.mid_stride = up8(a.shape.ff);
    const bool shared = a.shape.shared_ff > 0;
    if (shared) { p.shared_up = a.shared_up->data; p.shared_down = a.shared_down->data; p.shared_ld = a.shared_down->ld; }
    p.shared_mid = a.scratch + l.shared_mid; p.shared_stride = up8(a.shape.shared_ff);
    if (few(a.m, a.f32)) {
        if (p.correction || a.shape.identity) return a.f32 ? few_rows<float, true>(p, s, launches) : few_rows<__nv_bfloat16, true>(p, s, launches);
        return a.f32 ? few_rows<float, false>(p, s, launches) : few_rows<__nv_bfloat16, false>(p, s, launches);
    }

    const int all = a.m * a.shape.top, E = a.shape.experts;
    p.sorted = reinterpret_cast<__nv_bfloat16*>(a.scratch + l.sorted); p.sorted_stride = up8(a.shape.width);
    p.y = reinterpret_cast<float*>(a.scratch + l.y); p.y_stride = up8(a.shape.width);
    p.tiles = reinterpret_cast<int4*>(a.scratch + l.tiles); p.bn = grouped_bn(all, E); p.max_tiles = grouped_max_tiles(all, E);
    if ((a.x_stride & 7) || (reinterpret_cast<uintptr_t>(a.x) & 15)) { set_error("routed feed-forward: rows must be 16-byte aligned"); return SWLM_ERR_INVALID; }
    cudaError_t e = launch_k(routed_choose_kernel, dim3((a.m + kChooseWarps - 1) / kChooseWarps), dim3(kChooseWarps * 32), (size_t)kChooseWarps * (2 * a.shape.scored() + a.shape.groups) * 4, s, p);
    if (e != cudaSuccess) return cuda_fail(e, "routed choice launch");
    e = launch_k(routed_sort_kernel, dim3(std::min((all + kRtWarps - 1) / kRtWarps, 4 * 148)), dim3(kRtThreads), 0, s, p);
    if (e != cudaSuccess) return cuda_fail(e, "routed sort launch");
    ProductLaunch g;
    if (a.gate) { g.w = a.gate; g.w2 = a.up; g.act = a.act; }
    else { g.w = a.up; g.out.gelu = 1; }
    g.m = all; g.x = p.sorted; g.x_stride = p.sorted_stride; g.status = a.status;
    g.experts = E; g.tiles = p.tiles; g.max_tiles = p.max_tiles; g.group_bn = p.bn;
    g.out.y[0] = p.mid; g.out.stride[0] = p.mid_stride;
    for (int& end : g.out.end) end = a.shape.ff;
    int rc = launch_product(g, s);
    if (rc) return rc;
    ProductLaunch d = g;
    d.w = a.down; d.w2 = nullptr; d.out.gelu = 0; d.x = p.mid; d.x_stride = p.mid_stride;
    d.out.y[0] = p.y; d.out.stride[0] = p.y_stride; d.out.f32[0] = 1;
    for (int& end : d.out.end) end = a.shape.width;
    if ((rc = launch_product(d, s))) return rc;
    if (shared) {
        ProductLaunch u;
        u.w = a.shared_up; u.m = a.m; u.x = a.x; u.x_stride = a.x_stride; u.part = a.part; u.part_floats = a.part_floats; u.status = a.status;
        u.out.y[0] = p.shared_mid; u.out.stride[0] = p.shared_stride; u.out.gelu = 1;
        for (int& end : u.out.end) end = a.shape.shared_ff;
        if ((rc = launch_product(u, s))) return rc;
        *launches += product_launch_count(u);
        ProductLaunch w = u;
        w.w = a.shared_down; w.x = p.shared_mid; w.x_stride = p.shared_stride;
        p.shared_y = reinterpret_cast<const float*>(a.scratch + l.shared_y); p.shared_y_stride = up8(a.shape.width);
        w.out.y[0] = a.scratch + l.shared_y; w.out.stride[0] = p.shared_y_stride; w.out.f32[0] = 1; w.out.gelu = 0;
        for (int& end : w.out.end) end = a.shape.width;
        if ((rc = launch_product(w, s))) return rc;
        *launches += product_launch_count(w);
    }
    e = launch_k(routed_sum_kernel, dim3((a.shape.width + kRtThreads * 4 - 1) / (kRtThreads * 4), a.m), dim3(kRtThreads), 0, s, p);
    if (e != cudaSuccess) return cuda_fail(e, "routed sum launch");
    *launches += 5;
    return SWLM_OK;
}

}  // namespace swlm
