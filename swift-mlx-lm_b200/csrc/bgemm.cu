// Dense products of fp32-stream plans: Y[m][n] = X[m][k] . W[n][k]^T with bf16 weights and fp32 accumulation.
//
//   bgemv_kernel     1..kGemvRows activation rows: the weights are streamed once from HBM with 16-byte loads, four weight
//                    rows per warp and K cut across the warps of a CTA; the norm in front of the product can run in the
//                    prologue, gate and up in one launch with the gated activation in the epilogue. Activations bf16 or fp32
//                    (with fp32 ones the product is a true fp32 product: a bf16 weight is exact in fp32).
//   bgemm_tc_kernel  more rows, bf16 activations: tcgen05.mma with both operands staged by TMA (128-byte swizzle), two tiles
//                    of 128 weight rows side by side in tensor memory, K cut across CTAs when there are few tiles. The two
//                    tiles are 256 consecutive rows, or 128 rows of gate and the same rows of up. Grouped form: activation rows
//                    sorted by expert, a device table names the expert and the rows of every tile.
//   sgemm_kernel     more rows, fp32 activations: fp32 FMAs on 64 x 64 tiles.
#include <algorithm>
#include <cstdlib>

#include "swlm_internal.h"
#include "tc_device.cuh"

namespace swlm {
namespace {

__device__ __forceinline__ float b_lo(unsigned w) { return __uint_as_float(w << 16); }
__device__ __forceinline__ float b_hi(unsigned w) { return __uint_as_float(w & 0xFFFF0000u); }
__device__ __forceinline__ uint4 ldg_stream(const void* p) {
    uint4 v;
    asm volatile("ld.global.nc.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}

// Where the results of one weight row go: that of activation row m is m * stride bytes behind y.
struct ProductRow { unsigned char* y; size_t stride; bool f32; float bias; };
template <bool BIASED>
__device__ __forceinline__ ProductRow product_row(const ProductOut& o, int row) {
    void* y = o.y[0];
    const __nv_bfloat16* bias = BIASED ? o.bias[0] : nullptr;
    int first = 0, stride = o.stride[0], f32 = o.f32[0];
#pragma unroll
    for (int q = 1; q < kMaxProductSegs; ++q)
        if (q < o.count && row >= o.end[q - 1]) { y = o.y[q]; first = o.end[q - 1]; stride = o.stride[q]; f32 = o.f32[q]; if (BIASED) bias = o.bias[q]; }
    const int size = f32 ? 4 : 2;
    return ProductRow{static_cast<unsigned char*>(y) + (ptrdiff_t)(row - first) * size, (size_t)stride * size, f32 != 0,
                      BIASED && bias && row < o.end[o.count - 1] ? __bfloat162float(bias[row - first]) : 0.f};
}
template <bool BIASED>
__device__ __forceinline__ void product_store(const ProductOut& o, int m, int row, float val) {
    const ProductRow r = product_row<BIASED>(o, row);
    if (BIASED) val += r.bias;
    if (o.softcap > 0.f) val = o.softcap * tanhf(val / o.softcap);
    if (o.gelu) val = gelu_erf(val);
    if (r.f32) *reinterpret_cast<float*>(r.y + m * r.stride) = val;
    else *reinterpret_cast<__nv_bfloat16*>(r.y + m * r.stride) = __float2bfloat16_rn(val);
}

// ---- few rows ---------------------------------------------------------------------------------------------------------
constexpr int kGemvRows = 4;
constexpr int kGemvThreads = 256, kGemvWarps = kGemvThreads / 32;
constexpr int kGemvUnroll = 4;                       // 16-byte loads in flight per weight row and lane
constexpr size_t kGemvMaxSmem = 200 * 1024;

struct GemvParams {
    const __nv_bfloat16* w; const __nv_bfloat16* w2;
    int ld, n, k, m;
    GatedAct act;
    const void* x; int x_stride;
    const void* x2; int x2_stride, split;        // rows from `split` on (a multiple of four) meet a second input
    StreamNorm norm;
    ProductOut out;
};

__device__ __forceinline__ float cta_sum(float v, float* red) {
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.f;
#pragma unroll
    for (int i = 0; i < kGemvWarps; ++i) total += red[i];
    __syncthreads();
    return total;
}
__device__ __forceinline__ void put_x(float* p, float v) { *p = v; }
__device__ __forceinline__ void put_x(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
// eight consecutive activations
__device__ __forceinline__ void get_x8(const float* p, float (&f)[8]) {
    const float4 a = *reinterpret_cast<const float4*>(p), b = *reinterpret_cast<const float4*>(p + 4);
    f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
}
__device__ __forceinline__ void get_x8(const __nv_bfloat16* p, float (&f)[8]) {
    const uint4 v = *reinterpret_cast<const uint4*>(p);
    f[0] = b_lo(v.x); f[1] = b_hi(v.x); f[2] = b_lo(v.y); f[3] = b_hi(v.y); f[4] = b_lo(v.z); f[5] = b_hi(v.z); f[6] = b_lo(v.w); f[7] = b_hi(v.w);
}

// A warp takes groups of four weight rows (GATED: two of gate and the same two of up); WK warps share a group and cut K. MORE: biases
// and a second input are possible (others do without that code: its instructions have to be fetched, too).
template <typename T, int MR, int WK, bool GATED, bool MORE>
__global__ void __launch_bounds__(kGemvThreads, 2) bgemv_kernel(const GemvParams p) {
    pdl_launch_dependents();
    extern __shared__ __align__(16) unsigned char gemv_raw[];
    __shared__ float red[kGemvWarps];
    __shared__ float part[kGemvWarps][4 * MR];
    T* xs = reinterpret_cast<T*>(gemv_raw);                    // [MR][ld]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int kw = warp % WK, rg = warp / WK;
    constexpr int ROWS = GATED ? 2 : 4;                         // output rows of a group
    const int groups = (p.n + ROWS - 1) / ROWS, per_cta = kGemvWarps / WK;
    const int chunks = p.ld >> 3;                               // 16-byte chunks per weight row
    constexpr int STEP = 32 * WK;

    auto row_ptr = [&](int group, int i) -> const __nv_bfloat16* {
        const int r = min(group * ROWS + (GATED ? (i & 1) : i), p.n - 1);
        return (GATED && i >= 2 ? p.w2 : p.w) + (size_t)r * p.ld;
    };
    uint4 wv[4][kGemvUnroll];
    auto load = [&](int group, int c0) {
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const __nv_bfloat16* row = row_ptr(group, i);
#pragma unroll
            for (int u = 0; u < kGemvUnroll; ++u) {
                const int c = c0 + u * STEP;
                wv[i][u] = c < chunks ? ldg_stream(row + 8 * c) : make_uint4(0, 0, 0, 0);
            }
        }
    };
    const int first_chunk = kw * 32 + lane;
    int group = blockIdx.x * per_cta + rg;
    // the first weights (and a norm's) do not depend on the preceding kernel
    if (group < groups) load(group, first_chunk);
    // a norm over at most 4096 entries keeps its row in registers: entries 4 tid + 1024 j
    const bool norm_regs = p.norm.mode && p.k <= 16 * kGemvThreads && (p.k & 3) == 0;
    uint2 nw[4], npw[4];
    if (norm_regs) {
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int i = 4 * tid + 4 * kGemvThreads * j;
            nw[j] = i < p.k ? __ldg(reinterpret_cast<const uint2*>(p.norm.w + i)) : make_uint2(0, 0);
            npw[j] = i < p.k && p.norm.w_post ? __ldg(reinterpret_cast<const uint2*>(p.norm.w_post + i)) : make_uint2(0, 0);
        }
    }
    pdl_wait();

    // ---- activations to shared memory: plain rows, or the norm in front of the product (every CTA computes it; CTA 0 stores
    // the new residual) ----
    if (norm_regs) {
        for (int m = 0; m < MR; ++m) {
            T* xr = xs + (size_t)m * p.ld;
            const float* in = p.norm.in + (size_t)m * p.norm.in_stride;
            const float* res = p.norm.res_in ? p.norm.res_in + (size_t)m * p.norm.res_stride : nullptr;
            const __nv_bfloat16* joins = p.norm.table ? p.norm.table_row(m, p.k) : nullptr;
            float h[4][4], rv[4][4];
            float ss = 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int i = 4 * tid + 4 * kGemvThreads * j;
                const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
                const float4 a = i < p.k ? __ldcg(reinterpret_cast<const float4*>(in + i)) : z, b = i < p.k && res ? __ldcg(reinterpret_cast<const float4*>(res + i)) : z;
                h[j][0] = a.x; h[j][1] = a.y; h[j][2] = a.z; h[j][3] = a.w;
                rv[j][0] = b.x; rv[j][1] = b.y; rv[j][2] = b.z; rv[j][3] = b.w;
                if (joins && i < p.k) {
                    const uint2 v = __ldg(reinterpret_cast<const uint2*>(joins + i));
                    rv[j][0] += b_lo(v.x) * p.norm.table_scale; rv[j][1] += b_hi(v.x) * p.norm.table_scale;
                    rv[j][2] += b_lo(v.y) * p.norm.table_scale; rv[j][3] += b_hi(v.y) * p.norm.table_scale;
                }
            }
            if (p.norm.w_post) {
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int e = 0; e < 4; ++e) ss = fmaf(h[j][e], h[j][e], ss);
                const float sc = 1.0f / sqrtf(cta_sum(ss, red) / (float)p.k + p.norm.eps);
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float wf[4] = {b_lo(npw[j].x), b_hi(npw[j].x), b_lo(npw[j].y), b_hi(npw[j].y)};
#pragma unroll
                    for (int e = 0; e < 4; ++e) h[j][e] = h[j][e] * sc * (wf[e] + p.norm.weight_bias);
                }
            }
            ss = 0.f;
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) { h[j][e] += rv[j][e]; ss = fmaf(h[j][e], h[j][e], ss); }
            // (entries past k: zero input, zero residual)
            const float sc = 1.0f / sqrtf(cta_sum(ss, red) / (float)p.k + p.norm.eps);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int i = 4 * tid + 4 * kGemvThreads * j;
                const float wf[4] = {b_lo(nw[j].x), b_hi(nw[j].x), b_lo(nw[j].y), b_hi(nw[j].y)};
                if (i < p.k) {
                    if (p.norm.res_out && blockIdx.x == 0)
                        *reinterpret_cast<float4*>(p.norm.res_out + (size_t)m * p.norm.res_stride + i) = make_float4(h[j][0], h[j][1], h[j][2], h[j][3]);
#pragma unroll
                    for (int e = 0; e < 4; ++e) put_x(xr + i + e, h[j][e] * sc * (wf[e] + p.norm.weight_bias));
                } else if (i < p.ld) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) put_x(xr + i + e, 0.f);
                }
            }
        }
    } else if (p.norm.mode) {
        for (int m = 0; m < MR; ++m) {
            T* xr = xs + (size_t)m * p.ld;
            float* rowf = reinterpret_cast<float*>(gemv_raw + (size_t)MR * p.ld * sizeof(T));
            const float* in = p.norm.in + (size_t)m * p.norm.in_stride;
            const float* res = p.norm.res_in ? p.norm.res_in + (size_t)m * p.norm.res_stride : nullptr;
            const __nv_bfloat16* joins = p.norm.table ? p.norm.table_row(m, p.k) : nullptr;
            float post_scale = 1.f;
            float ss = 0.f;
            for (int i = tid; i < p.k; i += kGemvThreads) { const float v = in[i]; rowf[i] = v; ss = fmaf(v, v, ss); }
            if (p.norm.w_post) post_scale = 1.0f / sqrtf(cta_sum(ss, red) / (float)p.k + p.norm.eps);
            ss = 0.f;
            for (int i = tid; i < p.k; i += kGemvThreads) {
                float h = rowf[i];
                if (p.norm.w_post) h = h * post_scale * (__bfloat162float(p.norm.w_post[i]) + p.norm.weight_bias);
                if (res) h += res[i];
                if (joins) h += __bfloat162float(joins[i]) * p.norm.table_scale;
                if (p.norm.res_out && blockIdx.x == 0) p.norm.res_out[(size_t)m * p.norm.res_stride + i] = h;
                rowf[i] = h;
                ss = fmaf(h, h, ss);
            }
            const float sc = 1.0f / sqrtf(cta_sum(ss, red) / (float)p.k + p.norm.eps);
            for (int i = tid; i < p.ld; i += kGemvThreads)
                put_x(xr + i, i < p.k ? rowf[i] * sc * (__bfloat162float(p.norm.w[i]) + p.norm.weight_bias) : 0.f);
        }
    } else {
        for (int m = 0; m < MR; ++m) {
            const T* src = static_cast<const T*>(p.x) + (size_t)m * p.x_stride;
            for (int i = tid; i < p.ld; i += kGemvThreads) { T v = T(0.0f); if (i < p.k) v = src[i]; xs[(size_t)m * p.ld + i] = v; }
        }
        if (MORE && p.x2)
            for (int m = 0; m < MR; ++m) {
                const T* src = static_cast<const T*>(p.x2) + (size_t)m * p.x2_stride;
                for (int i = tid; i < p.ld; i += kGemvThreads) { T v = T(0.0f); if (i < p.k) v = src[i]; xs[(size_t)(MR + m) * p.ld + i] = v; }
            }
    }
    __syncthreads();

    const int rounds = (groups + gridDim.x * per_cta - 1) / (gridDim.x * per_cta);
    for (int it = 0; it < rounds; ++it) {
        float acc[4][MR];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int m = 0; m < MR; ++m) acc[i][m] = 0.f;
        const bool live = group < groups;
        const T* xg = xs + (MORE && p.x2 && group * ROWS >= p.split ? (size_t)MR * p.ld : 0);
        if (live) {
            for (int c0 = first_chunk; c0 < chunks; c0 += STEP * kGemvUnroll) {
                if (it > 0 || c0 != first_chunk) load(group, c0);
#pragma unroll
                for (int u = 0; u < kGemvUnroll; ++u) {
                    const int c = c0 + u * STEP;
                    if (c < chunks) {
                        float wf[4][8];
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            const uint4 v = wv[i][u];
                            wf[i][0] = b_lo(v.x); wf[i][1] = b_hi(v.x); wf[i][2] = b_lo(v.y); wf[i][3] = b_hi(v.y);
                            wf[i][4] = b_lo(v.z); wf[i][5] = b_hi(v.z); wf[i][6] = b_lo(v.w); wf[i][7] = b_hi(v.w);
                        }
#pragma unroll
                        for (int m = 0; m < MR; ++m) {
                            float xf[8];
                            get_x8(xg + (size_t)m * p.ld + 8 * c, xf);
#pragma unroll
                            for (int i = 0; i < 4; ++i)
#pragma unroll
                                for (int e = 0; e < 8; ++e) acc[i][m] = fmaf(wf[i][e], xf[e], acc[i][m]);
                        }
                    }
                }
            }
        }
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int m = 0; m < MR; ++m)
                for (int o = 16; o > 0; o >>= 1) acc[i][m] += __shfl_xor_sync(0xffffffffu, acc[i][m], o);
        if (WK > 1) {
            if (lane == 0) {
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int m = 0; m < MR; ++m) part[warp][i * MR + m] = acc[i][m];
            }
            __syncthreads();
            if (kw == 0) {
#pragma unroll
                for (int i = 0; i < 4; ++i)
#pragma unroll
                    for (int m = 0; m < MR; ++m) {
                        float v = 0.f;
#pragma unroll
                        for (int q = 0; q < WK; ++q) v += part[rg * WK + q][i * MR + m];
                        acc[i][m] = v;
                    }
            }
            __syncthreads();
        }
        if (live && kw == 0) {
            // lane (i * MR + m) stores one value
#pragma unroll
            for (int m = 0; m < MR; ++m) {
                if (GATED) {
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        const int row = group * 2 + i;
                        if (lane == i * MR + m && row < p.n) product_store<false>(p.out, m, row, gated_activation(acc[i][m], acc[2 + i][m], p.act));
                    }
                } else {
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        const int row = group * 4 + i;
                        if (lane == i * MR + m && row < p.n) product_store<MORE>(p.out, m, row, acc[i][m]);
                    }
                }
            }
        }
        group += gridDim.x * per_cta;
    }
}

// ---- many rows, bf16: tcgen05 -----------------------------------------------------------------------------------------
constexpr int kTileRows = 128;       // weight rows of one accumulator = UMMA M
constexpr int kTcK = 64;             // columns per stage = one 128-byte swizzle row
constexpr int kTcEpilogueWarps = 8;
constexpr int kTcWarps = 2 + kTcEpilogueWarps;   // TMA, MMA, epilogue
constexpr int kTcBlock = kTcWarps * 32;

struct TcParams {
    int n, m, steps;                 // weight rows, activation rows, 64-column steps of K
    int split;                       // weight rows from here on (a multiple of 256) meet the activations of wmap2's place
    int split_steps;                 // steps per K range (gridDim.z ranges); == steps when K is not cut
    GatedAct act;
    const int4* tiles;               // grouped form: (expert, first row, rows, 0) of tile blockIdx.x; n = rows of one expert's matrix
    ProductOut out;
    float* part;                     // [range][gated ? 2 : 1][m][n] when K is cut
    int* status;
};

// kind::f16: D fp32, A = B = bf16, both K-major, M = 128
__host__ __device__ constexpr unsigned tc_idesc(int bn) {
    return (1u << 4) | (1u << 7) | (1u << 10) | ((unsigned)(bn >> 3) << 17) | ((unsigned)(kTileRows >> 4) << 24);
}
__device__ __forceinline__ void umma_bf16(unsigned d_tmem, unsigned long long a_desc, unsigned long long b_desc, unsigned idesc, unsigned accumulate) {
    asm volatile(
        "{\n\t.reg .pred p;\n\t"
        "setp.ne.b32 p, %4, 0;\n\t"
        "tcgen05.mma.cta_group::1.kind::f16 [%0], %1, %2, %3, p;\n\t}"
        ::"r"(d_tmem), "l"(a_desc), "l"(b_desc), "r"(idesc), "r"(accumulate) : "memory");
}

__device__ __forceinline__ void tmem_ld16(unsigned (&v)[16], unsigned at) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0,%1,%2,%3,%4,%5,%6,%7,%8,%9,%10,%11,%12,%13,%14,%15}, [%16];"
        : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]), "=r"(v[4]), "=r"(v[5]), "=r"(v[6]), "=r"(v[7]),
          "=r"(v[8]), "=r"(v[9]), "=r"(v[10]), "=r"(v[11]), "=r"(v[12]), "=r"(v[13]), "=r"(v[14]), "=r"(v[15])
        : "r"(at) : "memory");
}

template <int BN, int STAGES, bool GATED>
__global__ void __launch_bounds__(kTcBlock) bgemm_tc_kernel(const TcParams p, const __grid_constant__ CUtensorMap xmap,
                                                           const __grid_constant__ CUtensorMap wmap, const __grid_constant__ CUtensorMap wmap2) {
    extern __shared__ __align__(1024) unsigned char tc_raw[];
    unsigned char* smem = tc_raw + ((1024 - (smem_u32(tc_raw) & 1023)) & 1023);   // swizzle atoms
    constexpr int A_BYTES = kTileRows * 128, B_BYTES = BN * 128;
    constexpr unsigned kCols = 2 * BN < 32 ? 32 : 2 * BN;
    __shared__ __align__(8) unsigned long long full_bar[STAGES], empty_bar[STAGES], done_bar;
    __shared__ unsigned tmem_base;
    __shared__ int failed;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    int tok0 = blockIdx.x * BN, tok_end = p.m, wrow0 = 0;     // wrow0: first row of the expert's matrix
    if (p.tiles) {
        pdl_wait();   // (the table is the preceding kernel's)
        const int4 tile = p.tiles[blockIdx.x];
        if (tile.z == 0) { pdl_launch_dependents(); return; }
        wrow0 = tile.x * p.n;
        tok0 = tile.y;
        tok_end = tile.y + tile.z;
    }
    const int row0 = blockIdx.y * (GATED ? kTileRows : 2 * kTileRows);
    const int nt = !GATED && row0 + kTileRows >= p.n ? 1 : 2;                       // accumulators in use
    const int stage_bytes = nt * A_BYTES + B_BYTES;
    constexpr int STAGE = 2 * A_BYTES + B_BYTES;
    const int step0 = blockIdx.z * p.split_steps;
    const int steps = min(p.split_steps, p.steps - step0);
    if (tid == 0) {
        for (int s = 0; s < STAGES; ++s) { mbar_init(&full_bar[s], 1); mbar_init(&empty_bar[s], 1); }
        mbar_init(&done_bar, 1);
        failed = 0;
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    if (warp == 1) {
        __syncwarp();
        asm volatile("tcgen05.alloc.cta_group::1.sync.aligned.shared::cta.b32 [%0], %1;" ::"r"(smem_u32(&tmem_base)), "r"(kCols) : "memory");
        asm volatile("tcgen05.relinquish_alloc_permit.cta_group::1.sync.aligned;" ::: "memory");
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
    const unsigned tmem = tmem_base;
    pdl_launch_dependents();   // behind the allocation: a successor that wants tensor memory cannot get in between

    if (warp == 0) {
        if (lane == 0) {
            // the weights of the first stages do not depend on the preceding kernel; the activations do
            const int ahead = min(STAGES, steps);
            auto weights = [&](int kt, int s) {
                const unsigned bar = smem_u32(&full_bar[s]), dst = smem_u32(smem + s * STAGE);
                mbar_expect(bar, (unsigned)stage_bytes);
                tma_load_2d(dst, &wmap, (step0 + kt) * kTcK, wrow0 + row0, bar);
                if (nt == 2) tma_load_2d(dst + A_BYTES, GATED ? &wmap2 : &wmap, (step0 + kt) * kTcK, wrow0 + (GATED ? row0 : row0 + kTileRows), bar);
            };
            auto activations = [&](int kt, int s) {
                tma_load_2d(smem_u32(smem + s * STAGE) + 2 * A_BYTES, !GATED && row0 >= p.split ? &wmap2 : &xmap, (step0 + kt) * kTcK, tok0, smem_u32(&full_bar[s]));
            };
            for (int kt = 0; kt < ahead; ++kt) weights(kt, kt);
            pdl_wait();
            for (int kt = 0; kt < ahead; ++kt) activations(kt, kt);
            int issued = ahead;
            for (int kt = ahead; kt < steps; ++kt) {
                const int s = kt % STAGES;
                if (!mbar_wait(&empty_bar[s], (unsigned)((kt / STAGES - 1) & 1))) { atomicExch(p.status, 31); failed = 1; break; }
                weights(kt, s);
                activations(kt, s);
                issued = kt + 1;
            }
            if (failed)   // copies already requested still write shared memory
                for (int kt = issued > STAGES ? issued - STAGES : 0; kt < issued; ++kt) mbar_wait(&full_bar[kt % STAGES], (unsigned)((kt / STAGES) & 1));
        }
        __syncwarp();
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr unsigned idesc = tc_idesc(BN);
            for (int kt = 0; kt < steps; ++kt) {
                const int s = kt % STAGES;
                if (!mbar_wait(&full_bar[s], (unsigned)((kt / STAGES) & 1))) { atomicExch(p.status, 32); failed = 1; break; }
                asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
                const unsigned a = smem_u32(smem + s * STAGE), b = a + 2 * A_BYTES;
#pragma unroll
                for (int j = 0; j < kTcK / 16; ++j) {
                    const unsigned acc = (kt > 0 || j > 0) ? 1u : 0u;
                    umma_bf16(tmem, umma_desc(a + 32 * j), umma_desc(b + 32 * j), idesc, acc);
                    if (nt == 2) umma_bf16(tmem + BN, umma_desc(a + A_BYTES + 32 * j), umma_desc(b + 32 * j), idesc, acc);
                }
                umma_commit(&empty_bar[s]);
            }
            umma_commit(&done_bar);   // also behind whatever was issued before a failure
        }
        __syncwarp();
    } else {
        // ---- epilogue: a warp reads the 32 accumulator lanes of its quarter (warp & 3), lane = weight row; the two warps of a
        // quarter take turns with the activation rows ----
        pdl_wait();   // the outputs may still be read by the kernel before this one
        const bool ok = mbar_wait(&done_bar, 0u);
        if (!ok) { atomicExch(p.status, 33); }
        asm volatile("tcgen05.fence::after_thread_sync;" ::: "memory");
        if (ok && !failed) {
            const int quarter = warp & 3;
            const bool cut = gridDim.z > 1;
#pragma unroll 1
            for (int t = 0; t < (GATED && !cut ? 1 : nt); ++t) {
                const int row = row0 + (GATED ? 0 : t * kTileRows) + quarter * 32 + lane;
                const ProductRow dst = cut ? ProductRow{reinterpret_cast<unsigned char*>(p.part + ((size_t)blockIdx.z * (GATED ? 2 : 1) + (GATED ? t : 0)) * p.m * p.n + row), (size_t)p.n * 4, true, 0.f}
                                           : product_row<true>(p.out, row);
#pragma unroll 1
                for (int c0 = 16 * ((warp - 2) >> 2); c0 < BN; c0 += 16 * (kTcEpilogueWarps / 4)) {
                    if (tok0 + c0 >= tok_end) break;   // uniform across the warp
                    unsigned v[16], u[16];
                    const unsigned at = tmem + ((unsigned)(quarter * 32) << 16) + (unsigned)(t * BN + c0);
                    tmem_ld16(v, at);
                    if (GATED && !cut) tmem_ld16(u, at + BN);
                    asm volatile("tcgen05.wait::ld.sync.aligned;" ::: "memory");
                    if (row < p.n) {
                        const int count = tok_end - tok0 - c0;
                        unsigned char* y = dst.y + (size_t)(tok0 + c0) * dst.stride;
#pragma unroll
                        for (int i = 0; i < 16; ++i) {
                            float val = __uint_as_float(v[i]);
                            if (GATED && !cut) val = gated_activation(val, __uint_as_float(u[i]), p.act);
                            val += dst.bias;
                            if (p.out.softcap > 0.f && !cut) val = p.out.softcap * tanhf(val / p.out.softcap);
                            if (p.out.gelu && !cut) val = gelu_erf(val);
                            if (i < count) {
                                if (dst.f32) *reinterpret_cast<float*>(y) = val;
                                else *reinterpret_cast<__nv_bfloat16*>(y) = __float2bfloat16_rn(val);
                            }
                            y += dst.stride;
                        }
                    }
                }
            }
        }
    }
    asm volatile("tcgen05.fence::before_thread_sync;" ::: "memory");
    __syncthreads();
    if (warp == 1) asm volatile("tcgen05.dealloc.cta_group::1.sync.aligned.b32 %0, %1;" ::"r"(tmem), "r"(kCols) : "memory");
}

// Sum of the K ranges in order, then the store (GATED: activation(gate sum) * up sum).
template <bool GATED>
__global__ void __launch_bounds__(256) bgemm_sum_kernel(const float* part, int ranges, int m, int n, GatedAct act, const ProductOut out) {
    pdl_launch_dependents();
    pdl_wait();
    const size_t total = (size_t)m * n;
    const int r = blockIdx.x * blockDim.x + threadIdx.x;
    if (r >= n) return;
    for (int t = blockIdx.y; t < m; t += gridDim.y) {
        const size_t i = (size_t)t * n + r;
        float a = 0.f, b = 0.f;
#pragma unroll 4
        for (int z = 0; z < ranges; ++z) {
            const float* base = part + (size_t)z * (GATED ? 2 : 1) * total;
            a += __ldcg(base + i);
            if (GATED) b += __ldcg(base + total + i);
        }
        product_store<!GATED>(out, t, r, GATED ? gated_activation(a, b, act) : a);
    }
}

// ---- many rows, fp32 --------------------------------------------------------------------------------------------------
__global__ void __launch_bounds__(256) sgemm_kernel(const __nv_bfloat16* w, int ld, int n, int k, int m, const float* x, int x_stride, const ProductOut out) {
    pdl_launch_dependents();
    pdl_wait();
    __shared__ float ws[16][68], xsm[16][68];
    const int n0 = blockIdx.x * 64, m0 = blockIdx.y * 64, tx = threadIdx.x & 15, ty = threadIdx.x >> 4;
    float acc[4][4] = {};
    for (int k0 = 0; k0 < k; k0 += 16) {
        for (int i = threadIdx.x; i < 64 * 16; i += 256) {
            const int r = i >> 4, c = i & 15;
            ws[c][r] = n0 + r < n && k0 + c < k ? __bfloat162float(w[(size_t)(n0 + r) * ld + k0 + c]) : 0.f;
            xsm[c][r] = m0 + r < m && k0 + c < k ? x[(size_t)(m0 + r) * x_stride + k0 + c] : 0.f;
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < 16; ++c) {
            float a[4], b[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) { a[i] = xsm[c][ty * 4 + i]; b[i] = ws[c][tx * 4 + i]; }
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int j = 0; j < 4; ++j) acc[i][j] = fmaf(a[i], b[j], acc[i][j]);
        }
        __syncthreads();
    }
    for (int i = 0; i < 4; ++i)
        for (int j = 0; j < 4; ++j) {
            const int mm = m0 + ty * 4 + i, nn = n0 + tx * 4 + j;
            if (mm < m && nn < n) product_store<true>(out, mm, nn, acc[i][j]);
        }
}

// ---- launches ---------------------------------------------------------------------------------------------------------
template <typename T, int MR, int WK, bool GATED, bool MORE = false>
int gemv_launch(const GemvParams& p, size_t smem, unsigned grid, cudaStream_t s) {
    static const cudaError_t attr = cudaFuncSetAttribute(bgemv_kernel<T, MR, WK, GATED, MORE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kGemvMaxSmem);
    if (attr != cudaSuccess) return cuda_fail(attr, "bgemv attributes");
    const cudaError_t e = launch_k(bgemv_kernel<T, MR, WK, GATED, MORE>, dim3(grid), dim3(kGemvThreads), smem, s, p);
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "bgemv launch");
}
template <typename T, int MR>
int gemv_pick(const GemvParams& p, bool gated, size_t smem, cudaStream_t s) {
    const int groups = (p.n + (gated ? 1 : 3)) / (gated ? 2 : 4);
    // warps that share a group: the fewest passes over the loop of 16-byte loads, a round of groups costing a little by itself
    const int max_grid = 148 * (smem > 100 * 1024 ? 1 : 2), chunks = p.ld >> 3;
    int wk = 1;
    float best = 0.f;
    for (int q = 1; q <= 8; q *= 2) {
        const int ctas = max_grid * (kGemvWarps / q), rounds = (groups + ctas - 1) / ctas, passes = (chunks + 32 * q * kGemvUnroll - 1) / (32 * q * kGemvUnroll);
        const float cost = rounds * (passes + 0.3f);
        if (q == 1 || cost < best) { best = cost; wk = q; }
    }
    const int per_cta = kGemvWarps / wk;
    const unsigned grid = (unsigned)std::min((groups + per_cta - 1) / per_cta, max_grid);
    if (gated) {
        switch (wk) {
        case 1: return gemv_launch<T, MR, 1, true>(p, smem, grid, s);
        case 2: return gemv_launch<T, MR, 2, true>(p, smem, grid, s);
        case 4: return gemv_launch<T, MR, 4, true>(p, smem, grid, s);
        default: return gemv_launch<T, MR, 8, true>(p, smem, grid, s);
        }
    }
    if (p.x2 || p.out.biased) {
        switch (wk) {
        case 1: return gemv_launch<T, MR, 1, false, true>(p, smem, grid, s);
        case 2: return gemv_launch<T, MR, 2, false, true>(p, smem, grid, s);
        case 4: return gemv_launch<T, MR, 4, false, true>(p, smem, grid, s);
        default: return gemv_launch<T, MR, 8, false, true>(p, smem, grid, s);
        }
    }
    switch (wk) {
    case 1: return gemv_launch<T, MR, 1, false>(p, smem, grid, s);
    case 2: return gemv_launch<T, MR, 2, false>(p, smem, grid, s);
    case 4: return gemv_launch<T, MR, 4, false>(p, smem, grid, s);
    default: return gemv_launch<T, MR, 8, false>(p, smem, grid, s);
    }
}
template <typename T>
int gemv_rows(const GemvParams& p, bool gated, size_t smem, cudaStream_t s) {
    switch (p.m) {
    case 1: return gemv_pick<T, 1>(p, gated, smem, s);
    case 2: return gemv_pick<T, 2>(p, gated, smem, s);
    case 3: return gemv_pick<T, 3>(p, gated, smem, s);
    default: return gemv_pick<T, 4>(p, gated, smem, s);
    }
}
size_t gemv_smem(int m, int ld, bool x_f32, bool norm) { return (size_t)m * ld * (x_f32 ? 4 : 2) + (norm ? (size_t)ld * 4 : 0); }

// bf16 matrix [rows][ld] as a 2-D tensor, k columns valid (beyond: zeros); box = 64 columns x box_rows, 128-byte swizzle
int bf16_map(const __nv_bfloat16* p, int ld, int rows, int k, int box_rows, CUtensorMap* map) {
    TensorMapEncodeFn fn = tensor_map_encode_fn();
    if (!fn) { set_error("dense product: cuTensorMapEncodeTiled is not available"); return SWLM_ERR_CUDA; }
    const cuuint64_t dims[2] = {(cuuint64_t)k, (cuuint64_t)rows};
    const cuuint64_t strides[1] = {(cuuint64_t)ld * 2};
    const cuuint32_t box[2] = {(cuuint32_t)kTcK, (cuuint32_t)box_rows};
    const cuuint32_t estr[2] = {1, 1};
    const CUresult r = fn(map, CU_TENSOR_MAP_DATA_TYPE_BFLOAT16, 2, const_cast<__nv_bfloat16*>(p), dims, strides, box, estr,
                          CU_TENSOR_MAP_INTERLEAVE_NONE, CU_TENSOR_MAP_SWIZZLE_128B, CU_TENSOR_MAP_L2_PROMOTION_L2_256B, CU_TENSOR_MAP_FLOAT_OOB_FILL_NONE);
    if (r != CUDA_SUCCESS) { set_error("dense product: cuTensorMapEncodeTiled failed (%d)", (int)r); return SWLM_ERR_CUDA; }
    return SWLM_OK;
}

struct TcShape { int bn, ranges, split_steps, tiles_m, tiles_n; };
TcShape tc_shape(int n, int k, int m, bool gated) {
    TcShape t;
    t.bn = m > 128 ? 256 : m > 64 ? 128 : m > 32 ? 64 : 32;
    // too few tiles to fill the GPU: half as many rows per tile before K is cut
    const int rows_n = gated ? kTileRows : 2 * kTileRows;
    if (t.bn == 256 && (m + 255) / 256 * ((n + rows_n - 1) / rows_n) < 100) t.bn = 128;
    t.tiles_m = (m + t.bn - 1) / t.bn;
    t.tiles_n = (n + (gated ? kTileRows : 2 * kTileRows) - 1) / (gated ? kTileRows : 2 * kTileRows);
    const int steps = (k + kTcK - 1) / kTcK, tiles = t.tiles_m * t.tiles_n;
    int ranges = tiles * 2 > 148 ? 1 : std::min(std::min(148 / tiles, std::max(1, steps / 4)), 16);
    t.split_steps = (steps + ranges - 1) / ranges;
    t.ranges = (steps + t.split_steps - 1) / t.split_steps;
    return t;
}

template <int BN, int STAGES>
constexpr size_t tc_smem() { return (size_t)STAGES * (2 * kTileRows * 128 + BN * 128) + 1024; }
template <int BN, int STAGES, bool GATED>
int tc_attr() {
    SWLM_CUDA(cudaFuncSetAttribute(bgemm_tc_kernel<BN, STAGES, GATED>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)tc_smem<BN, STAGES>()));
    return SWLM_OK;
}
template <int BN, int STAGES>
int tc_launch(const ProductLaunch& a, const TcShape& t, cudaStream_t s) {
    const bool gated = a.w2 != nullptr;
    TcParams p{};
    p.n = a.experts ? a.w->n / a.experts : a.w->n; p.tiles = a.tiles; p.m = a.m; p.steps = (a.w->k + kTcK - 1) / kTcK; p.split_steps = t.split_steps; p.act = a.act; p.out = a.out; p.part = a.part; p.status = a.status;
    CUtensorMap xmap, wmap, wmap2;
    int rc = bf16_map(static_cast<const __nv_bfloat16*>(a.x), a.x_stride, a.m, a.w->k, BN, &xmap);
    if (!rc) rc = bf16_map(a.w->data, a.w->ld, a.w->n, a.w->k, kTileRows, &wmap);
    wmap2 = wmap;
    p.split = a.x2 ? a.split : p.n;
    if (!rc && a.x2) rc = bf16_map(static_cast<const __nv_bfloat16*>(a.x2), a.x2_stride, a.m, a.w->k, BN, &wmap2);
    if (!rc && gated) rc = bf16_map(a.w2->data, a.w2->ld, a.w2->n, a.w2->k, kTileRows, &wmap2);
    if (rc) return rc;
    const dim3 grid((unsigned)t.tiles_m, (unsigned)t.tiles_n, (unsigned)t.ranges);
    cudaError_t e = gated ? launch_k(bgemm_tc_kernel<BN, STAGES, true>, grid, dim3(kTcBlock), tc_smem<BN, STAGES>(), s, p, xmap, wmap, wmap2)
                          : launch_k(bgemm_tc_kernel<BN, STAGES, false>, grid, dim3(kTcBlock), tc_smem<BN, STAGES>(), s, p, xmap, wmap, wmap2);
    if (e != cudaSuccess) return cuda_fail(e, "bgemm launch");
    if (t.ranges > 1) {
        const dim3 g((unsigned)((p.n + 255) / 256), (unsigned)std::min(p.m, std::max(64, 8 * 148 * 256 / p.n)));
        e = gated ? launch_k(bgemm_sum_kernel<true>, g, dim3(256), 0, s, (const float*)a.part, t.ranges, p.m, p.n, p.act, p.out)
                  : launch_k(bgemm_sum_kernel<false>, g, dim3(256), 0, s, (const float*)a.part, t.ranges, p.m, p.n, p.act, p.out);
        if (e != cudaSuccess) return cuda_fail(e, "bgemm sum launch");
    }
    return SWLM_OK;
}

TcShape grouped_shape(const ProductLaunch& a) {
    TcShape t;
    const int n = a.w->n / a.experts, rows_n = a.w2 ? kTileRows : 2 * kTileRows;
    t.bn = a.group_bn;
    t.tiles_m = a.max_tiles;
    t.tiles_n = (n + rows_n - 1) / rows_n;
    t.ranges = 1;
    t.split_steps = (a.w->k + kTcK - 1) / kTcK;
    return t;
}

bool gemv_fits(int m, int k, bool x_f32, bool norm) {
    const int ld = (k + 7) / 8 * 8;
    return m <= kGemvRows && gemv_smem(m, ld, x_f32, norm) <= kGemvMaxSmem;
}

}  // namespace

int bgemm_init() {
    int rc;
    if ((rc = tc_attr<32, 4, false>()) || (rc = tc_attr<32, 4, true>()) || (rc = tc_attr<64, 4, false>()) || (rc = tc_attr<64, 4, true>()) ||
        (rc = tc_attr<128, 4, false>()) || (rc = tc_attr<128, 4, true>()) || (rc = tc_attr<256, 3, false>()) || (rc = tc_attr<256, 3, true>())) return rc;
    return SWLM_OK;
}

bool product_takes_norm(int m, int k) { return m <= 2 && k <= 16384 && gemv_fits(m, k, true, true); }
// gate and up in one launch: always, except as true fp32 products over many rows
bool product_takes_gate(int m, int k, bool x_f32) { return !x_f32 || gemv_fits(m, k, true, false); }

bool product_takes_two(int m, int k, int split, bool x_f32) {
    if (gemv_fits(m, k, x_f32, false)) return !(split & 3) && gemv_smem(2 * m, (k + 7) / 8 * 8, x_f32, false) <= kGemvMaxSmem;
    return !x_f32 && split % (2 * kTileRows) == 0;   // no tile has rows of both
}

size_t product_part_floats(int n, int k, int m, bool gated) {
    if (gemv_fits(m, k, false, false)) return 0;
    const TcShape t = tc_shape(n, k, m, gated);
    return t.ranges > 1 ? (size_t)t.ranges * (gated ? 2 : 1) * m * n : 0;
}

// tiles about as tall as an expert has rows on average
int grouped_bn(int rows, int experts) {
    const int avg = rows / std::max(1, experts);
    return avg > 160 ? 256 : avg > 64 ? 128 : avg > 24 ? 64 : 32;
}
int grouped_max_tiles(int rows, int experts) { return std::min(rows, experts) + rows / grouped_bn(rows, experts); }

int product_launch_count(const ProductLaunch& a) {
    if (a.experts) return 1;
    if (gemv_fits(a.m, a.w->k, a.x_f32, a.norm.mode != 0) || a.x_f32) return 1;
    return tc_shape(a.w->n, a.w->k, a.m, a.w2 != nullptr).ranges > 1 ? 2 : 1;
}

int launch_product(const ProductLaunch& a, cudaStream_t s) {
    if (a.m <= 0) return SWLM_OK;
    const bool gated = a.w2 != nullptr;
    if (gated && (a.w2->n != a.w->n || a.w2->k != a.w->k)) { set_error("gated product: the two matrices differ in shape"); return SWLM_ERR_INVALID; }
    if (a.experts && (a.x_f32 || a.norm.mode || !a.tiles)) { set_error("a grouped product takes plain bf16 rows"); return SWLM_ERR_INVALID; }
    if (!a.experts && gemv_fits(a.m, a.w->k, a.x_f32, a.norm.mode != 0)) {
        GemvParams p{};
        p.w = a.w->data; p.w2 = gated ? a.w2->data : nullptr; p.ld = a.w->ld; p.n = a.w->n; p.k = a.w->k; p.m = a.m; p.act = a.act;
        p.x = a.x; p.x_stride = a.x_stride; p.norm = a.norm; p.out = a.out;
        if (a.x2 && (gated || a.norm.mode || !product_takes_two(a.m, a.w->k, a.split, a.x_f32))) { set_error("two inputs of a product over %d rows run one after the other", a.m); return SWLM_ERR_INVALID; }
        p.x2 = a.x2; p.x2_stride = a.x2_stride; p.split = a.split;
        const size_t smem = gemv_smem(a.x2 ? 2 * a.m : a.m, a.w->ld, a.x_f32, a.norm.mode != 0);
        return a.x_f32 ? gemv_rows<float>(p, gated, smem, s) : gemv_rows<__nv_bfloat16>(p, gated, smem, s);
    }
    if (a.x2 && (gated || a.experts || !product_takes_two(a.m, a.w->k, a.split, a.x_f32))) { set_error("two inputs of a product over %d rows run one after the other", a.m); return SWLM_ERR_INVALID; }
    if (a.norm.mode) { set_error("a norm in front of a product over %d rows runs on its own", a.m); return SWLM_ERR_INVALID; }
    if (a.x_f32) {
        if (gated) { set_error("gate and up of fp32 rows run one after the other"); return SWLM_ERR_INVALID; }
        const cudaError_t e = launch_k(sgemm_kernel, dim3((a.w->n + 63) / 64, (a.m + 63) / 64), dim3(256), 0, s, (const __nv_bfloat16*)a.w->data,
                                       a.w->ld, a.w->n, a.w->k, a.m, static_cast<const float*>(a.x), a.x_stride, a.out);
        return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "sgemm launch");
    }
    if (((a.x_stride | a.x2_stride) & 7) || ((reinterpret_cast<uintptr_t>(a.x) | reinterpret_cast<uintptr_t>(a.x2)) & 15)) { set_error("dense product: activation rows must be 16-byte aligned"); return SWLM_ERR_INVALID; }
    const TcShape t = a.experts ? grouped_shape(a) : tc_shape(a.w->n, a.w->k, a.m, gated);
    if (t.ranges > 1 && (!a.part || a.part_floats < (size_t)t.ranges * (gated ? 2 : 1) * a.m * a.w->n)) { set_error("dense product: scratch too small"); return SWLM_ERR_INVALID; }
    switch (t.bn) {
    case 32: return tc_launch<32, 4>(a, t, s);
    case 64: return tc_launch<64, 4>(a, t, s);
    case 128: return tc_launch<128, 4>(a, t, s);
    default: return tc_launch<256, 3>(a, t, s);
    }
}

}  // namespace swlm
