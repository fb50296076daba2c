// Row kernels of fp32-stream plans: embedding gather, norms, gated activation, soft cap of the logits. The residual
// stream, the norms and the logits stay in fp32; results that feed a product are stored in the plan's activation type.
#include "swlm_internal.h"

namespace swlm {
namespace {

__device__ __forceinline__ float stream_block_sum(float v, float* red) {
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    const int nw = blockDim.x >> 5;
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float total = 0.f;
    for (int i = 0; i < nw; ++i) total += red[i];   // the same order in every thread
    __syncthreads();
    return total;
}
__device__ __forceinline__ void put(float* p, float v) { *p = v; }
__device__ __forceinline__ void put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
__device__ __forceinline__ void put4(float* p, float a, float b, float c, float d) { *reinterpret_cast<float4*>(p) = make_float4(a, b, c, d); }
__device__ __forceinline__ void put4(__nv_bfloat16* p, float a, float b, float c, float d) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(a, b), hi = __floats2bfloat162_rn(c, d);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const unsigned*>(&lo), *reinterpret_cast<const unsigned*>(&hi));
}
__device__ __forceinline__ float get(const float* p) { return *p; }
__device__ __forceinline__ float get(const __nv_bfloat16* p) { return __bfloat162float(*p); }

// One CTA per output row; the row lives in shared memory between the passes.
template <typename T>
__global__ void __launch_bounds__(256) stream_norm_kernel(StreamNorm a, int dim, const int32_t* rows_idx, T* out, int out_stride) {
    pdl_launch_dependents();
    pdl_wait();
    extern __shared__ __align__(16) float row[];
    __shared__ float red[8];
    const int r = rows_idx ? rows_idx[blockIdx.x] : blockIdx.x;
    const float* in = a.in + (size_t)r * a.in_stride;
    const bool post = a.w_post != nullptr, add = a.res_in != nullptr;
    const __nv_bfloat16* joins = a.table ? a.table_row(r, dim) : nullptr;
    float post_scale = 1.f;
    if (post) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < dim; i += blockDim.x) { const float v = in[i]; row[i] = v; ss = fmaf(v, v, ss); }
        post_scale = 1.0f / sqrtf(stream_block_sum(ss, red) / (float)dim + a.eps);
    }
    float ss = 0.f;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) {
        float h = post ? row[i] * post_scale * (__bfloat162float(a.w_post[i]) + a.weight_bias) : in[i];
        if (add) h += a.res_in[(size_t)r * a.res_stride + i];
        if (joins) h += __bfloat162float(joins[i]) * a.table_scale;
        if (a.res_out) a.res_out[(size_t)r * a.res_stride + i] = h;
        row[i] = h;
        ss = fmaf(h, h, ss);
    }
    const float scale = 1.0f / sqrtf(stream_block_sum(ss, red) / (float)dim + a.eps);
    T* o = out + (size_t)blockIdx.x * out_stride;
    for (int i = threadIdx.x; i < dim; i += blockDim.x) put(o + i, row[i] * scale * (__bfloat162float(a.w[i]) + a.weight_bias));
}

// The same for rows of up to 4096 entries, a multiple of four: a thread keeps entries 4 tid + 1024 j in registers and asks for
// all it needs at once.
constexpr int kNormQuads = 4;
template <typename T>
__global__ void __launch_bounds__(256) stream_norm_quads_kernel(StreamNorm a, int dim, const int32_t* rows_idx, T* out, int out_stride) {
    pdl_launch_dependents();
    __shared__ float red[8];
    uint2 w[kNormQuads], wp[kNormQuads];
#pragma unroll
    for (int j = 0; j < kNormQuads; ++j) {
        const int i = 4 * threadIdx.x + 1024 * j;
        w[j] = i < dim ? __ldg(reinterpret_cast<const uint2*>(a.w + i)) : make_uint2(0, 0);
        wp[j] = i < dim && a.w_post ? __ldg(reinterpret_cast<const uint2*>(a.w_post + i)) : make_uint2(0, 0);
    }
    pdl_wait();
    const int r = rows_idx ? rows_idx[blockIdx.x] : blockIdx.x;
    const float* in = a.in + (size_t)r * a.in_stride;
    const __nv_bfloat16* joins = a.table ? a.table_row(r, dim) : nullptr;
    float h[kNormQuads][4], res[kNormQuads][4];
#pragma unroll
    for (int j = 0; j < kNormQuads; ++j) {
        const int i = 4 * threadIdx.x + 1024 * j;
        const float4 z = make_float4(0.f, 0.f, 0.f, 0.f);
        const float4 x = i < dim ? *reinterpret_cast<const float4*>(in + i) : z;
        const float4 y = i < dim && a.res_in ? *reinterpret_cast<const float4*>(a.res_in + (size_t)r * a.res_stride + i) : z;
        h[j][0] = x.x; h[j][1] = x.y; h[j][2] = x.z; h[j][3] = x.w;
        res[j][0] = y.x; res[j][1] = y.y; res[j][2] = y.z; res[j][3] = y.w;
        if (joins && i < dim) {
            const uint2 v = __ldg(reinterpret_cast<const uint2*>(joins + i));
            res[j][0] += __uint_as_float(v.x << 16) * a.table_scale; res[j][1] += __uint_as_float(v.x & 0xFFFF0000u) * a.table_scale;
            res[j][2] += __uint_as_float(v.y << 16) * a.table_scale; res[j][3] += __uint_as_float(v.y & 0xFFFF0000u) * a.table_scale;
        }
    }
    auto weights = [&](const uint2& v, float (&f)[4]) {
        f[0] = __uint_as_float(v.x << 16) + a.weight_bias; f[1] = __uint_as_float(v.x & 0xFFFF0000u) + a.weight_bias;
        f[2] = __uint_as_float(v.y << 16) + a.weight_bias; f[3] = __uint_as_float(v.y & 0xFFFF0000u) + a.weight_bias;
    };
    float ss = 0.f;
    if (a.w_post) {
#pragma unroll
        for (int j = 0; j < kNormQuads; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) ss = fmaf(h[j][e], h[j][e], ss);
        const float sc = 1.0f / sqrtf(stream_block_sum(ss, red) / (float)dim + a.eps);
#pragma unroll
        for (int j = 0; j < kNormQuads; ++j) {
            float f[4];
            weights(wp[j], f);
#pragma unroll
            for (int e = 0; e < 4; ++e) h[j][e] = h[j][e] * sc * f[e];
        }
    }
    ss = 0.f;
#pragma unroll
    for (int j = 0; j < kNormQuads; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) { h[j][e] += res[j][e]; ss = fmaf(h[j][e], h[j][e], ss); }   // (entries past dim: zeros)
    const float scale = 1.0f / sqrtf(stream_block_sum(ss, red) / (float)dim + a.eps);
    T* o = out + (size_t)blockIdx.x * out_stride;
#pragma unroll
    for (int j = 0; j < kNormQuads; ++j) {
        const int i = 4 * threadIdx.x + 1024 * j;
        if (i >= dim) continue;
        if (a.res_out) *reinterpret_cast<float4*>(a.res_out + (size_t)r * a.res_stride + i) = make_float4(h[j][0], h[j][1], h[j][2], h[j][3]);
        float f[4];
        weights(w[j], f);
        put4(o + i, h[j][0] * scale * f[0], h[j][1] * scale * f[1], h[j][2] * scale * f[2], h[j][3] * scale * f[3]);
    }
}

__global__ void __launch_bounds__(256) stream_embed_kernel(int dim, const int32_t* tokens, int vocab, const __nv_bfloat16* table,
                                                          float scale, float* out, int out_stride) {
    pdl_launch_dependents();
    pdl_wait();
    int tok = tokens[blockIdx.y];
    tok = tok < 0 ? 0 : (tok >= vocab ? vocab - 1 : tok);
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < dim) out[(size_t)blockIdx.y * out_stride + i] = __bfloat162float(table[(size_t)tok * dim + i]) * scale;
}

template <typename T>
__global__ void __launch_bounds__(256) stream_gated_kernel(int n, const T* gate, int g_stride, const T* up, int u_stride, T* out, int o_stride, GatedAct act) {
    pdl_launch_dependents();
    pdl_wait();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    const size_t r = blockIdx.y;
    put(out + r * o_stride + i, gated_activation(get(gate + r * g_stride + i), get(up + r * u_stride + i), act));
}

__global__ void __launch_bounds__(256) stream_softcap_kernel(int n, float* x, int stride, float cap) {
    pdl_launch_dependents();
    pdl_wait();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    float* v = x + (size_t)blockIdx.y * stride + i;
    *v = cap * tanhf(*v / cap);
}

}  // namespace

int launch_stream_norm(const StreamNorm& a, int m, int dim, const int32_t* rows_idx, void* out, int out_stride, bool out_f32, cudaStream_t s) {
    if (m <= 0) return SWLM_OK;
    cudaError_t e;
    // (buffer rows start at multiples of eight entries)
    if (dim <= 1024 * kNormQuads && !(dim & 3)) {
        if (out_f32) e = launch_k(stream_norm_quads_kernel<float>, dim3(m), dim3(256), 0, s, a, dim, rows_idx, static_cast<float*>(out), out_stride);
        else e = launch_k(stream_norm_quads_kernel<__nv_bfloat16>, dim3(m), dim3(256), 0, s, a, dim, rows_idx, static_cast<__nv_bfloat16*>(out), out_stride);
        return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "stream norm launch");
    }
    const size_t smem = (size_t)dim * 4;
    if (smem > 200 * 1024) { set_error("norm over %d entries does not fit shared memory", dim); return SWLM_ERR_UNSUPPORTED; }
    if (smem > 40 * 1024) {
        SWLM_CUDA(cudaFuncSetAttribute(stream_norm_kernel<float>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        SWLM_CUDA(cudaFuncSetAttribute(stream_norm_kernel<__nv_bfloat16>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    }
    if (out_f32) e = launch_k(stream_norm_kernel<float>, dim3(m), dim3(256), smem, s, a, dim, rows_idx, static_cast<float*>(out), out_stride);
    else e = launch_k(stream_norm_kernel<__nv_bfloat16>, dim3(m), dim3(256), smem, s, a, dim, rows_idx, static_cast<__nv_bfloat16*>(out), out_stride);
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "stream norm launch");
}

int launch_stream_embed(int m, int dim, const int32_t* tokens, int vocab, const __nv_bfloat16* table, float scale, float* out, int out_stride, cudaStream_t s) {
    const cudaError_t e = launch_k(stream_embed_kernel, dim3((dim + 255) / 256, m), dim3(256), 0, s, dim, tokens, vocab, table, scale, out, out_stride);
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "stream embed launch");
}

int launch_stream_gated(int m, int n, const void* gate, int g_stride, const void* up, int u_stride, void* out, int o_stride, bool f32, GatedAct act, cudaStream_t s) {
    cudaError_t e;
    const dim3 grid((n + 255) / 256, m);
    if (f32) e = launch_k(stream_gated_kernel<float>, grid, dim3(256), 0, s, n, static_cast<const float*>(gate), g_stride, static_cast<const float*>(up), u_stride, static_cast<float*>(out), o_stride, act);
    else e = launch_k(stream_gated_kernel<__nv_bfloat16>, grid, dim3(256), 0, s, n, static_cast<const __nv_bfloat16*>(gate), g_stride,
                      static_cast<const __nv_bfloat16*>(up), u_stride, static_cast<__nv_bfloat16*>(out), o_stride, act);
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "gated activation launch");
}

int launch_stream_softcap(int m, int n, float* logits, int stride, float cap, cudaStream_t s) {
    if (m <= 0) return SWLM_OK;
    const cudaError_t e = launch_k(stream_softcap_kernel, dim3((n + 255) / 256, m), dim3(256), 0, s, n, logits, stride, cap);
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "soft cap launch");
}

}  // namespace swlm
