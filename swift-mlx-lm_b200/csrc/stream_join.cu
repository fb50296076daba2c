// The residual stream between the sublayers of designs whose sublayers read the stream itself: what a sublayer returns is gated,
// normed and added, results of layers are averaged over the depth, and the next sublayer gets the stream with a short causal
// convolution over it. Everything that happens between two products is one launch over the batch's rows; all of it is fp32.
//
// The convolution needs the stream at the tokens in front of a row. Inside a portion those are rows of the same launch, so a CTA
// walks consecutive rows and keeps the last ones in shared memory; in front of its first row it works out as many rows of its
// neighbour again as the convolution reaches back. In front of a portion they come from the state of the sequence. The state is
// written by the launch that changes the stream next (it reads the same rows), so no CTA writes what another still reads.
#include <algorithm>

#include "swlm_internal.h"

namespace swlm {
namespace {

constexpr int kJoinWarpsMax = 16;
constexpr size_t kJoinMaxSmem = 200 * 1024;

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

// CTA: rows_per_cta consecutive rows. A thread keeps entries 4 (tid + NT j) .. + 3 of a row; the next row is requested while the
// present one waits for its norm. Shared memory: [taps - 1][width] last rows of the stream, then [taps][width] weights in bf16
// (a thread only ever touches its own columns of the rows).
template <typename T, int J, int NT>
__global__ void __launch_bounds__(NT) stream_join_kernel(const JoinLaunch p, int rows_per_cta) {
    extern __shared__ __align__(16) unsigned char join_smem[];
    __shared__ float red[2][kJoinWarpsMax];
    const int tid = threadIdx.x, width = p.width, pitch = (width + 3) / 4 * 4, past = max(0, p.taps - 1);
    float* hist = reinterpret_cast<float*>(join_smem);
    __nv_bfloat16* cw = reinterpret_cast<__nv_bfloat16*>(hist + (size_t)past * pitch);
    const bool whole = (width & 3) == 0;
    pdl_launch_dependents();
    float nw[J][4];
#pragma unroll
    for (int j = 0; j < J; ++j) {
        const int i = 4 * (tid + NT * j);
        if (p.in) jn_weights4(p.w, i, width, whole, nw[j]);
#pragma unroll
        for (int e = 0; e < 4; ++e) nw[j][e] += p.weight_bias;
        if (p.conv_out)
            for (int e = 0; e < 4; ++e)
                for (int k = 0; k < p.taps; ++k)
                    if (i + e < pitch) cw[(size_t)k * pitch + i + e] = i + e < width ? p.conv_w[(size_t)(i + e) * p.taps + k] : __float2bfloat16_rn(0.f);
    }
    pdl_wait();
    const int r0 = blockIdx.x * rows_per_cta, r1 = min(r0 + rows_per_cta, p.rows);
    int first = r0;   // rows in front of r0 that the convolution reaches
    for (int n = 0; n < past && p.conv_out && first > 0 && p.row_seq[first - 1] == p.row_seq[r0]; ++n) --first;

    float x[J][4], in[J][4], gate[J][4], sum[J][4];
    auto request = [&](int r) {
        const __nv_bfloat16* row = p.table ? p.table + (size_t)min(max(p.tokens[r], 0), p.vocab - 1) * width : nullptr;
#pragma unroll
        for (int j = 0; j < J; ++j) {
            const int i = 4 * (tid + NT * j);
            if (i >= width) continue;
            if (row) jn_weights4(row, i, width, whole, x[j]);
            else jn_get4(p.res_in + (size_t)r * p.res_stride + i, x[j]);
            if (p.in) jn_get4(p.in + (size_t)r * p.in_stride + i, in[j]);
            if (p.gate) jn_get4(p.gate + (size_t)r * p.gate_stride + i, gate[j]);
        }
        if (p.avg) {
#pragma unroll
            for (int j = 0; j < J; ++j) sum[j][0] = sum[j][1] = sum[j][2] = sum[j][3] = 0.f;
#pragma unroll 4
            for (int q = 0; q < p.avg - 1; ++q) {
                const float w = __bfloat162float(p.avg_w[q]);
                const float* result = p.results + q * p.result_step + (size_t)r * p.res_stride;
#pragma unroll
                for (int j = 0; j < J; ++j) {
                    const int i = 4 * (tid + NT * j);
                    if (i >= width) continue;
                    float v[4];
                    jn_get4(result + i, v);
#pragma unroll
                    for (int e = 0; e < 4; ++e) sum[j][e] = fmaf(w, v[e], sum[j][e]);
                }
            }
        }
    };
    request(first);
    const float own_w = p.avg ? __bfloat162float(p.avg_w[p.avg - 1]) : 1.f;
    int slot = 0;   // of the row in hist
    for (int r = first, turn = 0; r < r1; ++r, turn ^= 1) {
        float h[J][4], t[J][4], before[J][4];
        float ss = 0.f;
#pragma unroll
        for (int j = 0; j < J; ++j) {
            const int i = 4 * (tid + NT * j);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const bool live = i + e < width;
                h[j][e] = live ? x[j][e] * (p.table ? p.table_scale : 1.f) : 0.f;
                t[j][e] = !live || !p.in ? 0.f : p.gate ? in[j][e] * jn_sigmoid(gate[j][e]) : in[j][e];
                before[j][e] = p.avg ? sum[j][e] : 0.f;
                ss = fmaf(t[j][e], t[j][e], ss);
            }
        }
        const bool mine = r >= r0;
        const int seq = p.row_seq[r], pos = p.row_pos[r];
        if (p.keep_ring && mine && !(r + p.keep_taps - 1 < p.rows && p.row_seq[r + p.keep_taps - 1] == seq)) {
            float* keep = p.keep_ring + ((size_t)seq * (p.keep_taps - 1) + pos % (p.keep_taps - 1)) * width;
#pragma unroll
            for (int j = 0; j < J; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) { const int i = 4 * (tid + NT * j) + e; if (i < width) keep[i] = h[j][e]; }
        }
        if (r + 1 < r1) request(r + 1);
        if (p.in) {
            for (int o = 16; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
            if ((tid & 31) == 0) red[turn][tid >> 5] = ss;
            __syncthreads();
            float total = 0.f;
#pragma unroll
            for (int i = 0; i < NT / 32; ++i) total += red[turn][i];
            const float scale = 1.0f / sqrtf(total / (float)width + p.eps);
#pragma unroll
            for (int j = 0; j < J; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) h[j][e] = fmaf(t[j][e] * scale, nw[j][e], h[j][e]);
        }
        // a portion starts here: its past comes from the sequence's state
        const bool starts = r == 0 || p.row_seq[r - 1] != seq;
#pragma unroll
        for (int j = 0; j < J; ++j) {
            const int i = 4 * (tid + NT * j);
            if (i >= width) continue;
            if (p.store >= 0 && mine) jn_put4(p.results + p.store * p.result_step + (size_t)r * p.res_stride + i, h[j]);
            if (p.avg) {
#pragma unroll
                for (int e = 0; e < 4; ++e) h[j][e] = fmaf(own_w, h[j][e], before[j][e]);
            }
            if (p.res_out && mine) jn_put4(p.res_out + (size_t)r * p.res_stride + i, h[j]);
            if (p.copy_out && mine) jn_put4(static_cast<T*>(p.copy_out) + (size_t)r * p.copy_stride + i, h[j]);
            if (!p.conv_out) continue;
            if (starts)
                for (int d = 1; d <= past; ++d) {
                    const float* from = p.conv_ring + ((size_t)seq * past + (pos >= d ? (pos - d) % past : 0)) * width;
                    float v[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) v[e] = pos >= d && i + e < width ? from[i + e] : 0.f;
                    jn_put4(hist + (size_t)(slot >= d ? slot - d : slot - d + past) * pitch + i, v);
                }
            float y[4];
            const __nv_bfloat16* w = cw + i;
#pragma unroll
            for (int e = 0; e < 4; ++e) y[e] = fmaf(__bfloat162float(w[(size_t)past * pitch + e]), h[j][e], h[j][e]);
            for (int d = 1; d <= past; ++d) {
                float v[4];
                jn_get4(hist + (size_t)(slot >= d ? slot - d : slot - d + past) * pitch + i, v);
#pragma unroll
                for (int e = 0; e < 4; ++e) y[e] = fmaf(__bfloat162float(w[(size_t)(past - d) * pitch + e]), v[e], y[e]);
            }
            if (past) jn_put4(hist + (size_t)slot * pitch + i, h[j]);
            if (mine) jn_put4(static_cast<T*>(p.conv_out) + (size_t)r * p.conv_stride + i, y);
        }
        if (++slot >= past) slot = 0;
    }
}

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

size_t join_smem_bytes(int width, int taps) {
    const size_t pitch = (width + 3) / 4 * 4;
    return taps > 0 ? (size_t)(taps - 1) * pitch * 4 + (size_t)taps * pitch * 2 : 0;
}

template <typename T, int J, int NT>
int join_kernel(const JoinLaunch& a, int rows_per_cta, cudaStream_t s) {
    static const cudaError_t attr = cudaFuncSetAttribute(stream_join_kernel<T, J, NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)kJoinMaxSmem);
    if (attr != cudaSuccess) return cuda_fail(attr, "stream join attributes");
    const cudaError_t e = launch_k(stream_join_kernel<T, J, NT>, dim3((a.rows + rows_per_cta - 1) / rows_per_cta), dim3(NT), join_smem_bytes(a.width, a.conv_out ? a.taps : 0), s, a, rows_per_cta);
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "stream join launch");
}
template <typename T>
int join_rows(const JoinLaunch& a, cudaStream_t s) {
    // portions: a few rows per CTA, so that few are worked out twice
    const int rows = a.singles || !a.conv_out || a.taps < 2 ? 1 : std::min(16, std::max(a.taps - 1, (a.rows + 3 * 148 - 1) / (3 * 148)));
    if (a.width <= 4 * 128) return join_kernel<T, 1, 128>(a, rows, s);
    if (a.width <= 4 * 256) return join_kernel<T, 1, 256>(a, rows, s);
    if (a.width <= 4 * 512) return join_kernel<T, 2, 256>(a, rows, s);
    if (a.width <= 4 * 1024) return join_kernel<T, 2, 512>(a, rows, s);
    return join_kernel<T, 8, 512>(a, rows, s);
}

}  // namespace

int join_init() { return SWLM_OK; }
bool join_supported(int width, int taps) { return width > 0 && width <= 4 * 512 * 8 && taps >= 0 && join_smem_bytes(width, taps) <= kJoinMaxSmem; }

int launch_join(const JoinLaunch& a, cudaStream_t s) {
    if (a.rows <= 0) return SWLM_OK;
    if (!join_supported(a.width, a.conv_out ? a.taps : 0)) { set_error("stream of %d entries with convolutions of %d taps", a.width, a.taps); return SWLM_ERR_UNSUPPORTED; }
    return a.f32 ? join_rows<float>(a, s) : join_rows<__nv_bfloat16>(a, s);
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
