// Gated delta rule over an fp32 state per sequence and head: short causal convolutions with SiLU in front of q, k and v, unit q
// and k, one decay per head or per key channel, and a normed, gated read-out.
//
// Two ways through it, chosen per row of a batch:
//   * a single token of a sequence (decode steps): delta_step_kernel does all of it in one launch, a cluster of CTAs per head
//     that each own 32 columns of the state; state and convolution inputs are requested before the preceding kernel has
//     finished.
//   * portions: tokens are taken in blocks of kDeltaBlock. delta_prepare_kernel works out, for every block and head, what the
//     recurrence needs of the block with the decays folded in; delta_scan_kernel walks the blocks with the state in registers;
//     delta_gate_kernel norms and gates the rows.
//
// Inside a block, with S the state in front of it, G_t the product of the decays up to token t and D_ts the product of the
// decays of tokens s + 1 .. t (all at most 1, nothing is divided):
//   u_t = beta_t (v_t - S^T (G_t k_t)) - sum_{s < t} beta_t (k_s . D_ts k_t) u_s     (a triangular system)
//   o_t = S^T (G_t q_t) + sum_{s <= t} (k_s . D_ts q_t) u_s
//   S' = G_T S + sum_s (D_Ts k_s) u_s^T
// The products of k and q with each other do not depend on the state's column: they are formed once per head. Everything is
// fp32. Where a sequence is cut changes the blocks, and with them the order of sums, nothing else.
#include <cooperative_groups.h>

#include <algorithm>
#include <utility>

#include "swlm_internal.h"
#include "tc_device.cuh"

namespace cg = cooperative_groups;

namespace swlm {
namespace {

constexpr int TB = kDeltaBlock;
constexpr int kScanCols = 16, kScanWarpCols = 2, kScanWarps = kScanCols / kScanWarpCols, kScanThreads = (kScanWarps + 1) * 32;   // the last warp requests the records
constexpr int kStepCols = 32, kStepWarps = 8, kStepThreads = kStepWarps * 32, kStepCluster = 8;
constexpr int kPrepThreads = 128;

// copies in flight: a block is walked in a fraction of a copy's latency; two CTAs fit an SM at up to 256 key channels
__host__ __device__ constexpr int scan_stages(int regs) { return regs <= 4 ? 14 : regs <= 8 ? 8 : 6; }

struct DeltaParams {
    DeltaShape sh;
    int decay_dim, gate_act;
    float eps, unit_eps, q_scale;
    const void* qkv; int qkv_stride;
    const float* beta; int beta_stride;
    const float* decay; int decay_stride;
    const void* gate; int gate_stride;
    const __nv_bfloat16 *conv_q, *conv_k, *conv_v, *norm_w, *a_log, *dt_bias;
    void* ring; float* state;
    const int32_t* row_seq; const int32_t* row_pos;
    void* out; int out_stride;
    int n_single; const int32_t* single_rows;
    const RowRun* runs; const int32_t* block_run;   // runs == null: every single row is a run of one token
    float* rec; float* vrec; float* o;
    int dp, rec_floats, vblocks;                    // padded key channels, floats per block and head, column blocks of the scan
    int* status;
};

__device__ __forceinline__ float dl_get(const float* p) { return *p; }
__device__ __forceinline__ float dl_get(const __nv_bfloat16* p) { return __bfloat162float(*p); }
__device__ __forceinline__ void dl_put(float* p, float v) { *p = v; }
__device__ __forceinline__ void dl_put(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }
// With bf16 activations the hardware's approximations of exp, log and division are used (still fp32 numbers: their errors are a
// few units in the last place); fp32 plans use the functions of full accuracy.
template <typename T> struct Fn;
template <> struct Fn<float> {
    static __device__ __forceinline__ float exp(float x) { return expf(x); }
    static __device__ __forceinline__ float log1p(float x) { return log1pf(x); }
    static __device__ __forceinline__ float inv(float x) { return 1.0f / x; }
};
template <> struct Fn<__nv_bfloat16> {
    static __device__ __forceinline__ float exp(float x) { return __expf(x); }
    static __device__ __forceinline__ float log1p(float x) { return __logf(1.0f + x); }
    static __device__ __forceinline__ float inv(float x) { return __fdividef(1.0f, x); }   // (1 + exp(..) above 2^126 comes out as 0, as it should)
};
template <typename T> __device__ __forceinline__ float sigmoid(float x) { return Fn<T>::inv(1.0f + Fn<T>::exp(-x)); }
template <typename T> __device__ __forceinline__ float silu(float x) { return x * sigmoid<T>(x); }
template <typename T> __device__ __forceinline__ float softplus(float x) { return fmaxf(x, 0.f) + Fn<T>::log1p(Fn<T>::exp(-fabsf(x))); }
__device__ __forceinline__ float warp_sum(float v) {
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
template <typename T> __device__ __forceinline__ float gate_of(float x, int act) { return act == SWLM_GATE_SIGMOID ? sigmoid<T>(x) : silu<T>(x); }
// two fp32 numbers in one register pair: a * b + c and a * b on both
typedef unsigned long long pair_t;
__device__ __forceinline__ pair_t pair_of(float lo, float hi) { return (pair_t)__float_as_uint(lo) | ((pair_t)__float_as_uint(hi) << 32); }
__device__ __forceinline__ float pair_lo(pair_t v) { return __uint_as_float((unsigned)v); }
__device__ __forceinline__ float pair_hi(pair_t v) { return __uint_as_float((unsigned)(v >> 32)); }
__device__ __forceinline__ pair_t pair_fma(pair_t a, pair_t b, pair_t c) {
    pair_t d;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(d) : "l"(a), "l"(b), "l"(c));
    return d;
}
__device__ __forceinline__ pair_t pair_mul(pair_t a, pair_t b) {
    pair_t d;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(d) : "l"(a), "l"(b));
    return d;
}

__device__ __forceinline__ RowRun run_of(const DeltaParams& p, int i) {
    if (p.runs) return p.runs[i];
    const int row = p.single_rows ? p.single_rows[i] : i;
    return RowRun{row, 1, p.row_pos[row], p.row_seq[row], i};
}
// channel `ch` of q | k | v: its taps (q, k and v keep theirs in tensors of their own)
__device__ __forceinline__ const __nv_bfloat16* taps_of(const DeltaParams& p, int ch) {
    const int gk = p.sh.groups * p.sh.dim;
    return ch < gk ? p.conv_q + (size_t)ch * p.sh.taps : ch < 2 * gk ? p.conv_k + (size_t)(ch - gk) * p.sh.taps : p.conv_v + (size_t)(ch - 2 * gk) * p.sh.taps;
}
// input of channel ch at token i of a run; i < 0: what earlier batches left
template <typename T>
__device__ __forceinline__ float conv_input(const DeltaParams& p, const RowRun& run, int ch, int i) {
    if (i >= 0) return dl_get(static_cast<const T*>(p.qkv) + (size_t)(run.row0 + i) * p.qkv_stride + ch);
    const int pos = run.pos0 + i;
    if (pos < 0) return 0.f;
    return dl_get(static_cast<const T*>(p.ring) + ((size_t)run.seq * p.sh.taps + pos % p.sh.taps) * p.sh.channels() + ch);
}
template <typename T>
__device__ __forceinline__ float conv_silu(const DeltaParams& p, const RowRun& run, int ch, int i) {
    const __nv_bfloat16* w = taps_of(p, ch);
    float acc = 0.f;
    for (int j = 0; j < p.sh.taps; ++j) acc = fmaf(__bfloat162float(w[j]), conv_input<T>(p, run, ch, i - (p.sh.taps - 1) + j), acc);
    return silu<T>(acc);
}
template <typename T>
__device__ __forceinline__ float decay_of(const DeltaParams& p, int row, int h, int d, float rate) {
    const int i = p.decay_dim == 1 ? h : h * p.decay_dim + d;
    return Fn<T>::exp(-rate * softplus<T>(p.decay[(size_t)row * p.decay_stride + i] + __bfloat162float(p.dt_bias[i])));
}

// ---- portions: what a block needs of its tokens -----------------------------------------------------------------------
// CTA (block, head). Record: [TB][dp] beta_t G_t k_t, [TB][dp] G_t q_t, [TB][dp] D_Ts k_s, [dp] G_T, then two [TB][TB] matrices
// that turn w_s = beta_s v_s - S^T (beta_s G_s k_s) into u and into the block's own share of o: with A_ts = beta_t (k_s . D_ts k_t)
// for s < t and B_ts = k_s . D_ts q_t for s <= t, u = (I + A)^-1 w and the share is B u. Values: [column block][TB][kScanCols]
// beta_t v_t. Tokens past the end of the run: k = q = v = 0 and a decay of 1.
constexpr int kPrepTaps = 4;   // convolutions of up to this many taps read every input once
template <typename T>
__device__ __forceinline__ void conv_block(const DeltaParams& p, const RowRun& run, int ch, int t0, int nt, float (&y)[TB]) {
    if (p.sh.taps > kPrepTaps) {
#pragma unroll
        for (int t = 0; t < TB; ++t) y[t] = t < nt ? conv_silu<T>(p, run, ch, t0 + t) : 0.f;
        return;
    }
    const __nv_bfloat16* w = taps_of(p, ch);
    float wf[kPrepTaps], x[TB + kPrepTaps - 1];
#pragma unroll
    for (int j = 0; j < kPrepTaps; ++j) wf[j] = j < p.sh.taps ? __bfloat162float(w[p.sh.taps - 1 - j]) : 0.f;   // wf[j] meets the input j tokens back
    const T* in = static_cast<const T*>(p.qkv) + (size_t)(run.row0 + t0) * p.qkv_stride + ch;
    if (t0 >= kPrepTaps - 1) {
#pragma unroll
        for (int i = 0; i < TB + kPrepTaps - 1; ++i) {
            const int at = i - (kPrepTaps - 1);
            x[i] = at < nt ? dl_get(in + (ptrdiff_t)at * p.qkv_stride) : 0.f;
        }
    } else {
#pragma unroll
        for (int i = 0; i < TB + kPrepTaps - 1; ++i) {
            const int at = i - (kPrepTaps - 1);
            x[i] = at < nt && at > -p.sh.taps ? conv_input<T>(p, run, ch, t0 + at) : 0.f;
        }
    }
#pragma unroll
    for (int t = 0; t < TB; ++t) {
        float acc = 0.f;
#pragma unroll
        for (int j = kPrepTaps - 1; j >= 0; --j) acc = fmaf(wf[j], x[t + kPrepTaps - 1 - j], acc);
        y[t] = t < nt ? silu<T>(acc) : 0.f;
    }
}

// Sums over the warp of N values a lane (N a power of two up to 32); value lane * N / 32 is left in this lane. At every step half
// of the values go to the partner.
template <int N>
__device__ __forceinline__ float warp_sums(float (&v)[N], int lane) {
    int o = 16;
#pragma unroll
    for (int n = N / 2; n > 0; n >>= 1, o >>= 1) {
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

template <typename T>
__global__ void __launch_bounds__(kPrepThreads) delta_prepare_kernel(const DeltaParams p) {
    static_assert(TB == 4, "the pair sums of a block fill the lanes of a warp");
    pdl_wait();
    extern __shared__ __align__(16) float prep_smem[];
    __shared__ float beta_s[TB], decay_s[TB], norm_s[2 * TB], red[kPrepThreads / 32][2 * TB * TB], a_s[TB][TB], b_s[TB][TB], m_s[TB][TB];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, blk = blockIdx.x, h = blockIdx.y;
    const RowRun run = run_of(p, p.block_run ? p.block_run[blk] : blk);
    const int t0 = (blk - run.blk0) * TB, nt = min(TB, run.count - t0);
    const int dim = p.sh.dim, vdim = p.sh.vdim, grp = h / (p.sh.heads / p.sh.groups), gk = p.sh.groups * dim;
    const float rate = expf(__bfloat162float(p.a_log[h]));
    float* q = prep_smem;            // [TB][dim]
    float* k = q + TB * dim;         // [TB][dim]
    if (tid < TB) {
        const int row = run.row0 + t0 + tid;
        beta_s[tid] = tid < nt ? sigmoid<T>(p.beta[(size_t)row * p.beta_stride + h]) : 0.f;
        if (p.decay_dim == 1) decay_s[tid] = tid < nt ? decay_of<T>(p, row, h, 0, rate) : 1.f;
    }
    for (int i = tid; i < 2 * dim; i += kPrepThreads) {
        const int d = i < dim ? i : i - dim, ch = (i < dim ? 0 : gk) + grp * dim + d;
        float* dst = i < dim ? q : k;
        float y[TB];
        conv_block<T>(p, run, ch, t0, nt, y);
#pragma unroll
        for (int t = 0; t < TB; ++t) dst[t * dim + d] = y[t];
    }
    __syncthreads();
    float* vr = p.vrec + (size_t)(blk * p.sh.heads + h) * p.vblocks * TB * kScanCols;
    for (int c = tid; c < p.vblocks * kScanCols; c += kPrepThreads) {
        float y[TB] = {};
        if (c < vdim) conv_block<T>(p, run, 2 * gk + h * vdim + c, t0, nt, y);
#pragma unroll
        for (int t = 0; t < TB; ++t) vr[(c / kScanCols * TB + t) * kScanCols + c % kScanCols] = beta_s[t] * y[t];
    }
    for (int i = warp; i < 2 * TB; i += kPrepThreads / 32) {
        const float* x = (i < TB ? q : k) + (i % TB) * dim;
        float ss = 0.f;
        for (int d = lane; d < dim; d += 32) ss = fmaf(x[d], x[d], ss);
        ss = warp_sum(ss);
        if (lane == 0) norm_s[i] = (i < TB ? p.q_scale : 1.0f) / sqrtf(ss + p.unit_eps);
    }
    __syncthreads();
    float* rec = p.rec + (size_t)(blk * p.sh.heads + h) * p.rec_floats;
    float pairs[2 * TB * TB];   // A without beta, B
#pragma unroll
    for (int i = 0; i < 2 * TB * TB; ++i) pairs[i] = 0.f;
    for (int d = tid; d < p.dp; d += kPrepThreads) {
        float kv[TB], qv[TB], g[TB];
#pragma unroll
        for (int t = 0; t < TB; ++t) {
            const bool live = d < dim && t < nt;
            kv[t] = live ? k[t * dim + d] * norm_s[TB + t] : 0.f;
            qv[t] = live ? q[t * dim + d] * norm_s[t] : 0.f;
            g[t] = !live ? 1.f : p.decay_dim == 1 ? decay_s[t] : decay_of<T>(p, run.row0 + t0 + t, h, d, rate);
        }
        float gt = 1.f;
#pragma unroll
        for (int t = 0; t < TB; ++t) {
            gt *= g[t];
            rec[t * p.dp + d] = beta_s[t] * gt * kv[t];
            rec[(TB + t) * p.dp + d] = gt * qv[t];
        }
        rec[3 * TB * p.dp + d] = gt;
#pragma unroll
        for (int s = 0; s < TB; ++s) {
            float w = kv[s];
            pairs[TB * TB + s * TB + s] = fmaf(w, qv[s], pairs[TB * TB + s * TB + s]);
#pragma unroll
            for (int t = s + 1; t < TB; ++t) {
                w *= g[t];
                pairs[t * TB + s] = fmaf(w, kv[t], pairs[t * TB + s]);
                pairs[TB * TB + t * TB + s] = fmaf(w, qv[t], pairs[TB * TB + t * TB + s]);
            }
            rec[(2 * TB + s) * p.dp + d] = w;
        }
    }
    red[warp][lane] = warp_sums(pairs, lane);
    __syncthreads();
    if (tid < 2 * TB * TB) {
        float v = 0.f;
#pragma unroll
        for (int w = 0; w < kPrepThreads / 32; ++w) v += red[w][tid];
        const int t = tid % (TB * TB) / TB, s = tid % TB;
        if (tid < TB * TB) a_s[t][s] = beta_s[t] * v;
        else b_s[t][s] = v;
    }
    __syncwarp();
    if (tid < TB) {   // column tid of (I + A)^-1
        float m[TB];
#pragma unroll
        for (int t = 0; t < TB; ++t) {
            m[t] = t == tid ? 1.f : 0.f;
#pragma unroll
            for (int s = 0; s < t; ++s) m[t] = fmaf(-a_s[t][s], m[s], m[t]);
            m_s[t][tid] = m[t];
        }
    }
    __syncwarp();
    if (tid < 2 * TB * TB) {
        const int t = tid % (TB * TB) / TB, s = tid % TB;
        float v = m_s[t][s];
        if (tid >= TB * TB) {
            v = 0.f;
            for (int e = 0; e <= t; ++e) v = fmaf(b_s[t][e], m_s[e][s], v);
        }
        rec[(3 * TB + 1) * p.dp + tid] = v;
    }
}

// ---- portions: the recurrence -----------------------------------------------------------------------------------------
// CTA (16 columns of the state, head, run): a warp holds two columns, a lane key channels 4 lane + 128 i + (0 .. 3) of them, so
// that a record row is read once per two columns. The 16 products of a block with the state (w and o of four tokens and two
// columns) are summed across the warp in 16 exchanges that leave one in each pair of lanes. Records come through a ring of bulk copies.
// At the end the run's last inputs go to the convolution ring (all readers of the old ones have finished).
// Launched without overlap: CTAs that move in while another kernel drains would crowd together on the SMs that drain first.
template <typename T, int R>
__global__ void __launch_bounds__(kScanThreads) delta_scan_kernel(const DeltaParams p) {
    constexpr int DP = R * 32, REC = (3 * TB + 1) * DP + 2 * TB * TB, VREC = TB * kScanCols, STAGE = REC + VREC, WC = kScanWarpCols;
    constexpr int kScanStages = scan_stages(R);
    extern __shared__ __align__(128) float scan_smem[];
    __shared__ __align__(8) unsigned long long full_bar[kScanStages], empty_bar[kScanStages];
    __shared__ __align__(16) float u_s[kScanWarps][TB * WC];
    static_assert(WC == 2, "lane = 16 * (0: w, 1: o) + 4 * token + 2 * column + copy");
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int vb = blockIdx.x, h = blockIdx.y, col0 = vb * kScanCols + warp * WC;
    if (tid == 0) {
        for (int s = 0; s < kScanStages; ++s) { mbar_init(&full_bar[s], 1); mbar_init(&empty_bar[s], kScanWarps); }
        asm volatile("fence.mbarrier_init.release.cluster;" ::: "memory");
    }
    __syncthreads();
    pdl_wait();
    const RowRun run = run_of(p, blockIdx.z);
    const int nb = (run.count + TB - 1) / TB;
    auto request = [&](int b, int s) {
        const unsigned bar = smem_u32(&full_bar[s]), dst = smem_u32(scan_smem + (size_t)s * STAGE);
        const size_t at = (size_t)(run.blk0 + b) * p.sh.heads + h;
        mbar_expect(bar, STAGE * 4);
        bulk_load(dst, p.rec + at * REC, REC * 4, bar);
        bulk_load(dst + REC * 4, p.vrec + (at * p.vblocks + vb) * VREC, VREC * 4, bar);
    };
    if (warp == kScanWarps) {
        if (lane == 0) {
            int b = 0;
            for (int s = 0, round = 0; b < nb; ++b) {
                if (round > 0 && !mbar_wait(&empty_bar[s], (unsigned)((round - 1) & 1))) { atomicExch(p.status, 52); break; }
                request(b, s);
                if (++s == kScanStages) { s = 0; ++round; }
            }
            // leave only when the copies that may still be under way have landed (bounded)
            for (int q = max(0, b - kScanStages); q < b; ++q) mbar_wait(&full_bar[q % kScanStages], (unsigned)((q / kScanStages) & 1));
        }
        return;
    }
    float* st = p.state + ((size_t)run.seq * p.sh.heads + h) * p.sh.dim * p.sh.vdim + col0;
    auto channel = [&](int i) { return lane * 4 + 128 * (i >> 2) + (i & 3); };
    pair_t S[WC][R / 2];
    auto load = [&](int i, int c) { return run.pos0 > 0 && channel(i) < p.sh.dim && col0 + c < p.sh.vdim ? st[(size_t)channel(i) * p.sh.vdim + c] : 0.f; };
#pragma unroll
    for (int i = 0; i < R; i += 2)
#pragma unroll
        for (int c = 0; c < WC; ++c) S[c][i / 2] = pair_of(load(i, c), load(i + 1, c));
    // after the sums lane = 16 * (0: w, 1: o) + 4 * token + 2 * column + copy
    const int tok = (lane >> 2) & 3, lc = (lane >> 1) & 1, oc = col0 + lc;
    float* o_at = p.o + ((size_t)(run.row0 + tok) * p.sh.heads + h) * p.sh.vdim + oc;
    const size_t o_step = (size_t)TB * p.sh.heads * p.sh.vdim;
    for (int b = 0, s = 0, round = 0; b < nb; ++b) {
        if (!mbar_wait(&full_bar[s], (unsigned)(round & 1))) { atomicExch(p.status, 51); return; }   // (uniform; the requesting warp sees the copies out)
        const float* rec = scan_smem + (size_t)s * STAGE;
        const ulonglong2* r2 = reinterpret_cast<const ulonglong2*>(rec) + lane;
        const float4 coef = *reinterpret_cast<const float4*>(rec + (3 * TB + 1) * DP + (lane >> 2) * TB);
        const float vv = rec[REC + tok * kScanCols + warp * WC + lc];
        pair_t acc[2 * TB * WC];
#pragma unroll
        for (int i = 0; i < R / 4; ++i)
#pragma unroll
            for (int t = 0; t < 2 * TB; ++t) {
                const ulonglong2 y = r2[(t * DP + 128 * i) / 4];
#pragma unroll
                for (int c = 0; c < WC; ++c) {
                    pair_t& a = acc[t * WC + c];
                    a = i == 0 ? pair_mul(S[c][0], y.x) : pair_fma(S[c][2 * i], y.x, a);
                    a = pair_fma(S[c][2 * i + 1], y.y, a);
                }
            }
        float x[2 * TB * WC];
#pragma unroll
        for (int i = 0; i < 2 * TB * WC; ++i) x[i] = pair_lo(acc[i]) + pair_hi(acc[i]);
        const float sum = warp_sums(x, lane);
        const float w = vv - sum;                            // (of lanes 0 .. 15)
        float r = lane < 16 ? 0.f : sum;
        r = fmaf(coef.x, __shfl_sync(0xffffffffu, w, lane & 3), r);
        r = fmaf(coef.y, __shfl_sync(0xffffffffu, w, 4 + (lane & 3)), r);
        r = fmaf(coef.z, __shfl_sync(0xffffffffu, w, 8 + (lane & 3)), r);
        r = fmaf(coef.w, __shfl_sync(0xffffffffu, w, 12 + (lane & 3)), r);
        if (!(lane & 1)) {
            if (lane < 16) u_s[warp][lane >> 1] = r;
            else if (oc < p.sh.vdim && b * TB + tok < run.count) o_at[b * o_step] = r;
        }
        __syncwarp();
        float u[TB * WC];
#pragma unroll
        for (int t = 0; t < TB * WC; t += 4) {
            const float4 v = *reinterpret_cast<const float4*>(&u_s[warp][t]);
            u[t] = v.x; u[t + 1] = v.y; u[t + 2] = v.z; u[t + 3] = v.w;
        }
#pragma unroll
        for (int i = 0; i < R / 4; ++i) {
            const ulonglong2 g = r2[(3 * TB * DP + 128 * i) / 4];
#pragma unroll
            for (int c = 0; c < WC; ++c) { S[c][2 * i] = pair_mul(S[c][2 * i], g.x); S[c][2 * i + 1] = pair_mul(S[c][2 * i + 1], g.y); }
#pragma unroll
            for (int t = 0; t < TB; ++t) {
                const ulonglong2 kt = r2[((2 * TB + t) * DP + 128 * i) / 4];
#pragma unroll
                for (int c = 0; c < WC; ++c) {
                    const pair_t uu = pair_of(u[t * WC + c], u[t * WC + c]);
                    S[c][2 * i] = pair_fma(kt.x, uu, S[c][2 * i]);
                    S[c][2 * i + 1] = pair_fma(kt.y, uu, S[c][2 * i + 1]);
                }
            }
        }
        __syncwarp();
        if (lane == 0) asm volatile("mbarrier.arrive.shared::cta.b64 _, [%0];" ::"r"(smem_u32(&empty_bar[s])) : "memory");   // the stage is free
        if (++s == kScanStages) { s = 0; ++round; }
    }
#pragma unroll
    for (int i = 0; i < R; ++i)
#pragma unroll
        for (int c = 0; c < WC; ++c)
            if (channel(i) < p.sh.dim && col0 + c < p.sh.vdim) st[(size_t)channel(i) * p.sh.vdim + c] = i & 1 ? pair_hi(S[c][i / 2]) : pair_lo(S[c][i / 2]);
    if (vb == 0) {
        const int share = p.sh.heads / p.sh.groups, gk = p.sh.groups * p.sh.dim, ch_all = p.sh.channels();
        const int n_qk = h % share == 0 ? p.sh.dim : 0, grp = h / share;
        for (int back = 0; back < min(run.count, p.sh.taps); ++back) {
            const int tok = run.count - 1 - back, slot = (run.pos0 + tok) % p.sh.taps;
            const T* src = static_cast<const T*>(p.qkv) + (size_t)(run.row0 + tok) * p.qkv_stride;
            T* dst = static_cast<T*>(p.ring) + ((size_t)run.seq * p.sh.taps + slot) * ch_all;
            for (int i = tid; i < p.sh.vdim + 2 * n_qk; i += kScanWarps * 32) {
                const int ch = i < p.sh.vdim ? 2 * gk + h * p.sh.vdim + i : i < p.sh.vdim + n_qk ? grp * p.sh.dim + i - p.sh.vdim : gk + grp * p.sh.dim + i - p.sh.vdim - n_qk;
                dst[ch] = src[ch];
            }
        }
    }
}

// ---- portions: norm and gate ------------------------------------------------------------------------------------------
// CTA (block, head), a warp per token.
template <typename T>
__global__ void __launch_bounds__(TB * 32) delta_gate_kernel(const DeltaParams p) {
    pdl_launch_dependents();
    pdl_wait();
    const int lane = threadIdx.x & 31, t = threadIdx.x >> 5, blk = blockIdx.x, h = blockIdx.y, vdim = p.sh.vdim;
    const RowRun run = run_of(p, p.block_run ? p.block_run[blk] : blk);
    const int i = (blk - run.blk0) * TB + t;
    if (i >= run.count) return;
    const int row = run.row0 + i;
    const float* o = p.o + ((size_t)row * p.sh.heads + h) * vdim;
    float ss = 0.f;
    for (int c = lane; c < vdim; c += 32) ss = fmaf(o[c], o[c], ss);
    const float sc = 1.0f / sqrtf(warp_sum(ss) / (float)vdim + p.eps);
    const T* gate = static_cast<const T*>(p.gate) + (size_t)row * p.gate_stride + (size_t)h * vdim;
    T* out = static_cast<T*>(p.out) + (size_t)row * p.out_stride + (size_t)h * vdim;
    for (int c = lane; c < vdim; c += 32) dl_put(out + c, o[c] * sc * __bfloat162float(p.norm_w[c]) * gate_of<T>(dl_get(gate + c), p.gate_act));
}

// ---- single tokens ----------------------------------------------------------------------------------------------------
// Cluster of CTAs per (head, row), 32 state columns each: warp w holds key channels w, w + 8, ... of the CTA's columns, lane =
// column. Nothing of this layer's state is touched by the kernels in front of this one, so it is read ahead of them. The slot
// of the convolution ring that is written (position % taps) is none of those that are read.
template <typename T, int R>
__global__ void __launch_bounds__(kStepThreads, R <= 16 ? 3 : 2) delta_step_kernel(const DeltaParams p) {
    extern __shared__ __align__(16) float step_smem[];
    __shared__ float part_a[kStepWarps][kStepCols], part_b[kStepWarps][kStepCols], scal[4], v_s[kStepCols], ssq[kStepCluster];
    const cg::cluster_group cluster = cg::this_cluster();
    auto started = cluster.barrier_arrive();   // waited for before anything is written to another CTA's shared memory
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, vb = blockIdx.x, h = blockIdx.y;
    const int row = p.single_rows ? p.single_rows[blockIdx.z] : blockIdx.z, pos = p.row_pos[row], seq = p.row_seq[row];
    const int dim = p.sh.dim, vdim = p.sh.vdim, taps = p.sh.taps, share = p.sh.heads / p.sh.groups, grp = h / share, gk = p.sh.groups * dim, ch_all = p.sh.channels();
    const int col = vb * kStepCols + lane;
    const bool live = col < vdim;
    float* q = step_smem;        // [dim]
    float* k = q + dim;          // [dim]
    float* g = k + dim;          // [dim]
    float* st = p.state + ((size_t)seq * p.sh.heads + h) * dim * vdim + col;
    float S[R];
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = warp + kStepWarps * i;
        S[i] = live && pos > 0 && d < dim ? st[(size_t)d * vdim] : 0.f;
    }
    // channel tid + 256 j of q | k | this CTA's v: the past's share of the convolution
    constexpr int CH = (2 * R * kStepWarps + kStepCols + kStepThreads - 1) / kStepThreads;
    const T* ring = static_cast<const T*>(p.ring) + (size_t)seq * taps * ch_all;
    float acc[CH], w_last[CH];
    int chan[CH];
#pragma unroll
    for (int j = 0; j < CH; ++j) {
        const int i = tid + kStepThreads * j, vc = vb * kStepCols + i - 2 * dim;
        chan[j] = i < dim ? grp * dim + i : i < 2 * dim ? gk + grp * dim + i - dim : i < 2 * dim + kStepCols && vc < vdim ? 2 * gk + h * vdim + vc : -1;
        acc[j] = w_last[j] = 0.f;
        if (chan[j] >= 0) {
            const __nv_bfloat16* w = taps_of(p, chan[j]);
            for (int e = 0; e + 1 < taps; ++e) {
                const int at = pos - (taps - 1) + e;
                if (at >= 0) acc[j] = fmaf(__bfloat162float(w[e]), dl_get(ring + (size_t)(at % taps) * ch_all + chan[j]), acc[j]);
            }
            w_last[j] = __bfloat162float(w[taps - 1]);
        }
    }
    const float rate = expf(__bfloat162float(p.a_log[h]));
    const float nw = live ? __bfloat162float(p.norm_w[col]) : 0.f;
    pdl_wait();

    const bool keeps_qk = vb == 0 && h % share == 0;
#pragma unroll
    for (int j = 0; j < CH; ++j) {
        const int i = tid + kStepThreads * j;
        float y = 0.f;
        if (chan[j] >= 0) {
            const T x = static_cast<const T*>(p.qkv)[(size_t)row * p.qkv_stride + chan[j]];
            y = silu<T>(fmaf(w_last[j], dl_get(&x), acc[j]));
            if (i >= 2 * dim || keeps_qk) const_cast<T*>(ring)[(size_t)(pos % taps) * ch_all + chan[j]] = x;
        }
        if (i < dim) q[i] = y;
        else if (i < 2 * dim) k[i - dim] = y;
        else if (i < 2 * dim + kStepCols) v_s[i - 2 * dim] = y;
    }
    if (p.decay_dim == 1) {
        const float one = decay_of<T>(p, row, h, 0, rate);
        for (int d = tid; d < dim; d += kStepThreads) g[d] = one;
    } else {
        for (int d = tid; d < dim; d += kStepThreads) g[d] = decay_of<T>(p, row, h, d, rate);
    }
    const float gate = live && warp == 0 ? gate_of<T>(dl_get(static_cast<const T*>(p.gate) + (size_t)row * p.gate_stride + (size_t)h * vdim + col), p.gate_act) : 0.f;
    const float beta = sigmoid<T>(p.beta[(size_t)row * p.beta_stride + h]);
    __syncthreads();
    if (warp < 3) {
        const float* x = warp == 1 ? k : q;
        const float* y = warp == 0 ? q : k;
        float ss = 0.f;
        for (int d = lane; d < dim; d += 32) ss = fmaf(x[d], y[d], ss);
        ss = warp_sum(ss);
        if (lane == 0) scal[warp] = ss;
    }
    __syncthreads();
    const float qn = p.q_scale / sqrtf(scal[0] + p.unit_eps), kn = 1.0f / sqrtf(scal[1] + p.unit_eps);
    float a = 0.f, b = 0.f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = warp + kStepWarps * i;
        if (d < dim) {
            S[i] *= g[d];
            a = fmaf(S[i], k[d], a);
            b = fmaf(S[i], q[d], b);
        }
    }
    part_a[warp][lane] = a;
    part_b[warp][lane] = b;
    __syncthreads();
    a = b = 0.f;
#pragma unroll
    for (int w = 0; w < kStepWarps; ++w) { a += part_a[w][lane]; b += part_b[w][lane]; }
    const float u = beta * (v_s[lane] - a * kn), uk = u * kn;
    const float o = live ? fmaf(scal[2] * qn, uk, b * qn) : 0.f;
#pragma unroll
    for (int i = 0; i < R; ++i) {
        const int d = warp + kStepWarps * i;
        if (d < dim && live) st[(size_t)d * vdim] = fmaf(k[d], uk, S[i]);
    }
    const int nz = gridDim.x;
    cluster.barrier_wait(std::move(started));
    if (warp == 0) {
        const float ss = warp_sum(o * o);
        if (lane < nz) cluster.map_shared_rank(ssq, lane)[vb] = ss;
    }
    cluster.sync();
    if (warp == 0 && live) {
        float ss = 0.f;
        for (int i = 0; i < nz; ++i) ss += ssq[i];
        dl_put(static_cast<T*>(p.out) + (size_t)row * p.out_stride + (size_t)h * vdim + col, o / sqrtf(ss / (float)vdim + p.eps) * nw * gate);
    }
}

// ---- launches ---------------------------------------------------------------------------------------------------------
int scan_regs(int dim) { return dim <= 128 ? 4 : dim <= 256 ? 8 : dim <= 512 ? 16 : 0; }   // key channels per lane
int rec_floats(int dim) { return (3 * TB + 1) * scan_regs(dim) * 32 + 2 * TB * TB; }
int scan_vblocks(int vdim) { return (vdim + kScanCols - 1) / kScanCols; }
size_t scan_smem_bytes(int dim) { return (size_t)scan_stages(scan_regs(dim)) * (rec_floats(dim) + TB * kScanCols) * 4; }

template <typename T, int R>
int scan_launch(const DeltaParams& p, int runs, cudaStream_t s) {
    static const cudaError_t attr = cudaFuncSetAttribute(delta_scan_kernel<T, R>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)scan_smem_bytes(R * 32));
    if (attr != cudaSuccess) return cuda_fail(attr, "delta scan attributes");
    delta_scan_kernel<T, R><<<dim3(p.vblocks, p.sh.heads, runs), dim3(kScanThreads), scan_smem_bytes(R * 32), s>>>(p);
    const cudaError_t e = cudaGetLastError();
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "delta scan launch");
}
template <typename T>
int portions(const DeltaParams& p, int runs, int blocks, cudaStream_t s) {
    cudaError_t e = launch_k(delta_prepare_kernel<T>, dim3(blocks, p.sh.heads), dim3(kPrepThreads), (size_t)2 * TB * p.sh.dim * 4, s, p);
    if (e != cudaSuccess) return cuda_fail(e, "delta prepare launch");
    int rc;
    switch (scan_regs(p.sh.dim)) {
    case 4: rc = scan_launch<T, 4>(p, runs, s); break;
    case 8: rc = scan_launch<T, 8>(p, runs, s); break;
    default: rc = scan_launch<T, 16>(p, runs, s); break;
    }
    if (rc) return rc;
    e = launch_k(delta_gate_kernel<T>, dim3(blocks, p.sh.heads), dim3(TB * 32), 0, s, p);
    return e == cudaSuccess ? SWLM_OK : cuda_fail(e, "delta gate launch");
}
template <typename T, int R>
cudaError_t step_launch(const DeltaParams& p, cudaStream_t s) {
    const int nz = (p.sh.vdim + kStepCols - 1) / kStepCols;
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(nz, p.sh.heads, p.n_single); cfg.blockDim = dim3(kStepThreads); cfg.stream = s;
    cfg.dynamicSmemBytes = (size_t)3 * p.sh.dim * 4;
    cudaLaunchAttribute attr[2];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = nz; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = 1;
    attr[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    attr[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = attr;
    cfg.numAttrs = pdl_enabled() ? 2 : 1;
    return cudaLaunchKernelEx(&cfg, delta_step_kernel<T, R>, p);
}
template <typename T>
int run(const DeltaLaunch& a, DeltaParams p, cudaStream_t s, int* launches) {
    int rc;
    if (a.n_single > 0) {
        if (delta_step_fits(a.shape)) {
            const int regs = (a.shape.dim + kStepWarps - 1) / kStepWarps;
            const cudaError_t e = regs <= 8 ? step_launch<T, 8>(p, s) : regs <= 16 ? step_launch<T, 16>(p, s) : step_launch<T, 32>(p, s);
            if (e != cudaSuccess) return cuda_fail(e, "delta step launch");
            *launches += 1;
        } else {
            if ((rc = portions<T>(p, a.n_single, a.n_single, s))) return rc;
            *launches += 3;
        }
    }
    if (a.n_runs > 0) {
        p.runs = a.runs;
        p.block_run = a.block_run;
        if ((rc = portions<T>(p, a.n_runs, a.n_blocks, s))) return rc;
        *launches += 3;
    }
    return SWLM_OK;
}

}  // namespace

bool delta_supported(const DeltaShape& s) {
    return s.heads > 0 && s.groups > 0 && s.heads % s.groups == 0 && s.dim > 0 && s.vdim > 0 && s.taps > 0 && scan_regs(s.dim) > 0;
}
bool delta_step_fits(const DeltaShape& s) { return s.dim <= 32 * kStepWarps && s.vdim <= kStepCols * kStepCluster; }
size_t delta_scratch_floats(const DeltaShape& s, int blocks, int rows) {
    return (size_t)blocks * s.heads * (rec_floats(s.dim) + (size_t)scan_vblocks(s.vdim) * TB * kScanCols) + (size_t)rows * s.heads * s.vdim;
}

int launch_delta(const DeltaLaunch& a, cudaStream_t s, int* launches) {
    DeltaParams p{};
    p.sh = a.shape; p.decay_dim = a.decay_dim; p.gate_act = a.gate_act; p.eps = a.eps; p.unit_eps = a.unit_eps; p.q_scale = a.q_scale;
    p.qkv = a.qkv; p.qkv_stride = a.qkv_stride; p.beta = a.beta; p.beta_stride = a.beta_stride; p.decay = a.decay; p.decay_stride = a.decay_stride;
    p.gate = a.gate; p.gate_stride = a.gate_stride; p.conv_q = a.conv_q; p.conv_k = a.conv_k; p.conv_v = a.conv_v; p.norm_w = a.norm_w;
    p.a_log = a.a_log; p.dt_bias = a.dt_bias; p.ring = a.ring; p.state = a.state; p.row_seq = a.row_seq; p.row_pos = a.row_pos;
    p.out = a.out; p.out_stride = a.out_stride; p.n_single = a.n_single; p.single_rows = a.single_rows; p.status = a.status;
    p.dp = scan_regs(a.shape.dim) * 32; p.rec_floats = rec_floats(a.shape.dim); p.vblocks = scan_vblocks(a.shape.vdim);
    const int blocks = std::max(a.n_blocks, a.n_single);
    p.rec = a.scratch;
    p.vrec = p.rec + (size_t)blocks * a.shape.heads * p.rec_floats;
    p.o = p.vrec + (size_t)blocks * a.shape.heads * p.vblocks * TB * kScanCols;
    return a.f32 ? run<float>(a, p, s, launches) : run<__nv_bfloat16>(a, p, s, launches);
}

}  // namespace swlm
