// Executor of fp32-stream plans: step list -> launches, the paged pool of latent rows, and one row executor that runs decode
// steps, prompt chunks and mixed batches alike. A batch is a list of rows, each with its token, sequence and position; the
// only steps that look beyond their own row are latent and grouped attention, which find the cached rows through the page table,
// and the gated delta rule, retention and convolutions over the stream, which carry a state per sequence.
#include <cmath>
#include <cstdio>
#include <cstring>

#include "swlm_runtime.h"

namespace swlm {
namespace {

bool stored_f32(const swlm_plan* p, int buf) {
    return p->all_f32() || buf == SWLM_BUF_HIDDEN || buf == SWLM_BUF_RESIDUAL || buf == SWLM_BUF_SCRATCH3 || buf == SWLM_BUF_SCRATCH4 || buf == SWLM_BUF_LOGITS;
}
size_t stored_bytes(const swlm_plan* p, int buf) { return stored_f32(p, buf) ? 4 : 2; }
bool act_buf(const swlm_plan* p, int buf) { return buf >= SWLM_BUF_SCRATCH0 && buf <= SWLM_BUF_SCRATCH2; }   // buffers products read
bool any_buf(int b) { return b >= 0 && b < SWLM_BUF_COUNT; }

int find_matrix(swlm_ctx* ctx, const char* name, int n, int k, const Matrix** out) {
    auto it = ctx->matrices.find(name);
    if (it == ctx->matrices.end()) { set_error("matrix '%s' not in the weight store", name); return SWLM_ERR_NOT_FOUND; }
    if (it->second.n != n || it->second.k != k) { set_error("matrix '%s' is %d x %d, the step wants %d x %d", name, it->second.n, it->second.k, n, k); return SWLM_ERR_INVALID; }
    *out = &it->second;
    return SWLM_OK;
}
int find_vector(swlm_ctx* ctx, const char* name, int count, const DenseTensor** out) {
    auto it = ctx->dense.find(name);
    if (it == ctx->dense.end()) { set_error("tensor '%s' not in the weight store", name); return SWLM_ERR_NOT_FOUND; }
    if (it->second.rows * it->second.cols != count) { set_error("tensor '%s' holds %lld values, the step wants %d", name, (long long)(it->second.rows * it->second.cols), count); return SWLM_ERR_INVALID; }
    *out = &it->second;
    return SWLM_OK;
}

// The rows of several matrices one after the other; the parts become views of it, so nothing is stored twice.
int concat_matrices(swlm_ctx* ctx, const std::vector<std::string>& names, const Matrix** out) {
    std::string key = names[0];
    for (size_t i = 1; i < names.size(); ++i) key += "|" + names[i];
    auto hit = ctx->matrix_cat.find(key);
    if (hit != ctx->matrix_cat.end()) { *out = &hit->second; return SWLM_OK; }
    Matrix cat;
    cat.k = ctx->matrices.at(names[0]).k; cat.ld = ctx->matrices.at(names[0]).ld;
    for (const std::string& nm : names) cat.n += ctx->matrices.at(nm).n;
    int rc = dev_alloc(&cat.data, (size_t)cat.n * cat.ld, &ctx->bytes);
    if (rc) return rc;
    size_t row = 0;
    for (const std::string& nm : names) {
        Matrix& m = ctx->matrices.at(nm);
        if (m.ld != cat.ld) { set_error("matrix '%s' is already part of a product over side-by-side matrices", nm.c_str()); return SWLM_ERR_UNSUPPORTED; }
        SWLM_CUDA(cudaMemcpy(cat.data + row * cat.ld, m.data, (size_t)m.n * m.ld * 2, cudaMemcpyDeviceToDevice));
        if (!m.view) {
            // plans built earlier may hold the old address: their kernels are ordered before the free by the device
            SWLM_CUDA(cudaDeviceSynchronize());
            cudaFree(m.data);
            ctx->bytes -= (int64_t)m.n * m.ld * 2;
        }
        m.data = cat.data + row * cat.ld;
        m.view = true;
        row += m.n;
    }
    ctx->matrix_cat[key] = cat;
    *out = &ctx->matrix_cat[key];
    return SWLM_OK;
}

// Two matrices side by side, the second from a multiple of 8 columns on; both become views of the result.
int join_matrices(swlm_ctx* ctx, const char* left, const char* right, const Matrix** out) {
    const std::string key = std::string(left) + "&" + right;
    auto hit = ctx->matrix_cat.find(key);
    if (hit != ctx->matrix_cat.end()) { *out = &hit->second; return SWLM_OK; }
    Matrix* part[2] = {&ctx->matrices.at(left), &ctx->matrices.at(right)};
    const int at[2] = {0, (part[0]->k + 7) / 8 * 8};
    Matrix both;
    both.n = part[0]->n; both.k = at[1] + part[1]->k; both.ld = (both.k + 7) / 8 * 8;
    if (part[0]->view || part[1]->view || !strcmp(left, right)) { set_error("matrices '%s' and '%s' are already part of a concatenated matrix", left, right); return SWLM_ERR_UNSUPPORTED; }
    const int rc = dev_alloc(&both.data, (size_t)both.n * both.ld, &ctx->bytes);
    if (rc) return rc;
    SWLM_CUDA(cudaMemset(both.data, 0, (size_t)both.n * both.ld * 2));
    for (int i = 0; i < 2; ++i) {
        Matrix& m = *part[i];
        SWLM_CUDA(cudaMemcpy2D(both.data + at[i], (size_t)both.ld * 2, m.data, (size_t)m.ld * 2, (size_t)m.k * 2, m.n, cudaMemcpyDeviceToDevice));
        SWLM_CUDA(cudaDeviceSynchronize());
        cudaFree(m.data);
        ctx->bytes -= (int64_t)m.n * m.ld * 2;
        m.data = both.data + at[i];
        m.ld = both.ld;
        m.view = true;
    }
    ctx->matrix_cat[key] = both;
    *out = &ctx->matrix_cat[key];
    return SWLM_OK;
}

// Angle per position of every pair, interpolated by parts when the step says so, in double precision on the host.
int stream_rope_table(swlm_plan* plan, const swlm_step& st, int* index) {
    const float divisor = st.rope_divisor > 0.f ? st.rope_divisor : 1.f;
    for (size_t i = 0; i < plan->rope_tables.size(); ++i) {
        const RopeTable& t = plan->rope_tables[i];
        if (t.divisor == divisor && t.rope_dim == st.rope_dim && t.base == st.rope_base && t.factor == st.rope_factor && t.original == st.rope_original &&
            t.fast == st.rope_fast && t.slow == st.rope_slow) { *index = (int)i; return SWLM_OK; }
    }
    const int half = st.rope_dim / 2;
    std::vector<float> f(std::max(1, half));
    const double base = st.rope_base, dims = st.rope_dim;
    RopeTable t;
    t.rope_dim = st.rope_dim; t.base = st.rope_base; t.factor = st.rope_factor; t.original = st.rope_original; t.fast = st.rope_fast; t.slow = st.rope_slow; t.divisor = divisor;
    double lo = 0, hi = 0;
    if (st.rope_factor > 0.f) {
        auto dim_of = [&](double turns) { return dims * std::log((double)st.rope_original / (2.0 * M_PI * turns)) / (2.0 * std::log(base)); };
        lo = std::max(std::floor(dim_of(st.rope_fast)), 0.0);
        hi = std::min(std::ceil(dim_of(st.rope_slow)), dims - 1.0);
        t.magnitude = (float)(0.1 * std::log((double)st.rope_factor) + 1.0);
    }
    for (int i = 0; i < half; ++i) {
        const double plain = std::pow(base, -2.0 * i / dims);
        const double ramp = st.rope_factor > 0.f ? std::min(1.0, std::max(0.0, (i - lo) / std::max(hi - lo, 0.001))) : 0.0;
        f[i] = (float)((ramp > 0.0 ? plain / st.rope_factor * ramp + plain * (1.0 - ramp) : plain) / divisor);
    }
    int rc = dev_alloc(&t.inv_freq, f.size());
    if (rc) return rc;
    SWLM_CUDA(cudaMemcpy(t.inv_freq, f.data(), f.size() * 4, cudaMemcpyHostToDevice));
    plan->rope_tables.push_back(t);
    *index = (int)plan->rope_tables.size() - 1;
    return SWLM_OK;
}

bool is_norm(int kind) {
    return kind == SWLM_STEP_COPY_RMSNORM || kind == SWLM_STEP_RESADD_COPY_RMSNORM || kind == SWLM_STEP_RESADD_RMSNORM ||
           kind == SWLM_STEP_POSTNORM_RESADD_COPY_RMSNORM || kind == SWLM_STEP_POSTNORM_RESADD_RMSNORM;
}
bool is_postnorm(int kind) { return kind == SWLM_STEP_POSTNORM_RESADD_COPY_RMSNORM || kind == SWLM_STEP_POSTNORM_RESADD_RMSNORM; }
bool norm_stores(const swlm_step& s) { const int kind = s.kind; return (kind == SWLM_STEP_COPY_RMSNORM && s.in_buf != SWLM_BUF_RESIDUAL) || kind == SWLM_STEP_RESADD_COPY_RMSNORM || kind == SWLM_STEP_POSTNORM_RESADD_COPY_RMSNORM; }
bool reads(const Launch& L, int buf) {
    const swlm_step& s = L.st;
    if (s.in_buf == buf || L.x2_buf == buf) return true;
    if (L.kind == L_JOIN) return L.join.in_buf == buf || L.join.gate_buf == buf;
    return s.kind != SWLM_STEP_PRODUCT && !is_norm(s.kind) && (s.in2_buf == buf || s.in3_buf == buf || s.in4_buf == buf);
}
bool is_glu(int kind) { return kind == SWLM_STEP_SWIGLU || kind == SWLM_STEP_GEGLU || kind == SWLM_STEP_CLAMPED_GLU; }
GatedAct glu_of(const swlm_step& s) {
    GatedAct a;
    a.kind = s.kind == SWLM_STEP_GEGLU ? GATED_ACT_GELU_TANH : s.kind == SWLM_STEP_CLAMPED_GLU ? GATED_ACT_CLAMPED : GATED_ACT_SILU;
    a.alpha = s.scale;
    a.limit = s.limit;
    return a;
}
RoutedShape routed_shape(const swlm_step& s) { return RoutedShape{s.experts, s.top, s.groups, s.groups_keep, s.n, s.k, s.weight5[0] ? s.k2 : 0, s.identity}; }
bool is_join(const swlm_step& s) {
    return s.kind == SWLM_STEP_GATED_POSTNORM_ADD || s.kind == SWLM_STEP_DEPTH_AVG || s.kind == SWLM_STEP_STREAM_CONV || s.kind == SWLM_STEP_STREAM_COPY ||
           (s.kind == SWLM_STEP_EMBED && s.out_buf == SWLM_BUF_RESIDUAL);
}
DeltaShape retention_shape(const swlm_step& s) { return DeltaShape{s.heads, s.heads, s.key_dim, s.value_dim, 0}; }
const char* glu_name(int kind) { return kind == GATED_ACT_GELU_TANH ? "geglu" : kind == GATED_ACT_CLAMPED ? "clamped glu" : "swiglu"; }

// One step over the stream into the parts of a launch; false: it has to be a launch of its own (the parts are in order).
bool join_takes(const JoinParts& j, const swlm_step& s) {
    const bool out = j.copy_buf >= 0 || j.conv_buf >= 0;
    switch (s.kind) {
    case SWLM_STEP_EMBED: return !j.changes() && !out;
    case SWLM_STEP_GATED_POSTNORM_ADD: return !j.changes() && !out;
    case SWLM_STEP_DEPTH_AVG: return !j.table && !j.avg && !out;
    case SWLM_STEP_STREAM_CONV: return j.conv_buf < 0;
    default: return j.copy_buf < 0;
    }
}

int join_part(swlm_plan* plan, const swlm_step& s, JoinParts* j) {
    swlm_ctx* ctx = plan->ctx;
    const swlm_buffers_desc& d = plan->desc;
    int rc;
    if (s.n != d.hidden) { set_error("step over the stream: %d entries, the stream has %d", s.n, d.hidden); return SWLM_ERR_INVALID; }
    switch (s.kind) {
    case SWLM_STEP_EMBED: {
        auto it = ctx->dense.find(s.weight);
        if (it == ctx->dense.end()) { set_error("embedding table '%s' missing", s.weight); return SWLM_ERR_NOT_FOUND; }
        if (it->second.cols != s.n || it->second.rows != d.vocab) { set_error("embedding '%s': table %lld x %lld for vocabulary %d, width %d", s.weight, (long long)it->second.rows, (long long)it->second.cols, d.vocab, d.hidden); return SWLM_ERR_INVALID; }
        j->table = &it->second;
        j->table_scale = s.scale != 0.f ? s.scale : 1.f;
        if (d.depth_results > 0) j->store = 0;
        return SWLM_OK;
    }
    case SWLM_STEP_GATED_POSTNORM_ADD:
        if (s.in_buf != SWLM_BUF_HIDDEN || (s.in3_buf != SWLM_BUF_NONE && s.in3_buf != SWLM_BUF_SCRATCH3 && s.in3_buf != SWLM_BUF_SCRATCH4)) { set_error("gated norm '%s': reads hidden, gate in scratch 3 or 4", s.weight); return SWLM_ERR_INVALID; }
        if ((rc = find_vector(ctx, s.weight, s.n, &j->w))) return rc;
        j->adds = true; j->in_buf = s.in_buf; j->gate_buf = s.in3_buf; j->eps = s.eps; j->weight_bias = s.weight_bias;
        return SWLM_OK;
    case SWLM_STEP_DEPTH_AVG:
        if (s.k < 1 || s.k > d.depth_results) { set_error("average over %d results, %d are kept", s.k, d.depth_results); return SWLM_ERR_INVALID; }
        if ((rc = find_vector(ctx, s.weight, s.k, &j->avg_w))) return rc;
        j->avg = s.k; j->store = s.k - 1;
        return SWLM_OK;
    case SWLM_STEP_STREAM_CONV: {
        if (s.layer < 0 || s.layer >= d.stream_convs) { set_error("convolution over the stream: layer %d has no state", s.layer); return SWLM_ERR_INVALID; }
        if (!act_buf(plan, s.out_buf) || !join_supported(s.n, s.conv_kernel) || s.conv_kernel < 1) { set_error("convolution over the stream: %d taps, result in scratch 0..2", s.conv_kernel); return SWLM_ERR_UNSUPPORTED; }
        if ((rc = find_vector(ctx, s.weight, s.n * s.conv_kernel, &j->conv_w))) return rc;
        StreamConv& c = plan->convs[s.layer];
        if (c.taps && c.taps != s.conv_kernel) { set_error("convolution state %d is used with %d and %d taps", s.layer, c.taps, s.conv_kernel); return SWLM_ERR_INVALID; }
        c.taps = s.conv_kernel;
        j->conv = s.layer; j->conv_buf = s.out_buf;
        return SWLM_OK;
    }
    default:
        if (!act_buf(plan, s.out_buf)) { set_error("copy of the stream: into scratch 0..2"); return SWLM_ERR_INVALID; }
        j->copy_buf = s.out_buf;
        return SWLM_OK;
    }
}

}  // namespace

int stream_compile(swlm_plan* plan) {
    swlm_ctx* ctx = plan->ctx;
    const swlm_buffers_desc& d = plan->desc;
    const std::vector<swlm_step>& st = plan->steps;
    if (ctx->tp_size > 1) { set_error("fp32-stream plans run on one GPU"); return SWLM_ERR_UNSUPPORTED; }
    if (d.stream_dtype < 0 || d.stream_dtype > SWLM_STREAM_ALL_F32) { set_error("stream_dtype %d", d.stream_dtype); return SWLM_ERR_INVALID; }
    int rc;
    auto widen = [&](int buf, int n) { plan->stream_width[buf] = std::max(plan->stream_width[buf], (n + 7) / 8 * 8); };
    auto window_set = [&](int window) {
        const int at = (int)(std::find(plan->windows.begin(), plan->windows.end(), window) - plan->windows.begin());
        if (at == (int)plan->windows.size()) plan->windows.push_back(window);
        return at;
    };
    plan->latent.assign(std::max(0, d.latent_layers), LatentLayer{});
    plan->grouped.assign(std::max(0, d.grouped_layers), GroupedLayer{});
    plan->delta.assign(std::max(0, d.delta_layers), DeltaLayer{});
    for (const swlm_step& s : st) plan->biased |= s.kind == SWLM_STEP_PRODUCT && s.weight3[0];
    plan->convs.assign(std::max(0, d.stream_convs), StreamConv{});
    int unkept = -1;   // convolution whose state does not have its last inputs yet
    widen(SWLM_BUF_HIDDEN, d.hidden);
    widen(SWLM_BUF_RESIDUAL, d.hidden);
    widen(SWLM_BUF_LOGITS, d.vocab);
    for (size_t i = 0; i < st.size();) {
        const swlm_step& s = st[i];
        Launch L;
        L.st = s;
        if (is_join(s)) {
            L.kind = L_JOIN;
            L.label = "stream";
            L.steps_covered = 0;
            for (size_t j = i; j < st.size() && is_join(st[j]) && join_takes(L.join, st[j]); ++j) {
                if ((rc = join_part(plan, st[j], &L.join))) return rc;
                if (st[j].kind == SWLM_STEP_STREAM_CONV || st[j].kind == SWLM_STEP_STREAM_COPY) widen(st[j].out_buf, st[j].n);
                if (st[j].in3_buf != SWLM_BUF_NONE) widen(st[j].in3_buf, st[j].n);
                L.label += std::string(" + ") + (st[j].weight[0] ? st[j].weight : "copy");
                L.steps_covered += 1;
            }
            if (L.join.changes() && unkept >= 0) { L.join.keep = unkept; unkept = -1; }
            if (L.join.conv >= 0 && plan->convs[L.join.conv].taps > 1) {
                if (unkept >= 0) { set_error("two convolutions over the stream without a change of it between them"); return SWLM_ERR_UNSUPPORTED; }
                unkept = L.join.conv;
            }
            i += L.steps_covered;
            plan->launches.push_back(L);
            continue;
        }
        switch (s.kind) {
        case SWLM_STEP_EMBED: {
            L.kind = L_EMBED;
            auto it = ctx->dense.find(s.weight);
            if (it == ctx->dense.end()) { set_error("embedding table '%s' missing", s.weight); return SWLM_ERR_NOT_FOUND; }
            L.d1 = &it->second;
            if (s.out_buf != SWLM_BUF_HIDDEN || s.n != d.hidden || L.d1->cols != s.n || L.d1->rows != d.vocab) { set_error("embedding '%s': table %lld x %lld for vocabulary %d, width %d", s.weight, (long long)L.d1->rows, (long long)L.d1->cols, d.vocab, d.hidden); return SWLM_ERR_INVALID; }
            L.label = std::string("embed ") + s.weight;
            break;
        }
        case SWLM_STEP_COPY_RMSNORM: case SWLM_STEP_RESADD_COPY_RMSNORM: case SWLM_STEP_RESADD_RMSNORM:
        case SWLM_STEP_POSTNORM_RESADD_COPY_RMSNORM: case SWLM_STEP_POSTNORM_RESADD_RMSNORM:
            L.kind = L_RMSNORM;
            if ((s.in_buf != SWLM_BUF_HIDDEN && (s.in_buf != SWLM_BUF_RESIDUAL || s.kind != SWLM_STEP_COPY_RMSNORM)) || !act_buf(plan, s.out_buf) || s.n != d.hidden) { set_error("norm '%s': reads hidden, writes scratch 0..2, width %d", s.weight, d.hidden); return SWLM_ERR_INVALID; }
            if ((rc = find_vector(ctx, is_postnorm(s.kind) ? s.weight2 : s.weight, s.n, &L.d1))) return rc;
            if (is_postnorm(s.kind) && (rc = find_vector(ctx, s.weight, s.n, &L.norm_post))) return rc;
            if (is_postnorm(s.kind) && s.weight3[0]) {   // an embedding row joins
                auto it = ctx->dense.find(s.weight3);
                if (it == ctx->dense.end()) { set_error("embedding table '%s' missing", s.weight3); return SWLM_ERR_NOT_FOUND; }
                if (it->second.cols != s.n || it->second.rows != d.vocab) { set_error("norm '%s': table '%s' is %lld x %lld", s.weight, s.weight3, (long long)it->second.rows, (long long)it->second.cols); return SWLM_ERR_INVALID; }
                L.dv[0] = &it->second;
            }
            widen(s.out_buf, s.n);
            L.label = std::string(is_postnorm(s.kind) ? "postnorm+rmsnorm " : "rmsnorm ") + (is_postnorm(s.kind) ? s.weight2 : s.weight);
            break;
        case SWLM_STEP_PRODUCT: {
            L.kind = L_PRODUCT;
            if (!act_buf(plan, s.in_buf) || !any_buf(s.out_buf) || s.out_buf == s.in_buf || s.out_buf == SWLM_BUF_RESIDUAL) { set_error("product '%s': bad buffers", s.weight); return SWLM_ERR_INVALID; }
            if ((rc = find_matrix(ctx, s.weight, s.n, s.k, &L.m1))) return rc;
            if (s.weight3[0] && (rc = find_vector(ctx, s.weight3, s.n, &L.seg_bias[0]))) return rc;
            if (s.weight2[0]) {   // side by side with a second matrix
                const Matrix* right;
                if (s.k2 <= 0 || s.in_off < 0 || s.out_off < 0 || (s.in_off & 7)) { set_error("product '%s': bad columns", s.weight); return SWLM_ERR_INVALID; }
                if ((rc = find_matrix(ctx, s.weight2, s.n, s.k2, &right)) || (rc = join_matrices(ctx, s.weight, s.weight2, &L.m1))) return rc;
                widen(s.in_buf, s.in_off + L.m1->k);
                widen(s.out_buf, s.out_off + s.n);
                L.seg_buf[0] = s.out_buf; L.seg_off[0] = s.out_off; L.seg_end[0] = s.n;
                L.label = std::string("product ") + s.weight + " & " + s.weight2;
                break;
            }
            if (s.in_off < 0 || s.out_off < 0 || (s.in_off & 7) || (s.out_buf == SWLM_BUF_LOGITS && s.out_off)) { set_error("product '%s': input columns start at multiples of 8", s.weight); return SWLM_ERR_INVALID; }
            widen(s.in_buf, s.in_off + s.k);
            widen(s.out_buf, s.out_off + s.n);
            // gate, up, gated activation -> one launch
            if (i + 2 < st.size() && st[i + 1].kind == SWLM_STEP_PRODUCT && !st[i + 1].weight2[0] && !s.weight3[0] && !st[i + 1].weight3[0] && is_glu(st[i + 2].kind) && !s.in_off && !s.out_off && !st[i + 1].in_off && !st[i + 1].out_off &&
                st[i + 1].in_buf == s.in_buf && st[i + 1].k == s.k && st[i + 1].n == s.n && st[i + 2].in_buf == s.out_buf &&
                st[i + 2].in2_buf == st[i + 1].out_buf && st[i + 2].n == s.n && act_buf(plan, st[i + 2].out_buf) && st[i + 2].out_buf != s.in_buf &&
                act_buf(plan, s.out_buf) && act_buf(plan, st[i + 1].out_buf)) {
                if ((rc = find_matrix(ctx, st[i + 1].weight, s.n, s.k, &L.m2))) return rc;
                widen(st[i + 1].out_buf, s.n);
                widen(st[i + 2].out_buf, s.n);
                L.act = glu_of(st[i + 2]);
                L.seg_buf[0] = st[i + 2].out_buf; L.seg_end[0] = s.n;
                L.seg_buf[1] = s.out_buf; L.seg_buf[2] = st[i + 1].out_buf;   // where the halves go when they run apart
                L.steps_covered = 3;
                L.label = std::string("product+gate ") + s.weight + " ^ " + st[i + 1].weight;
                break;
            }
            std::vector<std::string> names{s.weight};
            L.seg_buf[0] = s.out_buf; L.seg_off[0] = s.out_off; L.seg_end[0] = s.n;
            L.label = std::string("product ") + s.weight;
            // the soft cap of the logits happens where they are stored
            if (s.out_buf == SWLM_BUF_LOGITS && i + 1 < st.size() && st[i + 1].kind == SWLM_STEP_SOFTCAP && st[i + 1].scale > 0.f && st[i + 1].n == s.n) {
                L.softcap = st[i + 1].scale;
                L.steps_covered = 2;
                L.label += " + softcap";
                break;
            }
            size_t j = i + 1;
            int rows = s.n;
            while (j < st.size() && (int)names.size() < kMaxProductSegs && st[j].kind == SWLM_STEP_PRODUCT && !st[j].weight2[0] && st[j].k == s.k &&
                   st[j].out_off >= 0 && st[j].out_buf != s.in_buf && any_buf(st[j].out_buf) && st[j].out_buf != SWLM_BUF_LOGITS && s.out_buf != SWLM_BUF_LOGITS) {
                // products of one input, and behind them of a second one (no result may go there)
                const bool same = st[j].in_buf == s.in_buf && st[j].in_off == s.in_off && L.x2_buf < 0;
                const bool second = act_buf(plan, st[j].in_buf) && st[j].in_buf != s.in_buf && !st[j].in_off && !s.in_off && (L.x2_buf < 0 || L.x2_buf == st[j].in_buf) && st[j].out_buf != st[j].in_buf;
                if (!same && !second) break;
                bool clash = false;
                for (size_t q = i; q < j; ++q)
                    clash |= (!same && st[q].out_buf == st[j].in_buf) || (st[q].out_buf == st[j].out_buf && st[q].out_off < st[j].out_off + st[j].n && st[j].out_off < st[q].out_off + st[q].n) || !strcmp(st[q].weight, st[j].weight);
                // a gate / up pair that starts here keeps its own launch
                if (clash || (j + 2 < st.size() && is_glu(st[j + 2].kind) && st[j + 2].in_buf == st[j].out_buf)) break;
                const Matrix* m;
                if ((rc = find_matrix(ctx, st[j].weight, st[j].n, st[j].k, &m))) return rc;
                widen(st[j].out_buf, st[j].out_off + st[j].n);
                const int q = (int)names.size();
                if (st[j].weight3[0] && (rc = find_vector(ctx, st[j].weight3, st[j].n, &L.seg_bias[q]))) return rc;
                if (!same && L.x2_buf < 0) { L.x2_buf = st[j].in_buf; L.first_segs = q; widen(st[j].in_buf, st[j].k); L.part[0].n = rows; }
                rows += st[j].n;
                L.seg_buf[q] = st[j].out_buf; L.seg_off[q] = st[j].out_off; L.seg_end[q] = L.seg_end[q - 1] + st[j].n;
                names.push_back(st[j].weight);
                L.label += std::string(" ") + st[j].weight;
                ++j;
            }
            L.n_seg = (int)names.size();
            L.steps_covered = L.n_seg;
            if (L.n_seg > 1 && (rc = concat_matrices(ctx, names, &L.m1))) return rc;
            if (L.x2_buf >= 0) {
                const int split = L.part[0].n;
                L.part[0] = L.part[1] = *L.m1;
                L.part[0].n = split;
                L.part[1].n = rows - split;
                L.part[1].data = L.m1->data + (size_t)split * L.m1->ld;
            }
            break;
        }
        case SWLM_STEP_SWIGLU: case SWLM_STEP_GEGLU: case SWLM_STEP_CLAMPED_GLU:
            L.kind = L_SWIGLU;
            L.act = glu_of(s);
            if (!act_buf(plan, s.in_buf) || !act_buf(plan, s.in2_buf) || !act_buf(plan, s.out_buf) || s.n <= 0) { set_error("gated activation: bad buffers"); return SWLM_ERR_INVALID; }
            widen(s.in_buf, s.n); widen(s.in2_buf, s.n); widen(s.out_buf, s.n);
            L.label = glu_name(L.act.kind);
            break;
        case SWLM_STEP_LATENT_ATTN: {
            L.kind = L_LATENT;
            if (s.layer < 0 || s.layer >= d.latent_layers) { set_error("latent attention: layer %d outside the pool", s.layer); return SWLM_ERR_INVALID; }
            if (s.heads <= 0 || s.head_dim <= 0 || s.key_dim < 0 || s.value_dim <= 0 || s.n <= 0 || s.rope_dim < 0 || s.rope_dim > s.key_dim || (s.rope_dim & 1)) { set_error("latent attention: bad sizes"); return SWLM_ERR_INVALID; }
            if (!act_buf(plan, s.in_buf) || !stored_f32(plan, s.in2_buf) || !any_buf(s.in2_buf) || !act_buf(plan, s.out_buf) || s.out_buf == s.in_buf ||
                (s.in3_buf != SWLM_BUF_NONE && (!any_buf(s.in3_buf) || !stored_f32(plan, s.in3_buf)))) { set_error("latent attention: q and the result in scratch 0..2, latent and gate in scratch 3 and 4"); return SWLM_ERR_INVALID; }
            if ((rc = find_vector(ctx, s.weight, s.n, &L.d1))) return rc;
            if (s.n > 8192 || s.head_dim + s.key_dim > 4096) { set_error("latent attention: latent of %d, query of %d entries per head", s.n, s.head_dim + s.key_dim); return SWLM_ERR_UNSUPPORTED; }
            const Matrix *uk, *uv;
            if ((rc = find_matrix(ctx, s.weight2, s.heads * s.head_dim, s.n, &uk)) || (rc = find_matrix(ctx, s.weight3, s.heads * s.value_dim, s.n, &uv))) return rc;
            const Matrix* both;
            const std::vector<std::string> pair{s.weight2, s.weight3};
            if ((rc = concat_matrices(ctx, pair, &both))) return rc;
            L.m1 = uk; L.m2 = uv;
            if ((rc = stream_rope_table(plan, s, &L.rope_table))) return rc;
            if (s.window_left < 0) { set_error("latent attention: window %d", s.window_left); return SWLM_ERR_INVALID; }
            if (s.weight4[0] && (rc = find_vector(ctx, s.weight4, s.heads, &L.dv[0]))) return rc;
            L.window_set = window_set(s.window_left);
            LatentLayer& ll = plan->latent[s.layer];
            if (ll.rank && (ll.rank != s.n || ll.rot != s.key_dim)) { set_error("latent layer %d is used with two row sizes", s.layer); return SWLM_ERR_INVALID; }
            ll.rank = s.n; ll.rot = s.key_dim; ll.row = latent_row(s.n, s.key_dim, plan->all_f32());
            widen(s.in_buf, s.heads * (s.head_dim + s.key_dim));
            widen(s.in2_buf, s.n + s.key_dim);
            if (s.in3_buf != SWLM_BUF_NONE) widen(s.in3_buf, s.heads);
            widen(s.out_buf, s.heads * s.value_dim);
            plan->latent_heads_max = std::max(plan->latent_heads_max, s.heads);
            plan->latent_q_floats = std::max(plan->latent_q_floats, (int)latent_qcat_floats(ll.row, s.heads));
            plan->latent_part_floats = std::max(plan->latent_part_floats, (int)latent_partial_floats(ll.row, s.heads));
            L.label = std::string("latent_attention ") + s.weight2;
            break;
        }
        case SWLM_STEP_GATED_DELTA: {
            L.kind = L_DELTA;
            if (s.layer < 0 || s.layer >= d.delta_layers) { set_error("gated delta rule: layer %d has no state", s.layer); return SWLM_ERR_INVALID; }
            DeltaShape shape;
            shape.heads = s.heads; shape.groups = s.groups; shape.dim = s.key_dim; shape.vdim = s.value_dim; shape.taps = s.conv_kernel;
            if (!delta_supported(shape) || (s.k != 1 && s.k != s.key_dim) || (s.gate_act != SWLM_GATE_SILU && s.gate_act != SWLM_GATE_SIGMOID)) { set_error("gated delta rule: %d heads over %d groups, %d x %d, %d taps, %d decays per head", s.heads, s.groups, s.key_dim, s.value_dim, s.conv_kernel, s.k); return SWLM_ERR_UNSUPPORTED; }
            const bool same_scalars = s.in2_buf == s.in3_buf && s.in2_off < s.in3_off + s.heads * s.k && s.in3_off < s.in2_off + s.heads;
            const bool same_rows = s.in4_buf == s.in_buf && s.in4_off < shape.channels();
            if (!act_buf(plan, s.in_buf) || !any_buf(s.in2_buf) || !stored_f32(plan, s.in2_buf) || !any_buf(s.in3_buf) || !stored_f32(plan, s.in3_buf) || same_scalars || same_rows ||
                s.in2_off < 0 || s.in3_off < 0 || s.in4_off < 0 || !act_buf(plan, s.in4_buf) || !act_buf(plan, s.out_buf) || s.out_buf == s.in_buf || (s.out_buf == s.in4_buf && s.in4_off)) { set_error("gated delta rule: q | k | v, gate and result in scratch 0..2, step sizes and decays in scratch 3 and 4"); return SWLM_ERR_INVALID; }
            const char* names[6] = {s.weight, s.weight2, s.weight3, s.weight4, s.weight5, s.weight6};
            const int counts[6] = {s.groups * s.key_dim * s.conv_kernel, s.groups * s.key_dim * s.conv_kernel, s.heads * s.value_dim * s.conv_kernel, s.value_dim, s.heads, s.heads * s.k};
            for (int q = 0; q < 6; ++q) if ((rc = find_vector(ctx, names[q], counts[q], &L.dv[q]))) return rc;
            DeltaLayer& dl = plan->delta[s.layer];
            if (dl.shape.heads && memcmp(&dl.shape, &shape, sizeof(shape))) { set_error("gated-delta layer %d is used with two shapes", s.layer); return SWLM_ERR_INVALID; }
            dl.shape = shape;
            widen(s.in_buf, shape.channels());
            widen(s.in2_buf, s.in2_off + s.heads);
            widen(s.in3_buf, s.in3_off + s.heads * s.k);
            widen(s.in4_buf, s.in4_off + s.heads * s.value_dim);
            widen(s.out_buf, s.heads * s.value_dim);
            L.label = std::string("gated_delta ") + s.weight4;
            break;
        }
        case SWLM_STEP_ROUTED_MLP: {
            L.kind = L_ROUTED;
            const bool gated = s.weight2[0], shared = s.weight5[0];
            const RoutedShape shape = routed_shape(s);
            if (!routed_supported(shape) || (shared && (s.k2 <= 0 || gated || s.identity)) || s.expert_act < 0 || s.expert_act > SWLM_EXPERT_SILU) { set_error("routed feed-forward: %d of %d experts, %d of %d groups, %d x %d, shared %d", s.top, s.experts, s.groups_keep, s.groups, s.n, s.k, s.k2); return SWLM_ERR_UNSUPPORTED; }
            if (s.score_act < 0 || s.score_act > SWLM_SCORE_SOFTMAX || s.group_best < 0 || s.group_best > 2) { set_error("routed feed-forward: scores %d, group %d", s.score_act, s.group_best); return SWLM_ERR_UNSUPPORTED; }
            if (!act_buf(plan, s.in_buf) || !any_buf(s.in2_buf) || !stored_f32(plan, s.in2_buf) || s.out_buf != SWLM_BUF_HIDDEN || s.n != d.hidden) { set_error("routed feed-forward: input in scratch 0..2, logits in scratch 3 or 4, result in hidden"); return SWLM_ERR_INVALID; }
            const char* suffix[3] = {s.weight2, s.weight3, s.weight4};
            const Matrix** into[3] = {&L.m1, &L.m2, &L.m3};
            for (int q = gated ? 0 : 1; q < 3; ++q) {
                std::vector<std::string> names;
                for (int e = 0; e < s.experts; ++e) {
                    names.push_back(std::string(s.weight) + std::to_string(e) + suffix[q]);
                    const Matrix* m;
                    if ((rc = find_matrix(ctx, names.back().c_str(), q < 2 ? s.k : s.n, q < 2 ? s.n : s.k, &m))) return rc;
                }
                if ((rc = concat_matrices(ctx, names, into[q]))) return rc;
            }
            if (shared && ((rc = find_matrix(ctx, s.weight5, s.k2, s.n, &L.m4)) || (rc = find_matrix(ctx, s.weight6, s.n, s.k2, &L.m5)))) return rc;
            if (s.weight7[0] && (rc = find_vector(ctx, s.weight7, shape.scored(), &L.dv[0]))) return rc;
            if (L.dv[0] && s.groups != 1) { set_error("routed feed-forward: a correction goes with one group"); return SWLM_ERR_UNSUPPORTED; }
            L.act.kind = s.expert_act == SWLM_EXPERT_SILU ? GATED_ACT_SILU : GATED_ACT_CLAMPED; L.act.alpha = s.glu_alpha; L.act.limit = s.limit;
            widen(s.in_buf, s.n);
            widen(s.in2_buf, shape.scored() + (shared ? 1 : 0));
            widen(s.out_buf, s.n);
            L.label = std::string("routed_mlp ") + s.weight;
            break;
        }
        case SWLM_STEP_GROUPED_ATTN: {
            L.kind = L_GROUPED;
            if (s.layer < 0 || s.layer >= d.grouped_layers) { set_error("grouped attention: layer %d outside the pool", s.layer); return SWLM_ERR_INVALID; }
            if (s.heads <= 0 || s.kv_heads <= 0 || s.heads % s.kv_heads || s.head_dim <= 0 || s.value_dim <= 0 || s.rope_dim < 0 || s.rope_dim > s.head_dim || (s.rope_dim & 1) ||
                s.window_left < 0 || s.chunk < 0) { set_error("grouped attention: bad sizes"); return SWLM_ERR_INVALID; }
            if (!act_buf(plan, s.in_buf) || !act_buf(plan, s.out_buf) || s.out_buf == s.in_buf || s.in_off < 0 || (s.in_off & 7) || s.out_off < 0 || (s.out_off & 7) ||
                (s.in3_buf != SWLM_BUF_NONE && (!any_buf(s.in3_buf) || !stored_f32(plan, s.in3_buf)))) { set_error("grouped attention: q | k | v and the result in scratch 0..2 from columns that are multiples of 8, gate in scratch 3 or 4"); return SWLM_ERR_INVALID; }
            if (s.weight[0] && (rc = find_vector(ctx, s.weight, s.head_dim, &L.dv[0]))) return rc;
            if (s.weight2[0] && (rc = find_vector(ctx, s.weight2, s.head_dim, &L.dv[1]))) return rc;
            if ((s.value_is_key && (s.value_dim != s.head_dim || s.rope_dim || s.weight[0] || s.weight2[0])) || (s.head_norm && (s.weight[0] || s.weight2[0])) || s.temp_every < 0) { set_error("grouped attention: values that are keys go without rotation and norm weights"); return SWLM_ERR_UNSUPPORTED; }
            const bool entry_gate = s.in4_buf != SWLM_BUF_NONE;
            const int kv_entries = s.kv_heads * (s.head_dim + (s.value_is_key ? 0 : s.value_dim));
            if (entry_gate && (!act_buf(plan, s.in4_buf) || s.in4_buf == s.out_buf || s.in4_off < 0 || (s.in4_buf == s.in_buf && s.in4_off < s.in_off + s.heads * s.head_dim + kv_entries))) { set_error("grouped attention: gates of the entries in scratch 0..2, behind q | k | v"); return SWLM_ERR_INVALID; }
            const GroupedRow row = grouped_row(s.kv_heads, s.head_dim, s.value_dim, plan->all_f32(), s.value_is_key);
            if (!grouped_supported(row)) { set_error("grouped attention: heads of %d and %d", s.head_dim, s.value_dim); return SWLM_ERR_UNSUPPORTED; }
            if ((rc = stream_rope_table(plan, s, &L.rope_table))) return rc;
            L.window_set = window_set(s.window_left);
            GroupedLayer& gl = plan->grouped[s.layer];
            if (gl.row.groups && memcmp(&gl.row, &row, sizeof(row))) { set_error("grouped layer %d is used with two row sizes", s.layer); return SWLM_ERR_INVALID; }
            gl.row = row;
            widen(s.in_buf, s.in_off + s.heads * s.head_dim + kv_entries);
            if (entry_gate) widen(s.in4_buf, s.in4_off + s.heads * s.value_dim);
            if (s.in3_buf != SWLM_BUF_NONE) widen(s.in3_buf, s.heads);
            widen(s.out_buf, s.out_off + s.heads * s.value_dim);
            L.label = std::string("grouped_attention ") + s.weight;
            break;
        }
        case SWLM_STEP_RETENTION: {
            L.kind = L_RETENTION;
            if (s.layer < 0 || s.layer >= d.delta_layers) { set_error("retention: layer %d has no state", s.layer); return SWLM_ERR_INVALID; }
            if (!retention_supported(s.heads, s.key_dim, s.value_dim)) { set_error("retention: %d heads of %d x %d", s.heads, s.key_dim, s.value_dim); return SWLM_ERR_UNSUPPORTED; }
            if (!act_buf(plan, s.in_buf) || !act_buf(plan, s.in4_buf) || !act_buf(plan, s.out_buf) || s.out_buf == s.in_buf || s.out_buf == s.in4_buf || s.in_off < 0 || s.in4_off < 0 || s.out_off < 0 ||
                ((s.in_off | s.in4_off | s.out_off) & 7)) { set_error("retention: q | k | v, gate and result in scratch 0..2, from columns that are multiples of 8"); return SWLM_ERR_INVALID; }
            auto decay = ctx->densef.find(s.weight);
            if (decay == ctx->densef.end() || decay->second.count != s.heads) { set_error("retention: decays '%s' missing or not one per head", s.weight); return SWLM_ERR_NOT_FOUND; }
            L.f1 = &decay->second;
            DeltaLayer& dl = plan->delta[s.layer];
            const DeltaShape shape = retention_shape(s);
            if (dl.shape.heads && memcmp(&dl.shape, &shape, sizeof(shape))) { set_error("state %d is used with two shapes", s.layer); return SWLM_ERR_INVALID; }
            dl.shape = shape;
            widen(s.in_buf, s.in_off + s.heads * (2 * s.key_dim + s.value_dim));
            widen(s.in4_buf, s.in4_off + s.heads * s.value_dim);
            widen(s.out_buf, s.out_off + s.heads * s.value_dim);
            L.label = std::string("retention ") + s.weight;
            break;
        }
        case SWLM_STEP_TOKEN_GATE: {
            L.kind = L_TOKEN_GATE;
            auto it = ctx->dense.find(s.weight);
            if (it == ctx->dense.end()) { set_error("table '%s' missing", s.weight); return SWLM_ERR_NOT_FOUND; }
            L.d1 = &it->second;
            if (s.n <= 0 || !act_buf(plan, s.in_buf) || !act_buf(plan, s.out_buf) || s.in2_off < 0 || L.d1->rows != d.vocab || L.d1->cols < s.in2_off + s.n) { set_error("token gate '%s': columns %d .. %d of a table %lld x %lld", s.weight, s.in2_off, s.in2_off + s.n, (long long)L.d1->rows, (long long)L.d1->cols); return SWLM_ERR_INVALID; }
            widen(s.in_buf, s.n); widen(s.out_buf, s.n);
            L.label = std::string("token gate ") + s.weight;
            break;
        }
        case SWLM_STEP_SOFTCAP:
            L.kind = L_SOFTCAP;
            if (s.in_buf != SWLM_BUF_LOGITS || s.n != d.vocab || !(s.scale > 0.f)) { set_error("soft cap: of the logits, by a positive number"); return SWLM_ERR_INVALID; }
            L.label = "softcap";
            break;
        case SWLM_STEP_ARGMAX:
            L.kind = L_ARGMAX;
            if (s.in_buf != SWLM_BUF_LOGITS || s.n != d.vocab) { set_error("argmax: reads the logits"); return SWLM_ERR_INVALID; }
            L.label = "argmax";
            break;
        default:
            set_error("step %zu: kind %d cannot be part of an fp32-stream plan", i, s.kind);
            return SWLM_ERR_UNSUPPORTED;
        }
        i += L.steps_covered;
        plan->launches.push_back(L);
    }
    if (unkept >= 0) {   // nothing changes the stream any more: a launch that only keeps its rows
        Launch L;
        L.kind = L_JOIN;
        L.join.keep = unkept;
        L.st.in_buf = L.st.in2_buf = L.st.in3_buf = L.st.in4_buf = L.st.out_buf = SWLM_BUF_NONE;
        L.label = "stream rows to their state";
        L.steps_covered = 0;
        plan->launches.push_back(L);
    }
    for (int l = 0; l < d.stream_convs; ++l)
        if (!plan->convs[l].taps && st.size() > 1) { set_error("convolution %d has no step", l); return SWLM_ERR_INVALID; }
    for (int l = 0; l < d.latent_layers; ++l)
        if (!plan->latent[l].rank && st.size() > 1) { set_error("latent layer %d has no step", l); return SWLM_ERR_INVALID; }
    for (int l = 0; l < d.grouped_layers; ++l)
        if (!plan->grouped[l].row.groups && st.size() > 1) { set_error("grouped layer %d has no step", l); return SWLM_ERR_INVALID; }
    for (int l = 0; l < d.delta_layers; ++l)
        if (!plan->delta[l].shape.heads && st.size() > 1) { set_error("state %d has no step", l); return SWLM_ERR_INVALID; }

    // A norm rides with the product behind it when that is its only reader: few rows compute it in the product's prologue,
    // more rows run it in front.
    for (size_t i = 0; i + 1 < plan->launches.size(); ++i) {
        const Launch A = plan->launches[i];
        Launch& B = plan->launches[i + 1];
        if (A.kind != L_RMSNORM || B.kind != L_PRODUCT || B.st.in_buf != A.st.out_buf || B.st.in_off || B.x2_buf >= 0) continue;
        bool ok = true;
        for (size_t j = i + 2; j < plan->launches.size(); ++j) {
            const Launch& C = plan->launches[j];
            if (reads(C, A.st.out_buf)) { ok = false; break; }
            bool writes = C.kind == L_JOIN ? C.join.conv_buf == A.st.out_buf || C.join.copy_buf == A.st.out_buf : C.st.out_buf == A.st.out_buf;
            for (int q = 0; q < C.n_seg; ++q) writes |= C.seg_buf[q] == A.st.out_buf;
            if (writes) break;
        }
        if (!ok) continue;
        B.norm = A.st; B.norm_w = A.d1; B.norm_post = A.norm_post; B.dv[0] = A.dv[0];
        B.label = A.label + " + " + B.label;
        B.steps_covered += 1;
        plan->launches.erase(plan->launches.begin() + i);
    }
    // A join that only hands the stream on to a token input, its two products, and the join behind them
    for (size_t i = 0; i + 4 < plan->launches.size(); ++i) {
        const Launch *q = &plan->launches[i], &A = q[0], &G = q[1], &T = q[2], &P = q[3], &B = q[4];
        if (A.kind != L_JOIN || G.kind != L_PRODUCT || T.kind != L_TOKEN_GATE || P.kind != L_PRODUCT || B.kind != L_JOIN) continue;
        const bool plain = G.n_seg == 1 && P.n_seg == 1 && !G.m2 && !P.m2 && !G.st.weight2[0] && !P.st.weight2[0] && !G.seg_bias[0] && !P.seg_bias[0] && !G.norm.kind && !P.norm.kind && !G.st.in_off && !P.st.in_off &&
                           !G.st.out_off && !P.st.out_off;
        const bool chain = A.join.adds && A.join.copy_buf >= 0 && A.join.conv < 0 && !A.join.avg && A.join.store < 0 && G.st.in_buf == A.join.copy_buf && T.st.in_buf == G.st.out_buf && T.st.n == G.st.n &&
                           P.st.in_buf == T.st.out_buf && P.st.k == T.st.n && P.st.out_buf == SWLM_BUF_HIDDEN && P.st.n == d.hidden && G.st.k == d.hidden && B.join.adds && B.join.gate_buf < 0 && B.join.keep < 0;
        bool again = false;   // does anything read the buffers that are not written then, before they are written again?
        for (const int buf : {A.join.copy_buf, T.st.out_buf, (int)G.st.out_buf})
            for (size_t j = i + 4; j < plan->launches.size(); ++j) {
                const Launch& C = plan->launches[j];
                if (j > i + 4 && reads(C, buf)) { again = true; break; }
                bool writes = C.kind == L_JOIN ? C.join.conv_buf == buf || C.join.copy_buf == buf : C.st.out_buf == buf;
                for (int s2 = 0; s2 < C.n_seg; ++s2) writes |= C.seg_buf[s2] == buf;
                if (writes) break;
            }
        if (plain && chain && !again) plan->launches[i].fused = 4;
    }
    // the residual stream alternates between two buffers, so that a norm computed by every CTA of a product can be stored by one
    int cur = 0;
    for (Launch& L : plan->launches) {
        const swlm_step* norm = L.kind == L_RMSNORM ? &L.st : L.kind == L_PRODUCT && L.norm.kind ? &L.norm : nullptr;
        L.res_in = L.res_out = cur;
        if ((norm && norm_stores(*norm)) || (L.kind == L_JOIN && L.join.changes())) { L.res_out = 1 - cur; cur = 1 - cur; }
    }
    plan->final_res = cur;
    return SWLM_OK;
}

// ---- pages -----------------------------------------------------------------------------------------------------------
int stream_reserve(swlm_state* s, int seq, int tokens, bool shrink) {
    if (tokens > s->plan->desc.max_seq) { set_error("sequence %d: %d tokens exceed max_seq %d", seq, tokens, s->plan->desc.max_seq); return SWLM_ERR_STATE; }
    std::vector<int>& have = s->seq_pages[seq];
    const size_t need = (size_t)(tokens + SWLM_PAGE_TOKENS - 1) / SWLM_PAGE_TOKENS;
    if (need > have.size() + s->free_pages.size()) {
        set_error("sequence %d needs %zu pages, %zu held and %zu free", seq, need, have.size(), s->free_pages.size());
        return SWLM_ERR_STATE;
    }
    while (have.size() < need) {
        s->page_table_host[(size_t)seq * s->pages_per_seq + have.size()] = s->free_pages.back();
        have.push_back(s->free_pages.back());
        s->free_pages.pop_back();
        s->page_table_dirty = true;
    }
    while (shrink && have.size() > need) {
        s->free_pages.push_back(have.back());
        have.pop_back();
    }
    return SWLM_OK;
}

void stream_release_all(swlm_state* s) {
    for (std::vector<int>& pages : s->seq_pages) pages.clear();
    s->free_pages.clear();
    for (int p = s->pool_pages - 1; p >= 0; --p) s->free_pages.push_back(p);   // page 0 is handed out first
}

int stream_upload_pages(swlm_state* s) {
    if (!s->page_table_dirty || s->page_table_host.empty()) return SWLM_OK;
    SWLM_CUDA(cudaMemcpyAsync(s->page_table, s->page_table_host.data(), s->page_table_host.size() * 4, cudaMemcpyHostToDevice, s->stream));
    s->page_table_dirty = false;
    return SWLM_OK;
}

namespace {

template <typename T>
int grow(T** p, size_t* cap, size_t need, cudaStream_t stream) {
    if (need <= *cap) return SWLM_OK;
    SWLM_CUDA(cudaStreamSynchronize(stream));
    cudaFree(*p);
    *p = nullptr; *cap = 0;
    const int rc = dev_alloc(p, need);
    if (!rc) *cap = need;
    return rc;
}

int bufs_rows(swlm_state* s, StreamBufs* b, int rows, int wants) {
    const swlm_plan* plan = s->plan;
    int rc;
    if (rows > b->rows) {
        SWLM_CUDA(cudaStreamSynchronize(s->stream));
        for (int i = 0; i < SWLM_BUF_COUNT; ++i) {
            if (i == SWLM_BUF_LOGITS) continue;
            cudaFree(b->buf[i]);
            b->buf[i] = nullptr;
            const size_t bytes = (size_t)rows * s->width[i] * stored_bytes(plan, i);
            unsigned char* p = nullptr;
            if ((rc = dev_alloc(&p, bytes))) return rc;
            b->buf[i] = p;
            if (bytes) SWLM_CUDA(cudaMemsetAsync(p, 0, bytes, s->stream));
        }
        cudaFree(b->res2);
        if ((rc = dev_alloc(&b->res2, (size_t)rows * s->width[SWLM_BUF_RESIDUAL]))) return rc;
        SWLM_CUDA(cudaMemsetAsync(b->res2, 0, (size_t)rows * s->width[SWLM_BUF_RESIDUAL] * 4, s->stream));
        cudaFree(b->results);
        const size_t results = (size_t)std::max(0, plan->desc.depth_results) * rows * s->width[SWLM_BUF_RESIDUAL];
        if ((rc = dev_alloc(&b->results, results))) return rc;
        if (results) SWLM_CUDA(cudaMemsetAsync(b->results, 0, results * 4, s->stream));
        b->rows = rows;
    }
    if (wants > b->wants) {
        SWLM_CUDA(cudaStreamSynchronize(s->stream));
        cudaFree(b->buf[SWLM_BUF_LOGITS]);
        cudaFree(b->argmax_out);
        b->buf[SWLM_BUF_LOGITS] = nullptr; b->argmax_out = nullptr; b->wants = 0;
        float* p = nullptr;
        if ((rc = dev_alloc(&p, (size_t)wants * s->width[SWLM_BUF_LOGITS]))) return rc;
        b->buf[SWLM_BUF_LOGITS] = p;
        if ((rc = dev_alloc(&b->argmax_out, wants))) return rc;
        b->wants = wants;
    }
    if (!b->argmax_val) {
        if ((rc = dev_alloc(&b->argmax_val, argmax_scratch_elems(kMaxSequences)))) return rc;
        if ((rc = dev_alloc(&b->argmax_idx, argmax_scratch_elems(kMaxSequences)))) return rc;
    }
    return SWLM_OK;
}

size_t part_need(const swlm_plan* plan, int rows, int wants) {
    size_t need = 0;
    if (plan->all_f32()) return 0;
    for (const Launch& L : plan->launches)
        if (L.kind == L_PRODUCT && L.x2_buf >= 0) for (const Matrix* m : {L.m1, &L.part[0], &L.part[1]}) need = std::max(need, product_part_floats(m->n, m->k, rows, false));
        else if (L.kind == L_PRODUCT) need = std::max(need, product_part_floats(L.m1->n, L.m1->k, L.seg_buf[0] == SWLM_BUF_LOGITS ? wants : rows, L.m2 != nullptr));
        else if (L.kind == L_ROUTED && L.m4) need = std::max(need, std::max(product_part_floats(L.m4->n, L.m4->k, rows, false), product_part_floats(L.m5->n, L.m5->k, rows, false)));
    return need;
}

// scratch of a batch; r.splits_pages bounds the splits
int bufs_scratch(swlm_state* s, StreamBufs* b, const RowBatch& r) {
    const swlm_plan* plan = s->plan;
    int rc;
    size_t part = part_need(plan, r.rows, r.wants), expand = 0;
    for (const Launch& L : plan->launches) {
        if (L.kind != L_LATENT || r.n_long == 0) continue;
        const LatentLayer& ll = plan->latent[L.st.layer];
        const int ctx = r.total_ctx[L.window_set];
        expand = std::max(expand, latent_expand_bytes(ll.row, L.st.heads, L.st.head_dim, L.st.value_dim, ctx));
        part = std::max(part, product_part_floats(L.st.heads * (L.st.head_dim + L.st.value_dim), ll.rank, ctx, false));
    }
    if ((rc = grow(&b->part, &b->part_cap, part, s->stream))) return rc;
    if ((rc = grow(&b->expand, &b->expand_cap, expand, s->stream))) return rc;
    size_t delta = 0, routed = 0;
    for (const Launch& L : plan->launches) {
        if (L.kind == L_DELTA) {
            const DeltaShape& sh = plan->delta[L.st.layer].shape;
            if (r.n_runs || (r.n_single && !delta_step_fits(sh))) delta = std::max(delta, delta_scratch_floats(sh, std::max(r.n_blocks, r.n_single), r.rows));
        } else if (L.kind == L_RETENTION) {
            if (r.n_runs || (r.n_single && !retention_step_fits(L.st.key_dim, L.st.value_dim))) delta = std::max(delta, (size_t)r.rows * L.st.heads * L.st.value_dim);
        } else if (L.kind == L_ROUTED) routed = std::max(routed, routed_scratch_bytes(routed_shape(L.st), r.rows, plan->all_f32()));
    }
    if ((rc = grow(&b->delta, &b->delta_cap, delta, s->stream))) return rc;
    if ((rc = grow(&b->routed, &b->routed_cap, routed, s->stream))) return rc;
    if ((rc = grow(&b->qcat, &b->qcat_cap, (size_t)r.n_short * plan->latent_q_floats, s->stream))) return rc;
    size_t partial = 0;
    for (const Launch& L : plan->launches)
        if (L.kind == L_LATENT)
            partial = std::max(partial, (size_t)r.n_short * latent_pick_splits(r.n_short, L.st.heads, r.splits_pages, L.st.window_left) * latent_partial_floats(plan->latent[L.st.layer].row, L.st.heads));
    return grow(&b->partial, &b->partial_cap, partial, s->stream);
}

void bufs_free(StreamBufs* b) {
    for (void* p : b->buf) cudaFree(p);
    cudaFree(b->res2); cudaFree(b->results); cudaFree(b->meta); cudaFree(b->argmax_out); cudaFree(b->qcat); cudaFree(b->partial); cudaFree(b->part);
    cudaFree(b->expand); cudaFree(b->delta); cudaFree(b->routed); cudaFree(b->argmax_val); cudaFree(b->argmax_idx);
    *b = StreamBufs{};
}

TokenInput token_input(const Launch* L) {
    TokenInput t;
    t.n = L[1].st.n;
    t.gate = L[1].m1->data; t.gate_ld = L[1].m1->ld; t.proj = L[3].m1->data; t.proj_ld = L[3].m1->ld;
    t.table = L[2].d1->data; t.cols = (int)L[2].d1->cols; t.col = L[2].st.in2_off;
    return t;
}

float* residual(StreamBufs* b, int phys) { return phys ? b->res2 : static_cast<float*>(b->buf[SWLM_BUF_RESIDUAL]); }

StreamNorm norm_of(swlm_state* s, StreamBufs* b, const RowBatch& r, const Launch& L, const swlm_step& st, const DenseTensor* w, int res_in, int res_out) {
    const DenseTensor* post = L.norm_post;
    StreamNorm n;
    n.mode = st.kind;
    n.in = st.in_buf == SWLM_BUF_RESIDUAL ? residual(b, res_in) : static_cast<const float*>(b->buf[st.in_buf]); n.in_stride = s->width[st.in_buf];
    n.res_stride = s->width[SWLM_BUF_RESIDUAL];
    if (st.kind != SWLM_STEP_COPY_RMSNORM) n.res_in = residual(b, res_in);
    if (norm_stores(st)) n.res_out = residual(b, res_out);
    n.w = w->data; n.w_post = post ? post->data : nullptr;
    n.eps = st.eps; n.weight_bias = st.weight_bias;
    if (is_postnorm(st.kind) && L.dv[0]) { n.table = L.dv[0]->data; n.tokens = r.tok; n.vocab = s->plan->desc.vocab; n.table_scale = st.scale; }
    return n;
}

// The plan's launches over one batch of rows. only_kind >= 0: those launches alone (timing hook; L_ATTN stands for the
// attention kernel of the latent steps).
int enqueue_rows_stream(swlm_state* s, StreamBufs* b, const RowBatch& r, bool body_only, cudaStream_t stream, int only_kind = -1) {
    const swlm_plan* plan = s->plan;
    const swlm_buffers_desc& d = plan->desc;
    const bool f32 = plan->all_f32();
    const int wants = body_only ? 0 : r.wants;
    bool advanced = false;
    int rc = SWLM_OK;
    auto column = [plan](StreamBufs* bufs, int buf, int off) -> void* { return static_cast<unsigned char*>(bufs->buf[buf]) + (size_t)off * stored_bytes(plan, buf); };
    s->last_bufs = b;
    s->last_res = plan->final_res;
    auto join_of = [&](const Launch& L) {
        const JoinParts& j = L.join;
        JoinLaunch a;
        a.rows = r.rows; a.width = d.hidden; a.f32 = f32; a.singles = r.n_runs == 0;
        a.row_seq = r.seq; a.row_pos = r.pos; a.tokens = r.tok; a.vocab = d.vocab;
        a.res_stride = s->width[SWLM_BUF_RESIDUAL];
        if (j.table) { a.table = j.table->data; a.table_scale = j.table_scale; }
        else a.res_in = residual(b, L.res_in);
        if (j.changes()) a.res_out = residual(b, L.res_out);
        if (j.keep >= 0) { a.keep_ring = s->conv_state[j.keep]; a.keep_taps = plan->convs[j.keep].taps; }
        if (j.adds) { a.in = static_cast<const float*>(b->buf[j.in_buf]); a.in_stride = s->width[j.in_buf]; a.w = j.w->data; a.eps = j.eps; a.weight_bias = j.weight_bias; }
        if (j.adds && j.gate_buf >= 0) { a.gate = static_cast<const float*>(b->buf[j.gate_buf]); a.gate_stride = s->width[j.gate_buf]; }
        a.results = b->results; a.result_step = (size_t)b->rows * a.res_stride; a.store = j.store;
        if (j.avg) { a.avg_w = j.avg_w->data; a.avg = j.avg; }
        if (j.conv >= 0) { a.conv_w = j.conv_w->data; a.conv_ring = s->conv_state[j.conv]; a.taps = plan->convs[j.conv].taps; a.conv_out = b->buf[j.conv_buf]; a.conv_stride = s->width[j.conv_buf]; }
        if (j.copy_buf >= 0) { a.copy_out = b->buf[j.copy_buf]; a.copy_stride = s->width[j.copy_buf]; }
        return a;
    };
    for (size_t li = 0; li < plan->launches.size(); ++li) {
        const Launch& L = plan->launches[li];
        const swlm_step& st = L.st;
        if (L.fused && r.n_runs == 0) {
            TokenInput t = token_input(&L);
            t.status = s->pf_status;
            if (token_input_fits(t, r.rows, d.hidden)) {
                li += L.fused;
                if (only_kind >= 0 && only_kind != L_JOIN) continue;
                if ((rc = launch_token_input(join_of(L), t, join_of(plan->launches[li]), stream))) return rc;
                s->launches += 1;
                continue;
            }
        }
        const bool latent_kernel = only_kind == L_ATTN && (L.kind == L_LATENT || L.kind == L_GROUPED);
        if (only_kind >= 0 && L.kind != only_kind && !latent_kernel) continue;
        switch (L.kind) {
        case L_EMBED:
            rc = launch_stream_embed(r.rows, st.n, r.tok, d.vocab, L.d1->data, st.scale != 0.f ? st.scale : 1.f, static_cast<float*>(b->buf[st.out_buf]), s->width[st.out_buf], stream);
            s->launches += 1;
            break;
        case L_RMSNORM:
            rc = launch_stream_norm(norm_of(s, b, r, L, st, L.d1, L.res_in, L.res_out), r.rows, st.n, nullptr, b->buf[st.out_buf], s->width[st.out_buf], f32, stream);
            s->launches += 1;
            break;
        case L_PRODUCT: {
            const bool head = L.seg_buf[0] == SWLM_BUF_LOGITS;
            const int m = head ? wants : r.rows;
            if (m == 0) break;
            const int32_t* idx = head ? r.wants_idx : nullptr;
            ProductLaunch a;
            a.w = L.m1; a.w2 = L.m2; a.act = L.act; a.m = m; a.x_f32 = f32;
            a.x = static_cast<unsigned char*>(b->buf[st.in_buf]) + (size_t)st.in_off * stored_bytes(plan, st.in_buf); a.x_stride = s->width[st.in_buf];
            a.part = b->part; a.part_floats = b->part_cap; a.status = s->pf_status;
            if (head && idx && !L.norm.kind) { set_error("the output head must follow a norm that nothing else reads"); return SWLM_ERR_UNSUPPORTED; }
            if (L.norm.kind) {
                const StreamNorm n = norm_of(s, b, r, L, L.norm, L.norm_w, L.res_in, L.res_out);
                if (!idx && product_takes_norm(m, L.m1->k)) a.norm = n;
                else {
                    rc = launch_stream_norm(n, m, L.norm.n, idx, b->buf[st.in_buf], s->width[st.in_buf], f32, stream);
                    s->launches += 1;
                    if (rc) return rc;
                }
            }
            a.out.softcap = L.softcap;
            a.out.biased = plan->biased;   // (one form of the kernel for all products of the plan: the fewer instructions, the sooner they are fetched)
            auto segment = [&](int q, int buf, int off, int end) {
                a.out.bias[q] = L.seg_bias[q] ? L.seg_bias[q]->data : nullptr;
                a.out.y[q] = static_cast<unsigned char*>(b->buf[buf]) + (size_t)off * stored_bytes(plan, buf); a.out.stride[q] = s->width[buf]; a.out.f32[q] = stored_f32(plan, buf) ? 1 : 0; a.out.end[q] = end;
            };
            if (L.m2 && !product_takes_gate(m, L.m1->k, f32)) {
                // gate and up one after the other, then the activation
                for (int h = 0; h < 2 && !rc; ++h) {
                    ProductLaunch c = a;
                    c.w = h ? L.m2 : L.m1; c.w2 = nullptr;
                    c.out.count = 1;
                    const int buf = L.seg_buf[1 + h];
                    c.out.y[0] = b->buf[buf]; c.out.stride[0] = s->width[buf]; c.out.f32[0] = stored_f32(plan, buf) ? 1 : 0; c.out.end[0] = c.w->n;
                    rc = launch_product(c, stream);
                    s->launches += product_launch_count(c);
                }
                if (!rc) rc = launch_stream_gated(m, L.m1->n, b->buf[L.seg_buf[1]], s->width[L.seg_buf[1]], b->buf[L.seg_buf[2]], s->width[L.seg_buf[2]],
                                                  b->buf[L.seg_buf[0]], s->width[L.seg_buf[0]], f32, L.act, stream);
                s->launches += 1;
                break;
            }
            a.out.count = L.n_seg;
            for (int q = 0; q < L.n_seg; ++q) segment(q, L.seg_buf[q], L.seg_off[q], L.seg_end[q]);
            for (int q = L.n_seg; q < kMaxProductSegs; ++q) a.out.end[q] = L.seg_end[L.n_seg - 1];
            if (L.x2_buf >= 0) {
                a.x2 = b->buf[L.x2_buf]; a.x2_stride = s->width[L.x2_buf]; a.split = L.part[0].n;
                if (!product_takes_two(m, L.m1->k, a.split, f32)) {   // one input after the other
                    for (int h = 0; h < 2 && !rc; ++h) {
                        ProductLaunch c = a;
                        c.w = &L.part[h]; c.x2 = nullptr;
                        if (h) { c.x = a.x2; c.x_stride = a.x2_stride; }
                        const int q0 = h ? L.first_segs : 0, q1 = h ? L.n_seg : L.first_segs;
                        c.out.count = q1 - q0;
                        for (int q = 0; q < kMaxProductSegs; ++q) {
                            const int from = std::min(q0 + q, q1 - 1);
                            c.out.y[q] = a.out.y[from]; c.out.stride[q] = a.out.stride[from]; c.out.f32[q] = a.out.f32[from]; c.out.bias[q] = a.out.bias[from];
                            c.out.end[q] = a.out.end[from] - (h ? a.split : 0);
                        }
                        rc = launch_product(c, stream);
                        s->launches += product_launch_count(c);
                    }
                    break;
                }
            }
            rc = launch_product(a, stream);
            s->launches += product_launch_count(a);
            break;
        }
        case L_SWIGLU:
            rc = launch_stream_gated(r.rows, st.n, b->buf[st.in_buf], s->width[st.in_buf], b->buf[st.in2_buf], s->width[st.in2_buf], b->buf[st.out_buf],
                                     s->width[st.out_buf], f32, L.act, stream);
            s->launches += 1;
            break;
        case L_SOFTCAP:
            rc = launch_stream_softcap(wants, st.n, static_cast<float*>(b->buf[SWLM_BUF_LOGITS]), s->width[SWLM_BUF_LOGITS], st.scale, stream);
            s->launches += wants > 0 ? 1 : 0;
            break;
        case L_DELTA: {
            DeltaLaunch a;
            a.shape = plan->delta[st.layer].shape;
            a.decay_dim = st.k; a.gate_act = st.gate_act; a.eps = st.eps; a.unit_eps = st.eps2; a.q_scale = st.scale; a.f32 = f32;
            a.qkv = b->buf[st.in_buf]; a.qkv_stride = s->width[st.in_buf];
            a.beta = static_cast<const float*>(column(b, st.in2_buf, st.in2_off)); a.beta_stride = s->width[st.in2_buf];
            a.decay = static_cast<const float*>(column(b, st.in3_buf, st.in3_off)); a.decay_stride = s->width[st.in3_buf];
            a.gate = column(b, st.in4_buf, st.in4_off); a.gate_stride = s->width[st.in4_buf];
            a.conv_q = L.dv[0]->data; a.conv_k = L.dv[1]->data; a.conv_v = L.dv[2]->data; a.norm_w = L.dv[3]->data; a.a_log = L.dv[4]->data; a.dt_bias = L.dv[5]->data;
            a.ring = s->delta_ring[st.layer]; a.state = s->delta_state[st.layer];
            a.row_seq = r.seq; a.row_pos = r.pos;
            a.out = b->buf[st.out_buf]; a.out_stride = s->width[st.out_buf];
            a.n_single = r.n_single; a.single_rows = r.single_rows; a.n_runs = r.n_runs; a.runs = r.runs; a.n_blocks = r.n_blocks; a.block_run = r.block_run;
            a.scratch = b->delta; a.status = s->pf_status;
            int n = 0;
            rc = launch_delta(a, stream, &n);
            s->launches += n;
            break;
        }
        case L_ROUTED: {
            RoutedLaunch a;
            a.shape = routed_shape(st); a.scale = st.scale; a.act = L.act; a.m = r.rows; a.f32 = f32;
            a.x = b->buf[st.in_buf]; a.x_stride = s->width[st.in_buf];
            a.z = static_cast<const float*>(b->buf[st.in2_buf]); a.z_stride = s->width[st.in2_buf];
            a.gate = L.m1; a.up = L.m2; a.down = L.m3; a.shared_up = L.m4; a.shared_down = L.m5;
            a.softmax = st.score_act == SWLM_SCORE_SOFTMAX; a.group_best = st.group_best == 1 ? 1 : 2; a.raw_weights = st.raw_weights;
            a.part = b->part; a.part_floats = b->part_cap; a.correction = L.dv[0] ? L.dv[0]->data : nullptr;
            a.out = static_cast<float*>(b->buf[st.out_buf]); a.out_stride = s->width[st.out_buf];
            a.scratch = b->routed; a.counts = s->routed_counts; a.status = s->pf_status;
            int n = 0;
            rc = launch_routed(a, stream, &n);
            s->launches += n;
            break;
        }
        case L_GROUPED: {
            GroupedLaunch a;
            const RopeTable& rope = plan->rope_tables[L.rope_table];
            a.row = plan->grouped[st.layer].row;
            a.heads = st.heads; a.rot_dims = st.rope_dim; a.rot_neighbours = st.rope_pairs == SWLM_ROPE_NEIGHBOURS; a.window = st.window_left; a.chunk = st.chunk; a.sink_one = st.sink_one;
            a.scale = st.scale; a.eps = st.eps; a.weight_bias = st.weight_bias; a.magnitude = rope.magnitude; a.inv_freq = rope.inv_freq; a.out_scale = st.out_scale; a.f32 = f32;
            a.head_norm = st.head_norm; a.temp_every = st.temp_every; a.temp_coef = st.temp_coef;
            if (st.in4_buf != SWLM_BUF_NONE) { a.entry_gate = column(b, st.in4_buf, st.in4_off); a.entry_gate_stride = s->width[st.in4_buf]; }
            a.q_norm = L.dv[0] ? L.dv[0]->data : nullptr; a.k_norm = L.dv[1] ? L.dv[1]->data : nullptr;
            a.qkv = column(b, st.in_buf, st.in_off); a.qkv_stride = s->width[st.in_buf];
            if (st.in3_buf != SWLM_BUF_NONE) { a.gate = static_cast<const float*>(b->buf[st.in3_buf]); a.gate_stride = s->width[st.in3_buf]; }
            a.pool = s->pool[plan->latent.size() + st.layer]; a.page_table = s->page_table; a.pages_per_seq = s->pages_per_seq;
            a.row_seq = r.seq; a.row_pos = r.pos;
            a.out = column(b, st.out_buf, st.out_off); a.out_stride = s->width[st.out_buf];
            a.n_rows = r.rows; a.n_short = r.n_short; a.short_rows = r.short_rows; a.max_pages = r.splits_pages;
            a.n_tiles = r.n_tiles; a.tiles = r.tiles; a.status = s->pf_status; a.only_attention = latent_kernel; a.singles = r.n_runs == 0;
            if (r.n_spans) a.spans = r.spans[L.window_set];
            int n = 0;
            rc = launch_grouped(a, stream, &n);
            s->launches += n;
            break;
        }
        case L_RETENTION: {
            RetentionLaunch a;
            a.heads = st.heads; a.dim = st.key_dim; a.vdim = st.value_dim; a.eps = st.eps; a.scale = st.scale; a.out_scale = st.out_scale; a.f32 = f32;
            a.decay = L.f1->data;
            a.qkv = column(b, st.in_buf, st.in_off); a.qkv_stride = s->width[st.in_buf];
            a.gate = column(b, st.in4_buf, st.in4_off); a.gate_stride = s->width[st.in4_buf];
            a.state = s->delta_state[st.layer]; a.row_seq = r.seq; a.row_pos = r.pos;
            a.out = column(b, st.out_buf, st.out_off); a.out_stride = s->width[st.out_buf];
            a.n_single = r.n_single; a.single_rows = r.single_rows; a.n_runs = r.n_runs; a.runs = r.runs; a.n_blocks = r.n_blocks; a.block_run = r.block_run;
            a.scratch = b->delta;
            int n = 0;
            rc = launch_retention(a, stream, &n);
            s->launches += n;
            break;
        }
        case L_LATENT: {
            LatentLaunch a;
            const RopeTable& rope = plan->rope_tables[L.rope_table];
            a.row = plan->latent[st.layer].row;
            a.heads = st.heads; a.dim = st.head_dim; a.vdim = st.value_dim; a.rot_dims = st.rope_dim; a.rot_neighbours = st.rope_pairs == SWLM_ROPE_NEIGHBOURS;
            a.scale = st.scale; a.eps = st.eps; a.weight_bias = st.weight_bias; a.magnitude = rope.magnitude; a.inv_freq = rope.inv_freq; a.f32 = f32;
            a.window = st.window_left; a.sink = L.dv[0] ? L.dv[0]->data : nullptr;
            a.q = b->buf[st.in_buf]; a.q_stride = s->width[st.in_buf];
            a.kv = static_cast<const float*>(b->buf[st.in2_buf]); a.kv_stride = s->width[st.in2_buf];
            if (st.in3_buf != SWLM_BUF_NONE) { a.gate = static_cast<const float*>(b->buf[st.in3_buf]); a.gate_stride = s->width[st.in3_buf]; }
            a.norm_w = L.d1->data; a.uk = L.m1; a.uv = L.m2;
            a.ukv = &plan->ctx->matrix_cat.at(std::string(st.weight2) + "|" + st.weight3);
            a.pool = s->pool[st.layer]; a.page_table = s->page_table; a.pages_per_seq = s->pages_per_seq;
            a.row_seq = r.seq; a.row_pos = r.pos;
            a.out = b->buf[st.out_buf]; a.out_stride = s->width[st.out_buf];
            a.n_short = r.n_short; a.short_rows = r.short_rows; a.splits = latent_pick_splits(r.n_short, st.heads, r.splits_pages, st.window_left);
            a.qcat = b->qcat; a.partial = b->partial;
            a.n_long = r.n_long; a.long_rows = r.long_rows; a.n_spans = r.n_spans; a.n_tiles = r.n_tiles; a.tiles = r.tiles;
            if (r.n_spans) { a.spans = r.spans[L.window_set]; a.total_ctx = r.total_ctx[L.window_set]; }
            a.expand = b->expand; a.part = b->part; a.part_floats = b->part_cap; a.status = s->pf_status;
            a.only_attention = latent_kernel;
            int n = 0;
            rc = launch_latent(a, stream, &n);
            s->launches += n;
            break;
        }
        case L_JOIN: {
            int n = 0;
            rc = launch_join(join_of(L), stream, &n);
            s->launches += n;
            break;
        }
        case L_TOKEN_GATE:
            rc = launch_token_gate(r.rows, st.n, b->buf[st.in_buf], s->width[st.in_buf], r.tok, d.vocab, L.d1->data, (int)L.d1->cols, st.in2_off, b->buf[st.out_buf], s->width[st.out_buf], f32, stream);
            s->launches += 1;
            break;
        case L_ARGMAX:
            if (wants == 0) break;
            if (r.advance) {
                rc = launch_argmax_f32(wants, st.n, static_cast<const float*>(b->buf[SWLM_BUF_LOGITS]), s->width[SWLM_BUF_LOGITS], s->token_out, s->token_in, s->ring,
                                       s->step_counter, s->ring_cap, s->position, 1, b->argmax_val, b->argmax_idx, stream);
                advanced = true;
            } else {
                rc = launch_argmax_f32(wants, st.n, static_cast<const float*>(b->buf[SWLM_BUF_LOGITS]), s->width[SWLM_BUF_LOGITS], b->argmax_out, nullptr, nullptr,
                                       s->step_counter, s->ring_cap, s->position, 0, b->argmax_val, b->argmax_idx, stream);
            }
            s->launches += 2 * ((wants + kMaxSequences - 1) / kMaxSequences);
            break;
        }
        if (rc) return rc;
    }
    if (r.advance && !advanced && only_kind < 0) {
        rc = launch_advance(r.rows, s->position, nullptr, stream);
        s->launches += 1;
    }
    return rc;
}

RowBatch identity_batch(const swlm_state* s) {
    RowBatch r;
    r.rows = r.wants = r.n_short = r.n_single = s->plan->desc.max_batch;
    r.tok = s->token_in; r.seq = s->seq_identity; r.pos = s->position;
    r.splits_pages = s->pages_per_seq;
    r.advance = true;
    return r;
}

// scratch of every decode step a graph may hold: 1 .. max_batch rows
int decode_scratch(swlm_state* s) {
    for (int n = 1; n <= s->plan->desc.max_batch; ++n) {
        RowBatch r;
        r.rows = r.wants = r.n_short = r.n_single = n;
        r.splits_pages = s->pages_per_seq;
        const int rc = bufs_scratch(s, &s->dec, r);
        if (rc) return rc;
    }
    return SWLM_OK;
}

}  // namespace

// ---- state -----------------------------------------------------------------------------------------------------------
int stream_state_create(swlm_state* s) {
    const swlm_plan* plan = s->plan;
    const swlm_buffers_desc& d = plan->desc;
    int rc;
    for (int i = 0; i < SWLM_BUF_COUNT; ++i) s->width[i] = plan->stream_width[i];
    s->pages_per_seq = (d.max_seq + SWLM_PAGE_TOKENS - 1) / SWLM_PAGE_TOKENS;
    s->pool_pages = d.kv_pool_tokens > 0 ? (d.kv_pool_tokens + SWLM_PAGE_TOKENS - 1) / SWLM_PAGE_TOKENS : s->pages_per_seq * d.max_batch;
    const size_t elem = plan->all_f32() ? 4 : 2;
    for (const LatentLayer& l : plan->latent) {
        const size_t bytes = (size_t)s->pool_pages * SWLM_PAGE_TOKENS * l.row.pitch * elem;
        unsigned char* p = nullptr;
        if ((rc = dev_alloc(&p, bytes))) return rc;
        s->pool.push_back(p);
        s->pool_bytes.push_back(bytes);
        // a page is read whole: rows nobody has written must hold finite numbers
        if (bytes) SWLM_CUDA(cudaMemset(p, 0, bytes));
    }
    for (const GroupedLayer& l : plan->grouped) {
        const size_t bytes = (size_t)s->pool_pages * l.row.groups * l.row.block * elem;
        unsigned char* p = nullptr;
        if ((rc = dev_alloc(&p, bytes))) return rc;
        s->pool.push_back(p);
        s->pool_bytes.push_back(bytes);
        if (bytes) SWLM_CUDA(cudaMemset(p, 0, bytes));
    }
    for (const DeltaLayer& l : plan->delta) {
        float* st = nullptr;
        unsigned char* ring = nullptr;
        const size_t bytes = (size_t)d.max_batch * l.ring_elems() * elem;
        if ((rc = dev_alloc(&st, (size_t)d.max_batch * l.state_elems()))) return rc;
        s->delta_state.push_back(st);
        if ((rc = dev_alloc(&ring, bytes))) return rc;
        s->delta_ring.push_back(ring);
        // (a sequence at position 0 starts from zeros whatever its slot holds; this is for positions that are set)
        if (bytes) SWLM_CUDA(cudaMemset(ring, 0, bytes));
        if (st) SWLM_CUDA(cudaMemset(st, 0, (size_t)d.max_batch * l.state_elems() * 4));
    }
    for (const StreamConv& c : plan->convs) {   // (as above: a sequence at position 0 starts from zeros)
        const size_t count = (size_t)d.max_batch * std::max(0, c.taps - 1) * d.hidden;
        float* p = nullptr;
        if ((rc = dev_alloc(&p, count))) return rc;
        s->conv_state.push_back(p);
        if (count) SWLM_CUDA(cudaMemset(p, 0, count * 4));
    }
    if ((rc = dev_alloc(&s->routed_counts, kMaxExperts))) return rc;
    SWLM_CUDA(cudaMemset(s->routed_counts, 0, kMaxExperts * 4));
    s->seq_pages.assign(d.max_batch, {});
    s->page_table_host.assign((size_t)d.max_batch * s->pages_per_seq, 0);
    if ((rc = dev_alloc(&s->page_table, s->page_table_host.size()))) return rc;
    s->page_table_dirty = true;
    stream_release_all(s);
    if ((rc = dev_alloc(&s->seq_identity, d.max_batch))) return rc;
    std::vector<int32_t> ident(d.max_batch);
    for (int i = 0; i < d.max_batch; ++i) ident[i] = i;
    SWLM_CUDA(cudaMemcpy(s->seq_identity, ident.data(), ident.size() * 4, cudaMemcpyHostToDevice));
    if (!s->pf_status) {
        if ((rc = dev_alloc(&s->pf_status, 1))) return rc;
        SWLM_CUDA(cudaMemset(s->pf_status, 0, sizeof(int)));
    }
    if ((rc = bufs_rows(s, &s->dec, d.max_batch, d.max_batch))) return rc;
    if ((rc = grow(&s->dec.meta, &s->dec.meta_cap, (size_t)3 * d.max_batch, s->stream))) return rc;
    s->last_bufs = &s->dec;
    return decode_scratch(s);
}

void stream_drop_graphs(swlm_state* s) {
    for (auto& g : s->row_graphs) cudaGraphExecDestroy(g.second);
    s->row_graphs.clear();
    s->row_graph_launches.clear();
}

void stream_state_free(swlm_state* s) {
    stream_drop_graphs(s);
    for (void* p : s->pool) cudaFree(p);
    for (float* p : s->delta_state) cudaFree(p);
    for (void* p : s->delta_ring) cudaFree(p);
    for (float* p : s->conv_state) cudaFree(p);
    cudaFree(s->routed_counts);
    cudaFree(s->page_table);
    cudaFree(s->seq_identity);
    bufs_free(&s->dec);
    bufs_free(&s->big);
    if (s->h_rows) cudaFreeHost(s->h_rows);
}

int stream_enqueue_step(swlm_state* s, bool body_only, cudaStream_t stream, int only_kind) {
    return enqueue_rows_stream(s, &s->dec, identity_batch(s), body_only, stream, only_kind);
}

int stream_launches_per_step(const swlm_plan* plan) {
    const int m = plan->desc.max_batch;
    int n = 0;
    for (size_t li = 0; li < plan->launches.size(); ++li) {
        const Launch& L = plan->launches[li];
        if (L.fused && token_input_fits(token_input(&L), m, plan->desc.hidden)) { n += 1; li += L.fused; continue; }
        if (L.kind == L_PRODUCT) {
            ProductLaunch a;
            a.w = L.m1; a.w2 = L.m2; a.m = m; a.x_f32 = plan->all_f32();
            const bool fused = L.norm.kind && product_takes_norm(m, L.m1->k);
            if (fused) a.norm.mode = L.norm.kind;
            else if (L.norm.kind) n += 1;
            if (L.m2 && !product_takes_gate(m, L.m1->k, a.x_f32)) { a.w2 = nullptr; n += 2 * product_launch_count(a) + 1; }
            else if (L.x2_buf >= 0 && !product_takes_two(m, L.m1->k, L.part[0].n, plan->all_f32()))
                for (const Matrix& part : L.part) { a.w = &part; n += product_launch_count(a); }
            else n += product_launch_count(a);
        } else if (L.kind == L_DELTA) n += delta_step_fits(plan->delta[L.st.layer].shape) ? 1 : 3;
        else if (L.kind == L_RETENTION) n += retention_step_fits(L.st.key_dim, L.st.value_dim) ? 1 : 2;
        else if (L.kind == L_GROUPED) n += grouped_appends(plan->grouped[L.st.layer].row, plan->all_f32(), L.st.rope_dim) ? 1 : 2;
        else if (L.kind == L_ROUTED) {
            n += m <= 4 || plan->all_f32() ? 2 : 5;
            if (L.m4 && m > 4 && !plan->all_f32())
                for (const Matrix* w : {L.m4, L.m5}) { ProductLaunch a; a.w = w; a.m = m; n += product_launch_count(a); }
        }
        else n += L.kind == L_LATENT ? 3 : L.kind == L_ARGMAX ? 2 : 1;
    }
    return n;
}

int stream_check_status(swlm_state* s) {
    int st = 0;
    SWLM_CUDA(cudaMemcpy(&st, s->pf_status, sizeof(int), cudaMemcpyDeviceToHost));
    if (!st) return SWLM_OK;
    SWLM_CUDA(cudaMemset(s->pf_status, 0, sizeof(int)));
    set_error("a bounded wait in a kernel expired (code %d)", st);
    return SWLM_ERR_TIMEOUT;
}

// ---- batches ---------------------------------------------------------------------------------------------------------
namespace {

struct Piece { int seq, pos0, count; const int32_t* tokens; };

int stage(swlm_state* s, StreamBufs* b, const std::vector<int32_t>& meta) {
    int rc;
    // (`dec` never grows: its capacity covers 3 * max_batch words from the start)
    if ((rc = grow(&b->meta, &b->meta_cap, meta.size(), s->stream))) return rc;
    if (meta.size() > s->h_rows_cap) {
        SWLM_CUDA(cudaStreamSynchronize(s->stream));
        if (s->h_rows) cudaFreeHost(s->h_rows);
        s->h_rows = nullptr; s->h_rows_cap = 0;
        const size_t cap = std::max<size_t>(4096, meta.size());
        SWLM_CUDA(cudaMallocHost((void**)&s->h_rows, cap * 4));
        s->h_rows_cap = cap;
    }
    memcpy(s->h_rows, meta.data(), meta.size() * 4);   // callers synchronise before the next batch is staged
    SWLM_CUDA(cudaMemcpyAsync(b->meta, s->h_rows, meta.size() * 4, cudaMemcpyHostToDevice, s->stream));
    return SWLM_OK;
}

// spans of at least this many rows are attended over expanded keys and values
constexpr int kSpanMinRows = 64;
static_assert(sizeof(LatentSpan) == 24 && sizeof(RowRun) == 20, "spans are staged as six words, runs as five");

// Rows of `pieces` in one pass; `want_rows` get logits and tokens in b->buf[LOGITS] / b->argmax_out.
int run_rows(swlm_state* s, const std::vector<Piece>& pieces, const std::vector<int32_t>& want_rows, StreamBufs** used, int only_kind = -1, int repeats = 1) {
    const swlm_plan* plan = s->plan;
    int rows = 0;
    bool single = true;
    for (const Piece& p : pieces) { rows += p.count; single &= p.count == 1; }
    bool every = (int)want_rows.size() == rows;
    for (int i = 0; i < (int)want_rows.size() && every; ++i) every = want_rows[i] == i;
    const bool graph = single && every && rows <= plan->desc.max_batch && only_kind < 0;
    StreamBufs* b = graph ? &s->dec : &s->big;
    *used = b;
    int rc;
    if ((rc = stream_upload_pages(s))) return rc;
    std::vector<int32_t> meta((size_t)3 * rows);
    int at = 0, longest = 0;
    for (const Piece& p : pieces) {
        longest = std::max(longest, p.pos0 + p.count);
        for (int i = 0; i < p.count; ++i, ++at) { meta[at] = p.tokens[i]; meta[rows + at] = p.seq; meta[2 * rows + at] = p.pos0 + i; }
    }
    RowBatch r;
    r.rows = rows;
    r.wants = (int)want_rows.size();
    if (graph) {
        if ((rc = stage(s, b, meta))) return rc;
        r.tok = b->meta; r.seq = b->meta + rows; r.pos = b->meta + 2 * rows;
        r.n_short = r.n_single = rows; r.splits_pages = s->pages_per_seq;
        auto it = s->row_graphs.find(rows);
        if (it == s->row_graphs.end()) {
            cudaGraph_t g = nullptr;
            const int64_t before = s->launches;
            SWLM_CUDA(cudaStreamBeginCapture(s->stream, cudaStreamCaptureModeThreadLocal));
            rc = enqueue_rows_stream(s, b, r, false, s->stream);
            cudaError_t e = cudaStreamEndCapture(s->stream, &g);
            const int n = (int)(s->launches - before);
            s->launches = before;   // capture does not execute
            if (rc) { if (g) cudaGraphDestroy(g); return rc; }
            if (e != cudaSuccess) return cuda_fail(e, "cudaStreamEndCapture");
            cudaGraphExec_t x = nullptr;
            e = cudaGraphInstantiate(&x, g, 0);
            cudaGraphDestroy(g);
            if (e != cudaSuccess) return cuda_fail(e, "cudaGraphInstantiate");
            it = s->row_graphs.emplace(rows, x).first;
            s->row_graph_launches[rows] = n;
        }
        SWLM_CUDA(cudaGraphLaunch(it->second, s->stream));
        s->launches += s->row_graph_launches[rows];
        s->last_bufs = b;
        return SWLM_OK;
    }

    // which pieces are attended in spans: every attention layer must allow it
    bool expands = true;
    for (const Launch& L : plan->launches)
        if (L.kind == L_LATENT) expands &= latent_expands(plan->latent[L.st.layer].row, L.st.head_dim, L.st.value_dim, plan->all_f32());
        else if (L.kind == L_GROUPED) expands &= grouped_spans(plan->grouped[L.st.layer].row, plan->all_f32());
    std::vector<int32_t> shorts, longs, singles, block_run;
    std::vector<LatentSpan> spans;
    std::vector<RowRun> runs;
    std::vector<std::pair<int, int2>> tiles;   // (context at the end of the tile, tile)
    int row0 = 0, short_longest = 0;
    for (const Piece& p : pieces) {
        if (expands && p.count >= kSpanMinRows) {
            const int sp = (int)spans.size();
            spans.push_back(LatentSpan{row0, p.count, p.pos0, p.seq, 0, 0});
            for (int i = 0; i < p.count; ++i) longs.push_back(row0 + i);
            for (int q = 0; q * kLatentQueryTile < p.count; ++q)
                tiles.push_back({p.pos0 + std::min(p.count, (q + 1) * kLatentQueryTile), int2{sp, q}});
        } else {
            for (int i = 0; i < p.count; ++i) shorts.push_back(row0 + i);
            short_longest = std::max(short_longest, p.pos0 + p.count);
        }
        if (p.count == 1) singles.push_back(row0);
        else {
            runs.push_back(RowRun{row0, p.count, p.pos0, p.seq, (int)block_run.size()});
            block_run.insert(block_run.end(), (p.count + kDeltaBlock - 1) / kDeltaBlock, (int)runs.size() - 1);
        }
        row0 += p.count;
    }
    std::stable_sort(tiles.begin(), tiles.end(), [](const std::pair<int, int2>& a, const std::pair<int, int2>& c) { return a.first > c.first; });   // the longest first
    const size_t o_want = meta.size();
    meta.insert(meta.end(), want_rows.begin(), want_rows.end());
    const size_t o_short = meta.size();
    meta.insert(meta.end(), shorts.begin(), shorts.end());
    const size_t o_long = meta.size();
    meta.insert(meta.end(), longs.begin(), longs.end());
    if (meta.size() & 1) meta.push_back(0);
    const size_t o_tiles = meta.size();
    for (const auto& tl : tiles) { meta.push_back(tl.second.x); meta.push_back(tl.second.y); }
    const size_t o_spans = meta.size();
    for (const int window : plan->windows) {
        int ctx = 0;
        for (const LatentSpan& sp : spans) {
            const int lo = window > 0 ? std::max(0, sp.pos0 - window + 1) / SWLM_PAGE_TOKENS * SWLM_PAGE_TOKENS : 0;
            const int32_t w[6] = {sp.row0, sp.count, sp.pos0, sp.seq, ctx, lo};
            meta.insert(meta.end(), w, w + 6);
            ctx += sp.pos0 + sp.count - lo;
        }
        r.total_ctx.push_back(ctx);
    }
    const size_t o_single = meta.size();
    meta.insert(meta.end(), singles.begin(), singles.end());
    const size_t o_runs = meta.size();
    for (const RowRun& run : runs) { const int32_t w[5] = {run.row0, run.count, run.pos0, run.seq, run.blk0}; meta.insert(meta.end(), w, w + 5); }
    const size_t o_blocks = meta.size();
    meta.insert(meta.end(), block_run.begin(), block_run.end());
    r.n_single = (int)singles.size();
    r.n_runs = (int)runs.size();
    r.n_blocks = (int)block_run.size();
    r.n_short = (int)shorts.size();
    r.n_long = (int)longs.size();
    r.n_spans = (int)spans.size();
    r.n_tiles = (int)tiles.size();
    r.splits_pages = std::max(1, (short_longest + SWLM_PAGE_TOKENS - 1) / SWLM_PAGE_TOKENS);
    if ((rc = bufs_rows(s, b, std::max(rows, r.wants), r.wants)) || (rc = bufs_scratch(s, b, r)) || (rc = stage(s, b, meta))) return rc;
    r.tok = b->meta; r.seq = b->meta + rows; r.pos = b->meta + 2 * rows;
    r.wants_idx = b->meta + o_want;
    r.short_rows = b->meta + o_short; r.long_rows = b->meta + o_long;
    r.tiles = reinterpret_cast<const int2*>(b->meta + o_tiles);
    for (size_t q = 0; q < plan->windows.size(); ++q) r.spans.push_back(reinterpret_cast<const LatentSpan*>(b->meta + o_spans + q * 6 * spans.size()));
    r.single_rows = b->meta + o_single;
    r.runs = reinterpret_cast<const RowRun*>(b->meta + o_runs);
    r.block_run = b->meta + o_blocks;
    for (int i = 0; i < repeats && !rc; ++i) rc = enqueue_rows_stream(s, b, r, false, s->stream, only_kind);
    return rc;
}

}  // namespace

int stream_profile(swlm_state* s, int seq, const int32_t* tokens, int n, int only_kind, int repeats) {
    const int rc = stream_reserve(s, seq, s->pos_host[seq] + n);
    if (rc) return rc;
    StreamBufs* b = nullptr;
    return run_rows(s, {Piece{seq, s->pos_host[seq], n, tokens}}, {}, &b, only_kind, repeats);
}

int stream_run(swlm_state* s, int n_entries, const int32_t* seqs, const int32_t* counts, const int32_t* tokens, const int32_t* want_counts,
               const int32_t* wants, float* logits_out, int32_t* tokens_out, int row_cap) {
    const swlm_buffers_desc& d = s->plan->desc;
    int rc;
    std::vector<char> seen(d.max_batch, 0);
    size_t n_tok = 0, n_want = 0, new_pages = 0;
    for (int e = 0; e < n_entries; ++e) {
        const int q = seqs[e];
        if (q < 0 || q >= d.max_batch || seen[q]) { set_error("entry %d: sequence %d outside 0..%d or named twice", e, q, d.max_batch - 1); return SWLM_ERR_INVALID; }
        seen[q] = 1;
        if (counts[e] <= 0 || (want_counts && want_counts[e] < 0)) { set_error("entry %d: no tokens", e); return SWLM_ERR_INVALID; }
        if (s->pos_host[q] + counts[e] > d.max_seq) { set_error("sequence %d: position %d + %d tokens exceeds max_seq %d", q, s->pos_host[q], counts[e], d.max_seq); return SWLM_ERR_STATE; }
        for (int i = 0; i < counts[e]; ++i)
            if (tokens[n_tok + i] < 0 || tokens[n_tok + i] >= d.vocab) { set_error("entry %d: token %d outside the vocabulary of %d", e, tokens[n_tok + i], d.vocab); return SWLM_ERR_INVALID; }
        for (int i = 0; want_counts && i < want_counts[e]; ++i)
            if (wants[n_want + i] < 0 || wants[n_want + i] >= counts[e]) { set_error("entry %d: place %d outside its %d tokens", e, wants[n_want + i], counts[e]); return SWLM_ERR_INVALID; }
        n_tok += counts[e];
        n_want += want_counts ? want_counts[e] : 0;
        const size_t need = (size_t)(s->pos_host[q] + counts[e] + SWLM_PAGE_TOKENS - 1) / SWLM_PAGE_TOKENS;
        new_pages += need > s->seq_pages[q].size() ? need - s->seq_pages[q].size() : 0;
    }
    if (new_pages > s->free_pages.size()) { set_error("the batch needs %zu more pages, %zu are free", new_pages, s->free_pages.size()); return SWLM_ERR_STATE; }
    for (int e = 0; e < n_entries; ++e)
        if ((rc = stream_reserve(s, seqs[e], s->pos_host[seqs[e]] + counts[e]))) return rc;

    const size_t vocab = d.vocab;
    std::vector<float> row_logits;
    std::vector<int32_t> row_tokens;
    int e = 0, off = 0;                 // next entry and how many of its tokens have run
    size_t tok0 = 0, want0 = 0;         // first token and first wanted place of entry e
    while (e < n_entries) {
        std::vector<Piece> pieces;
        std::vector<int32_t> want_rows;
        std::vector<size_t> slots;      // where a wanted row goes in the outputs
        int rows = 0;
        while (e < n_entries && rows < row_cap) {
            const int take = std::min(row_cap - rows, counts[e] - off);
            pieces.push_back(Piece{seqs[e], s->pos_host[seqs[e]] + off, take, tokens + tok0 + off});
            const int nw = want_counts ? want_counts[e] : 0;
            for (int i = 0; i < nw; ++i)
                if (wants[want0 + i] >= off && wants[want0 + i] < off + take) { want_rows.push_back(rows + wants[want0 + i] - off); slots.push_back(want0 + i); }
            rows += take;
            off += take;
            if (off == counts[e]) { tok0 += counts[e]; want0 += nw; off = 0; ++e; }
        }
        StreamBufs* b = nullptr;
        if ((rc = run_rows(s, pieces, want_rows, &b))) return rc;
        const size_t w = want_rows.size();
        if (w && logits_out) {
            const size_t pitch = (size_t)s->width[SWLM_BUF_LOGITS] * 4;
            bool straight = true;
            for (size_t i = 1; i < w; ++i) straight &= slots[i] == slots[i - 1] + 1;
            float* dst = logits_out + slots[0] * vocab;
            if (!straight) { row_logits.resize(w * vocab); dst = row_logits.data(); }
            SWLM_CUDA(cudaMemcpy2DAsync(dst, vocab * 4, b->buf[SWLM_BUF_LOGITS], pitch, vocab * 4, w, cudaMemcpyDeviceToHost, s->stream));
            SWLM_CUDA(cudaStreamSynchronize(s->stream));
            if (!straight) for (size_t i = 0; i < w; ++i) memcpy(logits_out + slots[i] * vocab, row_logits.data() + i * vocab, vocab * 4);
        }
        if (w && tokens_out) {
            row_tokens.resize(w);
            SWLM_CUDA(cudaMemcpyAsync(row_tokens.data(), b->argmax_out, w * 4, cudaMemcpyDeviceToHost, s->stream));
            SWLM_CUDA(cudaStreamSynchronize(s->stream));
            for (size_t i = 0; i < w; ++i) tokens_out[slots[i]] = row_tokens[i];
        }
        SWLM_CUDA(cudaStreamSynchronize(s->stream));
    }
    for (int q = 0; q < n_entries; ++q) s->pos_host[seqs[q]] += counts[q];
    SWLM_CUDA(cudaMemcpyAsync(s->position, s->pos_host.data(), sizeof(int32_t) * d.max_batch, cudaMemcpyHostToDevice, s->stream));
    SWLM_CUDA(cudaStreamSynchronize(s->stream));
    return stream_check_status(s);
}

int stream_run_step(swlm_state* s, const swlm_step* step, const int32_t* token_in, int32_t* token_out) {
    const int m = s->plan->desc.max_batch;
    swlm_plan tmp;
    tmp.ctx = s->plan->ctx;
    tmp.desc = s->plan->desc;
    tmp.steps.assign(step, step + 1);
    int rc = stream_compile(&tmp);
    auto done = [&](int code) { stream_plan_free(&tmp); return code; };
    if (rc) return done(rc);
    for (int i = 0; i < SWLM_BUF_COUNT; ++i)
        if (tmp.stream_width[i] > s->width[i]) { set_error("step: buffer %d is %d wide, the step needs %d", i, s->width[i], tmp.stream_width[i]); return done(SWLM_ERR_INVALID); }
    for (size_t l = 0; l < tmp.latent.size(); ++l)
        if (tmp.latent[l].rank && tmp.latent[l].row.pitch != s->plan->latent[l].row.pitch) { set_error("step: latent layer %zu has other rows", l); return done(SWLM_ERR_INVALID); }
    for (size_t l = 0; l < tmp.grouped.size(); ++l)
        if (tmp.grouped[l].row.groups && memcmp(&tmp.grouped[l].row, &s->plan->grouped[l].row, sizeof(GroupedRow))) { set_error("step: grouped layer %zu has other rows", l); return done(SWLM_ERR_INVALID); }
    for (size_t l = 0; l < tmp.convs.size(); ++l)
        if (tmp.convs[l].taps && tmp.convs[l].taps != s->plan->convs[l].taps) { set_error("step: convolution %zu has other taps", l); return done(SWLM_ERR_INVALID); }
    for (size_t l = 0; l < tmp.delta.size(); ++l)
        if (tmp.delta[l].shape.heads && memcmp(&tmp.delta[l].shape, &s->plan->delta[l].shape, sizeof(DeltaShape))) { set_error("step: gated-delta layer %zu has another shape", l); return done(SWLM_ERR_INVALID); }
    for (int b = 0; b < m; ++b)
        if ((rc = stream_reserve(s, b, s->pos_host[b] + 1))) return done(rc);
    if ((rc = stream_upload_pages(s))) return done(rc);
    if (token_in) SWLM_CUDA(cudaMemcpyAsync(s->token_in, token_in, sizeof(int32_t) * m, cudaMemcpyHostToDevice, s->stream));
    stream_drop_graphs(s);   // the step may need more scratch than the graphs were captured with
    if (s->graph_full) { cudaGraphExecDestroy(s->graph_full); s->graph_full = nullptr; }
    if (s->graph_body) { cudaGraphExecDestroy(s->graph_body); s->graph_body = nullptr; }
    swlm_plan* saved = s->plan;
    RowBatch r = identity_batch(s);
    r.advance = false;
    s->plan = &tmp;
    rc = bufs_scratch(s, &s->dec, r);
    if (!rc) rc = enqueue_rows_stream(s, &s->dec, r, false, s->stream);
    s->plan = saved;
    const cudaError_t e = cudaStreamSynchronize(s->stream);
    if (rc) return done(rc);
    if (e != cudaSuccess) return done(cuda_fail(e, "run_step sync"));
    if (token_out) SWLM_CUDA(cudaMemcpy(token_out, s->dec.argmax_out, sizeof(int32_t) * m, cudaMemcpyDeviceToHost));
    return done(stream_check_status(s));
}

void stream_plan_free(swlm_plan* plan) {
    for (RopeTable& t : plan->rope_tables) cudaFree(t.inv_freq);
    plan->rope_tables.clear();
}

}  // namespace swlm
