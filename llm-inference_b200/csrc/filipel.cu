// Model family "Filipel": a decoder of parallel layers, x <- x + m (mixer(N x) + ff(N x)), with ONE layer norm per layer (a
// weight, no bias) that both sublayers read and one residual multiplier m. Two kinds of mixer that config.json orders freely:
//   "latent_attention"  queries through a normed low-rank row; the cache holds one normed latent row per token plus one rotated
//                       key part shared by all heads, keys and values are up-projections of the latent; full causal softmax;
//                       element-wise sigmoid output gate. A layer with "kv_from": j has no cache of its own and reads layer j's
//                       rows with its own queries and up-projections.
//   "parallel"          two mixers beside each other. Left: grouped-query attention in a sliding window with a temperature per
//                       head, whose softmax weights are mixed across the heads (a learned matrix) before they meet the values;
//                       element-wise sigmoid output gate. Right: a state-space recurrence with one decay per head behind a
//                       short convolution, gated by silu(z) and then RMS-normed in equal parts. The mixer is half the sum of the
//                       two outputs, each RMS-normed over the model width with its own weight.
// Feed-forward: none, a dense one whose activation is a polynomial of RMS-normed powers, or a routed mixture of silu-gated
// experts (softmax over all experts, the choice limited to the best groups, renormalised weights).
//
// A step runs on the family-independent pieces of the library: StepRunner (streams and lanes, workspaces, graph replay of
// single-token steps, routed experts as dense products, results to the host), SequenceBatch / PagePool for slots, pages and
// the per-token tables, SlotState for what the recurrence carries, b200_linear_ex2 (tcgen05) and b200_gemm_grouped,
// b200_rope_angles, b200_latent_norms / b200_rotate_part / b200_latent_attention_ex, b200_qk_prepare, b200_paged_attention
// (window, temperatures, mix), b200_sigmoid_gate, b200_conv_act / b200_ssd_scan / b200_gated_group_rms,
// b200_moe_route_groups / b200_moe_dispatch, b200_poly_norm, b200_parallel_residual. The residual stream, all norms, rotary
// angles, scores and weights, the router, and the recurrence with everything that enters it after projections and convolution
// are fp32 in both serving dtypes; in B200_BF16 the GEMM operands and the cache pages are bfloat16.
//
// Launch order of a layer (T tokens of all entries packed; h = N x in the serving dtype). The sublayers read the same h, so
// they are enqueued on lanes of their own and meet in the residual update:
//   lane 1:  router -> counting sort -> gated up products per expert -> down products; or up -> normed powers -> down
//   lane 0:  latent: [dq | dkv | gate] = h W^T -> both low-rank norms, key part rotated, row to the pages -> q = cq W_uq^T ->
//              per head q W_uk beside the rotated query part -> attention over the rows -> per head W_uv, gated -> W_o
//            parallel: [q | k | v | gate | z | x B C | dt] = h W^T -> rotations, page stores -> attention -> gate -> W_o
//   lane 2:  (parallel) convolution + silu -> recurrence -> gated norm -> W_o
//   join:    x += m (mixer + ff), h = next layer's N x (one kernel).
#include <cuda_bf16.h>

#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstdlib>
#include <cstring>

#include "checkpoint_upload.h"
#include "common.cuh"
#include "launch_count.h"
#include "model_registry.h"
#include "safetensors.h"

namespace b200 {
namespace {

constexpr int kPageRows = 64;

struct FpFreq {
    std::vector<double> f;
    double* dev = nullptr;
};
struct FpLatent {
    int heads = 0, dim = 0, rot_dim = 0, vdim = 0, q_rank = 0, rank = 0, table = -1, kv_from = -1;
    double base = 0.0;
    float scale = 1.f;
    int kv_off = 0, g_off = 0;              // columns in the stacked input projection
    float *q_norm = nullptr, *kv_norm = nullptr;
    void *uq = nullptr, *uk = nullptr, *uv = nullptr;
    int nq() const { return heads * (dim + rot_dim); }
    int row() const { return rank + rot_dim; }
};
struct FpAttn {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, rot_dims = 0, window = 0, table = -1;
    double base = 0.0;
    float scale = 1.f;
    float *temp = nullptr, *mix = nullptr, *out_norm = nullptr;
    int nq() const { return heads * dim; }
    int nk() const { return kv_heads * dim; }
    int nv() const { return kv_heads * vdim; }
    int natt() const { return heads * vdim; }
};
struct FpSsd {
    int heads = 0, vdim = 0, state = 0, groups = 0, taps = 1, norm_parts = 1, in_off = 0;
    float *conv_w = nullptr, *conv_b = nullptr, *dt_b = nullptr, *A = nullptr, *Dv = nullptr, *norm = nullptr, *out_norm = nullptr;
    void* w_o = nullptr;
    int inner() const { return heads * vdim; }
    int channels() const { return inner() + 2 * groups * state; }   // x | B | C
};
enum { kFfNone = 0, kFfDense = 1, kFfRouted = 2 };

struct FpLayer {
    bool latent = false;
    FpLatent la;
    FpAttn at;
    FpSsd ss;
    int n_in = 0, n_mid = 0;                         // columns of the stacked input projection; inputs of W_o
    void *w_in = nullptr, *w_o = nullptr;
    float* n1 = nullptr;
    int ff_kind = kFfNone, ff = 0, experts = 0, top = 0, groups = 1, keep = 1;
    float *router = nullptr, *act = nullptr;
    void *w_up = nullptr, *w_down = nullptr;         // routed: [experts, 2 ff, D] (gate rows first) and [experts, D, ff]
    void *k_pool = nullptr, *v_pool = nullptr;       // latent: k_pool holds the rows [latent | key part], another layer's with kv_from
    SlotState ring, state;
};

class Filipel : public StepRunner {
public:
    ~Filipel() override {
        if (stream_) cudaStreamSynchronize(stream_);
        cudaFree(scratch_);
    }
    const char* family() const override { return "Filipel"; }
    int layer_count() const override { return (int)layers_.size(); }
    int load(const ModelDir& dir, const b200_model_options& opt, std::string& err);

private:
    int parse(const Json& ls, std::string& err);
    int parse_latent(const Json& mx, int i, const std::string& where, FpLayer& L, std::string& err);
    int parse_parallel(const Json& mx, const std::string& where, FpLayer& L, std::string& err);
    int parse_ff(const Json& ml, const std::string& where, FpLayer& L, std::string& err);
    int freq_table(double base, int dims, int& table, std::string& err);
    int ensure_scratch(int T, int W) override;
    int enqueue(int T, int W, int longest_entry, int longest_context, bool want_ids, std::string& err) override;
    int latent_mixer(FpLayer& L, int T, int longest_entry, int longest_context, std::string& err);
    int attention_side(FpLayer& L, int T, int longest_entry, int longest_context, std::string& err);
    int recurrent_side(FpLayer& L, int T, int longest_entry, std::string& err);
    size_t attention_bytes(int T) const;
    size_t scan_bytes(int T, int n_entries) const;
    // attention and recurrence run on different lanes: each has its own part of the shared workspace
    size_t step_workspace_bytes(int T, int n_entries) const override { return attention_bytes(T) + scan_bytes(T, n_entries); }
    const float* cos_of(int table) const { return cs_ + (size_t)seq_.n_tokens * freq_off_[table]; }
    const float* sin_of(int table) const { return cos_of(table) + (size_t)seq_.n_tokens * freqs_[table].f.size(); }

    float eps_ = 1e-6f, mult_ = 1.f;
    std::vector<FpLayer> layers_;
    std::vector<FpFreq> freqs_;
    void *embed_ = nullptr, *head_ = nullptr;
    float* fnw_ = nullptr;
    // scratch, grown to the largest step seen
    char* scratch_ = nullptr;
    int cap_T_ = 0, cap_W_ = 0;
    float *x_ = nullptr, *proj_ = nullptr, *y_ = nullptr, *y2_ = nullptr, *y3_ = nullptr, *qf_ = nullptr, *qa_ = nullptr, *oa_ = nullptr, *attf_ = nullptr,
          *conv_ = nullptr, *scan_ = nullptr, *up_ = nullptr, *eo_ = nullptr, *weight_ = nullptr, *cs_ = nullptr;
    void *h_ = nullptr, *cq_ = nullptr, *q_ = nullptr, *mid_ = nullptr, *sy_ = nullptr, *act_ = nullptr, *gath_ = nullptr, *hf_ = nullptr;
    int *chosen_ = nullptr, *group_off_ = nullptr, *src_row_ = nullptr, *dest_ = nullptr;
    // maxima over layers (scratch sizes)
    int max_in_ = 0, max_mid_ = 0, max_qf_ = 0, max_qa_ = 0, max_q_ = 0, max_attf_ = 0, max_cq_ = 0, max_ch_ = 0, max_inner_ = 0, max_dense_ = 0,
        max_act_ = 0, max_top_ = 0, max_experts_ = 0, freq_floats_ = 0;
    std::vector<int> freq_off_;
};

#define FP_TRY(call)                    \
    do {                                \
        const int rc_ = (call);         \
        if (rc_ != B200_OK) return rc_; \
    } while (0)
#define FP_OP(call)                                                             \
    do {                                                                        \
        const int rc_ = (call);                                                 \
        if (rc_ != B200_OK) { err = std::string(#call) + " failed (" + std::to_string(rc_) + ")"; return rc_; } \
    } while (0)

const Json* member(const Json& j, const char* name) {   // null counts as absent
    const Json* v = j.get(name);
    return v && !v->is_null() ? v : nullptr;
}

// f_i = base^(-2i/dims); layers with equal frequencies share one cos / sin table per step
int Filipel::freq_table(double base, int dims, int& table, std::string& err) {
    FpFreq fs;
    fs.f.resize(dims / 2);
    for (int i = 0; i < dims / 2; ++i) fs.f[i] = std::pow(base, -2.0 * i / dims);
    for (size_t k = 0; k < freqs_.size(); ++k)
        if (freqs_[k].f == fs.f) { table = (int)k; return B200_OK; }
    fs.dev = (double*)dalloc(fs.f.size() * sizeof(double));
    if (!fs.dev || cudaMemcpy(fs.dev, fs.f.data(), fs.f.size() * sizeof(double), cudaMemcpyHostToDevice) != cudaSuccess) { err = "out of device memory"; return B200_ENOMEM; }
    table = (int)freqs_.size();
    freqs_.push_back(fs);
    return B200_OK;
}

int Filipel::parse_latent(const Json& mx, int i, const std::string& where, FpLayer& L, std::string& err) {
    FpLatent& la = L.la;
    L.latent = true;
    la.heads = (int)mx.integer("heads", 0);
    la.dim = (int)mx.integer("dim", 0);
    la.vdim = (int)mx.integer("vdim", 0);
    la.q_rank = (int)mx.integer("q_rank", 0);
    la.rank = (int)mx.integer("kv_rank", 0);
    la.rot_dim = (int)mx.integer("rot_dim", 0);
    if (la.heads < 1 || la.dim < 1 || la.vdim < 1 || la.q_rank < 1 || la.rank < 1 || la.rot_dim < 0 || (la.rot_dim & 1) || !mx.has("scale")) {
        err = where + "latent attention needs heads, dim, vdim, q_rank, kv_rank, scale and an even rot_dim";
        return B200_EINVAL;
    }
    la.scale = (float)mx.number("scale", 1.0);
    if (la.row() > 640) { err = where + "cached rows wider than 640 are not supported by the latent attention kernels"; return B200_EUNSUPPORTED; }
    const Json* r = member(mx, "rot");
    if (la.rot_dim > 0) {
        if (!r || (int)r->integer("dims", la.rot_dim) != la.rot_dim || !(r->number("base", 0.0) > 0.0)) { err = where + "rot: dims must equal rot_dim, base must be positive"; return B200_EINVAL; }
        la.base = r->number("base", 0.0);
    }
    if (member(mx, "kv_from")) {
        la.kv_from = (int)mx.integer("kv_from", -1);
        const FpLayer* src = la.kv_from >= 0 && la.kv_from < i ? &layers_[la.kv_from] : nullptr;
        if (!src || !src->latent || src->la.kv_from >= 0) { err = where + "kv_from must name an earlier latent attention layer with rows of its own"; return B200_EINVAL; }
        if (src->la.rank != la.rank || src->la.rot_dim != la.rot_dim || src->la.base != la.base) { err = where + "kv_from: kv_rank, rot_dim and rotation must equal the other layer's"; return B200_EINVAL; }
    }
    la.kv_off = la.q_rank;
    la.g_off = la.kv_off + (la.kv_from < 0 ? la.row() : 0);
    L.n_mid = la.heads * la.vdim;
    L.n_in = la.g_off + L.n_mid;
    return B200_OK;
}

int Filipel::parse_parallel(const Json& mx, const std::string& where, FpLayer& L, std::string& err) {
    const Json *left = member(mx, "left"), *right = member(mx, "right");
    if (!left || !right) { err = where + "a parallel mixer needs left and right"; return B200_EINVAL; }
    FpAttn& at = L.at;
    at.heads = (int)left->integer("heads", 0);
    at.kv_heads = (int)left->integer("kv_heads", at.heads);
    at.dim = (int)left->integer("dim", 0);
    at.vdim = (int)left->integer("vdim", 0);
    if (at.heads < 1 || at.kv_heads < 1 || at.dim < 1 || at.vdim < 1 || !left->has("scale")) { err = where + "attention needs heads, kv_heads, dim, vdim and scale"; return B200_EINVAL; }
    if (at.heads % at.kv_heads) { err = where + "heads must be a multiple of kv_heads"; return B200_EINVAL; }
    at.scale = (float)left->number("scale", 1.0);
    const Json* mk = member(*left, "mask");
    at.window = mk ? (int)mk->integer("size", 0) : 0;
    if (mk && at.window < 1) { err = where + "mask.size must be positive"; return B200_EINVAL; }
    const Json* r = member(*left, "rot");
    at.rot_dims = r ? (int)r->integer("dims", 0) : 0;
    at.base = r ? r->number("base", 0.0) : 0.0;
    if (at.rot_dims < 0 || (at.rot_dims & 1) || at.rot_dims > at.dim || (at.rot_dims > 0 && !(at.base > 0.0))) { err = where + "rot: dims must be even and at most dim, base must be positive"; return B200_EINVAL; }
    FpSsd& ss = L.ss;
    ss.heads = (int)right->integer("heads", 0);
    ss.vdim = (int)right->integer("vdim", 0);
    ss.state = (int)right->integer("state", 0);
    ss.groups = (int)right->integer("groups", 1);
    ss.taps = (int)right->integer("conv", 1);
    ss.norm_parts = (int)right->integer("norm_groups", 1);
    if (ss.heads < 1 || ss.vdim < 1 || ss.state < 1 || ss.groups < 1 || ss.taps < 1 || ss.norm_parts < 1) { err = where + "the recurrence needs heads, vdim, state, groups, conv and norm_groups"; return B200_EINVAL; }
    if (ss.heads % ss.groups || ss.inner() % ss.norm_parts) { err = where + "heads must be a multiple of groups, heads * vdim of norm_groups"; return B200_EINVAL; }
    if (ss.state > 256) { err = where + "state above 256 is not supported by the recurrence kernels"; return B200_EUNSUPPORTED; }
    ss.in_off = at.nq() + at.nk() + at.nv() + at.natt();
    L.n_mid = at.natt();
    L.n_in = ss.in_off + ss.inner() + ss.channels() + ss.heads;
    return B200_OK;
}

int Filipel::parse_ff(const Json& ml, const std::string& where, FpLayer& L, std::string& err) {
    const std::string kind = ml.text("kind");
    if (kind == "dense") {
        L.ff_kind = kFfDense;
        L.ff = (int)ml.integer("ff", 0);
        if (L.ff < 1) { err = where + "mlp.ff is required"; return B200_EINVAL; }
    } else if (kind == "moe") {
        L.ff_kind = kFfRouted;
        const Json *ex = member(ml, "expert"), *ro = member(ml, "router");
        L.ff = ex ? (int)ex->integer("ff", 0) : 0;
        L.experts = ro ? (int)ro->integer("experts", 0) : 0;
        L.top = ro ? (int)ro->integer("top", 0) : 0;
        if (L.ff < 1 || L.experts < 1 || L.top < 1 || L.top > L.experts) { err = where + "a routed feed-forward needs expert.ff, router.experts and 1 <= router.top <= experts"; return B200_EINVAL; }
        if (const Json* gr = member(*ro, "groups")) {
            L.groups = (int)gr->integer("count", 0);
            L.keep = (int)gr->integer("keep", 0);
            if (L.groups < 1 || L.experts % L.groups || L.keep < 1 || L.keep > L.groups || L.top > L.keep * (L.experts / L.groups)) {
                err = where + "router.groups: count must divide the experts, 1 <= keep <= count, and the kept groups must hold `top` experts";
                return B200_EINVAL;
            }
        }
        if (L.top > 16) { err = where + "more than 16 experts per token are not supported"; return B200_EUNSUPPORTED; }
    } else {
        err = where + "feed-forward kind '" + kind + "' is not part of this family";
        return B200_EUNSUPPORTED;
    }
    return B200_OK;
}

// everything that can be refused from the configuration alone, before the first CUDA call
int Filipel::parse(const Json& ls, std::string& err) {
    layers_.resize(ls.arr.size());
    for (size_t i = 0; i < ls.arr.size(); ++i) {
        const Json& lj = ls.arr[i];
        const std::string type = lj.text("type"), where = "layer " + std::to_string(i) + ": ";
        const Json* mx = member(lj, "mixer");
        if (!mx) { err = where + "no mixer"; return B200_EINVAL; }
        if (type == "latent_attention") FP_TRY(parse_latent(*mx, (int)i, where, layers_[i], err));
        else if (type == "parallel") FP_TRY(parse_parallel(*mx, where, layers_[i], err));
        else { err = where + "mixer type '" + type + "' is not part of this family"; return B200_EUNSUPPORTED; }
        if (const Json* ml = member(lj, "mlp")) FP_TRY(parse_ff(*ml, where, layers_[i], err));
    }
    return B200_OK;
}

int Filipel::load(const ModelDir& dir, const b200_model_options& opt, std::string& err) {
    const Json& c = dir.config;
    dtype_ = opt.dtype;
    if (dtype_ != B200_BF16 && dtype_ != B200_F32) { err = "dtype must be bfloat16 or float32"; return B200_EINVAL; }
    vocab_ = (int)c.integer("vocab", 0);
    D_ = (int)c.integer("width", 0);
    const Json *norm = member(c, "norm"), *ls = c.get("layers");
    if (vocab_ < 1 || D_ < 1 || !norm || !norm->has("eps") || !ls || ls->kind != Json::Arr || ls->arr.empty()) {
        err = "config.json: vocab, width, norm.eps and layers are required";
        return B200_EINVAL;
    }
    eps_ = (float)norm->number("eps", 1e-6);
    mult_ = (float)c.number("residual_mult", 1.0);
    if (opt.max_tokens < 1 || opt.max_slots < 1) { err = "max_tokens and max_slots must be positive"; return B200_EINVAL; }
    FP_TRY(parse(*ls, err));

    FP_TRY(init_runner(err));
    SafeTensorsFile st;
    if (!st.open(dir.path + "/model.safetensors", err)) return B200_EINVAL;
    // the design has no position limit of its own: a sequence can grow as long as the pool has pages
    const int n_pages = (opt.max_tokens + kPageRows - 1) / kPageRows;
    FP_TRY(seq_.init(opt.max_tokens, kPageRows, opt.max_slots, n_pages * kPageRows, err));

    const size_t E = esz();
    const long long D = D_;
    auto f32 = [&](const std::string& name, std::vector<long long> shape, float*& dst) -> int {
        size_t cnt = 1;
        for (long long d : shape) cnt *= (size_t)d;
        dst = (float*)dalloc(cnt * 4);
        if (!dst) { err = "out of device memory"; return B200_ENOMEM; }
        return upload_tensor(st, name, shape, true, dtype_, dst, err);
    };
    // checkpoint matrices that read the same input (or the experts of one layer), stacked row-wise into one operand
    auto stacked = [&](const std::vector<std::pair<std::string, long long>>& parts, long long cols, void*& dst) -> int {
        long long rows = 0;
        for (auto& p : parts) rows += p.second;
        dst = dalloc((size_t)rows * cols * E);
        if (!dst) { err = "out of device memory"; return B200_ENOMEM; }
        long long at = 0;
        for (auto& p : parts) {
            FP_TRY(upload_tensor(st, p.first, {p.second, cols}, false, dtype_, (char*)dst + (size_t)at * cols * E, err));
            at += p.second;
        }
        return B200_OK;
    };
    auto mat = [&](const std::string& name, long long rows, long long cols, void*& dst) -> int { return stacked({{name, rows}}, cols, dst); };
    auto pages = [&](int row, void*& dst) -> int {
        const size_t bytes = (size_t)seq_.pool.n_pages() * kPageRows * row * E;
        dst = dalloc(bytes);
        if (!dst || cudaMemset(dst, 0, bytes) != cudaSuccess) { err = "out of device memory (cache pages)"; return B200_ENOMEM; }
        return B200_OK;
    };
    FP_TRY(mat("embed", vocab_, D, embed_));
    FP_TRY(mat("head", vocab_, D, head_));
    FP_TRY(f32("final.norm", {D}, fnw_));
    for (size_t i = 0; i < layers_.size(); ++i) {
        FpLayer& L = layers_[i];
        const std::string pre = "l" + std::to_string(i) + ".", mp = pre + "mix.";
        FP_TRY(f32(pre + "norm1", {D}, L.n1));
        if (L.latent) {
            FpLatent& la = L.la;
            std::vector<std::pair<std::string, long long>> parts = {{mp + "dq", la.q_rank}};
            if (la.kv_from < 0) {
                parts.push_back({mp + "dkv", la.row()});
                FP_TRY(f32(mp + "dkv.norm", {la.rank}, la.kv_norm));
                FP_TRY(pages(la.row(), L.k_pool));
            } else
                L.k_pool = layers_[la.kv_from].k_pool;
            parts.push_back({mp + "g", L.n_mid});
            FP_TRY(stacked(parts, D, L.w_in));
            FP_TRY(f32(mp + "dq.norm", {la.q_rank}, la.q_norm));
            FP_TRY(mat(mp + "uq", la.nq(), la.q_rank, la.uq));
            FP_TRY(mat(mp + "uk", (long long)la.heads * la.dim, la.rank, la.uk));
            FP_TRY(mat(mp + "uv", (long long)la.heads * la.vdim, la.rank, la.uv));
            FP_TRY(mat(mp + "o", D, L.n_mid, L.w_o));
            if (la.rot_dim > 0) FP_TRY(freq_table(la.base, la.rot_dim, la.table, err));
            max_qf_ = std::max(max_qf_, la.nq());
            max_qa_ = std::max(max_qa_, la.heads * la.row());
            max_cq_ = std::max(max_cq_, la.q_rank);
        } else {
            FpAttn& at = L.at;
            FpSsd& ss = L.ss;
            const std::string lp = mp + "left.", rp = mp + "right.";
            FP_TRY(stacked({{lp + "q", at.nq()}, {lp + "k", at.nk()}, {lp + "v", at.nv()}, {lp + "g", at.natt()},
                            {rp + "in", ss.inner() + ss.channels() + ss.heads}}, D, L.w_in));
            FP_TRY(f32(lp + "temp", {at.heads}, at.temp));
            FP_TRY(f32(lp + "talk", {at.heads, at.heads}, at.mix));
            FP_TRY(f32(lp + "out", {D}, at.out_norm));
            FP_TRY(mat(lp + "o", D, at.natt(), L.w_o));
            FP_TRY(pages(at.nk(), L.k_pool));
            FP_TRY(pages(at.nv(), L.v_pool));
            if (at.rot_dims > 0) FP_TRY(freq_table(at.base, at.rot_dims, at.table, err));
            FP_TRY(f32(rp + "conv", {ss.channels(), ss.taps}, ss.conv_w));
            FP_TRY(f32(rp + "conv.b", {ss.channels()}, ss.conv_b));
            FP_TRY(f32(rp + "dt_bias", {ss.heads}, ss.dt_b));
            FP_TRY(f32(rp + "D", {ss.heads}, ss.Dv));
            FP_TRY(f32(rp + "norm", {ss.inner()}, ss.norm));
            FP_TRY(f32(rp + "out", {D}, ss.out_norm));
            FP_TRY(mat(rp + "o", D, ss.inner(), ss.w_o));
            {   // A = -exp(A_log), formed once in double
                FP_TRY(f32(rp + "A_log", {ss.heads}, ss.A));
                const SafeTensor* t = st.find(rp + "A_log");
                std::vector<float> A(ss.heads);
                for (int k = 0; k < ss.heads; ++k) A[k] = (float)-std::exp((double)st_value(*t, k));
                if (cudaMemcpy(ss.A, A.data(), A.size() * 4, cudaMemcpyHostToDevice) != cudaSuccess) { err = "weight upload failed"; return B200_EINVAL; }
            }
            cudaError_t e = cudaSuccess;
            if (ss.taps > 1) e = L.ring.init(opt.max_slots, (size_t)(ss.taps - 1) * ss.channels());
            if (e == cudaSuccess) e = L.state.init(opt.max_slots, (size_t)ss.heads * ss.state * ss.vdim);
            if (e != cudaSuccess) { err = "out of device memory (carried state)"; return B200_ENOMEM; }
            max_q_ = std::max(max_q_, at.nq());
            max_attf_ = std::max(max_attf_, at.natt());
            max_ch_ = std::max(max_ch_, ss.channels());
            max_inner_ = std::max(max_inner_, ss.inner());
        }
        max_in_ = std::max(max_in_, L.n_in);
        max_mid_ = std::max(max_mid_, L.n_mid);
        if (L.ff_kind == kFfDense) {
            FP_TRY(mat(pre + "mlp.up", L.ff, D, L.w_up));
            FP_TRY(mat(pre + "mlp.down", D, L.ff, L.w_down));
            FP_TRY(f32(pre + "mlp.act", {4}, L.act));
            max_dense_ = std::max(max_dense_, L.ff);
            max_act_ = std::max(max_act_, L.ff);
        } else if (L.ff_kind == kFfRouted) {
            std::vector<std::pair<std::string, long long>> ups, downs;
            for (int e = 0; e < L.experts; ++e) {
                const std::string ep = pre + "mlp.e" + std::to_string(e) + ".";
                ups.push_back({ep + "gate", L.ff});
                ups.push_back({ep + "up", L.ff});
                downs.push_back({ep + "down", D});
            }
            FP_TRY(stacked(ups, D, L.w_up));
            FP_TRY(stacked(downs, L.ff, L.w_down));
            FP_TRY(f32(pre + "mlp.router", {L.experts, D}, L.router));
            max_act_ = std::max(max_act_, L.top * L.ff);
            max_top_ = std::max(max_top_, L.top);
            max_experts_ = std::max(max_experts_, L.experts);
        }
    }
    freq_off_.assign(freqs_.size(), 0);
    for (size_t k = 0; k < freqs_.size(); ++k) {
        freq_off_[k] = freq_floats_;
        freq_floats_ += 2 * (int)freqs_[k].f.size();   // cos and sin per token
    }
    if (cudaDeviceSynchronize() != cudaSuccess) { err = "weight upload failed"; return B200_EINVAL; }
    return B200_OK;
}

size_t Filipel::attention_bytes(int T) const {
    const int longest = seq_.length.empty() ? 0 : *std::max_element(seq_.length.begin(), seq_.length.end());
    size_t need = 0;
    for (const FpLayer& L : layers_) {
        if (!L.latent) {
            if (dtype_ == B200_BF16) need = std::max(need, b200_mixed_attention_workspace_bytes(T, L.at.heads, L.at.window, longest));
        } else if ((long long)T * L.la.heads <= 8192)   // only batches of few rows split their contexts
            need = std::max(need, b200_latent_attention_workspace_bytes(T, L.la.heads, L.la.row()));
    }
    return (need + 255) & ~(size_t)255;
}
size_t Filipel::scan_bytes(int T, int n_entries) const {
    size_t need = 0;
    if (dtype_ == B200_BF16)
        for (const FpLayer& L : layers_)
            if (!L.latent) need = std::max(need, b200_ssd_scan_workspace_bytes(T, n_entries, L.ss.heads, L.ss.groups, L.ss.vdim, L.ss.state));
    return need;
}

int Filipel::ensure_scratch(int T, int W) {
    if (T <= cap_T_ && W <= cap_W_) return B200_OK;
    const int cT = std::max(T, cap_T_), cW = std::max(W, cap_W_);
    cudaStreamSynchronize(stream_);
    buffers_moved();
    cudaFree(scratch_);
    scratch_ = nullptr;
    cap_T_ = cap_W_ = 0;
    auto al = [](size_t b) { return (std::max<size_t>(b, 1) + 255) & ~(size_t)255; };
    const size_t E = esz(), t = (size_t)cT, top = (size_t)std::max(1, max_top_), routed = max_top_ > 0;
    const size_t sizes[] = {
        al(t * D_ * 4),                            // x
        al(t * max_in_ * 4),                       // proj
        al(t * D_ * 4),                            // y
        al(t * D_ * 4),                            // y2
        al(t * D_ * 4),                            // y3
        al(t * max_qf_ * 4),                       // qf
        al(t * max_qa_ * 4),                       // qa
        al(t * max_qa_ * 4),                       // oa
        al(t * max_attf_ * 4),                     // attf
        al(t * max_ch_ * 4),                       // conv
        al(t * max_inner_ * 4),                    // scan
        al(t * max_dense_ * 4),                    // up
        al(routed * t * top * D_ * 4),             // eo
        al(t * top * 4),                           // weight
        al((size_t)cW * vocab_ * 4),               // logits
        al(t * freq_floats_ * 4),                  // cos / sin tables
        al(t * D_ * E),                            // h
        al(t * max_cq_ * E),                       // cq
        al(t * max_q_ * E),                        // q
        al(t * max_mid_ * E),                      // mid
        al(t * max_inner_ * E),                    // sy
        al(t * max_act_ * E),                      // act
        al(routed * t * top * D_ * E),             // gath
        al((size_t)cW * D_ * E),                   // hf
        al(t * top * 4),                           // chosen
        al((size_t)(max_experts_ + 2) * 4),        // group_off
        al(t * top * 4),                           // src_row
        al(t * top * 4),                           // dest
        al((size_t)cW * 4),                        // ids
    };
    size_t total = 0;
    for (size_t s : sizes) total += s;
    if (cudaMalloc(&scratch_, total) != cudaSuccess) return B200_ENOMEM;
    char* p = scratch_;
    int k = 0;
    auto take = [&](auto*& dst) { dst = reinterpret_cast<std::remove_reference_t<decltype(dst)>>(p); p += sizes[k++]; };
    take(x_); take(proj_); take(y_); take(y2_); take(y3_); take(qf_); take(qa_); take(oa_); take(attf_); take(conv_); take(scan_); take(up_);
    take(eo_); take(weight_); take(logits_); take(cs_);
    take(h_); take(cq_); take(q_); take(mid_); take(sy_); take(act_); take(gath_); take(hf_);
    take(chosen_); take(group_off_); take(src_row_); take(dest_); take(ids_dev_);
    cap_T_ = cT;
    cap_W_ = cW;
    return ensure_logits_host(cW);
}

int Filipel::latent_mixer(FpLayer& L, int T, int longest_entry, int longest_context, std::string& err) {
    const FpLatent& la = L.la;
    const int H = la.heads, R = la.rank, dr = la.rot_dim, row = la.row(), dt = dtype_, dq = la.dim + dr;
    const int* pages = seq_.pool.device();
    const int max_pages = seq_.pool.max_pages();
    const float *cs = dr > 0 ? cos_of(la.table) : nullptr, *sn = dr > 0 ? sin_of(la.table) : nullptr;
    FP_OP(gemm(h_, L.w_in, proj_, B200_F32, T, L.n_in, D_));
    {
        b200_latent_norms_args n{};
        n.raw = proj_; n.ld_raw = L.n_in; n.q_off = 0; n.kv_off = la.kv_off;
        n.q_norm = la.q_norm; n.q_rank = la.q_rank; n.q_out = cq_;
        n.kv_norm = la.kv_norm; n.eps = eps_; n.pool = la.kv_from < 0 ? L.k_pool : nullptr;
        n.pages = pages; n.max_pages = max_pages; n.page_rows = kPageRows; n.slot = seq_.d_slot(); n.pos = seq_.d_pos();
        n.n_tokens = T; n.rank = R; n.extra = dr; n.cos = cs; n.sin = sn; n.rot_layout = B200_ROPE_HALF; n.dtype = dt;
        FP_OP(b200_latent_norms(&n, stream_));
    }
    FP_OP(gemm(cq_, la.uq, qf_, B200_F32, T, la.nq(), la.q_rank));
    {   // qa[t, h, 0:R] = sum_d q[t, h, d] W_uk[h*dim + d, :]
        b200_gemm_grouped_args g{};
        g.A = qf_; g.lda = la.nq(); g.stride_a = dq;
        g.W = la.uk; g.ldw = R; g.stride_w = (long long)la.dim * R; g.trans_b = 0;
        g.C = qa_; g.ldc = (long long)H * row; g.stride_c = row;
        g.M = T; g.N = R; g.K = la.dim; g.batch = H;
        g.a_dtype = B200_F32; g.w_dtype = dt; g.c_dtype = B200_F32;
        FP_OP(b200_gemm_grouped(&g, stream_));
    }
    if (dr > 0)   // qa[t, h, R:R+dr] = the head's rotated query part
        FP_OP(b200_rotate_part(qf_, la.nq(), la.dim, dq, qa_, (long long)H * row, R, row, cs, sn, B200_ROPE_HALF, T, H, dr, stream_));
    b200_latent_attention_args at{};
    at.qa = qa_; at.out = oa_; at.pool = L.k_pool; at.pages = pages; at.max_pages = max_pages; at.page_rows = kPageRows;
    at.slot = seq_.d_slot(); at.pos = seq_.d_pos(); at.sink = nullptr; at.scale = la.scale;
    at.n_tokens = T; at.heads = H; at.rank = row; at.window = 0; at.dtype = dt;
    at.longest_entry = longest_entry; at.longest_context = longest_context;
    at.workspace = attn_ws_; at.workspace_bytes = std::min(attn_ws_bytes_, attention_bytes(T));
    at.out_cols = R;   // the value up-projection reads the latent columns only
    FP_OP(b200_latent_attention_ex(&at, stream_));
    {   // mid[t, h, :] = (W_uv,h oa[t, h, 0:R]) * sigmoid(gate[t, h, :])
        b200_gemm_grouped_args g{};
        g.A = oa_; g.lda = (long long)H * row; g.stride_a = row;
        g.W = la.uv; g.ldw = R; g.stride_w = (long long)la.vdim * R; g.trans_b = 1;
        g.C = mid_; g.ldc = L.n_mid; g.stride_c = la.vdim;
        g.aux = proj_ + la.g_off; g.ld_aux = L.n_in; g.stride_aux = la.vdim; g.epi = B200_GG_SIGMOID_MUL;
        g.M = T; g.N = la.vdim; g.K = R; g.batch = H;
        g.a_dtype = B200_F32; g.w_dtype = dt; g.c_dtype = dt;
        FP_OP(b200_gemm_grouped(&g, stream_));
    }
    FP_OP(gemm(mid_, L.w_o, y_, B200_F32, T, D_, L.n_mid));
    return B200_OK;
}

int Filipel::attention_side(FpLayer& L, int T, int longest_entry, int longest_context, std::string& err) {
    const FpAttn& at = L.at;
    const int dt = dtype_;
    b200_qk_prepare_args qa{};
    qa.proj = proj_; qa.ld_proj = L.n_in;
    if (at.rot_dims > 0) { qa.cos = cos_of(at.table); qa.sin = sin_of(at.table); }
    qa.rot_dims = at.rot_dims; qa.rot_layout = B200_ROPE_HALF;
    qa.q_out = q_; qa.k_pool = L.k_pool; qa.v_pool = L.v_pool;
    qa.pages = seq_.pool.device(); qa.max_pages = seq_.pool.max_pages(); qa.page_rows = kPageRows;
    qa.slot = seq_.d_slot(); qa.pos = seq_.d_pos(); qa.start = seq_.d_start();
    qa.n_tokens = T; qa.heads = at.heads; qa.kv_heads = at.kv_heads; qa.dim = at.dim; qa.dtype = dt;
    qa.v_heads = at.kv_heads; qa.vdim = at.vdim; qa.v_off = at.nq() + at.nk();
    FP_OP(b200_qk_prepare(&qa, stream_));
    b200_paged_attention_args pa{};
    pa.q = q_; pa.out = attf_; pa.k_pool = L.k_pool; pa.v_pool = L.v_pool;
    pa.pages = qa.pages; pa.max_pages = qa.max_pages; pa.page_rows = kPageRows;
    pa.slot = seq_.d_slot(); pa.pos = seq_.d_pos();
    pa.n_tokens = T; pa.heads = at.heads; pa.kv_heads = at.kv_heads; pa.dim = at.dim; pa.vdim = at.vdim;
    pa.scale = at.scale; pa.dtype = dt; pa.longest_entry = longest_entry; pa.longest_context = longest_context;
    pa.workspace = attn_ws_; pa.workspace_bytes = std::min(attn_ws_bytes_, attention_bytes(T));
    pa.out_f32 = 1; pa.window = at.window; pa.head_temp = at.temp; pa.head_mix = at.mix;
    FP_OP(b200_paged_attention(&pa, stream_));
    FP_OP(b200_sigmoid_gate(attf_, proj_ + at.nq() + at.nk() + at.nv(), L.n_in, mid_, T, at.natt(), dt, stream_));
    FP_OP(gemm(mid_, L.w_o, y_, B200_F32, T, D_, L.n_mid));
    return B200_OK;
}

int Filipel::recurrent_side(FpLayer& L, int T, int longest_entry, std::string& err) {
    const FpSsd& ss = L.ss;
    const int dt = dtype_;
    cudaStream_t s = lane(2);
    const float* z = proj_ + ss.in_off;
    const float* u = z + ss.inner();
    b200_conv_act_args ca{};
    ca.u = u; ca.ld_u = L.n_in; ca.w = ss.conv_w; ca.bias = ss.conv_b; ca.taps = ss.taps; ca.conv_state = L.ring.data();
    ca.out32 = conv_; ca.out_dtype = dt;
    ca.slot = seq_.d_slot(); ca.pos = seq_.d_pos(); ca.start = seq_.d_start();
    ca.n_tokens = T; ca.channels = ss.channels(); ca.update_state_inline = longest_entry == 1;
    FP_OP(b200_conv_act(&ca, s));
    if (ss.taps > 1 && longest_entry != 1)
        FP_OP(b200_conv_state_update(u, L.n_in, L.ring.data(), seq_.d_slot(), seq_.d_pos(), seq_.d_end(), T, ss.channels(), ss.taps, s));
    b200_ssd_scan_args sa{};
    sa.u = conv_; sa.ld_u = ss.channels(); sa.x_off = 0; sa.b_off = ss.inner(); sa.c_off = ss.inner() + ss.groups * ss.state;
    sa.dt_raw = u + ss.channels(); sa.ld_dt = L.n_in; sa.dt_bias = ss.dt_b; sa.A = ss.A; sa.D = ss.Dv;
    sa.state = L.state.data(); sa.out = scan_;
    sa.ent_row = seq_.d_ent_row(); sa.ent_len = seq_.d_ent_len(); sa.slot = seq_.d_slot(); sa.pos = seq_.d_pos();
    sa.n_entries = seq_.n_entries; sa.n_tokens = T; sa.heads = ss.heads; sa.groups = ss.groups; sa.vdim = ss.vdim; sa.n_state = ss.state;
    sa.longest_entry = longest_entry; sa.chunked = dt == B200_BF16;
    const size_t skip = attention_bytes(T);
    if (attn_ws_bytes_ > skip) { sa.workspace = (char*)attn_ws_ + skip; sa.workspace_bytes = attn_ws_bytes_ - skip; }
    FP_OP(b200_ssd_scan(&sa, s));
    FP_OP(b200_gated_group_rms(scan_, z, L.n_in, ss.norm, sy_, T, ss.inner(), ss.norm_parts, eps_, dt, s));
    FP_OP(gemm(sy_, ss.w_o, y2_, B200_F32, T, D_, ss.inner(), B200_GG_NONE, 0.f, 2));
    return B200_OK;
}

// every launch of a step, in order, on stream_ and the lanes beside it (no allocation; prompt steps wait for the sizes of the
// expert groups, single-token steps for nothing: capturable into a graph)
int Filipel::enqueue(int T, int W, int longest_entry, int longest_context, bool want_ids, std::string& err) {
    const int D = D_, dt = dtype_;
    for (size_t k = 0; k < freqs_.size(); ++k)
        FP_OP(b200_rope_angles(seq_.d_pos(), T, freqs_[k].dev, (int)freqs_[k].f.size(), const_cast<float*>(cos_of((int)k)), const_cast<float*>(sin_of((int)k)), stream_));
    FP_OP(b200_embed_positions(seq_.d_ids(), nullptr, embed_, nullptr, x_, T, D, dt, stream_));
    FP_OP(b200_layernorm_pair(x_, nullptr, T, D, eps_, layers_[0].n1, nullptr, h_, nullptr, nullptr, nullptr, dt, stream_));
    for (size_t li = 0; li < layers_.size(); ++li) {
        FpLayer& L = layers_[li];
        const bool routed = L.ff_kind == kFfRouted;
        bool products_later = false;
        ExpertGroups eg{h_, T, L.top, L.experts, L.ff, B200_GG_GLU, group_off_, src_row_, L.w_up, L.w_down, gath_, act_, eo_};
        // ---- feed-forward, lane 1
        if (L.ff_kind != kFfNone) FP_TRY(fork(1, err));
        if (L.ff_kind == kFfDense) {
            FP_OP(gemm(h_, L.w_up, up_, B200_F32, T, L.ff, D, B200_GG_NONE, 0.f, 1));
            FP_OP(b200_poly_norm(up_, L.act, eps_, act_, T, L.ff, dt, lane(1)));
            FP_OP(gemm(act_, L.w_down, y3_, B200_F32, T, D, L.ff, B200_GG_NONE, 0.f, 1));
        } else if (routed) {
            FP_OP(b200_moe_route_groups(h_, dt, L.router, T, D, L.experts, L.top, L.groups, L.keep, chosen_, weight_, lane(1)));
            FP_OP(b200_moe_dispatch(chosen_, T, L.top, L.experts, group_off_, src_row_, dest_, lane(1)));
            products_later = experts_fit_streams(T, L.ff, true);
            if (products_later)
                FP_TRY(expert_rows(eg, 1, err));
            else {
                b200_gemm_grouped_args g{};
                g.A = h_; g.lda = D; g.a_rows = src_row_; g.group_off = group_off_;
                g.W = L.w_up; g.ldw = D; g.stride_w = (long long)2 * L.ff * D; g.trans_b = 1; g.epi = B200_GG_GLU;
                g.C = act_; g.ldc = L.ff;
                g.M = T; g.N = L.ff; g.K = D; g.batch = L.experts;   // an expert owns at most one row per token
                g.a_dtype = dt; g.w_dtype = dt; g.c_dtype = dt;
                FP_OP(b200_gemm_grouped(&g, lane(1)));
                b200_gemm_grouped_args d{};
                d.A = act_; d.lda = L.ff; d.group_off = group_off_;
                d.W = L.w_down; d.ldw = L.ff; d.stride_w = (long long)D * L.ff; d.trans_b = 1;
                d.C = eo_; d.ldc = D;
                d.M = T; d.N = D; d.K = L.ff; d.batch = L.experts;
                d.a_dtype = dt; d.w_dtype = dt; d.c_dtype = B200_F32;
                FP_OP(b200_gemm_grouped(&d, lane(1)));
            }
        }
        // ---- mixer, lane 0 (and 2)
        if (L.latent) {
            FP_TRY(latent_mixer(L, T, longest_entry, longest_context, err));
        } else {
            FP_OP(gemm(h_, L.w_in, proj_, B200_F32, T, L.n_in, D));
            FP_TRY(fork(2, err));
            FP_TRY(recurrent_side(L, T, longest_entry, err));
            FP_TRY(attention_side(L, T, longest_entry, longest_context, err));
            FP_TRY(join(2, err));
        }
        if (products_later) FP_TRY(expert_products(eg, 1, err));
        if (L.ff_kind != kFfNone) FP_TRY(join(1, err));
        // ---- both sublayers join the residual; h = what the next layer reads
        b200_parallel_residual_args ra{};
        ra.x = x_; ra.mult = mult_; ra.y1 = y_; ra.s1 = 1.f;
        if (!L.latent) { ra.w1 = L.at.out_norm; ra.y2 = y2_; ra.w2 = L.ss.out_norm; ra.s1 = ra.s2 = 0.5f; }
        if (L.ff_kind == kFfDense) ra.y3 = y3_;
        if (routed) { ra.expert_out = eo_; ra.dest = dest_; ra.weight = weight_; ra.top = L.top; }
        ra.ln_w = li + 1 < layers_.size() ? layers_[li + 1].n1 : nullptr;
        ra.eps = eps_; ra.out = h_; ra.out_dtype = dt; ra.n_rows = T; ra.width = D;
        FP_OP(b200_parallel_residual(&ra, stream_));
        keep_layer(li, x_, T);
    }
    if (W > 0) {
        FP_OP(b200_layernorm_pair(x_, seq_.d_want_rows(), W, D, eps_, fnw_, nullptr, hf_, nullptr, nullptr, nullptr, dt, stream_));
        FP_OP(gemm(hf_, head_, logits_, B200_F32, W, vocab_, D));
        if (want_ids) FP_OP(b200_argmax(logits_, ids_dev_, W, vocab_, B200_F32, stream_));
    }
    return B200_OK;
}

Model* make_filipel(const ModelDir& dir, const b200_model_options& opt, std::string& err) {
    Filipel* m = new Filipel();
    if (m->load(dir, opt, err) != B200_OK) {
        delete m;
        return nullptr;
    }
    return m;
}

FamilyRegistrar reg_filipel("Filipel", make_filipel);

}  // namespace
}  // namespace b200
