// Model family "Mazotar": a decoder whose residual is `streams` parallel rows per token with learned connections. Sublayer q of a
// layer (1: mixer, 2: feed-forward) reads u = sum_s in[s] x_s through an RMS norm and writes x_t <- sum_s mix[s, t] x_s + out[t] y
// into all streams at once; the streams start as equal copies of the scaled embedding plus fixed sinusoids and are summed at the
// end. Two kinds of mixer that config.json orders freely:
//   "attention"  grouped-query attention without rotation: one RMS norm over the whole query and the whole key projection, queries
//                multiplied by a temperature that grows with the logarithm of the position, a learned bias per bucket of the distance
//                (exact for short distances, logarithmic up to bias_max), a softmax with a learned sink per head. A layer with
//                "kv_from": j has no keys and values of its own and reads layer j's pages with its own queries, table and sink.
//   "mlstm"      a matrix memory with exponential input and sigmoid forget gates, stabilised by a running maximum; each head's output
//                RMS-normed, weighted and gated by sigmoid(W_g h).
// Feed-forward: none, a dense silu-gated one, or a routed mixture of such experts whose sigmoid weights multiply the experts' INPUT,
// beside a shared expert with a sigmoid gate per token.
//
// A step runs on the family-independent pieces of the library: StepRunner (streams and lanes, workspaces, graph replay of
// single-token steps, routed experts as dense products, results to the host), SequenceBatch / PagePool for slots, pages and the
// per-token tables, SlotState for what the memory carries, b200_linear_ex2 (tcgen05) and b200_gemm_grouped, b200_embed_streams,
// b200_hyper_residual, b200_qk_prepare (row norms, temperature), b200_paged_attention (distance bias, sink), b200_mlstm,
// b200_head_rms_gate, b200_moe_route_sigmoid / b200_moe_dispatch_weighted. The streams, all norms, angles, temperatures, scores and
// weights, the router, and the memory with its gates are fp32 in both serving dtypes; in B200_BF16 the GEMM operands and the cache
// pages are bfloat16.
//
// Launch order of a layer (T tokens of all entries packed):
//   attention: [q | k | v] = h W^T -> row norms, temperature, page stores -> attention over the pages -> W_o
//   mlstm:     [q | k | v | g | i | f] = h W^T -> memory -> head norm, weight, gate -> W_o
//   streams <- mixer output; h = N2 of the next weighted sum (one kernel)
//   lane 0: router (+ the shared expert's gate) -> counting sort -> gated up products per expert, rows scaled -> down products; or the
//   dense gated unit;  lane 1: the shared expert;  streams <- both; h = the next layer's N1 (one kernel)
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
constexpr int kStreamRows = 256;   // up to here a stacked [gate; up] streams once through the split-K GEMM
constexpr double kPi = 3.14159265358979323846;

struct MzConnect {   // one sublayer's connections to the streams
    float *w_in = nullptr, *w_out = nullptr, *mix = nullptr;
};
struct MzAttn {
    int heads = 0, kv_heads = 0, dim = 0, vdim = 0, kv_from = -1, bias_max = 0, dist_n = 0, temp_every = 0;
    float scale = 1.f, temp_coef = 0.f;
    float *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr, *dist_bias = nullptr;
    int nq() const { return heads * dim; }
    int nk() const { return kv_heads * dim; }
    int nv() const { return kv_heads * vdim; }
};
struct MzMemory {
    int heads = 0, dim = 0, vdim = 0;
    float cap = 1.f;
    float *i_bias = nullptr, *f_bias = nullptr, *norm = nullptr;
    int nq() const { return heads * dim; }
    int nv() const { return heads * vdim; }
    int v_off() const { return 2 * nq(); }
    int g_off() const { return v_off() + nv(); }
    int i_off() const { return g_off() + nv(); }
    int f_off() const { return i_off() + heads; }
};
enum { kFfNone = 0, kFfDense = 1, kFfRouted = 2 };

struct MzLayer {
    bool memory = false;
    MzAttn at;
    MzMemory me;
    int n_in = 0, n_mid = 0;                         // columns of the stacked input projection (whole groups of 8); inputs of W_o
    void *w_in = nullptr, *w_o = nullptr;
    float *n1 = nullptr, *n2 = nullptr;
    MzConnect hc1, hc2;
    int ff_kind = kFfNone, ff = 0, experts = 0, top = 0, shared_ff = 0;
    float* router = nullptr;                         // [experts (+ 1 with a shared expert: its gate), D]
    void *w_gu = nullptr, *w_down = nullptr;         // [2 ff, D] (gate rows first), [D, ff]; routed: one per expert, back to back
    void *s_gu = nullptr, *s_down = nullptr;
    void *k_pool = nullptr, *v_pool = nullptr;       // another layer's with kv_from
    SlotState state, norm_state;
};

class Mazotar : public StepRunner {
public:
    ~Mazotar() override {
        if (stream_) cudaStreamSynchronize(stream_);
        cudaFree(scratch_);
    }
    const char* family() const override { return "Mazotar"; }
    int layer_count() const override { return (int)layers_.size(); }
    int load(const ModelDir& dir, const b200_model_options& opt, std::string& err);

private:
    int parse(const Json& ls, std::string& err);
    int parse_attention(const Json& mx, int i, const std::string& where, MzLayer& L, std::string& err);
    int parse_memory(const Json& mx, const std::string& where, MzLayer& L, std::string& err);
    int parse_ff(const Json& ml, const std::string& where, MzLayer& L, std::string& err);
    int load_distance_bias(const SafeTensorsFile& st, const std::string& name, MzAttn& at, std::string& err);
    int ensure_scratch(int T, int W) override;
    int enqueue(int T, int W, int longest_entry, int longest_context, bool want_ids, std::string& err) override;
    int attention_mixer(MzLayer& L, int T, int longest_entry, int longest_context, std::string& err);
    int memory_mixer(MzLayer& L, int T, int longest_entry, std::string& err);
    int gated_unit(const void* w_gu, const void* w_down, int ff, int T, float* gu, void* act, float* out, int k, std::string& err);
    int feed_forward(MzLayer& L, int T, std::string& err);
    size_t step_workspace_bytes(int T, int n_entries) const override {
        size_t need = 0;
        for (const MzLayer& L : layers_)
            if (!L.memory) need = std::max(need, b200_paged_attention_workspace_bytes(T, L.at.heads, L.at.vdim));
            else if (dtype_ == B200_BF16) need = std::max(need, b200_mlstm_workspace_bytes(T, n_entries, L.me.heads, L.me.dim, L.me.vdim));
        return need;
    }

    float eps_ = 1e-6f, embed_scale_ = 1.f;
    int streams_ = 1;
    std::vector<MzLayer> layers_;
    void *embed_ = nullptr, *head_ = nullptr;
    float* fnw_ = nullptr;
    double* turns_ = nullptr;
    // scratch, grown to the largest step seen
    char* scratch_ = nullptr;
    int cap_T_ = 0, cap_W_ = 0;
    float *x_ = nullptr, *sum_ = nullptr, *proj_ = nullptr, *y_ = nullptr, *y2_ = nullptr, *mem_ = nullptr, *gu_ = nullptr, *gu2_ = nullptr, *eo_ = nullptr,
          *weight_ = nullptr, *row_weight_ = nullptr, *gate_ = nullptr;
    void *h_ = nullptr, *q_ = nullptr, *mid_ = nullptr, *act_ = nullptr, *act2_ = nullptr, *gath_ = nullptr, *hf_ = nullptr;
    int *chosen_ = nullptr, *group_off_ = nullptr, *src_row_ = nullptr, *dest_ = nullptr;
    // maxima over layers (scratch sizes)
    int max_in_ = 0, max_q_ = 0, max_mid_ = 0, max_mem_ = 0, max_dense_ = 0, max_shared_ = 0, max_act_ = 0, max_top_ = 0, max_experts_ = 0;
};

#define MZ_TRY(call)                    \
    do {                                \
        const int rc_ = (call);         \
        if (rc_ != B200_OK) return rc_; \
    } while (0)
#define MZ_OP(call)                                                             \
    do {                                                                        \
        const int rc_ = (call);                                                 \
        if (rc_ != B200_OK) { err = std::string(#call) + " failed (" + std::to_string(rc_) + ")"; return rc_; } \
    } while (0)

const Json* member(const Json& j, const char* name) {   // null counts as absent
    const Json* v = j.get(name);
    return v && !v->is_null() ? v : nullptr;
}

int Mazotar::parse_attention(const Json& mx, int i, const std::string& where, MzLayer& L, std::string& err) {
    MzAttn& at = L.at;
    at.heads = (int)mx.integer("heads", 0);
    at.kv_heads = (int)mx.integer("kv_heads", at.heads);
    at.dim = (int)mx.integer("dim", 0);
    at.vdim = (int)mx.integer("vdim", 0);
    at.bias_max = (int)mx.integer("bias_max", 0);
    if (at.heads < 1 || at.kv_heads < 1 || at.dim < 1 || at.vdim < 1 || at.bias_max < 1 || !mx.has("scale")) { err = where + "attention needs heads, kv_heads, dim, vdim, scale and bias_max"; return B200_EINVAL; }
    if (at.heads % at.kv_heads) { err = where + "heads must be a multiple of kv_heads"; return B200_EINVAL; }
    if (at.vdim > 256) { err = where + "vdim above 256 is not supported by the attention kernels"; return B200_EUNSUPPORTED; }
    at.scale = (float)mx.number("scale", 1.0);
    if (const Json* qt = member(mx, "q_temp")) {
        at.temp_every = (int)qt->integer("every", 0);
        at.temp_coef = (float)qt->number("coef", 0.0);
        if (at.temp_every < 1) { err = where + "q_temp.every must be positive"; return B200_EINVAL; }
    }
    if (member(mx, "kv_from")) {
        at.kv_from = (int)mx.integer("kv_from", -1);
        const MzLayer* src = at.kv_from >= 0 && at.kv_from < i ? &layers_[at.kv_from] : nullptr;
        if (!src || src->memory || src->at.kv_from >= 0) { err = where + "kv_from must name an earlier attention layer with keys and values of its own"; return B200_EINVAL; }
        if (src->at.kv_heads != at.kv_heads || src->at.dim != at.dim || src->at.vdim != at.vdim) { err = where + "kv_from: kv_heads, dim and vdim must equal the other layer's"; return B200_EINVAL; }
    }
    L.n_mid = at.heads * at.vdim;
    L.n_in = at.nq() + (at.kv_from < 0 ? at.nk() + at.nv() : 0);
    return B200_OK;
}

int Mazotar::parse_memory(const Json& mx, const std::string& where, MzLayer& L, std::string& err) {
    MzMemory& me = L.me;
    L.memory = true;
    me.heads = (int)mx.integer("heads", 0);
    me.dim = (int)mx.integer("dim", 0);
    me.vdim = (int)mx.integer("vdim", 0);
    me.cap = (float)mx.number("gate_cap", 0.0);
    if (me.heads < 1 || me.dim < 1 || me.vdim < 1 || !(me.cap > 0.f)) { err = where + "a matrix memory needs heads, dim, vdim and a positive gate_cap"; return B200_EINVAL; }
    if (me.dim > 512) { err = where + "dim above 512 is not supported by the memory kernels"; return B200_EUNSUPPORTED; }
    L.n_mid = me.nv();
    L.n_in = me.f_off() + me.heads;
    return B200_OK;
}

int Mazotar::parse_ff(const Json& ml, const std::string& where, MzLayer& L, std::string& err) {
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
        if (L.top > 16) { err = where + "more than 16 experts per token are not supported"; return B200_EUNSUPPORTED; }
        if (const Json* sh = member(ml, "shared")) {
            L.shared_ff = (int)sh->integer("ff", 0);
            if (L.shared_ff < 1) { err = where + "mlp.shared.ff is required"; return B200_EINVAL; }
        }
    } else {
        err = where + "feed-forward kind '" + kind + "' is not part of this family";
        return B200_EUNSUPPORTED;
    }
    return B200_OK;
}

// everything that can be refused from the configuration alone, before the first CUDA call
int Mazotar::parse(const Json& ls, std::string& err) {
    layers_.resize(ls.arr.size());
    for (size_t i = 0; i < ls.arr.size(); ++i) {
        const Json& lj = ls.arr[i];
        const std::string type = lj.text("type"), where = "layer " + std::to_string(i) + ": ";
        const Json* mx = member(lj, "mixer");
        if (!mx) { err = where + "no mixer"; return B200_EINVAL; }
        if (type == "attention") MZ_TRY(parse_attention(*mx, (int)i, where, layers_[i], err));
        else if (type == "mlstm") MZ_TRY(parse_memory(*mx, where, layers_[i], err));
        else { err = where + "mixer type '" + type + "' is not part of this family"; return B200_EUNSUPPORTED; }
        if (const Json* ml = member(lj, "mlp")) MZ_TRY(parse_ff(*ml, where, layers_[i], err));
    }
    return B200_OK;
}

// The checkpoint's table has a row per bucket of distances; the kernels read one number per distance and head up to the first
// distance of the last bucket. Bucket of n with B rows, h = B / 2: n below h, else min(B - 1, h + floor(ln(n / h) / ln(bias_max / h)
// (B - h))).
int Mazotar::load_distance_bias(const SafeTensorsFile& st, const std::string& name, MzAttn& at, std::string& err) {
    const SafeTensor* t = st.find(name);
    if (!t) { err = "tensor " + name + " is missing"; return B200_EINVAL; }
    if (t->shape.size() != 2 || t->shape[1] != at.heads || (t->dtype != "BF16" && t->dtype != "F32")) { err = "tensor " + name + " needs the shape [buckets, " + std::to_string(at.heads) + "]"; return B200_EINVAL; }
    const int B = (int)t->shape[0], half = B / 2;
    if (half < 1 || at.bias_max <= half) { err = "tensor " + name + ": at least two buckets, and bias_max above half of them, are needed"; return B200_EINVAL; }
    auto bucket = [&](int n) {
        if (n < half) return n;
        const double r = std::floor(std::log((double)n / half) / std::log((double)at.bias_max / half) * (B - half));
        return r >= B - half ? B - 1 : std::min(B - 1, half + (int)r);
    };
    int last = 0;
    while (bucket(last) < B - 1) ++last;
    at.dist_n = last + 1;
    std::vector<float> v((size_t)at.heads * at.dist_n);
    for (int h = 0; h < at.heads; ++h)
        for (int n = 0; n < at.dist_n; ++n) v[(size_t)h * at.dist_n + n] = st_value(*t, (size_t)bucket(n) * at.heads + h);
    at.dist_bias = (float*)dalloc(v.size() * 4);
    if (!at.dist_bias || cudaMemcpy(at.dist_bias, v.data(), v.size() * 4, cudaMemcpyHostToDevice) != cudaSuccess) { err = "out of device memory"; return B200_ENOMEM; }
    return B200_OK;
}

int Mazotar::load(const ModelDir& dir, const b200_model_options& opt, std::string& err) {
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
    if (const Json* em = member(c, "embedding")) embed_scale_ = (float)em->number("scale", 1.0);
    streams_ = (int)c.integer("streams", 1);
    if (streams_ < 1) { err = "streams must be positive"; return B200_EINVAL; }
    if (streams_ > 16) { err = "more than 16 streams are not supported"; return B200_EUNSUPPORTED; }
    if (opt.max_tokens < 1 || opt.max_slots < 1) { err = "max_tokens and max_slots must be positive"; return B200_EINVAL; }
    MZ_TRY(parse(*ls, err));

    MZ_TRY(init_runner(err));
    SafeTensorsFile st;
    if (!st.open(dir.path + "/model.safetensors", err)) return B200_EINVAL;
    // the design has no position limit of its own: a sequence can grow as long as the pool has pages
    const int n_pages = (opt.max_tokens + kPageRows - 1) / kPageRows;
    MZ_TRY(seq_.init(opt.max_tokens, kPageRows, opt.max_slots, n_pages * kPageRows, err));

    const size_t E = esz();
    const long long D = D_;
    auto f32 = [&](const std::string& name, std::vector<long long> shape, float*& dst) -> int {
        size_t cnt = 1;
        for (long long d : shape) cnt *= (size_t)d;
        dst = (float*)dalloc(cnt * 4);
        if (!dst) { err = "out of device memory"; return B200_ENOMEM; }
        return upload_tensor(st, name, shape, true, dtype_, dst, err);
    };
    // checkpoint matrices that read the same input (or the experts of one layer), stacked row-wise into one operand; `pad_to`: zero
    // rows behind them
    auto stacked = [&](const std::vector<std::pair<std::string, long long>>& parts, long long cols, void*& dst, long long pad_to = 0) -> int {
        long long rows = 0;
        for (auto& p : parts) rows += p.second;
        const size_t total = (size_t)std::max(rows, pad_to) * cols * E;
        dst = dalloc(total);
        if (!dst) { err = "out of device memory"; return B200_ENOMEM; }
        if (pad_to > rows) cudaMemset((char*)dst + (size_t)rows * cols * E, 0, total - (size_t)rows * cols * E);
        long long at = 0;
        for (auto& p : parts) {
            MZ_TRY(upload_tensor(st, p.first, {p.second, cols}, false, dtype_, (char*)dst + (size_t)at * cols * E, err));
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
    auto connect = [&](const std::string& pre, MzConnect& hc) -> int {
        MZ_TRY(f32(pre + "in", {streams_}, hc.w_in));
        MZ_TRY(f32(pre + "out", {streams_}, hc.w_out));
        return f32(pre + "mix", {streams_, streams_}, hc.mix);
    };
    {   // angle of one position over pi, per pair of columns
        std::vector<double> turns((D_ + 1) / 2);
        for (size_t i = 0; i < turns.size(); ++i) turns[i] = std::pow(10000.0, -2.0 * (double)i / D_) / kPi;
        turns_ = (double*)dalloc(turns.size() * sizeof(double));
        if (!turns_ || cudaMemcpy(turns_, turns.data(), turns.size() * sizeof(double), cudaMemcpyHostToDevice) != cudaSuccess) { err = "out of device memory"; return B200_ENOMEM; }
    }
    MZ_TRY(mat("embed", vocab_, D, embed_));
    MZ_TRY(mat("head", vocab_, D, head_));
    MZ_TRY(f32("final.norm", {D}, fnw_));
    for (size_t i = 0; i < layers_.size(); ++i) {
        MzLayer& L = layers_[i];
        const std::string pre = "l" + std::to_string(i) + ".", mp = pre + "mix.";
        MZ_TRY(f32(pre + "norm1", {D}, L.n1));
        MZ_TRY(connect(pre + "hc1.", L.hc1));
        std::vector<std::pair<std::string, long long>> parts;
        if (L.memory) {
            const MzMemory& me = L.me;
            parts = {{mp + "q", me.nq()}, {mp + "k", me.nq()}, {mp + "v", me.nv()}, {mp + "g", me.nv()}, {mp + "i", me.heads}, {mp + "f", me.heads}};
            MZ_TRY(f32(mp + "i.b", {me.heads}, L.me.i_bias));
            MZ_TRY(f32(mp + "f.b", {me.heads}, L.me.f_bias));
            MZ_TRY(f32(mp + "norm", {me.nv()}, L.me.norm));
            cudaError_t e = L.state.init(opt.max_slots, (size_t)me.heads * me.dim * me.vdim);
            if (e == cudaSuccess) e = L.norm_state.init(opt.max_slots, (size_t)me.heads * b200_mlstm_norm_floats(me.dim, me.vdim));
            if (e != cudaSuccess) { err = "out of device memory (carried state)"; return B200_ENOMEM; }
            max_mem_ = std::max(max_mem_, me.nv());
        } else {
            const MzAttn& at = L.at;
            parts = {{mp + "q", at.nq()}};
            MZ_TRY(f32(mp + "q.norm", {at.nq()}, L.at.q_norm));
            if (at.kv_from < 0) {
                parts.push_back({mp + "k", at.nk()});
                parts.push_back({mp + "v", at.nv()});
                MZ_TRY(f32(mp + "k.norm", {at.nk()}, L.at.k_norm));
                MZ_TRY(pages(at.nk(), L.k_pool));
                MZ_TRY(pages(at.nv(), L.v_pool));
            } else {
                L.k_pool = layers_[at.kv_from].k_pool;
                L.v_pool = layers_[at.kv_from].v_pool;
            }
            MZ_TRY(f32(mp + "sink", {at.heads}, L.at.sink));
            MZ_TRY(load_distance_bias(st, mp + "rel", L.at, err));
            max_q_ = std::max(max_q_, at.nq());
        }
        L.n_in = (L.n_in + 7) & ~7;   // rows of the projection stay on 16-byte boundaries
        MZ_TRY(stacked(parts, D, L.w_in, L.n_in));
        MZ_TRY(mat(mp + "o", D, L.n_mid, L.w_o));
        max_in_ = std::max(max_in_, L.n_in);
        max_mid_ = std::max(max_mid_, L.n_mid);
        if (L.ff_kind == kFfNone) continue;
        MZ_TRY(f32(pre + "norm2", {D}, L.n2));
        MZ_TRY(connect(pre + "hc2.", L.hc2));
        const std::string fp = pre + "mlp.";
        if (L.ff_kind == kFfDense) {
            MZ_TRY(stacked({{fp + "gate", L.ff}, {fp + "up", L.ff}}, D, L.w_gu));
            MZ_TRY(mat(fp + "down", D, L.ff, L.w_down));
            max_dense_ = std::max(max_dense_, L.ff);
            max_act_ = std::max(max_act_, L.ff);
            continue;
        }
        std::vector<std::pair<std::string, long long>> ups, downs;
        for (int e = 0; e < L.experts; ++e) {
            const std::string ep = fp + "e" + std::to_string(e) + ".";
            ups.push_back({ep + "gate", L.ff});
            ups.push_back({ep + "up", L.ff});
            downs.push_back({ep + "down", D});
        }
        MZ_TRY(stacked(ups, D, L.w_gu));
        MZ_TRY(stacked(downs, L.ff, L.w_down));
        const int n_gates = L.shared_ff > 0 ? 1 : 0;
        L.router = (float*)dalloc((size_t)(L.experts + n_gates) * D * 4);
        if (!L.router) { err = "out of device memory"; return B200_ENOMEM; }
        MZ_TRY(upload_tensor(st, fp + "router", {L.experts, D}, true, dtype_, L.router, err));
        if (n_gates) {
            MZ_TRY(upload_tensor(st, fp + "shared.sg", {1, D}, true, dtype_, L.router + (size_t)L.experts * D, err));
            MZ_TRY(stacked({{fp + "shared.gate", L.shared_ff}, {fp + "shared.up", L.shared_ff}}, D, L.s_gu));
            MZ_TRY(mat(fp + "shared.down", D, L.shared_ff, L.s_down));
            max_shared_ = std::max(max_shared_, L.shared_ff);
        }
        max_act_ = std::max(max_act_, L.top * L.ff);
        max_top_ = std::max(max_top_, L.top);
        max_experts_ = std::max(max_experts_, L.experts);
    }
    if (cudaDeviceSynchronize() != cudaSuccess) { err = "weight upload failed"; return B200_EINVAL; }
    return B200_OK;
}

int Mazotar::ensure_scratch(int T, int W) {
    if (T <= cap_T_ && W <= cap_W_) return B200_OK;
    const int cT = std::max(T, cap_T_), cW = std::max(W, cap_W_);
    cudaStreamSynchronize(stream_);
    buffers_moved();
    cudaFree(scratch_);
    scratch_ = nullptr;
    cap_T_ = cap_W_ = 0;
    auto al = [](size_t b) { return (std::max<size_t>(b, 1) + 255) & ~(size_t)255; };
    const size_t E = esz(), t = (size_t)cT, top = (size_t)std::max(1, max_top_), routed = max_top_ > 0, few = std::min(cT, kStreamRows);
    const size_t sizes[] = {
        al(t * streams_ * D_ * 4),                 // x
        al(t * D_ * 4),                            // sum
        al(t * max_in_ * 4),                       // proj
        al(t * D_ * 4),                            // y
        al(t * D_ * 4),                            // y2
        al(t * max_mem_ * 4),                      // mem
        al(few * 2 * max_dense_ * 4),              // gu
        al(few * 2 * max_shared_ * 4),             // gu2
        al(routed * t * top * D_ * 4),             // eo
        al(t * top * 4),                           // weight
        al(t * top * 4),                           // row_weight
        al(t * 4),                                 // gate
        al((size_t)cW * vocab_ * 4),               // logits
        al(t * D_ * E),                            // h
        al(t * max_q_ * E),                        // q
        al(t * max_mid_ * E),                      // mid
        al(t * max_act_ * E),                      // act
        al(t * max_shared_ * E),                   // act2
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
    take(x_); take(sum_); take(proj_); take(y_); take(y2_); take(mem_); take(gu_); take(gu2_); take(eo_); take(weight_); take(row_weight_); take(gate_);
    take(logits_);
    take(h_); take(q_); take(mid_); take(act_); take(act2_); take(gath_); take(hf_);
    take(chosen_); take(group_off_); take(src_row_); take(dest_); take(ids_dev_);
    cap_T_ = cT;
    cap_W_ = cW;
    return ensure_logits_host(cW);
}

int Mazotar::attention_mixer(MzLayer& L, int T, int longest_entry, int longest_context, std::string& err) {
    const MzAttn& at = L.at;
    const int dt = dtype_;
    const bool own = at.kv_from < 0;
    MZ_OP(gemm(h_, L.w_in, proj_, B200_F32, T, L.n_in, D_));
    b200_qk_prepare_args qa{};
    qa.proj = proj_; qa.ld_proj = L.n_in;
    qa.norm_rows = 1; qa.q_norm = at.q_norm; qa.k_norm = own ? at.k_norm : nullptr; qa.eps = eps_;
    qa.temp_coef = at.temp_coef; qa.temp_every = at.temp_every;
    qa.q_out = q_; qa.k_pool = own ? L.k_pool : nullptr; qa.v_pool = own ? L.v_pool : nullptr;
    qa.pages = seq_.pool.device(); qa.max_pages = seq_.pool.max_pages(); qa.page_rows = kPageRows;
    qa.slot = seq_.d_slot(); qa.pos = seq_.d_pos(); qa.start = seq_.d_start();
    qa.n_tokens = T; qa.heads = at.heads; qa.kv_heads = at.kv_heads; qa.dim = at.dim; qa.dtype = dt;
    if (own) { qa.v_heads = at.kv_heads; qa.vdim = at.vdim; qa.v_off = at.nq() + at.nk(); }
    MZ_OP(b200_qk_prepare(&qa, stream_));
    b200_paged_attention_args pa{};
    pa.q = q_; pa.out = mid_; pa.k_pool = L.k_pool; pa.v_pool = L.v_pool;
    pa.pages = qa.pages; pa.max_pages = qa.max_pages; pa.page_rows = kPageRows;
    pa.slot = seq_.d_slot(); pa.pos = seq_.d_pos();
    pa.n_tokens = T; pa.heads = at.heads; pa.kv_heads = at.kv_heads; pa.dim = at.dim; pa.vdim = at.vdim;
    pa.scale = at.scale; pa.dtype = dt; pa.longest_entry = longest_entry; pa.longest_context = longest_context;
    pa.workspace = attn_ws_; pa.workspace_bytes = attn_ws_bytes_;
    pa.sink = at.sink; pa.dist_bias = at.dist_bias; pa.dist_n = at.dist_n;
    MZ_OP(b200_paged_attention(&pa, stream_));
    MZ_OP(gemm(mid_, L.w_o, y_, B200_F32, T, D_, L.n_mid));
    return B200_OK;
}

int Mazotar::memory_mixer(MzLayer& L, int T, int longest_entry, std::string& err) {
    const MzMemory& me = L.me;
    MZ_OP(gemm(h_, L.w_in, proj_, B200_F32, T, L.n_in, D_));
    b200_mlstm_args ma{};
    ma.proj = proj_; ma.ld_proj = L.n_in; ma.q_off = 0; ma.k_off = me.nq(); ma.v_off = me.v_off(); ma.i_off = me.i_off(); ma.f_off = me.f_off();
    ma.i_bias = me.i_bias; ma.f_bias = me.f_bias; ma.gate_cap = me.cap; ma.q_scale = (float)(1.0 / std::sqrt((double)me.dim));
    ma.state = L.state.data(); ma.norm = L.norm_state.data(); ma.out = mem_;
    ma.ent_row = seq_.d_ent_row(); ma.ent_len = seq_.d_ent_len(); ma.slot = seq_.d_slot(); ma.pos = seq_.d_pos();
    ma.n_entries = seq_.n_entries; ma.n_tokens = T; ma.heads = me.heads; ma.dim = me.dim; ma.vdim = me.vdim;
    ma.longest_entry = longest_entry; ma.chunked = dtype_ == B200_BF16;
    ma.workspace = attn_ws_; ma.workspace_bytes = attn_ws_bytes_;
    MZ_OP(b200_mlstm(&ma, stream_));
    MZ_OP(b200_head_rms_gate(mem_, proj_ + me.g_off(), L.n_in, me.norm, 1, mid_, T, me.heads, me.vdim, eps_, dtype_, stream_));
    MZ_OP(gemm(mid_, L.w_o, y_, B200_F32, T, D_, L.n_mid));
    return B200_OK;
}

// out = W_down (silu(W_gate h) * (W_up h)) on lane k
int Mazotar::gated_unit(const void* w_gu, const void* w_down, int ff, int T, float* gu, void* act, float* out, int k, std::string& err) {
    if (dtype_ == B200_BF16 && T <= kStreamRows) {   // few rows: the stacked [gate; up] streams once through the split-K GEMM
        MZ_OP(gemm(h_, w_gu, gu, B200_F32, T, 2 * ff, D_, B200_GG_NONE, 0.f, k));
        MZ_OP(b200_glu_act(gu, act, T, ff, B200_GG_GLU, dtype_, lane(k)));
    } else
        MZ_OP(gemm(h_, w_gu, act, dtype_, T, ff, D_, B200_GG_GLU, 0.f, k));
    MZ_OP(gemm(act, w_down, out, B200_F32, T, D_, ff, B200_GG_NONE, 0.f, k));
    return B200_OK;
}

int Mazotar::feed_forward(MzLayer& L, int T, std::string& err) {
    const int D = D_, dt = dtype_;
    if (L.ff_kind == kFfDense) return gated_unit(L.w_gu, L.w_down, L.ff, T, gu_, act_, y_, 0, err);
    const bool shared = L.shared_ff > 0;
    if (shared) {
        MZ_TRY(fork(1, err));
        MZ_TRY(gated_unit(L.s_gu, L.s_down, L.shared_ff, T, gu2_, act2_, y2_, 1, err));
    }
    MZ_OP(b200_moe_route_sigmoid(h_, dt, L.router, T, D, L.experts, L.top, shared ? 1 : 0, chosen_, weight_, shared ? gate_ : nullptr, stream_));
    MZ_OP(b200_moe_dispatch_weighted(chosen_, weight_, T, L.top, L.experts, group_off_, src_row_, dest_, row_weight_, stream_));
    if (experts_fit_streams(T, L.ff, true)) {
        const ExpertGroups eg{h_, T, L.top, L.experts, L.ff, B200_GG_GLU, group_off_, src_row_, L.w_gu, L.w_down, gath_, act_, eo_, row_weight_};
        MZ_TRY(expert_rows(eg, 0, err));
        MZ_TRY(expert_products(eg, 0, err));
    } else {
        b200_gemm_grouped_args g{};
        g.A = h_; g.lda = D; g.a_rows = src_row_; g.group_off = group_off_; g.row_scale = row_weight_;
        g.W = L.w_gu; g.ldw = D; g.stride_w = (long long)2 * L.ff * D; g.trans_b = 1; g.epi = B200_GG_GLU;
        g.C = act_; g.ldc = L.ff;
        g.M = T; g.N = L.ff; g.K = D; g.batch = L.experts;   // an expert owns at most one row per token
        g.a_dtype = dt; g.w_dtype = dt; g.c_dtype = dt;
        MZ_OP(b200_gemm_grouped(&g, stream_));
        b200_gemm_grouped_args d{};
        d.A = act_; d.lda = L.ff; d.group_off = group_off_;
        d.W = L.w_down; d.ldw = L.ff; d.stride_w = (long long)D * L.ff; d.trans_b = 1;
        d.C = eo_; d.ldc = D;
        d.M = T; d.N = D; d.K = L.ff; d.batch = L.experts;
        d.a_dtype = dt; d.w_dtype = dt; d.c_dtype = B200_F32;
        MZ_OP(b200_gemm_grouped(&d, stream_));
    }
    if (shared) MZ_TRY(join(1, err));
    return B200_OK;
}

// every launch of a step, in order, on stream_ and the lane beside it (no allocation; prompt steps wait for the sizes of the expert
// groups, single-token steps for nothing: capturable into a graph)
int Mazotar::enqueue(int T, int W, int longest_entry, int longest_context, bool want_ids, std::string& err) {
    const int D = D_, dt = dtype_;
    // the boundary behind a sublayer (done: its connections; NULL before the first one) and in front of the next (reads: its
    // connections and norm; nw NULL: nobody reads yet)
    auto boundary = [&](const MzConnect* done, const MzLayer* routed, const MzConnect* reads, const float* nw) -> int {
        b200_hyper_residual_args a{};
        a.x = x_; a.streams = streams_;
        if (done) {
            a.mix = done->mix; a.w_out = done->w_out;
            if (routed) {
                a.expert_out = eo_; a.dest = dest_; a.top = routed->top;
                if (routed->shared_ff > 0) { a.y2 = y2_; a.gate2 = gate_; }
            } else
                a.y1 = y_;
        }
        if (reads) a.w_in = reads->w_in;
        a.w = nw; a.eps = eps_; a.out = h_; a.out_dtype = dt;
        a.n_rows = T; a.width = D;
        return b200_hyper_residual(&a, stream_);
    };
    MZ_OP(b200_embed_streams(seq_.d_ids(), seq_.d_pos(), embed_, embed_scale_, turns_, x_, streams_, T, D, dt, stream_));
    MZ_OP(boundary(nullptr, nullptr, &layers_[0].hc1, layers_[0].n1));
    for (size_t li = 0; li < layers_.size(); ++li) {
        MzLayer& L = layers_[li];
        const MzLayer* next = li + 1 < layers_.size() ? &layers_[li + 1] : nullptr;
        if (L.memory) MZ_TRY(memory_mixer(L, T, longest_entry, err));
        else MZ_TRY(attention_mixer(L, T, longest_entry, longest_context, err));
        const MzConnect* after = next ? &next->hc1 : nullptr;
        const float* after_norm = next ? next->n1 : nullptr;
        if (L.ff_kind == kFfNone) {
            MZ_OP(boundary(&L.hc1, nullptr, after, after_norm));
        } else {
            MZ_OP(boundary(&L.hc1, nullptr, &L.hc2, L.n2));
            MZ_TRY(feed_forward(L, T, err));
            MZ_OP(boundary(&L.hc2, L.ff_kind == kFfRouted ? &L : nullptr, after, after_norm));
        }
        if (capture_on_) {   // the residual of a layer is the sum of its streams
            b200_hyper_residual_args a{};
            a.x = x_; a.streams = streams_; a.sum_out = sum_; a.n_rows = T; a.width = D;
            MZ_OP(b200_hyper_residual(&a, stream_));
            keep_layer(li, sum_, T);
        }
    }
    if (W > 0) {
        b200_hyper_residual_args a{};
        a.x = x_; a.streams = streams_; a.rows = seq_.d_want_rows(); a.w = fnw_; a.eps = eps_; a.out = hf_; a.out_dtype = dt; a.n_rows = W; a.width = D;
        MZ_OP(b200_hyper_residual(&a, stream_));
        MZ_OP(gemm(hf_, head_, logits_, B200_F32, W, vocab_, D));
        if (want_ids) MZ_OP(b200_argmax(logits_, ids_dev_, W, vocab_, B200_F32, stream_));
    }
    return B200_OK;
}

Model* make_mazotar(const ModelDir& dir, const b200_model_options& opt, std::string& err) {
    Mazotar* m = new Mazotar();
    if (m->load(dir, opt, err) != B200_OK) {
        delete m;
        return nullptr;
    }
    return m;
}

FamilyRegistrar reg_mazotar("Mazotar", make_mazotar);

}  // namespace
}  // namespace b200
