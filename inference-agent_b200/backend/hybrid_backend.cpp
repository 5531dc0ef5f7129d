// Decoder-only models whose layers are listed one by one in their configuration, each with a mixer of its own kind -
// recurrent, attention, or several side by side - and an optional gated feed-forward ("Besudra" and designs like it).
//
// Reading guide.
//   Mixer           one kind of sequence mixer: its weights, its per-sequence state, its launches. A new kind is a class
//                   here plus a line in make_mixer().
//   LayerOps        what every mixer is written in: projections (with the RMS norm of their input or the residual add of
//                   their output folded in), scratch activations, weight upload. It picks the kernel by the number of
//                   tokens: weight-streaming GEMV for one token, tcgen05 GEMM for more (f32 kernels in the 32-bit form).
//   HybridBackend   the step: one ragged batch of portions of several sequences, state slots and cache pages, logits.
//
// Precision. Weights are bf16. In the 16-bit form the tensor-core products take bf16 activations (a hi + lo pair where the
// product feeds a recurrence's gates or step sizes, and in small batches) and accumulate in f32; everything between products - residual stream,
// norms, scores and softmax, gates, recurrent states - is f32, and single tokens multiply f32 activations. In the f32 form
// every product is f32 FMA on widened weights and the attention cache is f32.
//
// Padding. Every vector is stored with a length that is a multiple of 8 (heads and gate blocks each padded on their own):
// padded weight rows and columns are zero, so padded activations are zero and only means need the true count.
#include <cuda_runtime.h>

#include <algorithm>
#include <cmath>
#include <cstdio>
#include <cstdlib>
#include <cstring>
#include <map>
#include <memory>
#include <string>
#include <vector>

#include "block_pool.h"
#include "cuda_util.h"
#include "ingot_cuda.h"
#include "model_registry.h"
#include "weight_streamer.h"

extern "C" {
cudaError_t ingot_support_embed_rows_bf16(float* out, const void* table, int n_in, int n_rows_table, const int32_t* rows_dev, int n_rows,
                                          int* status_dev, cudaStream_t s);
cudaError_t ingot_support_rmsnorm_rows(float* out, const float* x, const float* w, const int32_t* rows_dev, int n_rows, int n, int n_mean,
                                       float eps, cudaStream_t s);
cudaError_t ingot_support_linear_bf16(float* out, const void* w, const float* x, int x_ld, int n_in, int n_out, int rows_per_block,
                                      int n_tok, int accumulate, cudaStream_t s);
cudaError_t ingot_support_gemv_bf16(float* out, const void* w, int n_out, int n_in, const float* x, const float* norm_w, float eps, int n_mean,
                                    int gated, int act, int accumulate, cudaStream_t s);
cudaError_t ingot_support_gated_act(float* out, const float* in, int n_rows, int n, int act, cudaStream_t s);
struct ingot_linear_ws;
cudaError_t ingot_linear_ws_create_bf16(ingot_linear_ws** out, int max_tok, int max_in, int max_out);
void ingot_linear_ws_destroy(ingot_linear_ws* ws);
int* ingot_linear_ws_status_dev(ingot_linear_ws* ws);
void ingot_linear_ws_planes(ingot_linear_ws* ws, void** hi, void** lo);
cudaError_t ingot_linear_tc_prepared(ingot_linear_ws* ws, int n_in, int n_tok, int planes);
cudaError_t ingot_linear_tc_prepare_bf16(ingot_linear_ws* ws, const float* x, int x_ld, int n_in, int n_tok, int planes, cudaStream_t s);
cudaError_t ingot_linear_tc_prepare_norm_bf16(ingot_linear_ws* ws, const float* x, const float* norm_w, float eps, int n_in, int n_mean, int n_tok,
                                              int planes, cudaStream_t s);
cudaError_t ingot_linear_tc_run(ingot_linear_ws* ws, float* out, const void* w, int n_in, int n_out, int accumulate, cudaStream_t s);
cudaError_t ingot_linear_tc_run_blocks(ingot_linear_ws* ws, float* out, const void* w, int k_block, int n_out, int rows_per_block, cudaStream_t s);
cudaError_t ingot_linear_tc_run_partial(ingot_linear_ws* ws, const void* w, int n_in, int n_out, int slot, cudaStream_t s);
cudaError_t ingot_linear_tc_finish_residual_norm_bf16(ingot_linear_ws* ws, float* x, const float* norm_w, float eps, int n_mean, int planes,
                                                      cudaStream_t s);
cudaError_t ingot_linear_tc_finish_gated_bf16(ingot_linear_ws* ws, int act, int planes, cudaStream_t s);
}

namespace {

constexpr int kMinTcTokens = 2;  // from two tokens on, a 128-token tile that is mostly padding still only streams the weights once

// Up to this many tokens a product is bound by streaming the weights, so the activations go in as a hi + lo pair at no cost: a
// decoded token's logits then hardly depend on whether it is alone (f32 activations) or in a batch.
constexpr int kPairTokens = 64;

int round_up(int v, int q) { return (v + q - 1) / q * q; }

int get_int(const Json& j, const char* key, int lo = 1, int hi = 1 << 28) {
    const int64_t v = j.at(key).integer();
    if (v < lo || v > hi) throw std::runtime_error(std::string("model config: \"") + key + "\" is out of range");
    return int(v);
}
float get_float(const Json& j, const char* key) { return float(j.at(key).number()); }

// A dimension of n groups of `size` values, each stored with `padded` places.
struct Groups {
    int n, size, padded;
    int count() const { return n * size; }
    int width() const { return n * padded; }
};
Groups flat(int size) { return {1, size, round_up(size, 8)}; }

// A bf16 matrix on the device, [n_out][n_in] row-major, both padded. rows_per_block > 0: block-diagonal, n_in per block.
struct Matrix {
    void* data = nullptr;
    int n_out = 0, n_in = 0, rows_per_block = 0;
    const void* rows_from(int r) const { return static_cast<const char*>(data) + size_t(r) * n_in * 2; }
};

// One tensor's place in a matrix: its logical rows (from row src_row0 on) and columns go to r0 + row groups, c0 + column groups.
struct Part {
    std::string name;
    std::vector<int64_t> shape;
    Groups rows, cols;
    int r0 = 0, c0 = 0, src_row0 = 0;
};

enum Buf { kProj, kConv, kStateIn, kDt, kGates, kMix, kGateUp, kMid, kNormed, kQuery, kBufCount };

// The step as the launches see it.
struct StepCtx {
    ingot_step st = {};
    ingot_scan_plan scan = {}, lru = {};
    bool tc = false;  // products on the tensor cores (16-bit form, more than one token)
    int planes = 1;   // bf16 planes an activation is given as there
};

// Shared-row attention caches of equal shape live in one handle with one page pool.
struct CacheGroup {
    int kv_heads, dim, chunk, n_layer = 0;
    ingot_skv* kv = nullptr;
    BlockPool pool;
    int pages_per_chunk = 0;
    const int32_t *tables = nullptr, *first_page = nullptr;  // device, of the current step
    int width = 0;
    int page(int pos) const { return ingot_skv_pages(chunk, pos + 1) - 1; }
    int first_visible(int pos) const { return chunk > 0 ? pos / chunk * chunk : 0; }
};

class LayerOps {
public:
    LayerOps(const ModelDir& dir, const EngineOptions& opt, int max_step) : dir(dir), opt(opt), max_step(max_step) {
        cuda_check(cudaStreamCreateWithFlags(&stream, cudaStreamNonBlocking), "cudaStreamCreate");
    }
    ~LayerOps() {
        cudaStreamSynchronize(stream);
        ingot_linear_ws_destroy(ws);
        for (void* p : allocs_) cudaFree(p);
        cudaStreamDestroy(stream);
    }

    // ---- construction ----
    void* alloc(size_t bytes, bool zero = false) {
        void* p = nullptr;
        cuda_check(cudaMalloc(&p, std::max<size_t>(bytes, 16)), "cudaMalloc");
        allocs_.push_back(p);
        if (zero) cuda_check(cudaMemset(p, 0, std::max<size_t>(bytes, 16)), "cudaMemset");
        return p;
    }
    void need(Buf b, int columns) { columns_[b] = std::max(columns_[b], columns); }
    void tc_shape(int n_in, int n_out) { tc_in_ = std::max(tc_in_, n_in); tc_out_ = std::max(tc_out_, n_out); }
    void allocate() {
        for (int b = 0; b < kBufCount; b++) bufs_[b] = columns_[b] ? static_cast<float*>(alloc(size_t(max_step) * columns_[b] * 4, true)) : nullptr;
        if (!opt.f32 && max_step >= kMinTcTokens) cuda_check(ingot_linear_ws_create_bf16(&ws, max_step, tc_in_, tc_out_), "linear workspace");
        loader_.finish();
        cuda_check(cudaDeviceSynchronize(), "model upload");
    }
    float* upload(const std::vector<float>& v) {
        float* d = static_cast<float*>(alloc(v.size() * 4));
        cuda_check(cudaMemcpy(d, v.data(), v.size() * 4, cudaMemcpyHostToDevice), "cudaMemcpy");
        return d;
    }
    // A vector tensor with each group padded with zeros.
    std::vector<float> host_vector(const std::string& name, const std::vector<int64_t>& shape, Groups g) {
        const std::vector<float> v = tensor_f32(dir.tensor(name, shape));
        if (int(v.size()) != g.count()) throw std::runtime_error("model: tensor " + name + " does not have " + std::to_string(g.count()) + " values");
        std::vector<float> out(size_t(g.width()), 0.f);
        for (int i = 0; i < g.n; i++) std::copy(v.begin() + i * g.size, v.begin() + (i + 1) * g.size, out.begin() + i * g.padded);
        return out;
    }
    float* vector(const std::string& name, const std::vector<int64_t>& shape, Groups g) { return upload(host_vector(name, shape, g)); }
    float* vector(const std::string& name, int n) { return vector(name, {n}, flat(n)); }
    Matrix matrix(int n_out, int n_in, const std::vector<Part>& parts, int rows_per_block = 0) {
        std::vector<uint16_t> host(size_t(n_out) * n_in, 0);
        for (const Part& p : parts) {
            const TensorView& t = dir.tensor(p.name, p.shape);
            if (t.dtype != "BF16") throw std::runtime_error("model: tensor " + p.name + " has type " + t.dtype + ", expected BF16");
            if (t.elems() < int64_t(p.src_row0 + p.rows.count()) * p.cols.count() || t.elems() % p.cols.count() != 0)
                throw std::runtime_error("model: tensor " + p.name + " has an unexpected size");
            const int nr = p.rows.count();
            for (int r = 0; r < nr; r++) {
                uint16_t* dst = host.data() + size_t(p.r0 + r / p.rows.size * p.rows.padded + r % p.rows.size) * n_in + p.c0;
                const unsigned char* src = t.data + size_t(p.src_row0 + r) * p.cols.count() * 2;
                for (int g = 0; g < p.cols.n; g++) memcpy(dst + g * p.cols.padded, src + size_t(g) * p.cols.size * 2, size_t(p.cols.size) * 2);
            }
        }
        Matrix m;
        m.n_out = n_out;
        m.n_in = n_in;
        m.rows_per_block = rows_per_block;
        m.data = alloc(host.size() * 2);
        loader_.copy(m.data, host.data(), host.size() * 2);
        weight_bytes += host.size() * 2;
        tc_shape(rows_per_block > 0 ? n_in * (n_out / rows_per_block) : n_in, n_out);
        return m;
    }
    Matrix matrix(const std::string& name, Groups rows, Groups cols) {
        return matrix(rows.width(), cols.width(), {Part{name, {rows.count(), cols.count()}, rows, cols}});
    }

    // ---- the step ----
    float* buf(Buf b) const { return bufs_[b]; }
    // Output of a kernel that feeds a product: the operand planes on the tensor-core path (and f32 rows if `keep`), else f32.
    ingot_act_out operand(const StepCtx& s, float* f32, int ld, bool keep, int planes = 0) const {
        ingot_act_out o = {};
        o.ld = ld;
        if (!s.tc || keep) o.f32 = f32;
        if (s.tc) {
            ingot_linear_ws_planes(ws, &o.hi, &o.lo);
            if (std::max(planes, s.planes) < 2) o.lo = nullptr;
        }
        return o;
    }
    void operand_ready(const StepCtx& s, int n_in, int planes = 0) const {
        if (s.tc) cuda_check(ingot_linear_tc_prepared(ws, n_in, s.st.n_tok, std::max(planes, s.planes)), "operand");
    }
    static bool streams(const Matrix& w) { return w.n_in % 256 == 0 && w.n_in <= 12032 && w.rows_per_block == 0; }

    // out [n_tok][w.n_out] = W rmsnorm(x)
    void norm_project(const StepCtx& s, float* out, const Matrix& w, const float* norm) {
        if (s.tc) {
            prepare_norm(s, w, norm);
            cuda_check(ingot_linear_tc_run(ws, out, w.data, w.n_in, w.n_out, 0, stream), "projection");
        } else if (s.st.n_tok == 1 && streams(w)) {
            cuda_check(ingot_support_gemv_bf16(out, w.data, w.n_out, w.n_in, x, norm, eps, width, 0, 0, 0, stream), "projection");
        } else {
            norm_rows(s, norm);
            cuda_check(ingot_support_linear_bf16(out, w.data, buf(kNormed), w.n_in, w.n_in, w.n_out, 0, s.st.n_tok, 0, stream), "projection");
        }
    }
    // out = W in. Tensor-core path: the operand planes must hold `in` (operand_ready).
    void project(const StepCtx& s, float* out, const Matrix& w, const float* in, int in_ld) {
        if (s.tc) {
            if (w.rows_per_block > 0) cuda_check(ingot_linear_tc_run_blocks(ws, out, w.data, w.n_in, w.n_out, w.rows_per_block, stream), "block projection");
            else cuda_check(ingot_linear_tc_run(ws, out, w.data, w.n_in, w.n_out, 0, stream), "projection");
        } else if (s.st.n_tok == 1 && streams(w) && w.n_out > 2048) {  // few rows: ingot_support_linear_bf16 gives each a CTA
            cuda_check(ingot_support_gemv_bf16(out, w.data, w.n_out, w.n_in, in, nullptr, 0.f, w.n_in, 0, 0, 0, stream), "projection");
        } else {
            cuda_check(ingot_support_linear_bf16(out, w.data, in, in_ld, w.n_in, w.n_out, w.rows_per_block, s.st.n_tok, 0, stream), "projection");
        }
    }
    // The same for f32 rows that are not in the planes yet.
    void project_rows(const StepCtx& s, float* out, const Matrix& w, const float* in, int in_ld, int planes) {
        if (s.tc) cuda_check(ingot_linear_tc_prepare_bf16(ws, in, in_ld, w.n_in, s.st.n_tok, planes, stream), "operand");
        project(s, out, w, in, in_ld);
    }
    // x += W in; next_norm: the norm that the following product reads x through (null: none), folded into the same kernel.
    void project_residual(const StepCtx& s, const Matrix& w, const float* in, const float* next_norm) {
        norm_ready_ = nullptr;
        if (s.tc) {
            cuda_check(ingot_linear_tc_run_partial(ws, w.data, w.n_in, w.n_out, 0, stream), "output projection");
            cuda_check(ingot_linear_tc_finish_residual_norm_bf16(ws, x, next_norm, eps, width, s.planes, stream), "residual");
            norm_ready_ = next_norm;
        } else if (s.st.n_tok == 1 && streams(w)) {
            cuda_check(ingot_support_gemv_bf16(x, w.data, w.n_out, w.n_in, in, nullptr, 0.f, w.n_in, 0, 0, 1, stream), "output projection");
        } else {
            cuda_check(ingot_support_linear_bf16(x, w.data, in, w.n_in, w.n_in, w.n_out, 0, s.st.n_tok, 1, stream), "output projection");
        }
    }
    // kMid (or the operand planes) = gelu(W_gate h) * (W_up h), h = rmsnorm(x); w holds the gate rows and then the up rows
    void gated_project(const StepCtx& s, const Matrix& w, const float* norm) {
        const int ff = w.n_out / 2;
        if (s.tc) {
            prepare_norm(s, w, norm);
            cuda_check(ingot_linear_tc_run_partial(ws, w.data, w.n_in, w.n_out, 0, stream), "gate / up");
            cuda_check(ingot_linear_tc_finish_gated_bf16(ws, 1, s.planes, stream), "gate");
        } else if (s.st.n_tok == 1 && streams(w)) {
            cuda_check(ingot_support_gemv_bf16(buf(kMid), w.data, ff, w.n_in, x, norm, eps, width, 1, 1, 0, stream), "gate / up");
        } else {
            norm_rows(s, norm);
            cuda_check(ingot_support_linear_bf16(buf(kGateUp), w.data, buf(kNormed), w.n_in, w.n_in, w.n_out, 0, s.st.n_tok, 0, stream), "gate / up");
            cuda_check(ingot_support_gated_act(buf(kMid), buf(kGateUp), s.st.n_tok, ff, 1, stream), "gate");
        }
    }
    void begin() { norm_ready_ = nullptr; }

    const ModelDir& dir;
    const EngineOptions opt;
    const int max_step;
    cudaStream_t stream = nullptr;
    ingot_linear_ws* ws = nullptr;
    float* x = nullptr;  // residual stream [n_tok][round_up(width, 8)]
    int width = 0;
    float eps = 0.f;
    size_t weight_bytes = 0;
    std::vector<std::unique_ptr<CacheGroup>> caches;

    CacheGroup* cache_group(int kv_heads, int dim, int chunk, int* layer) {
        for (auto& g : caches)
            if (g->kv_heads == kv_heads && g->dim == dim && g->chunk == chunk) { *layer = g->n_layer++; return g.get(); }
        caches.push_back(std::make_unique<CacheGroup>());
        CacheGroup* g = caches.back().get();
        g->kv_heads = kv_heads; g->dim = dim; g->chunk = chunk; g->n_layer = 1;
        *layer = 0;
        return g;
    }

private:
    void norm_rows(const StepCtx& s, const float* norm) {
        cuda_check(ingot_support_rmsnorm_rows(buf(kNormed), x, norm, nullptr, s.st.n_tok, round_up(width, 8), width, eps, stream), "rmsnorm");
    }
    void prepare_norm(const StepCtx& s, const Matrix& w, const float* norm) {
        if (norm_ready_ == norm && norm) return;  // the kernel that finished x already normalised it for this product
        cuda_check(ingot_linear_tc_prepare_norm_bf16(ws, x, norm, eps, w.n_in, width, s.st.n_tok, s.planes, stream), "rmsnorm");
    }
    WeightStreamer loader_;
    std::vector<void*> allocs_;
    int columns_[kBufCount] = {};
    float* bufs_[kBufCount] = {};
    int tc_in_ = 8, tc_out_ = 8;
    const float* norm_ready_ = nullptr;  // the norm weights x has been prepared with
};

// ---- mixers ----------------------------------------------------------------------------------------------------------

class Mixer {
public:
    virtual ~Mixer() = default;
    // x += mixer(rmsnorm(x; norm)); next_norm as in LayerOps::project_residual.
    virtual void run(LayerOps& ops, const StepCtx& s, const float* norm, const float* next_norm) = 0;
    // Threads one time chunk of a recurrence of this mixer occupies (0: none); sizes the chunks of a step.
    virtual int scan_threads() const { return 0; }
    virtual int lru_threads() const { return 0; }
    virtual size_t scan_scratch_per_chunk() const { return 0; }
    virtual size_t lru_scratch_per_chunk() const { return 0; }
};

// Selective scan (Mamba): [x | z] = W_in h; x <- silu(conv(x)); [dt | B | C] = W_x x; dt <- W_dt dt; scan; W_o (y silu(z)).
std::vector<float> pad_rows(const std::vector<float>& v, int rows, int cols, int rows_p, int cols_p) {
    std::vector<float> out(size_t(rows_p) * cols_p, 0.f);
    for (int r = 0; r < rows; r++) std::copy(v.begin() + size_t(r) * cols, v.begin() + size_t(r + 1) * cols, out.begin() + size_t(r) * cols_p);
    return out;
}

class SelectiveScanMixer : public Mixer {
public:
    SelectiveScanMixer(LayerOps& ops, const Json& c, const std::string& p) {
        inner_ = get_int(c, "inner");
        states_ = get_int(c, "state", 1, 256);
        taps_ = get_int(c, "conv", 1, 16);
        const int rank = get_int(c, "dt_rank"), d = ops.width;
        const Groups in = flat(inner_), rk = flat(rank);
        ip_ = in.padded;
        np_ = ingot_scan_state_pad(states_);
        rank_p_ = rk.padded;
        w_in_ = ops.matrix(2 * ip_, flat(d).padded, {Part{p + "in", {2 * inner_, d}, {2, inner_, ip_}, flat(d)}});
        conv_w_ = ops.upload(pad_rows(tensor_f32(ops.dir.tensor(p + "conv", {inner_, taps_})), inner_, taps_, ip_, taps_));
        conv_b_ = ops.vector(p + "conv.b", inner_);
        // rows of W_x: dt, B and C each start on a padded place, so that B and C rows can be fetched 16 bytes at a time
        const std::vector<int64_t> x_shape = {rank + 2 * states_, inner_};
        const Groups st = {1, states_, np_};
        w_x_ = ops.matrix(rank_p_ + 2 * np_, ip_, {Part{p + "x", x_shape, rk, in, 0, 0, 0}, Part{p + "x", x_shape, st, in, rank_p_, 0, rank},
                                                   Part{p + "x", x_shape, st, in, rank_p_ + np_, 0, rank + states_}});
        w_dt_ = ops.matrix(ip_, rank_p_, {Part{p + "dt", {inner_, rank}, in, rk}});
        dt_b_ = ops.vector(p + "dt.b", inner_);
        std::vector<float> a = tensor_f32(ops.dir.tensor(p + "A_log", {inner_, states_}));
        for (float& v : a) v = float(-std::exp(double(v)) * 1.4426950408889634);  // exp(dt A) = 2^(dt A log2 e)
        a2_ = ops.upload(pad_rows(a, inner_, states_, ip_, np_));
        d_ = ops.vector(p + "D", inner_);
        w_o_ = ops.matrix(p + "o", flat(d), in);
        conv_state_ = static_cast<float*>(ops.alloc(size_t(ops.opt.max_seqs) * (taps_ - 1) * ip_ * 4, true));
        state_ = static_cast<float*>(ops.alloc(size_t(ops.opt.max_seqs) * ip_ * np_ * 4, true));
        ops.need(kProj, 2 * ip_);
        ops.need(kConv, ip_);
        ops.need(kStateIn, rank_p_ + 2 * np_);
        ops.need(kDt, ip_);
        ops.need(kMix, ip_);
    }
    void run(LayerOps& ops, const StepCtx& s, const float* norm, const float* next_norm) override {
        float *xz = ops.buf(kProj), *xc = ops.buf(kConv), *dbc = ops.buf(kStateIn), *dt = ops.buf(kDt);
        const int ld_bc = rank_p_ + 2 * np_;
        ops.norm_project(s, xz, w_in_, norm);
        const ingot_act_out conv = ops.operand(s, xc, ip_, true);
        ingot_check(ingot_causal_conv(&s.st, xz, 2 * ip_, nullptr, conv_w_, conv_b_, taps_, ip_, ops.opt.f32 ? 1 : 2, conv_state_, &conv, ops.stream));
        ops.operand_ready(s, ip_);
        ops.project(s, dbc, w_x_, xc, ip_);
        ops.project_rows(s, dt, w_dt_, dbc, ld_bc, 2);
        const ingot_act_out y = ops.operand(s, ops.buf(kMix), ip_, false);
        ingot_check(ingot_selective_scan(&s.st, &s.scan, xc, ip_, dt, ip_, dt_b_, dbc, ld_bc, rank_p_, rank_p_ + np_, xz + ip_, 2 * ip_, a2_, d_,
                                         state_, ip_, states_, ops.opt.f32 ? 1 : 0, &y, ops.stream));
        ops.operand_ready(s, ip_);
        ops.project_residual(s, w_o_, ops.buf(kMix), next_norm);
    }
    int scan_threads() const override { return ip_ * 2; }
    size_t scan_scratch_per_chunk() const override { return size_t(ip_) * (np_ + 1); }

private:
    int inner_, states_, taps_, ip_, np_, rank_p_;
    Matrix w_in_, w_x_, w_dt_, w_o_;
    float *conv_w_, *conv_b_, *dt_b_, *a2_, *d_, *conv_state_, *state_;
};

// Attention beside a gated linear recurrent unit, both reading the same normalised input:
//   left   chunk-local attention over shared key/value rows (ingot_skv_*)
//   right  y = gelu(W_y h + b), u = conv(W_x h + b), gates from block-diagonal products of u, S; output S * y
// x += W_left (left_scale * attention) + W_right (right_scale * recurrence): one input product for the four input matrices
// and one output product over the two results side by side.
class ParallelMixer : public Mixer {
public:
    ParallelMixer(LayerOps& ops, const Json& c, const std::string& p) {
        const Json &l = c.at("left"), &r = c.at("right");
        const int d = ops.width;
        left_scale_ = get_float(c, "left_scale");
        right_scale_ = get_float(c, "right_scale");
        heads_ = get_int(l, "heads");
        kv_heads_ = get_int(l, "kv_heads");
        dim_ = get_int(l, "dim");
        if (heads_ % kv_heads_ != 0) throw std::runtime_error("model config: \"heads\" is not a multiple of \"kv_heads\"");
        if (l.has("vdim") && get_int(l, "vdim") != dim_) throw std::runtime_error("model config: values that are the keys need \"vdim\" equal to \"dim\"");
        scale_ = get_float(l, "scale");
        const int chunk = l.has("mask") && !l.at("mask").is_null() ? get_int(l.at("mask"), "size") : 0;
        const int row = ops.opt.f32 ? round_up(dim_, 8) : ingot_skv_row_length(dim_);
        if (row < 2 || row > 512) throw std::runtime_error("model config: heads of more than 512 values are not supported");
        row_ = row;
        cache_ = ops.cache_group(kv_heads_, row, chunk, &cache_layer_);

        width_ = get_int(r, "width");
        const int blocks = get_int(r, "blocks");
        taps_ = get_int(r, "conv", 1, 16);
        if (width_ % blocks != 0) throw std::runtime_error("model config: \"width\" is not a multiple of \"blocks\"");
        const int m = width_ / blocks, mp = round_up(m, 8);
        const Groups q = {heads_, dim_, row}, k = {kv_heads_, dim_, row}, w = {blocks, m, mp}, in = flat(d);
        wp_ = w.width();
        block_ = mp;
        const std::string L = p + "left.", R = p + "right.";
        k_off_ = q.width();
        y_off_ = k_off_ + k.width();
        x_off_ = y_off_ + wp_;
        proj_ld_ = x_off_ + wp_;
        w_in_ = ops.matrix(proj_ld_, in.padded, {Part{L + "q", {q.count(), d}, q, in, 0}, Part{L + "k", {k.count(), d}, k, in, k_off_},
                                                 Part{R + "y", {width_, d}, w, in, y_off_}, Part{R + "x", {width_, d}, w, in, x_off_}});
        q_norm_ = ops.vector(L + "q.norm", {q.count()}, q);
        k_norm_ = ops.vector(L + "k.norm", {k.count()}, k);
        y_b_ = ops.vector(R + "y.b", {width_}, w);
        x_b_ = ops.vector(R + "x.b", {width_}, w);
        std::vector<float> cw = tensor_f32(ops.dir.tensor(R + "conv", {width_, taps_})), cw_p(size_t(wp_) * taps_, 0.f);
        for (int i = 0; i < width_; i++) std::copy(cw.begin() + size_t(i) * taps_, cw.begin() + size_t(i + 1) * taps_, cw_p.begin() + size_t(i / m * mp + i % m) * taps_);
        conv_w_ = ops.upload(cw_p);
        conv_b_ = ops.vector(R + "conv.b", {width_}, w);
        // block b: m rows of the recurrence gate, then m rows of the input gate
        const Groups gate_rows = {blocks, m, 2 * mp}, gate_cols = {1, m, mp};
        w_gates_ = ops.matrix(2 * wp_, mp, {Part{R + "ra", {blocks, m, m}, gate_rows, gate_cols, 0}, Part{R + "ri", {blocks, m, m}, gate_rows, gate_cols, mp}}, 2 * mp);
        r_b_ = ops.vector(R + "ra.b", {blocks, m}, w);
        i_b_ = ops.vector(R + "ri.b", {blocks, m}, w);
        std::vector<float> lam = ops.host_vector(R + "lam", {width_}, w);
        for (float& v : lam) v = float(double(v) > 30 ? double(v) : std::log1p(std::exp(double(v))));
        softplus_lam_ = ops.upload(lam);
        const Groups heads_out = flat(q.count());
        attn_cols_ = heads_out.padded;
        mix_ld_ = attn_cols_ + wp_;
        w_o_ = ops.matrix(in.padded, mix_ld_, {Part{L + "o", {d, q.count()}, in, heads_out, 0, 0}, Part{R + "o", {d, width_}, in, w, 0, attn_cols_}});
        conv_state_ = static_cast<float*>(ops.alloc(size_t(ops.opt.max_seqs) * (taps_ - 1) * wp_ * 4, true));
        state_ = static_cast<float*>(ops.alloc(size_t(ops.opt.max_seqs) * wp_ * 4, true));
        ops.need(kProj, proj_ld_);
        ops.need(kConv, wp_);
        ops.need(kGates, 2 * wp_);
        ops.need(kMix, mix_ld_);
        ops.need(kQuery, q.width());
    }
    void run(LayerOps& ops, const StepCtx& s, const float* norm, const float* next_norm) override {
        float *proj = ops.buf(kProj), *u = ops.buf(kConv), *gates = ops.buf(kGates), *mix = ops.buf(kMix);
        const CacheGroup& g = *cache_;
        ops.norm_project(s, proj, w_in_, norm);
        const ingot_act_out conv = ops.operand(s, u, wp_, true, 2);
        ingot_check(ingot_causal_conv(&s.st, proj + x_off_, proj_ld_, x_b_, conv_w_, conv_b_, taps_, wp_, 0, conv_state_, &conv, ops.stream));
        ops.operand_ready(s, wp_, 2);
        ops.project(s, gates, w_gates_, u, wp_);
        ingot_check(ingot_skv_append(g.kv, cache_layer_, &s.st, proj, proj_ld_, 0, k_off_, heads_, dim_, q_norm_, k_norm_, ops.eps, ops.buf(kQuery),
                                     g.tables, g.first_page, g.width, ops.stream));
        // the two results side by side are the operand of the output product
        const ingot_act_out left = ops.operand(s, mix, mix_ld_, false);
        ingot_check(ingot_skv_attend(g.kv, cache_layer_, &s.st, ops.buf(kQuery), heads_, dim_, scale_, left_scale_, &left, g.tables, g.first_page, g.width,
                                     0, ops.stream));
        ingot_act_out right = left;
        if (right.f32) right.f32 += attn_cols_;
        if (right.hi) right.hi = static_cast<char*>(right.hi) + size_t(attn_cols_) * 2;
        if (right.lo) right.lo = static_cast<char*>(right.lo) + size_t(attn_cols_) * 2;
        ingot_check(ingot_gated_lru(&s.st, &s.lru, u, wp_, gates, 2 * wp_, block_, r_b_, i_b_, softplus_lam_, proj + y_off_, proj_ld_, y_b_, state_, wp_,
                                    right_scale_, ops.opt.f32 ? 1 : 0, &right, ops.stream));
        ops.operand_ready(s, mix_ld_);
        ops.project_residual(s, w_o_, mix, next_norm);
    }
    int lru_threads() const override { return wp_; }
    size_t lru_scratch_per_chunk() const override { return 2 * size_t(wp_); }

private:
    int heads_, kv_heads_, dim_, row_, width_, wp_, block_, taps_, cache_layer_ = 0;
    int k_off_, y_off_, x_off_, proj_ld_, attn_cols_, mix_ld_;
    float scale_, left_scale_, right_scale_;
    CacheGroup* cache_;
    Matrix w_in_, w_gates_, w_o_;
    float *q_norm_, *k_norm_, *y_b_, *x_b_, *conv_w_, *conv_b_, *r_b_, *i_b_, *softplus_lam_, *conv_state_, *state_;
};

std::unique_ptr<Mixer> make_mixer(const std::string& type, LayerOps& ops, const Json& config, const std::string& prefix) {
    if (type == "mamba1") return std::make_unique<SelectiveScanMixer>(ops, config, prefix);
    if (type == "parallel") return std::make_unique<ParallelMixer>(ops, config, prefix);
    throw std::runtime_error("model config: unknown layer type \"" + type + "\"");
}

// Gated feed-forward: W_down (gelu(W_gate h) * (W_up h)).
class GatedFeedForward {
public:
    GatedFeedForward(LayerOps& ops, const Json& c, const std::string& p) {
        if (c.at("kind").str() != "dense") throw std::runtime_error("model config: unknown feed-forward kind \"" + c.at("kind").str() + "\"");
        const Groups ff = flat(get_int(c, "ff")), d = flat(ops.width);
        w_gu_ = ops.matrix(2 * ff.padded, d.padded, {Part{p + "gate", {ff.count(), d.count()}, ff, d, 0}, Part{p + "up", {ff.count(), d.count()}, ff, d, ff.padded}});
        w_down_ = ops.matrix(p + "down", d, ff);
        ops.need(kGateUp, 2 * ff.padded);
        ops.need(kMid, ff.padded);
        ops.tc_shape(ff.padded, 2 * ff.padded);
    }
    void run(LayerOps& ops, const StepCtx& s, const float* norm, const float* next_norm) {
        ops.gated_project(s, w_gu_, norm);
        ops.project_residual(s, w_down_, ops.buf(kMid), next_norm);
    }

private:
    Matrix w_gu_, w_down_;
};

// ---- the model -------------------------------------------------------------------------------------------------------

class HybridBackend : public ModelBackend {
public:
    HybridBackend(const ModelDir& dir, const EngineOptions& opt)
        : ops_(dir, opt, opt.max_step_tokens > 0 ? opt.max_step_tokens : opt.max_tokens), max_seqs_(opt.max_seqs), max_ctx_(opt.max_tokens) {
        if (opt.max_tokens < 1 || opt.max_seqs < 1) throw std::runtime_error("engine: needs at least one token and one sequence");
        int device = 0;
        cuda_check(cudaGetDevice(&device), "cudaGetDevice");
        cuda_check(cudaDeviceGetAttribute(&num_sms_, cudaDevAttrMultiProcessorCount, device), "device attribute");
        const Json& c = dir.config();
        n_vocab_ = get_int(c, "vocab");
        ops_.width = get_int(c, "width");
        ops_.eps = get_float(c.at("norm"), "eps");
        const Groups d = flat(ops_.width);
        ops_.x = static_cast<float*>(ops_.alloc(size_t(ops_.max_step) * d.padded * 4, true));
        ops_.need(kNormed, d.padded);
        ops_.tc_shape(d.padded, round_up(n_vocab_, 8));
        embed_ = ops_.matrix("embed", Groups{1, n_vocab_, n_vocab_}, d);
        const size_t embed_bytes = ops_.weight_bytes;
        const auto& layers = c.at("layers").items();
        for (size_t i = 0; i < layers.size(); i++) {
            const std::string p = "l" + std::to_string(i) + ".";
            Layer L;
            L.type = layers[i].at("type").str();
            L.norm1 = ops_.vector(p + "norm1", ops_.width);
            L.mixer = make_mixer(L.type, ops_, layers[i].at("mixer"), p + "mix.");
            if (layers[i].has("mlp") && !layers[i].at("mlp").is_null()) {
                L.norm2 = ops_.vector(p + "norm2", ops_.width);
                L.mlp = std::make_unique<GatedFeedForward>(ops_, layers[i].at("mlp"), p + "mlp.");
            }
            scan_threads_ = std::max(scan_threads_, L.mixer->scan_threads());
            lru_threads_ = std::max(lru_threads_, L.mixer->lru_threads());
            scan_scratch_ = std::max(scan_scratch_, L.mixer->scan_scratch_per_chunk());
            lru_scratch_ = std::max(lru_scratch_, L.mixer->lru_scratch_per_chunk());
            layers_.push_back(std::move(L));
        }
        final_norm_ = ops_.vector("final.norm", ops_.width);
        head_ = ops_.matrix("head", flat(n_vocab_), d);
        weight_bytes_ = ops_.weight_bytes - embed_bytes;
        for (auto& g : ops_.caches) {
            g->pages_per_chunk = g->chunk > 0 ? (g->chunk + INGOT_BLOCK_TOKENS - 1) / INGOT_BLOCK_TOKENS : 0;
            // the pool holds max_tokens tokens of live sequences however they are spread over max_seqs of them
            // (whole chunks, and one begun chunk and one begun page per sequence)
            const long long whole = g->chunk > 0 ? (long long)(max_ctx_ / g->chunk) * g->pages_per_chunk : 0, pages = (long long)max_ctx_ / INGOT_BLOCK_TOKENS + max_seqs_;
            const long long blocks = g->chunk > 0 ? whole + std::min(pages, (long long)max_seqs_ * g->pages_per_chunk) : pages;
            if (blocks > (1 << 26)) throw std::runtime_error("engine: cache pool too large");
            ingot_check(ingot_skv_create(&g->kv, g->n_layer, g->kv_heads, g->dim, opt.f32 ? INGOT_F32 : INGOT_F16, g->chunk, int(blocks)));
            g->pool = BlockPool(int(blocks), max_seqs_, ingot_skv_pages(g->chunk, max_ctx_));
        }
        embed_status_ = static_cast<int*>(ops_.alloc(sizeof(int), true));
        ops_.allocate();
        cuda_check(cudaMallocHost(&status_host_, kMaxStatus * sizeof(int)), "cudaMallocHost");
        cuda_check(cudaEventCreate(&ev0_), "cudaEventCreate");
        cuda_check(cudaEventCreate(&ev1_), "cudaEventCreate");
        lens_.assign(size_t(max_seqs_), 0);
        status_words_.push_back(embed_status_);
        if (ops_.ws) status_words_.push_back(ingot_linear_ws_status_dev(ops_.ws));
        for (auto& g : ops_.caches) status_words_.push_back(ingot_skv_status_dev(g->kv));
        if (status_words_.size() > kMaxStatus) throw std::runtime_error("engine: too many cache groups");
    }
    ~HybridBackend() override {
        cudaStreamSynchronize(ops_.stream);
        drop_graphs();
        for (auto& g : ops_.caches) ingot_skv_destroy(g->kv);
        cudaFree(meta_dev_);
        cudaFree(logits_dev_);
        cudaFree(scan_scratch_dev_);
        cudaFree(lru_scratch_dev_);
        cudaFreeHost(meta_host_);
        cudaFreeHost(logits_);
        cudaFreeHost(status_host_);
        if (ev0_) cudaEventDestroy(ev0_);
        if (ev1_) cudaEventDestroy(ev1_);
    }

    const float* forward_multi(const int32_t* tokens, const int32_t* seq_ids, const int32_t* positions, int n) override {
        static const int32_t zero = 0;
        std::vector<StepEntry> e(size_t(std::max(n, 0)));
        for (int i = 0; i < n; i++) e[size_t(i)] = StepEntry{seq_ids[i], positions[i], tokens + i, 1, &zero, 1};
        return forward_step(e.data(), n, n_vocab_);
    }

    const float* forward_step(const StepEntry* entries, int n, int n_vocab) override {
        if (n_vocab != n_vocab_) throw std::runtime_error("engine: vocabulary size mismatch");
        Step step = check(entries, n);
        reserve_pages(entries, n);
        const StepCtx s = upload_step(entries, n, step);
        reserve_logits(step.n_want);
        // Steps of single decoded tokens are the same launches every time but for what the metadata says: captured once per
        // batch size and replayed. The first such step of a size runs eagerly.
        const bool replay = step.decode && !tap_ && use_graphs_;
        cuda_check(cudaEventRecord(ev0_, ops_.stream), "cudaEventRecord");
        if (replay && graphs_.count(n) && graphs_[n].exec) {
            cuda_check(cudaGraphLaunch(graphs_[n].exec, ops_.stream), "cudaGraphLaunch");
        } else if (replay && graphs_[n].seen++ > 0) {
            cuda_check(cudaStreamBeginCapture(ops_.stream, cudaStreamCaptureModeThreadLocal), "cudaStreamBeginCapture");
            try {
                encode(s, step);
            } catch (...) {
                cudaGraph_t dead = nullptr;
                cudaStreamEndCapture(ops_.stream, &dead);
                if (dead) cudaGraphDestroy(dead);
                throw;
            }
            cuda_check(cudaStreamEndCapture(ops_.stream, &graphs_[n].graph), "cudaStreamEndCapture");
            cuda_check(cudaGraphInstantiate(&graphs_[n].exec, graphs_[n].graph, 0), "cudaGraphInstantiate");
            cuda_check(cudaGraphLaunch(graphs_[n].exec, ops_.stream), "cudaGraphLaunch");
        } else {
            encode(s, step);
        }
        cuda_check(cudaEventRecord(ev1_, ops_.stream), "cudaEventRecord");
        const int ld = head_.n_out;
        if (step.n_want)
            cuda_check(cudaMemcpy2DAsync(logits_, size_t(n_vocab_) * 4, logits_dev_, size_t(ld) * 4, size_t(n_vocab_) * 4, size_t(step.n_want),
                                         cudaMemcpyDeviceToHost, ops_.stream), "D2H logits");
        for (size_t i = 0; i < status_words_.size(); i++)
            cuda_check(cudaMemcpyAsync(status_host_ + i, status_words_[i], sizeof(int), cudaMemcpyDeviceToHost, ops_.stream), "D2H status");
        cuda_check(cudaStreamSynchronize(ops_.stream), "step");
        cudaEventElapsedTime(&last_ms_, ev0_, ev1_);
        for (size_t i = 0; i < status_words_.size(); i++)
            if (status_host_[i]) {
                const int word = status_host_[i];
                cudaMemset(status_words_[i], 0, sizeof(int));
                throw std::runtime_error("engine: a kernel reported status " + std::to_string(word));
            }
        for (int i = 0; i < n; i++) {
            const int seq = entries[i].seq_id, next = entries[i].pos0 + entries[i].n_tokens;
            lens_[size_t(seq)] = next;
            // pages of chunks that lie wholly in the past can never be seen again
            for (auto& g : ops_.caches)
                if (g->chunk > 0 && next < max_ctx_) g->pool.release(seq, 0, g->page(g->first_visible(next)));
        }
        return step.n_want ? logits_ : nullptr;
    }

    void release_sequence(int seq_id) override {
        if (seq_id < 0 || seq_id >= max_seqs_) throw std::runtime_error("engine: sequence id out of range");
        lens_[size_t(seq_id)] = 0;
        for (auto& g : ops_.caches) g->pool.release(seq_id);
    }
    int max_seqs() const override { return max_seqs_; }
    int n_ctx_per_seq() const override { return max_ctx_; }
    int max_portion() const override { return ops_.max_step; }
    int max_step_tokens() const override { return ops_.max_step; }
    int n_vocab() const override { return n_vocab_; }
    void tap_residuals(std::vector<float>* out) override { tap_ = out; }
    size_t weight_bytes() const override { return weight_bytes_; }
    float last_step_ms() const override { return last_ms_; }
    std::string describe() const override {
        std::map<std::string, int> kinds;
        for (const Layer& l : layers_) kinds[l.type]++;
        std::string t = std::to_string(layers_.size()) + " layers (";
        bool first = true;
        for (const auto& [k, v] : kinds) { t += (first ? "" : ", ") + std::to_string(v) + " " + k; first = false; }
        return t + "), width " + std::to_string(ops_.width) + ", vocabulary " + std::to_string(n_vocab_) + ", " + (ops_.opt.f32 ? "float32" : "bfloat16");
    }

private:
    struct Layer {
        std::string type;
        float *norm1 = nullptr, *norm2 = nullptr;
        std::unique_ptr<Mixer> mixer;
        std::unique_ptr<GatedFeedForward> mlp;
    };
    struct Step {
        int n_tok = 0, max_len = 0, n_want = 0;
        bool decode = true;           // one token of every sequence, its logits wanted
        const int32_t* want_rows = nullptr;  // device
        const int32_t* tokens = nullptr;     // device
        int first_want = 0;           // host copy of want_rows[0]
    };
    struct Graph {
        int seen = 0;
        cudaGraph_t graph = nullptr;
        cudaGraphExec_t exec = nullptr;
    };
    static constexpr size_t kMaxStatus = 64;

    Step check(const StepEntry* entries, int n) const {
        if (n < 1 || n > max_seqs_) throw std::runtime_error("engine: batch size out of range");
        Step step;
        std::vector<char> seen(size_t(max_seqs_), 0);
        for (int i = 0; i < n; i++) {
            const StepEntry& e = entries[i];
            if (e.seq_id < 0 || e.seq_id >= max_seqs_) throw std::runtime_error("engine: sequence id out of range");
            if (seen[size_t(e.seq_id)]++) throw std::runtime_error("engine: a sequence appears twice in one step");
            if (e.n_tokens < 1) throw std::runtime_error("engine: empty portion");
            if (e.pos0 < 0 || e.pos0 > max_ctx_ - e.n_tokens) throw std::runtime_error("context window exceeded");
            // a recurrent state only exists at the end of what has been run: go on from there, or start again
            if (e.pos0 != 0 && e.pos0 != lens_[size_t(e.seq_id)]) throw std::runtime_error("engine: a sequence must continue where it stands or restart at 0");
            for (int t = 0; t < e.n_tokens; t++)
                if (e.tokens[t] < 0 || e.tokens[t] >= n_vocab_) throw std::runtime_error("token id out of range");
            for (int w = 0; w < e.n_want; w++)
                if (e.want[w] < 0 || e.want[w] >= e.n_tokens) throw std::runtime_error("engine: wanted place outside the portion");
            step.n_tok += e.n_tokens;
            step.max_len = std::max(step.max_len, e.n_tokens);
            step.n_want += e.n_want;
            step.decode = step.decode && e.n_tokens == 1 && e.n_want == 1;
        }
        if (step.n_tok > ops_.max_step) throw std::runtime_error("engine: more tokens than a step may carry");
        return step;
    }

    void reserve_pages(const StepEntry* entries, int n) {
        for (int i = 0; i < n; i++)
            for (auto& g : ops_.caches) {
                if (entries[i].pos0 == 0) g->pool.release(entries[i].seq_id);  // a restart leaves what it held
                g->pool.ensure(entries[i].seq_id, g->page(g->first_visible(entries[i].pos0)), g->page(entries[i].pos0 + entries[i].n_tokens - 1));
            }
    }

    // INGOT_SCAN_THREADS: threads per SM the chunks of a recurrence aim for (tuning).
    // Length of the time chunks of a recurrence one token-chunk of which occupies `threads` threads: as few chunks as fill the GPU.
    int chunk_tokens(int n_tok, int threads) const {
        const int chunks = std::max(1, num_sms_ * scan_threads_per_sm_ / std::max(threads, 1));
        return std::max(32, round_up((n_tok + chunks - 1) / chunks, 16));
    }

    StepCtx upload_step(const StepEntry* entries, int n, Step& step) {
        std::vector<int32_t>& m = meta_;
        m.clear();
        auto mark = [&] { while (m.size() % 4) m.push_back(0); return m.size(); };
        const size_t o_tok = mark();
        for (int i = 0; i < n; i++) m.insert(m.end(), entries[i].tokens, entries[i].tokens + entries[i].n_tokens);
        const size_t o_rowseq = mark();
        for (int i = 0; i < n; i++) m.insert(m.end(), size_t(entries[i].n_tokens), i);
        const size_t o_start = mark();
        for (int i = 0, r = 0; i < n; r += entries[i].n_tokens, i++) m.push_back(r);
        const size_t o_len = mark();
        for (int i = 0; i < n; i++) m.push_back(entries[i].n_tokens);
        const size_t o_pos = mark();
        for (int i = 0; i < n; i++) m.push_back(entries[i].pos0);
        const size_t o_slot = mark();
        for (int i = 0; i < n; i++) m.push_back(entries[i].seq_id);
        const size_t o_want = mark();
        for (int i = 0; i < n; i++)
            for (int w = 0; w < entries[i].n_want; w++) m.push_back(m[o_start + size_t(i)] + entries[i].want[w]);
        step.first_want = step.n_want ? m[o_want] : 0;
        struct PlanAt { size_t seq, t0, len, first; int n_chunks, max_chunks; };
        auto plan = [&](int threads) {
            PlanAt p = {};
            const int L = chunk_tokens(step.n_tok, threads);
            std::vector<int32_t> seq, t0, len, first;
            for (int i = 0; i < n; i++) {
                first.push_back(int32_t(seq.size()));
                for (int t = 0; t < entries[i].n_tokens; t += L) {
                    seq.push_back(i);
                    t0.push_back(t);
                    len.push_back(std::min(L, entries[i].n_tokens - t));
                }
                p.max_chunks = std::max(p.max_chunks, int(seq.size()) - first.back());
            }
            first.push_back(int32_t(seq.size()));
            p.n_chunks = int(seq.size());
            p.seq = mark(); m.insert(m.end(), seq.begin(), seq.end());
            p.t0 = mark(); m.insert(m.end(), t0.begin(), t0.end());
            p.len = mark(); m.insert(m.end(), len.begin(), len.end());
            p.first = mark(); m.insert(m.end(), first.begin(), first.end());
            return p;
        };
        const PlanAt scan = plan(scan_threads_), lru = plan(lru_threads_);
        std::vector<std::pair<size_t, size_t>> table_at;
        for (auto& g : ops_.caches) {
            const size_t o_first = mark();
            int width = 1;
            for (int i = 0; i < n; i++) {
                const int first = g->page(g->first_visible(entries[i].pos0));
                width = std::max(width, g->page(entries[i].pos0 + entries[i].n_tokens - 1) - first + 1);
                m.push_back(first);
            }
            if (step.decode) width = g->chunk > 0 ? std::min(g->pages_per_chunk, g->pool.pages_per_seq()) : g->pool.pages_per_seq();  // the same at every step
            const size_t o_table = mark();
            for (int i = 0; i < n; i++) {
                const int first = m[o_first + size_t(i)];
                const int32_t* row = g->pool.row(entries[i].seq_id);
                for (int k = 0; k < width; k++) m.push_back(first + k < g->pool.pages_per_seq() ? row[first + k] : -1);
            }
            g->width = width;
            table_at.emplace_back(o_first, o_table);
        }
        mark();
        if (m.size() > meta_cap_) {
            drop_graphs();
            cudaFree(meta_dev_);
            cudaFreeHost(meta_host_);
            meta_dev_ = meta_host_ = nullptr;
            meta_cap_ = std::max<size_t>(m.size() * 2, 65536);
            cuda_check(cudaMalloc(&meta_dev_, meta_cap_ * 4), "cudaMalloc(step metadata)");
            cuda_check(cudaMallocHost(&meta_host_, meta_cap_ * 4), "cudaMallocHost(step metadata)");
        }
        memcpy(meta_host_, m.data(), m.size() * 4);
        cuda_check(cudaMemcpyAsync(meta_dev_, meta_host_, m.size() * 4, cudaMemcpyHostToDevice, ops_.stream), "H2D step metadata");

        StepCtx s;
        s.st.n_tok = step.n_tok;
        s.st.n_seq = n;
        s.st.max_len = step.max_len;
        s.st.row_seq = meta_dev_ + o_rowseq;
        s.st.row_start = meta_dev_ + o_start;
        s.st.len = meta_dev_ + o_len;
        s.st.pos0 = meta_dev_ + o_pos;
        s.st.slot = meta_dev_ + o_slot;
        step.tokens = meta_dev_ + o_tok;
        step.want_rows = meta_dev_ + o_want;
        auto fill = [&](ingot_scan_plan& p, const PlanAt& at, size_t per_chunk, float** scratch, size_t* cap) {
            p.n_chunks = at.n_chunks;
            p.max_chunks = at.max_chunks;
            p.chunk_seq = meta_dev_ + at.seq;
            p.chunk_t0 = meta_dev_ + at.t0;
            p.chunk_len = meta_dev_ + at.len;
            p.seq_chunk0 = meta_dev_ + at.first;
            const size_t floats = at.max_chunks > 1 ? per_chunk * size_t(at.n_chunks) : 0;
            if (floats > *cap) {
                drop_graphs();
                cuda_check(cudaStreamSynchronize(ops_.stream), "scratch");
                cudaFree(*scratch);
                *scratch = nullptr;
                cuda_check(cudaMalloc(scratch, floats * 4), "cudaMalloc(scan scratch)");
                *cap = floats;
            }
            p.scratch_dev = *scratch;
            p.scratch_floats = *cap;
        };
        fill(s.scan, scan, scan_scratch_, &scan_scratch_dev_, &scan_cap_);
        fill(s.lru, lru, lru_scratch_, &lru_scratch_dev_, &lru_cap_);
        for (size_t i = 0; i < ops_.caches.size(); i++) {
            ops_.caches[i]->first_page = meta_dev_ + table_at[i].first;
            ops_.caches[i]->tables = meta_dev_ + table_at[i].second;
        }
        s.tc = ops_.ws != nullptr && step.n_tok >= kMinTcTokens;
        s.planes = s.tc && step.n_tok <= kPairTokens ? 2 : 1;
        return s;
    }

    void reserve_logits(int rows) {
        if (rows <= logit_rows_) return;
        drop_graphs();
        cuda_check(cudaStreamSynchronize(ops_.stream), "logits");
        cudaFree(logits_dev_);
        cudaFreeHost(logits_);
        logits_dev_ = nullptr;
        logits_ = nullptr;
        logit_rows_ = std::max(rows, max_seqs_);
        cuda_check(cudaMalloc(&logits_dev_, size_t(logit_rows_) * head_.n_out * 4), "cudaMalloc(logits)");
        cuda_check(cudaMallocHost(&logits_, size_t(logit_rows_) * n_vocab_ * 4), "cudaMallocHost(logits)");
    }
    void drop_graphs() {
        if (graphs_.empty()) return;
        cudaStreamSynchronize(ops_.stream);
        for (auto& [n, g] : graphs_) {
            if (g.exec) cudaGraphExecDestroy(g.exec);
            if (g.graph) cudaGraphDestroy(g.graph);
        }
        graphs_.clear();
    }

    // Every launch of a step, from the token ids to the logits of the wanted rows.
    void encode(const StepCtx& s, const Step& step) {
        cuda_check(ingot_support_embed_rows_bf16(ops_.x, embed_.data, embed_.n_in, n_vocab_, step.tokens, s.st.n_tok, embed_status_, ops_.stream), "embedding rows");
        ops_.begin();
        for (size_t i = 0; i < layers_.size(); i++) {
            const Layer& L = layers_[i];
            const float* following = i + 1 < layers_.size() ? layers_[i + 1].norm1 : nullptr;
            L.mixer->run(ops_, s, L.norm1, L.mlp ? L.norm2 : following);
            if (L.mlp) L.mlp->run(ops_, s, L.norm2, following);
            if (tap_) tap(s.st.n_tok);
        }
        if (!step.n_want) return;
        const int ld = embed_.n_in;
        if (step.n_want == 1 && LayerOps::streams(head_)) {
            cuda_check(ingot_support_gemv_bf16(logits_dev_, head_.data, head_.n_out, head_.n_in, ops_.x + size_t(step.first_want) * ld, final_norm_, ops_.eps,
                                               ops_.width, 0, 0, 0, ops_.stream), "logits");
            return;
        }
        cuda_check(ingot_support_rmsnorm_rows(ops_.buf(kNormed), ops_.x, final_norm_, step.want_rows, step.n_want, ld, ops_.width, ops_.eps, ops_.stream), "final norm");
        if (ops_.ws && step.n_want >= kMinTcTokens) {
            cuda_check(ingot_linear_tc_prepare_bf16(ops_.ws, ops_.buf(kNormed), ld, ld, step.n_want, step.n_want <= kPairTokens ? 2 : 1, ops_.stream), "final norm");
            cuda_check(ingot_linear_tc_run(ops_.ws, logits_dev_, head_.data, head_.n_in, head_.n_out, 0, ops_.stream), "logits");
        } else {
            cuda_check(ingot_support_linear_bf16(logits_dev_, head_.data, ops_.buf(kNormed), ld, ld, head_.n_out, 0, step.n_want, 0, ops_.stream), "logits");
        }
    }

    void tap(int n_tok) {
        const int ld = embed_.n_in, w = ops_.width;
        std::vector<float> rows(size_t(n_tok) * ld);
        cuda_check(cudaStreamSynchronize(ops_.stream), "tap");
        cuda_check(cudaMemcpy(rows.data(), ops_.x, rows.size() * 4, cudaMemcpyDeviceToHost), "tap");
        for (int t = 0; t < n_tok; t++) tap_->insert(tap_->end(), rows.begin() + size_t(t) * ld, rows.begin() + size_t(t) * ld + w);
    }

    LayerOps ops_;
    int max_seqs_, max_ctx_, num_sms_ = 0, n_vocab_ = 0;
    std::vector<Layer> layers_;
    Matrix embed_, head_;
    float* final_norm_ = nullptr;
    int* embed_status_ = nullptr;
    size_t weight_bytes_ = 0;
    int scan_threads_ = 0, lru_threads_ = 0;
    size_t scan_scratch_ = 0, lru_scratch_ = 0;
    float *scan_scratch_dev_ = nullptr, *lru_scratch_dev_ = nullptr;
    size_t scan_cap_ = 0, lru_cap_ = 0;
    std::vector<int> lens_;            // tokens each sequence has run = position of its next one
    std::vector<int32_t> meta_;
    int32_t *meta_dev_ = nullptr, *meta_host_ = nullptr;
    size_t meta_cap_ = 0;
    float *logits_dev_ = nullptr, *logits_ = nullptr;
    int logit_rows_ = 0;
    std::vector<int*> status_words_;
    int* status_host_ = nullptr;
    std::map<int, Graph> graphs_;      // by batch size
    const bool use_graphs_ = !(getenv("INGOT_DECODE_GRAPH") && atoi(getenv("INGOT_DECODE_GRAPH")) == 0);
    const int scan_threads_per_sm_ = getenv("INGOT_SCAN_THREADS") ? std::max(1, atoi(getenv("INGOT_SCAN_THREADS"))) : 1024;
    std::vector<float>* tap_ = nullptr;
    cudaEvent_t ev0_ = nullptr, ev1_ = nullptr;
    float last_ms_ = 0.f;
};

const RegisterModel kBesudra("Besudra", [](const ModelDir& dir, const EngineOptions& opt) -> std::unique_ptr<ModelBackend> {
    return std::make_unique<HybridBackend>(dir, opt);
});

}  // namespace
