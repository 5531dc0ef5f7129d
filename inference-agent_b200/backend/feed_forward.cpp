// Feed-forwards of the model-folder backend: gated, and a mixture of experts (kernels: csrc/moe.cu, linear_sm100.cu).
#include "layer_ops.h"

namespace {

// Gated feed-forward: W_down (gelu(W_gate h) * (W_up h)).
class GatedFeedForward : public FeedForward {
public:
    GatedFeedForward(LayerOps& ops, const Json& c, const std::string& p) {
        const Groups ff = flat(get_int(c, "ff")), d = flat(ops.width);
        w_gu_ = ops.matrix(2 * ff.padded, d.padded, {Part{p + "gate", {ff.count(), d.count()}, ff, d, 0}, Part{p + "up", {ff.count(), d.count()}, ff, d, ff.padded}});
        w_down_ = ops.matrix(p + "down", d, ff);
        ops.need(kGateUp, 2 * ff.padded);
        ops.need(kMid, ff.padded);
        ops.need(kBranch, d.padded);
        ops.tc_shape(ff.padded, 2 * ff.padded);
    }
    void run(LayerOps& ops, const StepCtx& s, const float* norm, const float* next_norm) override {
        ops.gated_project(s, w_gu_, norm);
        ops.project_residual(s, w_down_, ops.buf(kMid), next_norm);
    }
    void branch(LayerOps& ops, const StepCtx& s, const float* norm) override {
        ops.gated_project(s, w_gu_, norm);
        ops.project(s, ops.buf(kBranch), w_down_, ops.buf(kMid), w_down_.n_in);
        ops.set_branch(Branch{ops.buf(kBranch), nullptr, 1});
    }

private:
    Matrix w_gu_, w_down_;
};

// Mixture of experts: router scores sigmoid(W_router h), the `top` experts with the largest; expert e on w h, w its score:
// W_down,e relu(W_up,e (w h))^2. The weight is applied to the product W_up h, which is the same and keeps h in one copy. Tensor-core
// path: rows gathered by expert, two grouped products with the activation in the first one's epilogue; the rows of the second go into
// the residual sum where the mixer's output does.
class MixtureFeedForward : public FeedForward {
public:
    MixtureFeedForward(LayerOps& ops, const Json& c, const std::string& p) {
        experts_ = get_int(c.at("router"), "experts", 1, 1 << 16);
        top_ = get_int(c.at("router"), "top", 1, experts_);
        const Groups ff = flat(get_int(c.at("expert"), "ff")), d = flat(ops.width), e = flat(experts_);
        std::vector<Part> up, down;
        for (int i = 0; i < experts_; i++) {
            const std::string q = p + "e" + std::to_string(i) + ".";
            up.push_back(Part{q + "up", {ff.count(), d.count()}, ff, d, i * ff.padded});
            down.push_back(Part{q + "down", {d.count(), ff.count()}, d, ff, i * d.padded});
        }
        w_router_ = ops.matrix(p + "router", e, d);
        w_up_ = ops.matrix(experts_ * ff.padded, d.padded, up, 0, true);
        w_down_ = ops.matrix(experts_ * d.padded, ff.padded, down, 0, true);
        ff_ = ff.padded;
        d_ = d.padded;
        const size_t pairs = size_t(ops.max_step) * top_;
        auto ints = [&](size_t n) { return static_cast<int32_t*>(ops.alloc(n * 4, true)); };
        expert_of_ = ints(pairs);
        row_of_ = ints(pairs);
        pair_of_ = ints(pairs);
        start_ = ints(size_t(experts_) + 1);
        weight_of_ = static_cast<float*>(ops.alloc(pairs * 4, true));
        row_weight_ = static_cast<float*>(ops.alloc(pairs * 4, true));
        ops.need(kRouter, e.padded);
        ops.need(kExpertMid, top_ * ff_);   // f32, or two bf16 planes
        ops.need(kExpertOut, top_ * d_);
        if (!ops.opt.f32) ops.need(kExpertIn, top_ * d_);
    }
    void branch(LayerOps& ops, const StepCtx& s, const float* norm) override {
        const int rows = s.st.n_tok * top_;
        float *mid = ops.buf(kExpertMid), *out = ops.buf(kExpertOut), *z = ops.buf(kRouter);
        if (s.tc) {
            ops.prepare_norm(s, w_router_, norm);
            ops.project(s, z, w_router_, nullptr, 0);
        } else {
            ops.norm_rows(s, norm);
            ops.project(s, z, w_router_, ops.buf(kNormed), d_);
        }
        ingot_check(ingot_moe_route(z, w_router_.n_out, s.st.n_tok, experts_, top_, expert_of_, weight_of_, start_, row_of_, pair_of_, row_weight_, ops.stream));
        if (s.tc) {
            void *h_hi, *h_lo;
            ingot_linear_ws_planes(ops.ws, &h_hi, &h_lo);
            const bool pair = s.planes > 1;
            char *in_hi = reinterpret_cast<char*>(ops.buf(kExpertIn)), *mid_hi = reinterpret_cast<char*>(mid);
            void *in_lo = pair ? in_hi + size_t(rows) * d_ * 2 : nullptr, *mid_lo = pair ? mid_hi + size_t(rows) * ff_ * 2 : nullptr;
            ingot_check(ingot_moe_gather(in_hi, in_lo, h_hi, h_lo, pair_of_, rows, top_, d_, ops.stream));
            ingot_grouped_gemm g = {};
            g.n_rows = rows;
            g.rows_per_group = s.st.n_tok;
            g.n_groups = experts_;
            g.group_start = start_;
            g.a_hi = in_hi; g.a_lo = in_lo; g.w = w_up_.data; g.n_in = d_; g.n_out = ff_;
            g.row_scale = row_weight_; g.act = INGOT_ACT_RELU2; g.out_hi = mid_hi; g.out_lo = mid_lo;
            cuda_check(ingot_grouped_tc_run(ops.ws, &g, ops.stream), "experts");
            g.a_hi = mid_hi; g.a_lo = mid_lo; g.w = w_down_.data; g.n_in = ff_; g.n_out = d_;
            g.row_scale = nullptr; g.act = INGOT_ACT_NONE; g.out_hi = g.out_lo = nullptr; g.out = out;
            cuda_check(ingot_grouped_tc_run(ops.ws, &g, ops.stream), "experts");
        } else {
            ingot_check(ingot_moe_linear(mid, w_up_.data, ops.buf(kNormed), d_, d_, ff_, experts_, rows, start_, pair_of_, top_, row_weight_, INGOT_ACT_RELU2, ops.stream));
            ingot_check(ingot_moe_linear(out, w_down_.data, mid, ff_, ff_, d_, experts_, rows, start_, nullptr, top_, nullptr, INGOT_ACT_NONE, ops.stream));
        }
        ops.set_branch(Branch{out, row_of_, top_});
    }
    void run(LayerOps& ops, const StepCtx& s, const float* norm, const float*) override {
        branch(ops, s, norm);
        ops.add_branch(s);
    }

private:
    int experts_, top_, ff_, d_;
    Matrix w_router_, w_up_, w_down_;
    int32_t *expert_of_, *row_of_, *pair_of_, *start_;
    float *weight_of_, *row_weight_;
};

}  // namespace

std::unique_ptr<FeedForward> make_gated_feed_forward(LayerOps& ops, const Json& config, const std::string& prefix) {
    return std::make_unique<GatedFeedForward>(ops, config, prefix);
}
std::unique_ptr<FeedForward> make_mixture(LayerOps& ops, const Json& config, const std::string& prefix) {
    return std::make_unique<MixtureFeedForward>(ops, config, prefix);
}
