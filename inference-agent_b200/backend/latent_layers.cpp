// Latent attention of the model-folder backend (kernels: csrc/attn_latent.cu).
#include "layer_ops.h"

namespace {

// q = W_q h, [c' | k'] = W_dkv h; c = rmsnorm(c'), k = rot(k') shared by all heads; head i scores (q_i . U_i c + rot(q_i') . k) * scale
// under a softmax with a sink and averages V_i c; W_o over the heads side by side. W_q and W_dkv are one product. The cache holds
// [c | k] per token; here the attention runs on those rows: U_i^T takes the query into the latent space, V_i follows once per token.
class LatentAttentionMixer : public Mixer {
public:
    LatentAttentionMixer(LayerOps& ops, const Json& c, const std::string& p) {
        heads_ = get_int(c, "heads");
        dim_ = get_int(c, "dim");
        const int rot = get_int(c, "rot_dim"), rank = get_int(c, "kv_rank"), vdim = get_int(c, "vdim"), d = ops.width;
        scale_ = get_float(c, "scale");
        const int rot_dims = get_int(c.at("rot"), "dims");
        const double base = c.at("rot").at("base").number();
        if (rot_dims % 2 != 0 || rot_dims > rot) throw std::runtime_error("model config: \"rot.dims\" must be even and at most \"rot_dim\"");
        const int window = c.has("mask") && !c.at("mask").is_null() ? get_int(c.at("mask"), "size") : 0;
        const Groups in = flat(d), latent = {1, rank, round_up(rank, 16)}, v = {heads_, vdim, round_up(vdim, 8)};
        shape_.n_head = heads_;
        shape_.dim = round_up(dim_, 8);
        shape_.rot = round_up(rot, 8);
        shape_.rank = latent.padded;
        shape_.rank_count = rank;
        shape_.rot_dims = rot_dims;
        row_ = round_up(shape_.rank + shape_.rot, 32);
        if (row_ > 1024) throw std::runtime_error("model config: latent rows of more than 1024 values are not supported");
        cache_ = ops.cache_group(1, row_, 0, window, false, &cache_layer_);

        const int per = shape_.dim + shape_.rot;
        latent_off_ = heads_ * per;
        proj_ld_ = latent_off_ + shape_.rank + shape_.rot;
        const std::vector<int64_t> q_shape = {heads_ * (dim_ + rot), d}, dkv_shape = {rank + rot, d};
        w_in_ = ops.matrix(proj_ld_, in.padded, {Part{p + "q", q_shape, {heads_, dim_, per}, in, 0, 0, 0, dim_ + rot},
                                                 Part{p + "q", q_shape, {heads_, rot, per}, in, shape_.dim, 0, dim_, dim_ + rot},
                                                 Part{p + "dkv", dkv_shape, latent, in, latent_off_, 0, 0},
                                                 Part{p + "dkv", dkv_shape, {1, rot, shape_.rot}, in, latent_off_ + shape_.rank, 0, rank}});
        norm_ = ops.vector(p + "dkv.norm", {rank}, latent);
        sink_ = ops.vector(p + "sink", {heads_}, {1, heads_, heads_});
        {   // U^T, head by head: row r of head i holds column r of U_i
            const TensorView& t = ops.bf16(p + "uk", {heads_ * dim_, rank});
            std::vector<uint16_t> host(size_t(heads_) * shape_.rank * shape_.dim, 0);
            for (int h = 0; h < heads_; h++)
                for (int r = 0; r < rank; r++)
                    for (int k = 0; k < dim_; k++)
                        memcpy(&host[(size_t(h) * shape_.rank + r) * shape_.dim + k], t.data + ((size_t(h) * dim_ + k) * rank + r) * 2, 2);
            w_query_ = ops.matrix(host, heads_ * shape_.rank, shape_.dim, shape_.rank);
        }
        w_value_ = ops.matrix(v.width(), latent.padded, {Part{p + "uv", {v.count(), rank}, v, latent}}, v.padded);
        w_o_ = ops.matrix(p + "o", in, v);
        std::vector<double> turns;
        for (int i = 0; i < rot_dims / 2; i++) turns.push_back(std::pow(base, -2.0 * i / rot_dims) / (2 * 3.14159265358979323846));
        turns_ = static_cast<double*>(ops.alloc(turns.size() * sizeof(double)));
        cuda_check(cudaMemcpy(turns_, turns.data(), turns.size() * sizeof(double), cudaMemcpyHostToDevice), "cudaMemcpy");

        plain_ld_ = heads_ * shape_.dim;
        latent_ld_ = heads_ * shape_.rank;
        value_ld_ = v.width();
        ops.need(kProj, proj_ld_);
        ops.need(kQueryPlain, plain_ld_);
        ops.need(kQuery, ops.opt.f32 ? heads_ * row_ : heads_ * row_ / 2);
        ops.need(kLatent, latent_ld_);
        ops.need(kValue, value_ld_);
    }
    void run(LayerOps& ops, const StepCtx& s, const float* norm, const float* next_norm) override {
        float *proj = ops.buf(kProj), *latent = ops.buf(kLatent), *value = ops.buf(kValue);
        void* rows = ops.buf(kQuery);
        const CacheGroup& g = *cache_;
        const int layer = cache_layer_ + ops.pass;
        ops.norm_project(s, proj, w_in_, norm);
        const ingot_act_out plain = ops.operand(s, ops.buf(kQueryPlain), plain_ld_, false);
        ingot_check(ingot_latent_append(g.kv, layer, &s.st, proj, proj_ld_, 0, latent_off_, &shape_, norm_, ops.eps, turns_, &plain, rows, g.tables, g.first_page,
                                        g.width, ops.stream));
        ops.operand_ready(s, plain_ld_);
        if (s.tc) {
            cuda_check(ingot_linear_tc_run_half(ops.ws, rows, heads_ * row_, row_, w_query_.data, w_query_.n_in, w_query_.n_out, shape_.rank, ops.stream), "latent queries");
        } else {
            ops.project(s, latent, w_query_, ops.buf(kQueryPlain), plain_ld_);
            ingot_check(ingot_latent_queries(g.kv, latent, s.st.n_tok, heads_, shape_.rank, rows, ops.stream));
        }
        const ingot_act_out mixed = ops.operand(s, latent, latent_ld_, false);
        ingot_check(ingot_latent_attend(g.kv, layer, &s.st, rows, heads_, shape_.rank, scale_, sink_, &mixed, g.tables, g.first_page, g.width, 0, 0, ops.stream));
        ops.operand_ready(s, latent_ld_);
        ops.project(s, value, w_value_, latent, latent_ld_);
        if (s.tc) ops.prepare_rows(s, value, value_ld_, value_ld_);
        ops.project_residual(s, w_o_, value, next_norm);
    }

private:
    int heads_, dim_, row_, latent_off_, proj_ld_, plain_ld_, latent_ld_, value_ld_, cache_layer_ = 0;
    ingot_latent_shape shape_ = {};
    float scale_;
    CacheGroup* cache_;
    Matrix w_in_, w_query_, w_value_, w_o_;
    float *norm_, *sink_;
    double* turns_;
};

}  // namespace

std::unique_ptr<Mixer> make_latent_attention(LayerOps& ops, const Json& config, const std::string& prefix) {
    return std::make_unique<LatentAttentionMixer>(ops, config, prefix);
}
