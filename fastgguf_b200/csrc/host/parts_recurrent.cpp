// Mixers that carry a state of fixed size from token to token instead of keys and values per position: retention, gated
// linear attention, and - behind a short convolution, with one decay per head and token - the state-space form and the gated
// delta rule.
//
// "retention": linear attention with a fixed decay per head and neither softmax nor denominator.  With the layer's
// normalised input h, per head (q, k of size head_dim, v of size v_head_dim):
//     q = W_q h, k = W_k h, v = W_v h, g = W_g h       no biases; the four projections are ONE contraction
//     q, k rotated by the position encoding (if any); k times k_scale afterwards
//     S_t = decay_head S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t
//     y = concat_heads(o / sqrt(mean(o^2) + eps)) * silu(g),  output W_o y
// The state S [heads, head_dim, v_head_dim] is float32 whatever the engine's dtype, one row of the engine's state pool
// per sequence slot (zeroed when a sequence takes the slot), and so are the projections' results that enter the
// recurrence: the contraction writes float32 and the kernels of retention.cu keep rotation, decay powers, scores, the
// unit norm and the gate in float32; y takes the engine's dtype for the output projection.
// Options: "qkv_activation": "silu" - q, k and v each pass silu (before a rotation); "norm": "whole" - instead of the unit norm per
// head, y = o / sqrt(mean(o^2) + eps) * w over all heads' outputs at once, with a weight [heads * v_head_dim]; "gate_activation":
// "sigmoid" - sigmoid(g) in place of silu(g) (with "norm": "whole").  k_scale 1 and no position: nothing else happens to k.
// A decode step and short portions walk their tokens one after another with S in shared memory; portions of
// `chunk_threshold` tokens and more run in chunks over all sequences at once (retention.cu says how).
#include <cmath>

#include "parts.hpp"

namespace fg {

class RetentionMixer : public Mixer {
public:
    RetentionMixer(const Json &p, BuildContext &ctx) {
        const char *me = "retention";
        E_ = (int)param_int(p, "hidden_size", me);
        H_ = (int)param_int(p, "n_heads", me);
        dk_ = (int)param_int(p, "head_dim", me);
        dv_ = (int)param_int(p, "v_head_dim", dk_, me);
        eps_ = (float)param_float(p, "eps", me);
        k_scale_ = (float)param_float(p, "k_scale", 1.0 / std::sqrt((double)dk_), me);
        if (E_ <= 0 || H_ <= 0 || dk_ <= 0 || dv_ <= 0) fail(FG_E_CONFIG, "retention: sizes must be positive");
        if (!(eps_ > 0.f)) fail(FG_E_CONFIG, "retention: eps must be positive");
        const Json &d = p.get("decay");
        if (!d.is_array() || (int)d.size() != H_) fail(FG_E_CONFIG, format("retention: 'decay' must list one number for each of the %d heads", H_));
        for (auto &v : d.items()) {
            if (!v.is_number() || v.is_bool() || !(v.as_double() >= 0.0) || !(v.as_double() <= 1.0))
                fail(FG_E_CONFIG, "retention: a decay must be a number in [0, 1], got " + v.dump());
            decay_.push_back((float)v.as_double());
            all_positive_ = all_positive_ && v.as_double() > 0.0;
        }
        auto option = [&](const char *key, const char *plain, const char *other) {
            const Json &v = p.get(key);
            if (v.is_null() || (v.is_string() && v.as_string() == plain)) return false;
            if (!v.is_string() || v.as_string() != other)
                fail(FG_E_CONFIG, format("retention: %s %s is not known (known: %s, %s)", key, v.dump().c_str(), plain, other));
            return true;
        };
        silu_ = option("qkv_activation", "none", "silu");
        whole_norm_ = option("norm", "head", "whole");
        sigmoid_gate_ = option("gate_activation", "silu", "sigmoid");
        if (!whole_norm_ && dv_ > 256) fail(FG_E_CONFIG, format("retention: v_head_dim %d exceeds 256, the largest the kernels take", dv_));
        if (!whole_norm_ && (size_t)dk_ * dv_ > 40 * 1024) fail(FG_E_CONFIG, "retention: a head's state exceeds what the kernels hold in shared memory");
        if (sigmoid_gate_ && !whole_norm_) fail(FG_E_CONFIG, "retention: a sigmoid gate needs norm 'whole'");
        const Json &pos = p.get("position");
        if (!pos.is_null()) {
            position_ = dynamic_cast<PositionEncoding *>(ctx.nested(FG_ROLE_POSITION, pos));
            if (!position_) fail(FG_E_CONFIG, "retention: 'position' is not a position encoding");
            if (position_->head_dim() != dk_)
                fail(FG_E_CONFIG, format("retention: the position encoding is built for head_dim %d, the mixer has %d", position_->head_dim(), dk_));
        }
    }
    std::vector<TensorDecl> tensor_decls() const override {
        int64_t Q = (int64_t)H_ * dk_, V = (int64_t)H_ * dv_;
        std::vector<TensorDecl> d = {{"q_proj.weight", {Q, E_}}, {"k_proj.weight", {Q, E_}}, {"v_proj.weight", {V, E_}}, {"g_proj.weight", {V, E_}},
                                     {"o_proj.weight", {E_, V}}};
        if (whole_norm_) d.push_back({"norm.weight", {V}, false, 1, 0.01f});
        return d;
    }
    bool can_overwrite() const override { return true; }
    bool supports_deferred_norm() const override { return true; }
    int64_t state_bytes() const override { return (int64_t)H_ * dk_ * dv_ * (int64_t)sizeof(float); }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        Weight q = tensor_of(tensors, "q_proj.weight"), k = tensor_of(tensors, "k_proj.weight");
        const Weight &v = tensor_of(tensors, "v_proj.weight"), &g = tensor_of(tensors, "g_proj.weight");
        if (position_ && !position_->permutation().empty()) {
            // the kernels rotate pairs (j, j + head_dim / 2); q . k does not change under a common permutation of both
            const std::vector<int> &perm = position_->permutation();
            std::vector<int64_t> rows;
            for (int h = 0; h < H_; h++)
                for (int i = 0; i < dk_; i++) rows.push_back((int64_t)h * dk_ + perm[(size_t)i]);
            q = gather_rows(q, rows, rt.stream);
            k = gather_rows(k, rows, rt.stream);
        }
        bool same = q.t.dtype == k.t.dtype && k.t.dtype == v.t.dtype && v.t.dtype == g.t.dtype;
        proj_ = Linear(concat_rows({q, k, v, g}, same ? q.t.dtype : FG_F32, rt.stream));
        o_ = Linear(tensor_of(tensors, "o_proj.weight"));
        if (whole_norm_) {
            const Weight &w = tensor_of(tensors, "norm.weight");
            norm_w_ = w.t.dtype == FG_F32 ? w : concat_rows({w}, FG_F32, rt.stream);
        }
        decay_dev_ = make_weight(1, H_, FG_F32, "retention decays");
        FG_CUDA(cudaMemcpyAsync(decay_dev_.t.data, decay_.data(), decay_.size() * sizeof(float), cudaMemcpyHostToDevice, rt.stream));
        FG_CUDA(cudaStreamSynchronize(rt.stream));
    }
    void prepare(Runtime &rt, int max_positions) override { if (position_) position_->prepare(rt, max_positions); }
    DeferredNorm forward(Runtime &rt, const Tensor &xn, const DeferredNorm *deferred, const Batch &b, const LayerIO &io, Tensor &residual,
                         Norm *emit_norm) override {
        if (!io.state || io.state_bytes < state_bytes()) fail(FG_E_INTERNAL, "retention: the schedule entry has no state rows");
        const float *cos_t = position_ ? position_->cos_table() : nullptr;
        const float *sin_t = position_ ? position_->sin_table() : nullptr;
        const int *host_cu = b.host_cu_rows.empty() ? nullptr : b.host_cu_rows.data();
        // activations of the engine's dtype and sums taken as they are: the tensor-core forms
        if (rt.dtype == FG_BF16 && !rt.plain_kernels && silu_ && whole_norm_ && !position_ && k_scale_ == 1.f && all_positive_ &&
            H_ * dv_ % 8 == 0 && H_ * dv_ <= 8192 && FG_KERNEL("mix", fg_decay_attention_ok)(dk_, dv_))
            return forward_on_activations(rt, xn, deferred, b, io, residual, emit_norm, host_cu);
        // what enters the recurrence stays float32: the contraction accumulates in float32 and writes it as it is
        Tensor proj = proj_.forward(rt, xn, deferred, Tensor(), FG_F32, false, nullptr, nullptr);
        const int M = (int)proj.rows;
        Tensor y = rt.arena->matrix(M, (int64_t)H_ * dv_, rt.dtype);
        // (a norm over all heads: the recurrence's sums stay float32 until that norm is done)
        Tensor o = whole_norm_ ? rt.arena->matrix(M, (int64_t)H_ * dv_, FG_F32) : y;
        const int opts = (silu_ ? 1 : 0) | (whole_norm_ ? 2 : 0);
        const int RC = FG_KERNEL("mix", fg_retention_chunk_tokens)();
        bool chunked = host_cu && !b.single_token && all_positive_ && b.max_new >= chunk_threshold_ &&
                       FG_KERNEL("mix", fg_retention_chunked_ok)(dk_, dv_);
        if (chunked) {
            // the host knows only how many chunks the step has; the kernels plan them from the step's row offsets
            int n_chunks = 0;
            for (int s = 0; s < b.n_seq; s++) n_chunks += (host_cu[s + 1] - host_cu[s] + RC - 1) / RC;
            int *plan = (int *)rt.arena->alloc(((size_t)2 * n_chunks + b.n_seq + 1) * sizeof(int));
            float *U = (float *)rt.arena->alloc((size_t)n_chunks * H_ * dk_ * dv_ * sizeof(float));
            FG_LAUNCH("mix", fg_retention_chunked, proj.ptr<float>(), (int)proj.ld, o.data, o.dtype, (int)o.ld, b.positions, b.cu_rows,
                      b.slots, cos_t, sin_t, decay_dev_.t.ptr<float>(), (float *)io.state, plan, U, b.n_seq, n_chunks, H_, dk_, dv_,
                      k_scale_, eps_, opts, rt.stream);
        } else {
            FG_LAUNCH("mix", fg_retention, proj.ptr<float>(), (int)proj.ld, o.data, o.dtype, (int)o.ld, b.positions, b.cu_rows, b.slots, cos_t,
                      sin_t, decay_dev_.t.ptr<float>(), (float *)io.state, b.n_seq, H_, dk_, dv_, k_scale_, eps_, opts, rt.stream);
        }
        if (whole_norm_)
            FG_LAUNCH("mix", fg_gated_group_norm, o.ptr<float>(), (int)o.ld, proj.ptr<float>() + (int64_t)2 * H_ * dk_ + (int64_t)H_ * dv_, (int)proj.ld,
                      norm_w_.t.ptr<float>(), H_ * dv_, y.data, y.dtype, (int)y.ld, M, H_ * dv_, H_ * dv_, eps_, 0, sigmoid_gate_ ? 1 : 0, rt.stream);
        DeferredNorm started;
        o_.forward(rt, y, nullptr, residual, FG_F32, !rt.overwrite, emit_norm, &started);
        return started;
    }

private:
    DeferredNorm forward_on_activations(Runtime &rt, const Tensor &xn, const DeferredNorm *deferred, const Batch &b, const LayerIO &io, Tensor &residual,
                                        Norm *emit_norm, const int *host_cu) {
        Tensor proj = proj_.forward(rt, xn, deferred, Tensor(), FG_BF16, false, nullptr, nullptr);
        const int M = (int)proj.rows, V = H_ * dv_, DC = FG_KERNEL("mix", fg_decay_attention_chunk_tokens)();
        Tensor o = rt.arena->matrix(M, V, FG_F32), y = rt.arena->matrix(M, V, FG_BF16);
        if (host_cu && !b.single_token && b.max_new >= DC / 2) {
            int n_chunks = 0;
            for (int s = 0; s < b.n_seq; s++) n_chunks += (host_cu[s + 1] - host_cu[s] + DC - 1) / DC;
            int *plan = (int *)rt.arena->alloc(((size_t)2 * n_chunks + b.n_seq + 1) * sizeof(int));
            float *U = (float *)rt.arena->alloc((size_t)n_chunks * H_ * dk_ * dv_ * sizeof(float));
            void *P = rt.arena->alloc((size_t)n_chunks * H_ * dk_ * dv_ * 3 * 2);      // the states in front of the chunks, three bfloat16 pieces each
            FG_LAUNCH("mix", fg_decay_attention_chunked, proj.data, (int)proj.ld, o.ptr<float>(), (int)o.ld, b.cu_rows, b.slots, decay_dev_.t.ptr<float>(),
                      (float *)io.state, plan, U, P, b.n_seq, n_chunks, H_, dk_, dv_, rt.stream);
        } else {
            FG_LAUNCH("mix", fg_decay_attention_step, proj.data, (int)proj.ld, o.ptr<float>(), (int)o.ld, b.cu_rows, b.slots, decay_dev_.t.ptr<float>(),
                      (float *)io.state, b.n_seq, H_, dk_, dv_, rt.stream);
        }
        const uint16_t *g = (const uint16_t *)proj.data + (int64_t)2 * H_ * dk_ + V;
        FG_LAUNCH("mix", fg_row_norm_gate, o.ptr<float>(), (int)o.ld, g, (int)proj.ld, norm_w_.t.ptr<float>(), y.data, (int)y.ld, M, V, eps_, sigmoid_gate_ ? 1 : 0,
                  rt.stream);
        DeferredNorm started;
        o_.forward(rt, y, nullptr, residual, FG_F32, !rt.overwrite, emit_norm, &started);
        return started;
    }
    int E_ = 0, H_ = 0, dk_ = 0, dv_ = 0, chunk_threshold_ = 16;
    float eps_ = 0.f, k_scale_ = 1.f;
    bool all_positive_ = true, silu_ = false, whole_norm_ = false, sigmoid_gate_ = false;
    std::vector<float> decay_;
    PositionEncoding *position_ = nullptr;
    Linear proj_, o_;
    Weight decay_dev_, norm_w_;
};

// "gated_linear_attention": linear attention whose state decays per key channel by a factor the token itself decides.
// With the layer's normalised input h, per head (q, k of size head_dim, v of size v_head_dim):
//     q = W_q h * q_scale, k = W_k h, v = W_v h, g = W_g h       no biases
//     a = sigmoid(W_a2 (W_a1 h) + b_a2)^(1 / tau)                 a decay per key channel, through a low-rank pair
//     S_t = diag(a_t) S_(t-1) + k_t v_t^T,  o_t = S_t^T q_t
//     y = concat_heads(o / sqrt(mean(o^2) + eps) * w_norm) * silu(g),  output W_o y
// decay_rank (the inner size of the low-rank pair) may be left to the checkpoint's tensor shapes.  q, k, v, g and the
// low-rank input are ONE contraction with float32 output; the decay logits, their log-sigmoid, the state, the unit norm and
// the gate stay float32 in every engine dtype (gla.cu), y takes the engine's dtype for the output projection.
class GatedLinearAttention : public Mixer {
public:
    GatedLinearAttention(const Json &p, BuildContext &) {
        const char *me = "gated_linear_attention";
        E_ = (int)param_int(p, "hidden_size", me);
        H_ = (int)param_int(p, "n_heads", me);
        dk_ = (int)param_int(p, "head_dim", me);
        dv_ = (int)param_int(p, "v_head_dim", dk_, me);
        rank_ = (int)param_int(p, "decay_rank", -1, me);
        eps_ = (float)param_float(p, "eps", me);
        tau_ = (float)param_float(p, "tau", 1.0, me);
        q_scale_ = (float)param_float(p, "q_scale", 1.0 / std::sqrt((double)dk_), me);
        if (E_ <= 0 || H_ <= 0 || dk_ <= 0 || dv_ <= 0 || rank_ == 0 || rank_ < -1) fail(FG_E_CONFIG, "gated_linear_attention: sizes must be positive");
        if (dv_ > 256) fail(FG_E_CONFIG, format("gated_linear_attention: v_head_dim %d exceeds 256, the largest the kernels take", dv_));
        if ((size_t)dk_ * dv_ > 40 * 1024) fail(FG_E_CONFIG, "gated_linear_attention: a head's state exceeds what the kernels hold in shared memory");
        if (!(eps_ > 0.f) || !(tau_ > 0.f)) fail(FG_E_CONFIG, "gated_linear_attention: eps and tau must be positive");
    }
    std::vector<TensorDecl> tensor_decls() const override {
        int64_t Q = (int64_t)H_ * dk_, V = (int64_t)H_ * dv_, R = rank_;
        return {{"q_proj.weight", {Q, E_}}, {"k_proj.weight", {Q, E_}}, {"v_proj.weight", {V, E_}}, {"g_proj.weight", {V, E_}},
                {"o_proj.weight", {E_, V}}, {"decay_down.weight", {R, E_}}, {"decay_up.weight", {Q, R}}, {"decay_up.bias", {Q}, false, 0, 1.0f},
                {"norm.weight", {dv_}, false, 1, 0.01f}};
    }
    bool can_overwrite() const override { return true; }
    bool supports_deferred_norm() const override { return true; }
    int64_t state_bytes() const override { return (int64_t)H_ * dk_ * dv_ * (int64_t)sizeof(float); }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        const Weight &q = tensor_of(tensors, "q_proj.weight"), &k = tensor_of(tensors, "k_proj.weight");
        const Weight &v = tensor_of(tensors, "v_proj.weight"), &g = tensor_of(tensors, "g_proj.weight");
        const Weight &a1 = tensor_of(tensors, "decay_down.weight"), &a2 = tensor_of(tensors, "decay_up.weight");
        if (a1.t.rows != a2.t.cols)
            fail(FG_E_WEIGHTS, format("gated_linear_attention: the decay's low-rank pair disagrees on its inner size (%lld against %lld)",
                                      (long long)a1.t.rows, (long long)a2.t.cols));
        rank_ = (int)a1.t.rows;
        bool same = q.t.dtype == k.t.dtype && k.t.dtype == v.t.dtype && v.t.dtype == g.t.dtype && g.t.dtype == a1.t.dtype;
        proj_ = Linear(concat_rows({q, k, v, g, a1}, same ? q.t.dtype : FG_F32, rt.stream));
        up_ = Linear(a2);
        o_ = Linear(tensor_of(tensors, "o_proj.weight"));
        bias_ = concat_rows({tensor_of(tensors, "decay_up.bias")}, FG_F32, rt.stream);
        norm_ = concat_rows({tensor_of(tensors, "norm.weight")}, FG_F32, rt.stream);
    }
    DeferredNorm forward(Runtime &rt, const Tensor &xn, const DeferredNorm *deferred, const Batch &b, const LayerIO &io, Tensor &residual,
                         Norm *emit_norm) override {
        if (!io.state || io.state_bytes < state_bytes()) fail(FG_E_INTERNAL, "gated_linear_attention: the schedule entry has no state rows");
        // what enters the recurrence stays float32: the contraction accumulates in float32 and writes it as it is
        Tensor proj = proj_.forward(rt, xn, deferred, Tensor(), FG_F32, false, nullptr, nullptr);
        const int M = (int)proj.rows;
        const int64_t low_at = (int64_t)2 * H_ * dk_ + (int64_t)2 * H_ * dv_;
        Tensor low = proj;
        low.data = proj.ptr<float>() + low_at;
        low.cols = rank_;
        Tensor z = up_.forward(rt, low, nullptr, Tensor(), FG_F32, false, nullptr, nullptr);
        Tensor y = rt.arena->matrix(M, (int64_t)H_ * dv_, rt.dtype);
        const int *host_cu = b.host_cu_rows.empty() ? nullptr : b.host_cu_rows.data();
        const int GC = FG_KERNEL("mix", fg_gla_chunk_tokens)();
        bool chunked = host_cu && !b.single_token && b.max_new >= chunk_threshold_ && FG_KERNEL("mix", fg_gla_chunked_ok)(dk_, dv_);
        if (chunked) {
            int n_chunks = 0;
            for (int s = 0; s < b.n_seq; s++) n_chunks += (host_cu[s + 1] - host_cu[s] + GC - 1) / GC;
            int *plan = (int *)rt.arena->alloc(((size_t)2 * n_chunks + b.n_seq + 1) * sizeof(int));
            float *U = (float *)rt.arena->alloc((size_t)n_chunks * H_ * dk_ * dv_ * sizeof(float));
            float *D = (float *)rt.arena->alloc((size_t)n_chunks * H_ * dk_ * (1 + GC) * sizeof(float));     // decays and cumulative log decays
            FG_LAUNCH("mix", fg_gla_chunked, proj.ptr<float>(), (int)proj.ld, z.ptr<float>(), (int)z.ld, bias_.t.ptr<float>(), norm_.t.ptr<float>(),
                      y.data, y.dtype, (int)y.ld, b.cu_rows, b.slots, (float *)io.state, plan, U, D, b.n_seq, n_chunks, H_, dk_, dv_, tau_,
                      q_scale_, eps_, rt.stream);
        } else {
            FG_LAUNCH("mix", fg_gla, proj.ptr<float>(), (int)proj.ld, z.ptr<float>(), (int)z.ld, bias_.t.ptr<float>(), norm_.t.ptr<float>(), y.data,
                      y.dtype, (int)y.ld, b.cu_rows, b.slots, (float *)io.state, b.n_seq, H_, dk_, dv_, tau_, q_scale_, eps_, rt.stream);
        }
        DeferredNorm started;
        o_.forward(rt, y, nullptr, residual, FG_F32, !rt.overwrite, emit_norm, &started);
        return started;
    }

private:
    int E_ = 0, H_ = 0, dk_ = 0, dv_ = 0, rank_ = -1, chunk_threshold_ = 32;
    float eps_ = 0.f, tau_ = 1.f, q_scale_ = 1.f;
    Linear proj_, up_, o_;
    Weight bias_, norm_;
};

// What the two mixers below share: a short causal convolution with SiLU in front of the recurrence, whose last taps - 1 inputs
// are the first part of the mixer's state row, and the recurrence of recurrence.cu behind it, whose state is the second part.
static Weight f32_rows(const std::vector<Weight> &parts, cudaStream_t s) { return concat_rows(parts, FG_F32, s); }
// Floats of a sequence's recurrence state, as recurrence.cu lays it out: a column of a head's [d, dv] state is shared by R
// lanes, the smallest power of two that leaves a lane at most 16 rows, and rows are padded to a multiple of R.  (Computed
// here so that sizing a cache needs no kernel library; load() checks it against the library's own answer.)
static int64_t recurrence_state_floats(int H, int d, int dv, const char *who) {
    int R = 1;
    while (R < 32 && (d + R - 1) / R > 16) R *= 2;
    if ((d + R - 1) / R > 16) fail(FG_E_CONFIG, std::string(who) + ": the state of a head exceeds what the kernel takes");
    return (int64_t)H * ((d + R - 1) / R) * dv * R;
}
static void check_state_floats(int H, int d, int dv, const char *who) {
    if (FG_KERNEL("mix", fg_decay_recurrence_state_floats)(H, d, dv) != recurrence_state_floats(H, d, dv, who))
        fail(FG_E_INTERNAL, std::string(who) + ": host and kernel library disagree on the size of a state row");
}

// "state_space": the state-space form with a scalar decay per head and token ("duality").  With the normalised input h,
// inner = n_heads * v_head_dim, N = state_size and G = n_groups (head h uses group h / (n_heads / G)):
//     W_in h = [z: inner | x: inner | B: G N | C: G N | dt: n_heads]
//     (x, B, C) <- silu(causal convolution over time per channel + bias)          weights [inner + 2 G N, taps]
//     dt <- softplus(dt + dt_bias);  S_t = exp(-exp(A_log) dt) S_(t-1) + dt B_t x_t^T (S: [N, v_head_dim]);  y_t = S_t^T C_t + D x_t
//     y <- y * silu(z), then an RMS norm in norm_groups equal parts of the inner channels, times a weight [inner]; output W_o y
// Projections leave their contraction as float32; convolution, decays, steps, state, gate and norm are float32 on the FMA units
// in every engine dtype; only the normalised y takes the engine's dtype, as the output projection's input.
class StateSpaceMixer : public Mixer {
public:
    StateSpaceMixer(const Json &p, BuildContext &) {
        const char *me = "state_space";
        E_ = (int)param_int(p, "hidden_size", me);
        H_ = (int)param_int(p, "n_heads", me);
        dv_ = (int)param_int(p, "v_head_dim", me);
        N_ = (int)param_int(p, "state_size", me);
        G_ = (int)param_int(p, "n_groups", 1, me);
        taps_ = (int)param_int(p, "conv_taps", 1, me);
        norm_groups_ = (int)param_int(p, "norm_groups", 1, me);
        eps_ = (float)param_float(p, "eps", me);
        if (E_ <= 0 || H_ <= 0 || dv_ <= 0 || N_ <= 0 || G_ <= 0 || taps_ <= 0 || norm_groups_ <= 0) fail(FG_E_CONFIG, "state_space: sizes must be positive");
        if (H_ % G_) fail(FG_E_CONFIG, format("state_space: %d heads are not a multiple of %d groups", H_, G_));
        if ((H_ * dv_) % norm_groups_) fail(FG_E_CONFIG, format("state_space: %d inner channels do not split into %d norm groups", H_ * dv_, norm_groups_));
        if (N_ > 512) fail(FG_E_CONFIG, format("state_space: state_size %d exceeds 512, the largest the kernel takes", N_));
        if (!(eps_ > 0.f)) fail(FG_E_CONFIG, "state_space: eps must be positive");
    }
    int64_t inner() const { return (int64_t)H_ * dv_; }
    int64_t conv_channels() const { return inner() + (int64_t)2 * G_ * N_; }
    int64_t conv_floats() const { return (int64_t)(taps_ - 1) * conv_channels(); }
    std::vector<TensorDecl> tensor_decls() const override {
        const int64_t I = inner(), C = conv_channels();
        return {{"in_proj.weight", {2 * I + 2 * G_ * N_ + H_, E_}}, {"conv.weight", {C, (int64_t)taps_}, false, 0, 0.5f}, {"conv.bias", {C}, false, 0, 0.3f},
                {"dt_bias", {(int64_t)H_}, false, 0, 1.0f}, {"A_log", {(int64_t)H_}, false, 0, 1.0f}, {"D", {(int64_t)H_}, false, 1, 0.3f},
                {"norm.weight", {I}, false, 1, 0.01f}, {"o_proj.weight", {E_, I}}};
    }
    bool can_overwrite() const override { return true; }
    bool strided_state() const override { return true; }
    int64_t state_bytes() const override {
        return (conv_floats() + recurrence_state_floats(H_, N_, dv_, "state_space")) * (int64_t)sizeof(float);
    }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        check_state_floats(H_, N_, dv_, "state_space");
        in_ = Linear(tensor_of(tensors, "in_proj.weight"));
        o_ = Linear(tensor_of(tensors, "o_proj.weight"));
        conv_w_ = f32_rows({tensor_of(tensors, "conv.weight")}, rt.stream);
        conv_b_ = f32_rows({tensor_of(tensors, "conv.bias")}, rt.stream);
        dt_bias_ = f32_rows({tensor_of(tensors, "dt_bias")}, rt.stream);
        a_log_ = f32_rows({tensor_of(tensors, "A_log")}, rt.stream);
        skip_ = f32_rows({tensor_of(tensors, "D")}, rt.stream);
        norm_ = f32_rows({tensor_of(tensors, "norm.weight")}, rt.stream);
    }
    DeferredNorm forward(Runtime &rt, const Tensor &xn, const DeferredNorm *, const Batch &b, const LayerIO &io, Tensor &residual,
                         Norm *emit_norm) override {
        if (!io.state || io.state_bytes < state_bytes()) fail(FG_E_INTERNAL, "state_space: the schedule entry has no state rows");
        const long long stride = (long long)(io.state_stride / (int64_t)sizeof(float));
        const int I = (int)inner(), C = (int)conv_channels(), GN = G_ * N_;
        Tensor proj = in_.forward(rt, xn, nullptr, Tensor(), FG_F32, false, nullptr, nullptr);
        const int M = (int)proj.rows, ld = (int)proj.ld;
        float *state = (float *)io.state;
        Tensor xbc = rt.arena->matrix(M, C, FG_F32);
        FG_LAUNCH("mix", fg_conv1d_silu, proj.ptr<float>() + I, ld, conv_w_.t.ptr<float>(), conv_b_.t.ptr<float>(), taps_, state, stride, b.row_seq, b.cu_rows,
                  b.slots, xbc.ptr<float>(), (int)xbc.ld, M, C, rt.stream);
        if (taps_ > 1)
            FG_LAUNCH("mix", fg_conv1d_state, proj.ptr<float>() + I, ld, taps_, state, stride, b.cu_rows, b.slots, b.n_seq, C, rt.stream);
        float *decay = (float *)rt.arena->alloc((size_t)2 * M * H_ * sizeof(float)), *step = decay + (size_t)M * H_;
        FG_LAUNCH("mix", fg_decay_gates, proj.ptr<float>() + I + C, ld, nullptr, 0, a_log_.t.ptr<float>(), dt_bias_.t.ptr<float>(), 0, decay, step, M, H_,
                  rt.stream);
        Tensor y = rt.arena->matrix(M, I, FG_F32);
        const int xl = (int)xbc.ld;
        FG_LAUNCH("mix", fg_decay_recurrence, xbc.ptr<float>() + I + GN, xl, xbc.ptr<float>() + I, xl, xbc.ptr<float>(), xl, decay, step, skip_.t.ptr<float>(),
                  y.ptr<float>(), (int)y.ld, b.cu_rows, b.slots, state + conv_floats(), stride, b.n_seq, H_, G_, N_, dv_, 0, rt.stream);
        Tensor yn = rt.arena->matrix(M, I, rt.dtype);
        FG_LAUNCH("mix", fg_gated_group_norm, y.ptr<float>(), (int)y.ld, proj.ptr<float>(), ld, norm_.t.ptr<float>(), I, yn.data, yn.dtype, (int)yn.ld, M, I,
                  I / norm_groups_, eps_, 1, 0, rt.stream);
        DeferredNorm started;
        o_.forward(rt, yn, nullptr, residual, FG_F32, !rt.overwrite, emit_norm, &started);
        return started;
    }

private:
    int E_ = 0, H_ = 0, dv_ = 0, N_ = 0, G_ = 1, taps_ = 1, norm_groups_ = 1;
    float eps_ = 0.f;
    Linear in_, o_;
    Weight conv_w_, conv_b_, dt_bias_, a_log_, skip_, norm_;
};

// "gated_delta": the gated delta rule.  With the normalised input h, n_kv_heads heads of q and k (size head_dim) and n_heads
// heads of v (size v_head_dim), head h using q/k head h / (n_heads / n_kv_heads):
//     q, k, v <- silu(causal convolution over time per channel of W_q h, W_k h, W_v h)      weights [channels, taps], no bias
//     q <- q / sqrt(sum(q^2) + unit_eps) * q_scale and k <- k / sqrt(sum(k^2) + unit_eps), per head
//     beta = sigmoid(W_b h), g = exp(-exp(A_log) softplus(W_a h + dt_bias)), one each per head
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q                          (S: [head_dim, v_head_dim])
//     y = o / sqrt(mean(o^2) + eps) * w (w [v_head_dim], shared by heads) * silu(W_g h); output W_o y
// The six projections are ONE contraction with float32 output; everything up to y is float32 in every engine dtype.
class GatedDeltaMixer : public Mixer {
public:
    GatedDeltaMixer(const Json &p, BuildContext &) {
        const char *me = "gated_delta";
        E_ = (int)param_int(p, "hidden_size", me);
        H_ = (int)param_int(p, "n_heads", me);
        G_ = (int)param_int(p, "n_kv_heads", H_, me);
        d_ = (int)param_int(p, "head_dim", me);
        dv_ = (int)param_int(p, "v_head_dim", d_, me);
        taps_ = (int)param_int(p, "conv_taps", 1, me);
        eps_ = (float)param_float(p, "eps", me);
        unit_eps_ = (float)param_float(p, "unit_eps", 1e-6, me);
        q_scale_ = (float)param_float(p, "q_scale", 1.0 / std::sqrt((double)d_), me);
        if (E_ <= 0 || H_ <= 0 || G_ <= 0 || d_ <= 0 || dv_ <= 0 || taps_ <= 0) fail(FG_E_CONFIG, "gated_delta: sizes must be positive");
        if (H_ % G_) fail(FG_E_CONFIG, format("gated_delta: %d heads are not a multiple of %d key heads", H_, G_));
        if (d_ > 512) fail(FG_E_CONFIG, format("gated_delta: head_dim %d exceeds 512, the largest the kernel takes", d_));
        if (!(eps_ > 0.f) || !(unit_eps_ >= 0.f)) fail(FG_E_CONFIG, "gated_delta: eps must be positive");
    }
    int64_t conv_channels() const { return (int64_t)2 * G_ * d_ + (int64_t)H_ * dv_; }
    int64_t conv_floats() const { return (int64_t)(taps_ - 1) * conv_channels(); }
    std::vector<TensorDecl> tensor_decls() const override {
        const int64_t Q = (int64_t)G_ * d_, V = (int64_t)H_ * dv_;
        return {{"q_proj.weight", {Q, E_}}, {"k_proj.weight", {Q, E_}}, {"v_proj.weight", {V, E_}}, {"b_proj.weight", {(int64_t)H_, E_}},
                {"a_proj.weight", {(int64_t)H_, E_}}, {"g_proj.weight", {V, E_}}, {"o_proj.weight", {E_, V}},
                {"q_conv.weight", {Q, (int64_t)taps_}, false, 0, 0.5f}, {"k_conv.weight", {Q, (int64_t)taps_}, false, 0, 0.5f},
                {"v_conv.weight", {V, (int64_t)taps_}, false, 0, 0.5f}, {"A_log", {(int64_t)H_}, false, 0, 1.0f}, {"dt_bias", {(int64_t)H_}, false, 0, 1.0f},
                {"norm.weight", {(int64_t)dv_}, false, 1, 0.01f}};
    }
    bool can_overwrite() const override { return true; }
    bool strided_state() const override { return true; }
    int64_t state_bytes() const override {
        return (conv_floats() + recurrence_state_floats(H_, d_, dv_, "gated_delta")) * (int64_t)sizeof(float);
    }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        check_state_floats(H_, d_, dv_, "gated_delta");
        std::vector<Weight> rows;
        bool same = true;
        for (const char *n : {"q_proj.weight", "k_proj.weight", "v_proj.weight", "b_proj.weight", "a_proj.weight", "g_proj.weight"}) {
            rows.push_back(tensor_of(tensors, n));
            same = same && rows.back().t.dtype == rows.front().t.dtype;
        }
        proj_ = Linear(concat_rows(rows, same ? rows.front().t.dtype : FG_F32, rt.stream));
        o_ = Linear(tensor_of(tensors, "o_proj.weight"));
        // [channels, taps] row-major: the three lie one after another
        conv_w_ = make_weight(conv_channels(), taps_, FG_F32, "convolution weights of the delta rule");
        size_t at = 0;
        for (const char *n : {"q_conv.weight", "k_conv.weight", "v_conv.weight"}) {
            const Weight &w = tensor_of(tensors, n);
            dev_convert(w.t.data, w.t.dtype, (char *)conv_w_.t.data + at * 4, FG_F32, w.t.numel(), rt.stream);
            at += (size_t)w.t.numel();
        }
        a_log_ = f32_rows({tensor_of(tensors, "A_log")}, rt.stream);
        dt_bias_ = f32_rows({tensor_of(tensors, "dt_bias")}, rt.stream);
        norm_ = f32_rows({tensor_of(tensors, "norm.weight")}, rt.stream);
    }
    DeferredNorm forward(Runtime &rt, const Tensor &xn, const DeferredNorm *, const Batch &b, const LayerIO &io, Tensor &residual,
                         Norm *emit_norm) override {
        if (!io.state || io.state_bytes < state_bytes()) fail(FG_E_INTERNAL, "gated_delta: the schedule entry has no state rows");
        const long long stride = (long long)(io.state_stride / (int64_t)sizeof(float));
        const int Q = G_ * d_, V = H_ * dv_, C = (int)conv_channels();
        Tensor proj = proj_.forward(rt, xn, nullptr, Tensor(), FG_F32, false, nullptr, nullptr);
        const int M = (int)proj.rows, ld = (int)proj.ld;
        float *state = (float *)io.state;
        Tensor qkv = rt.arena->matrix(M, C, FG_F32);
        const int xl = (int)qkv.ld;
        FG_LAUNCH("mix", fg_conv1d_silu, proj.ptr<float>(), ld, conv_w_.t.ptr<float>(), nullptr, taps_, state, stride, b.row_seq, b.cu_rows, b.slots,
                  qkv.ptr<float>(), xl, M, C, rt.stream);
        if (taps_ > 1) FG_LAUNCH("mix", fg_conv1d_state, proj.ptr<float>(), ld, taps_, state, stride, b.cu_rows, b.slots, b.n_seq, C, rt.stream);
        FG_LAUNCH("mix", fg_unit_heads, qkv.ptr<float>(), xl, G_, d_, unit_eps_, q_scale_, M, rt.stream);
        FG_LAUNCH("mix", fg_unit_heads, qkv.ptr<float>() + Q, xl, G_, d_, unit_eps_, 1.0f, M, rt.stream);
        float *decay = (float *)rt.arena->alloc((size_t)2 * M * H_ * sizeof(float)), *step = decay + (size_t)M * H_;
        FG_LAUNCH("mix", fg_decay_gates, proj.ptr<float>() + C + H_, ld, proj.ptr<float>() + C, ld, a_log_.t.ptr<float>(), dt_bias_.t.ptr<float>(), 1, decay,
                  step, M, H_, rt.stream);
        Tensor o = rt.arena->matrix(M, V, FG_F32);
        FG_LAUNCH("mix", fg_decay_recurrence, qkv.ptr<float>(), xl, qkv.ptr<float>() + Q, xl, qkv.ptr<float>() + 2 * Q, xl, decay, step, nullptr, o.ptr<float>(),
                  (int)o.ld, b.cu_rows, b.slots, state + conv_floats(), stride, b.n_seq, H_, G_, d_, dv_, 1, rt.stream);
        Tensor y = rt.arena->matrix(M, V, rt.dtype);
        FG_LAUNCH("mix", fg_gated_group_norm, o.ptr<float>(), (int)o.ld, proj.ptr<float>() + C + 2 * H_, ld, norm_.t.ptr<float>(), dv_, y.data, y.dtype,
                  (int)y.ld, M, V, dv_, eps_, 0, 0, rt.stream);
        DeferredNorm started;
        o_.forward(rt, y, nullptr, residual, FG_F32, !rt.overwrite, emit_norm, &started);
        return started;
    }

private:
    int E_ = 0, H_ = 0, G_ = 0, d_ = 0, dv_ = 0, taps_ = 1;
    float eps_ = 0.f, unit_eps_ = 1e-6f, q_scale_ = 1.f;
    Linear proj_, o_;
    Weight conv_w_, a_log_, dt_bias_, norm_;
};

// "rglru": a recurrent block around the real-gated linear recurrent unit.  With the mixer's input h, C = width channels and
// n_blocks equal parts of them:
//     y = gelu_tanh(W_y h + b_y),  u = causal convolution over time per channel of (W_x h + b_x), plus a bias   weights [C, taps]
//     r = sigmoid(R u + b_r), i = sigmoid(I u + b_i)                     R, I: one square matrix a part
//     log a = -gain r softplus(lam);  S_t = a S_(t-1) + sqrt(1 - a^2) i u;  output W_o (S y)
// W_y and W_x are ONE contraction with float32 output; convolution, gates (their matrix products included), decays and state are
// 32-bit in every engine dtype (rglru.cu); only S y takes the engine's dtype, as the output projection's input.
class RecurrentUnitMixer : public Mixer {
public:
    RecurrentUnitMixer(const Json &p, BuildContext &) {
        const char *me = "rglru";
        E_ = (int)param_int(p, "hidden_size", me);
        C_ = (int)param_int(p, "width", me);
        B_ = (int)param_int(p, "n_blocks", 1, me);
        taps_ = (int)param_int(p, "conv_taps", 1, me);
        gain_ = (float)param_float(p, "gain", 8.0, me);
        if (E_ <= 0 || C_ <= 0 || B_ <= 0 || taps_ <= 0) fail(FG_E_CONFIG, "rglru: sizes must be positive");
        if (C_ % B_) fail(FG_E_CONFIG, format("rglru: %d channels do not split into %d equal blocks", C_, B_));
        if (!(gain_ > 0.f)) fail(FG_E_CONFIG, "rglru: gain must be positive");
    }
    std::vector<TensorDecl> tensor_decls() const override {
        const int64_t C = C_, B = B_, s = C_ / B_;
        return {{"y_proj.weight", {C, E_}}, {"y_proj.bias", {C}, false, 0, 0.1f}, {"x_proj.weight", {C, E_}}, {"x_proj.bias", {C}, false, 0, 0.1f},
                {"conv.weight", {C, (int64_t)taps_}, false, 0, 0.5f}, {"conv.bias", {C}, false, 0, 0.1f},
                {"r_gate.weight", {B, s, s}, false, 0, 0.1f}, {"r_gate.bias", {B, s}, false, 0, 0.5f}, {"i_gate.weight", {B, s, s}, false, 0, 0.1f},
                {"i_gate.bias", {B, s}, false, 0, 0.5f}, {"lam", {C}, false, 0, 1.0f}, {"o_proj.weight", {E_, C}}};
    }
    bool can_overwrite() const override { return true; }
    bool supports_deferred_norm() const override { return true; }
    bool strided_state() const override { return true; }
    int64_t state_bytes() const override { return (int64_t)(taps_ > 1 ? taps_ + 1 : 1) * C_ * (int64_t)sizeof(float); }
    void load(const std::map<std::string, Weight> &tensors, Runtime &rt) override {
        if (FG_KERNEL("mix", fg_rglru_state_floats)(C_, taps_) * (int64_t)sizeof(float) != state_bytes())
            fail(FG_E_INTERNAL, "rglru: host and kernel library disagree on the size of a state row");
        const Weight &y = tensor_of(tensors, "y_proj.weight"), &x = tensor_of(tensors, "x_proj.weight");
        in_ = Linear(concat_rows({y, x}, y.t.dtype == x.t.dtype ? y.t.dtype : FG_F32, rt.stream));
        o_ = Linear(tensor_of(tensors, "o_proj.weight"));
        in_b_ = f32_rows({flat(tensors, "y_proj.bias"), flat(tensors, "x_proj.bias")}, rt.stream);
        // [C, taps] -> [taps][C], so that neighbouring channels' weights of a tap lie side by side
        const Weight cw = f32_rows({tensor_of(tensors, "conv.weight")}, rt.stream);
        conv_w_ = make_weight(taps_, C_, FG_F32, "convolution weights of a recurrent block");
        for (int t = 0; t < taps_; t++)
            FG_CUDA(cudaMemcpy2DAsync(conv_w_.t.ptr<float>() + (size_t)t * C_, sizeof(float), cw.t.ptr<float>() + t, (size_t)taps_ * sizeof(float), sizeof(float),
                                      (size_t)C_, cudaMemcpyDeviceToDevice, rt.stream));
        conv_b_ = f32_rows({tensor_of(tensors, "conv.bias")}, rt.stream);
        lam_ = f32_rows({tensor_of(tensors, "lam")}, rt.stream);
        // part by part: the rows of R, then those of I
        const int64_t s = C_ / B_;
        Weight r = tensor_of(tensors, "r_gate.weight"), i = tensor_of(tensors, "i_gate.weight");
        if (r.t.dtype != i.t.dtype) { r = f32_rows({r}, rt.stream); i = f32_rows({i}, rt.stream); }
        gates_ = by_part(r, i, s * s, r.t.dtype, rt.stream);
        gates_.t.rows = 2 * C_; gates_.t.cols = s; gates_.t.ld = s;
        gate_b_ = by_part(f32_rows({tensor_of(tensors, "r_gate.bias")}, rt.stream), f32_rows({tensor_of(tensors, "i_gate.bias")}, rt.stream), s, FG_F32, rt.stream);
        if (rt.dtype == FG_BF16 && !rt.plain_kernels && gates_.t.dtype == FG_BF16 && s % 8 == 0) {
            // the matrix three times side by side: it meets u as three bfloat16 numbers (rglru.cu)
            wide_ = make_weight(2 * C_, 3 * s, FG_BF16, "gates of a recurrent unit");
            for (int k = 0; k < 3; k++)
                FG_CUDA(cudaMemcpy2DAsync((char *)wide_.t.data + (size_t)k * s * 2, (size_t)3 * s * 2, gates_.t.data, (size_t)s * 2, (size_t)s * 2, (size_t)2 * C_,
                                          cudaMemcpyDeviceToDevice, rt.stream));
        }
        FG_CUDA(cudaStreamSynchronize(rt.stream));
    }
    DeferredNorm forward(Runtime &rt, const Tensor &xn, const DeferredNorm *deferred, const Batch &b, const LayerIO &io, Tensor &residual,
                         Norm *emit_norm) override {
        if (!io.state || io.state_bytes < state_bytes()) fail(FG_E_INTERNAL, "rglru: the schedule entry has no state rows");
        const long long stride = (long long)(io.state_stride / (int64_t)sizeof(float));
        const int s = C_ / B_;
        float *state = (float *)io.state;
        Tensor proj = in_.forward(rt, xn, deferred, Tensor(), FG_F32, false, nullptr, nullptr);
        const int M = (int)proj.rows, ld = (int)proj.ld;
        const float *in_b = in_b_.t.ptr<float>(), *conv_w = conv_w_.t.ptr<float>(), *conv_b = conv_b_.t.ptr<float>(), *gate_b = gate_b_.t.ptr<float>(),
                    *lam = lam_.t.ptr<float>();
        Tensor y = rt.arena->matrix(M, C_, rt.dtype);
        if (b.single_token && FG_KERNEL("mix", fg_rglru_step_ok)(s)) {
            FG_LAUNCH("mix", fg_rglru_step, proj.ptr<float>(), ld, in_b, conv_w, conv_b, taps_, gates_.t.data, gates_.t.dtype, gate_b, lam, gain_, b.positions,
                      b.row_seq, b.slots, state, stride, y.data, y.dtype, (int)y.ld, M, C_, s, rt.stream);
        } else {
            Tensor u = rt.arena->matrix(M, C_, FG_F32), z;
            int z_row = 2 * C_;
            long long z_part = 2 * s;
            const bool tc = wide_.t.defined() && !b.single_token && M >= tensor_cores_from_;
            if (tc) {
                Tensor pieces = rt.arena->matrix((int64_t)B_ * M, (int64_t)3 * s, FG_BF16);
                z = rt.arena->matrix((int64_t)B_ * M, (int64_t)2 * s, FG_F32);
                z_row = 2 * s; z_part = (long long)M * 2 * s;
                const int bn = FG_KERNEL("tc", fg_gemm_tc_grouped_bn)(2 * s), n_tiles = FG_KERNEL("mix", fg_rglru_tiles)(M, C_, s, bn);
                void *tiles = rt.arena->alloc((size_t)n_tiles * 4 * sizeof(int));
                FG_LAUNCH("mix", fg_rglru_conv, proj.ptr<float>(), ld, in_b, conv_w, conv_b, taps_, state, stride, b.positions, b.row_seq, b.cu_rows, b.slots,
                          u.ptr<float>(), (int)u.ld, pieces.data, tiles, bn, M, C_, s, rt.stream);
                FG_LAUNCH("tc", fg_gemm_tc_grouped, pieces.data, (int)pieces.ld, (int)pieces.rows, wide_.t.data, (int)wide_.t.ld, (int)wide_.t.rows,
                          z.ptr<float>(), (int)z.ld, 2 * s, 3 * s, tiles, n_tiles, rt.stream);
            } else {
                z = rt.arena->matrix(M, (int64_t)2 * C_, FG_F32);
                FG_LAUNCH("mix", fg_rglru_conv, proj.ptr<float>(), ld, in_b, conv_w, conv_b, taps_, state, stride, b.positions, b.row_seq, b.cu_rows, b.slots,
                          u.ptr<float>(), (int)u.ld, nullptr, nullptr, 0, M, C_, s, rt.stream);
                FG_LAUNCH("mix", fg_head_gemm, u.data, FG_F32, (int)u.ld, s, gates_.t.data, gates_.t.dtype, s, 0, z.data, FG_F32, (int)z.ld, 2 * s, nullptr, 0, M,
                          2 * s, s, B_, rt.stream);
            }
            FG_LAUNCH("mix", fg_rglru_scan, z.ptr<float>(), z_row, z_part, gate_b, u.ptr<float>(), (int)u.ld, lam, gain_, proj.ptr<float>(), ld, in_b, y.data,
                      y.dtype, (int)y.ld, b.cu_rows, b.slots, b.positions, state, stride, b.n_seq, b.max_new, C_, s, taps_, rt.stream);
        }
        DeferredNorm started;
        o_.forward(rt, y, nullptr, residual, FG_F32, !rt.overwrite, emit_norm, &started);
        return started;
    }

private:
    static Weight flat(const std::map<std::string, Weight> &tensors, const char *name) {
        Weight w = tensor_of(tensors, name);
        w.t.rows = w.t.numel(); w.t.cols = 1; w.t.ld = 1;
        return w;
    }
    // [parts][2][n]: part p of a, then part p of b
    Weight by_part(const Weight &a, const Weight &b, int64_t n, int dtype, cudaStream_t st) const {
        const size_t bytes = (size_t)n * elem_size(dtype);
        Weight out = make_weight(2 * B_, n, dtype, "gates of a recurrent unit");
        int at = 0;
        for (const Weight *w : {&a, &b})
            FG_CUDA(cudaMemcpy2DAsync((char *)out.t.data + bytes * at++, 2 * bytes, w->t.data, bytes, bytes, (size_t)B_, cudaMemcpyDeviceToDevice, st));
        FG_CUDA(cudaStreamSynchronize(st));            // a and b may go away with the caller's expression
        return out;
    }
    int E_ = 0, C_ = 0, B_ = 1, taps_ = 1;
    int tensor_cores_from_ = 64;             // rows from which the gates run on the tensor cores
    float gain_ = 8.f;
    Linear in_, o_;
    Weight in_b_, conv_w_, conv_b_, lam_, gates_, gate_b_, wide_;
};

void add_recurrent_kinds(std::map<std::string, PartFactory> &mixers) {
    mixers["gated_linear_attention"] = [](Runtime &, const Json &p, BuildContext &c) { return std::make_unique<GatedLinearAttention>(p, c); };
    mixers["rglru"] = [](Runtime &, const Json &p, BuildContext &c) { return std::make_unique<RecurrentUnitMixer>(p, c); };
    mixers["retention"] = [](Runtime &, const Json &p, BuildContext &c) { return std::make_unique<RetentionMixer>(p, c); };
    mixers["state_space"] = [](Runtime &, const Json &p, BuildContext &c) { return std::make_unique<StateSpaceMixer>(p, c); };
    mixers["gated_delta"] = [](Runtime &, const Json &p, BuildContext &c) { return std::make_unique<GatedDeltaMixer>(p, c); };
}

}  // namespace fg
